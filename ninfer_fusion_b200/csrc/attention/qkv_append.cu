// Per-head RMS norm and rotation of the query and key heads of a fused projection, the mix of the values with those of an
// earlier layer, and the append of k / v rows to their cache pages, for layers whose query / key and value widths differ and whose element type is bf16 or fp32.  One warp per
// (token, head row); values stay in registers between the two passes of the norm.
#include "head_mix.h"

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "rotary.cuh"

namespace nfb {

namespace {

constexpr int kMaxChunks = 4;   // 32 lanes x 8 values x 4 = rows of up to 1024 values

template <typename A>
__global__ void __launch_bounds__(256) qkv_append_kernel(const QkvAppendArgs p) {
  pdl_launch_next();
  pdl_wait_prior();
  const int lane = threadIdx.x & 31;
  const int rows = p.n_heads + 2 * p.n_kv;
  const long long item = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= static_cast<long long>(p.T) * rows) return;
  const int t = static_cast<int>(item / rows);
  int r = static_cast<int>(item % rows);
  const int kind = r < p.n_heads ? 0 : (r < p.n_heads + p.n_kv ? 1 : 2);
  if (kind == 1) r -= p.n_heads;
  if (kind == 2) r -= p.n_heads + p.n_kv;
  const int width = kind == 2 ? p.vdim : p.dim;
  const A* src = static_cast<const A*>(p.proj) + t * p.ldp + (kind == 0 ? p.q_off : (kind == 1 ? p.k_off : p.v_off)) + r * width;
  A* dst;
  const int pos = p.cache_pos[t];
  if (kind == 0) {
    dst = static_cast<A*>(p.q_out) + t * p.ldq + r * width;
  } else {
    const int page = p.block_table[static_cast<long long>(p.table_row[t]) * p.table_ld + pos / p.page_size];
    if (page < 0) return;
    dst = static_cast<A*>(kind == 1 ? p.k_pages : p.v_pages) +
          ((static_cast<long long>(page) * p.n_kv + r) * p.page_size + pos % p.page_size) * width;
  }
  const float* w = kind == 0 ? p.q_norm : (kind == 1 ? p.k_norm : nullptr);
  float v[kMaxChunks][8];
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < kMaxChunks; ++c) {
    const int at = (c * 32 + lane) * 8;
    if (at < width) {
      load8(src + at, v[c]);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v[c][j] * v[c][j];
    }
  }
  float inv = 1.f;
  const bool normed = w != nullptr || (p.unit && kind != 2);
  if (normed) inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.dim_true) + p.eps);
#pragma unroll
  for (int c = 0; c < kMaxChunks; ++c) {
    const int at = (c * 32 + lane) * 8;
    if (at < width) {
      if (normed) {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[c][j] = v[c][j] * inv * (w != nullptr ? w[at + j] : 1.f);
      }
      if (kind == 2 && p.v_first != nullptr) {
        A* first = static_cast<A*>(p.v_first) + t * p.ld_first + r * width + at;
        if (p.v_lambda == nullptr) {
          store8(first, v[c]);
        } else {
          const float lambda = *p.v_lambda;
          float u[8];
          load8(first, u);
#pragma unroll
          for (int j = 0; j < 8; ++j) v[c][j] = (1.f - lambda) * v[c][j] + lambda * u[j];
        }
      }
      if (kind != 2 && at < p.rot) {
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
          if (at + j < p.rot) {
            float cs, sn;
            rotary_angle(pos, p.freq[(at + j) / 2], cs, sn);
            const float a = v[c][j], b = v[c][j + 1];
            v[c][j] = a * cs - b * sn;
            v[c][j + 1] = b * cs + a * sn;
          }
        }
      }
      store8(dst + at, v[c]);
    }
  }
}

}  // namespace

const char* qkv_append(const QkvAppendArgs& a) {
  if (a.T <= 0) return nullptr;
  if (a.dim % 16 || a.vdim % 16 || a.dim > 1024 || a.vdim > 1024 || a.dim_true <= 0 || a.dim_true > a.dim)
    return "qkv_append: head widths must be multiples of 16 up to 1024";
  if (a.rot < 0 || a.rot % 2 || a.rot > a.dim_true || (a.rot > 0 && a.freq == nullptr)) return "qkv_append: bad rotation";
  const int align = a.f32 ? 4 : 8;
  if (a.ldp % align || a.ldq % align || a.q_off % 8 || a.k_off % 8 || a.v_off % 8 || a.ld_first % 8) return "qkv_append: misaligned rows";
  const long long items = static_cast<long long>(a.T) * (a.n_heads + 2 * a.n_kv);
  const dim3 grid(static_cast<unsigned>((items + 7) / 8));
  const cudaError_t e = a.f32 ? launch_kernel(qkv_append_kernel<float>, grid, dim3(256), 0, a.stream, a.pdl, 1, a)
                              : launch_kernel(qkv_append_kernel<__nv_bfloat16>, grid, dim3(256), 0, a.stream, a.pdl, 1, a);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
