// Latent attention: norms of the query latent (if there is one) and the key / value latent, rotation of the shared key part and append of the row
// [latent | rotated part] to its cache page.  One warp per (token, latent); a row is read twice, the second time from L1.
#include "latent.h"

#include "../common/elem.cuh"
#include "../common/launch.h"

namespace nfb {

namespace {

template <typename A>
__device__ __forceinline__ void norm_row(const A* src, A* dst, const float* w, int width, int width_true, float eps, int lane) {
  float ss = 0.f;
  for (int c = lane * 8; c < width; c += 256) {
    float v[8];
    load8(src + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(width_true) + eps);
  for (int c = lane * 8; c < width; c += 256) {
    float v[8], g[8];
    load8(src + c, v);
    load8(w + c, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = v[j] * inv * g[j];
    store8(dst + c, v);
  }
}

template <typename A>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrepArgs p) {
  pdl_launch_next();
  pdl_wait_prior();
  const int lane = threadIdx.x & 31;
  const long long item = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int per = p.q_rank > 0 ? 2 : 1;
  if (item >= static_cast<long long>(per) * p.T) return;
  const int t = static_cast<int>(item / per);
  const A* row = static_cast<const A*>(p.proj) + t * p.ldp;
  if (item % per != per - 1) {
    norm_row(row, static_cast<A*>(p.q_latent) + t * p.ldq, p.q_norm, p.q_rank, p.q_rank_true, p.eps, lane);
    return;
  }
  const int pos = p.cache_pos[t];
  const int page = p.block_table[static_cast<long long>(p.table_row[t]) * p.table_ld + pos / p.page_size];
  if (page < 0) return;
  A* dst = static_cast<A*>(p.pages) + (static_cast<long long>(page) * p.page_size + pos % p.page_size) * (p.rank + p.rot);
  norm_row(row + p.kv_off, dst, p.kv_norm, p.rank, p.rank_true, p.eps, lane);
  const A* r = row + p.kv_off + p.rank;
  for (int i = lane; i < p.rot / 2; i += 32) {
    float u = 0.f, v = 0.f;
    if (2 * i < p.rot_true) {
      float c, s;
      rotary_angle(pos, p.freq[i], c, s);
      const float a = elem_to_f(r[2 * i]), b = elem_to_f(r[2 * i + 1]);
      u = a * c - b * s;
      v = b * c + a * s;
    }
    dst[p.rank + 2 * i] = elem_from_f<A>(u);
    dst[p.rank + 2 * i + 1] = elem_from_f<A>(v);
  }
}

}  // namespace

const char* latent_prep(const LatentPrepArgs& a) {
  if (a.T <= 0) return nullptr;
  if (a.q_rank % 16 || a.rank % 16 || a.rot % 16 || a.rot_true % 2 || a.rot_true > a.rot || a.rank_true > a.rank ||
      a.q_rank_true > a.q_rank)
    return "latent_prep: widths must be multiples of 16";
  if (a.ldp % 8 || a.ldq % 8 || a.kv_off % 8) return "latent_prep: misaligned rows";
  const dim3 grid(static_cast<unsigned>(((a.q_rank > 0 ? 2LL : 1LL) * a.T + 7) / 8));
  const cudaError_t e = a.f32 ? launch_kernel(latent_prep_kernel<float>, grid, dim3(256), 0, a.stream, a.pdl, 1, a)
                              : launch_kernel(latent_prep_kernel<__nv_bfloat16>, grid, dim3(256), 0, a.stream, a.pdl, 1, a);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
