// Absorbed latent attention on the FP32 pipes: one CTA per (token, head).  A warp scores one key at a time, 128 keys per
// round; then the threads hold latent columns and add the weighted rows up.  For 32-bit runs.
#include "latent.h"

#include <math_constants.h>

#include "../common/elem.cuh"
#include "../common/launch.h"

namespace nfb {

namespace {

constexpr int kThreads = 256, kKeys = 128, kMaxCols = 4;   // latents of up to kThreads * kMaxCols

template <typename A>
__global__ void __launch_bounds__(kThreads) latent_token_kernel(const LatentArgs p) {
  extern __shared__ __align__(16) float smem[];
  const int W = p.rank + p.rot;
  float* q = smem;              // [W]
  float* s = q + W;             // [kKeys] scores, then weights
  long long* at = reinterpret_cast<long long*>(s + kKeys);   // [kKeys] row offsets, -1: not mapped
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_launch_next();
  pdl_wait_prior();
  const int t = blockIdx.x, h = blockIdx.y, len = p.kv_len[t];
  const A* ql = static_cast<const A*>(p.q_latent) + t * p.ldl + static_cast<long long>(h) * p.rank;
  const A* qr = static_cast<const A*>(p.q) + t * p.ldq + static_cast<long long>(h) * (p.dim + p.rot) + p.dim;
  for (int i = tid; i < p.rank; i += kThreads) q[i] = elem_to_f(ql[i]);
  for (int i = tid; i < p.rot / 2; i += kThreads) {
    float u = 0.f, v = 0.f;
    if (2 * i < p.rot_true) {
      float c, sn;
      rotary_angle(len - 1, p.freq[i], c, sn);
      const float a = elem_to_f(qr[2 * i]), b = elem_to_f(qr[2 * i + 1]);
      u = a * c - b * sn;
      v = b * c + a * sn;
    }
    q[p.rank + 2 * i] = u;
    q[p.rank + 2 * i + 1] = v;
  }
  const A* pages = static_cast<const A*>(p.pages);
  const int* table = p.block_table + static_cast<long long>(p.table_row[t]) * p.table_ld;
  const float sink = p.sink != nullptr ? p.sink[h] : -CUDART_INF_F;
  float m = sink, l = p.sink != nullptr ? 1.f : 0.f, o[kMaxCols] = {};
  for (int k0 = latent_first(len, p.window); k0 < len; k0 += kKeys) {
    const int n = min(kKeys, len - k0);
    __syncthreads();
    if (tid < n) {
      const int key = k0 + tid, page = table[key / p.page_size];
      at[tid] = page < 0 ? -1 : (static_cast<long long>(page) * p.page_size + key % p.page_size) * W;
    }
    __syncthreads();
    for (int j = warp; j < n; j += kThreads / 32) {
      float d = 0.f;
      if (at[j] >= 0)
        for (int c = lane * 8; c < W; c += 256) {
          float v[8];
          load8(pages + at[j] + c, v);
#pragma unroll
          for (int e = 0; e < 8; ++e) d = fmaf(q[c + e], v[e], d);
        }
      d = warp_sum(d);
      if (lane == 0) s[j] = at[j] >= 0 ? d * p.scale : -CUDART_INF_F;
    }
    __syncthreads();
    float mx = m;
    for (int j = lane; j < n; j += 32) mx = fmaxf(mx, s[j]);
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    if (!(mx > -CUDART_INF_F)) continue;      // nothing seen yet (the same for every thread)
    __syncthreads();
    if (tid < n) s[tid] = expf(s[tid] - mx);
    __syncthreads();
    float sum = 0.f;
    for (int j = lane; j < n; j += 32) sum += s[j];
    const float f = m > -CUDART_INF_F ? expf(m - mx) : 0.f;
    l = l * f + warp_sum(sum);
    m = mx;
#pragma unroll
    for (int i = 0; i < kMaxCols; ++i) o[i] *= f;
    for (int j = 0; j < n; ++j) {
      const float w = s[j];
      if (at[j] < 0) continue;
#pragma unroll
      for (int i = 0; i < kMaxCols; ++i) {
        const int c = tid + i * kThreads;
        if (c < p.rank) o[i] = fmaf(w, elem_to_f(pages[at[j] + c]), o[i]);
      }
    }
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  A* out = static_cast<A*>(p.out) + t * p.ldo + static_cast<long long>(h) * p.rank;
#pragma unroll
  for (int i = 0; i < kMaxCols; ++i) {
    const int c = tid + i * kThreads;
    if (c < p.rank) out[c] = elem_from_f<A>(o[i] * inv);
  }
}

}  // namespace

const char* latent_token_attention(const LatentArgs& a) {
  if (a.T <= 0) return nullptr;
  if (a.rank % 16 || a.rot % 16 || a.rank > kThreads * kMaxCols || a.rot_true > a.rot || a.rot_true % 2)
    return "latent attention: widths must be multiples of 16, the latent at most 1024 wide";
  if (a.n_heads > 65535) return "latent attention: too many heads";
  const size_t smem = sizeof(float) * (a.rank + a.rot + kKeys) + sizeof(long long) * kKeys;
  const dim3 grid(a.T, a.n_heads);
  const cudaError_t e = a.f32 ? launch_kernel(latent_token_kernel<float>, grid, dim3(kThreads), smem, a.stream, a.pdl, 1, a)
                              : launch_kernel(latent_token_kernel<__nv_bfloat16>, grid, dim3(kThreads), smem, a.stream, a.pdl, 1, a);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
