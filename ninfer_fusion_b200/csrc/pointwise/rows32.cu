// Row kernels on a 32-bit residual stream: embedding gather and the norm-after-the-sum step
//   y = alpha * x + delta;   x <- y / sqrt(mean(y^2) + eps) * gain        (one gain for all columns)
// fused with the copy of the new row in the activation type that the next GEMM consumes and, after the last
// sublayer, with the model's final norm.  One CTA per row, 16-byte accesses, the row held in registers.
#include "rows32.h"

#include "../common/elem.cuh"
#include "../common/launch.h"

namespace nfb {

namespace {

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = (lane < static_cast<int>(blockDim.x >> 5)) ? red[lane] : 0.f;
  t = warp_sum(t);
  __syncthreads();
  return t;
}

template <typename A>
__global__ void __launch_bounds__(256) embed_rows32_kernel(const int* __restrict__ ids, const A* __restrict__ table,
                                                            float* __restrict__ x32, A* __restrict__ xa, int N, long long ld_xa,
                                                            float scale, int vocab, const int* __restrict__ pos,
                                                            const A* __restrict__ places, int n_places) {
  pdl_launch_next();
  pdl_wait_prior();
  const long long row = blockIdx.x;
  int id = ids[row];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const A* src = table + static_cast<long long>(id) * N;
  const A* place = places == nullptr ? nullptr : places + static_cast<long long>(min(max(pos[row], 0), n_places - 1)) * N;
  for (int c = threadIdx.x * 8; c < N; c += blockDim.x * 8) {
    float v[8];
    load8(src + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= scale;
    if (place != nullptr) {
      float u[8];
      load8(place + c, u);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] += u[j];
    }
    store8(x32 + row * N + c, v);
    store8(xa + row * ld_xa + c, v);
  }
}

constexpr int kMaxVec = 4;   // 8-wide vectors per thread: 8192 columns with 256 threads, 32768 with 1024

template <typename A>
__global__ void __launch_bounds__(1024) post_norm_kernel(const PostNormArgs p) {
  __shared__ float red[32];
  pdl_launch_next();
  pdl_wait_prior();
  const long long row = blockIdx.x;
  float v[kMaxVec][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kMaxVec; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c < p.N) {
      load8(p.x32 + row * p.N + c, v[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= p.alpha;
      if (p.delta != nullptr) {
        float d[8];
        load8(p.delta + row * p.N + c, d);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] += d[j];
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v[i][j] * v[i][j];
    }
  }
  const float inv_n = 1.f / static_cast<float>(p.n_true);
  float s1 = 1.f;
  if (p.gain != nullptr) s1 = *p.gain / sqrtf(block_sum(ss, red) * inv_n + p.eps);
  float s2 = 1.f;
  if (p.final_gain != nullptr) {
    float ss2 = 0.f;   // of the new row, as it is stored
#pragma unroll
    for (int i = 0; i < kMaxVec; ++i)
      if (static_cast<int>(threadIdx.x + i * blockDim.x) * 8 < p.N) {
#pragma unroll
        for (int j = 0; j < 8; ++j) ss2 += (v[i][j] * s1) * (v[i][j] * s1);
      }
    s2 = *p.final_gain / sqrtf(block_sum(ss2, red) * inv_n + p.eps);
  }
#pragma unroll
  for (int i = 0; i < kMaxVec; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c < p.N) {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= s1;
      store8(p.x32 + row * p.N + c, v[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] *= s2;
      store8(static_cast<A*>(p.xa) + row * p.N + c, v[i]);
    }
  }
}

}  // namespace

const char* embed_rows32(const int* ids, const void* table, float* x32, void* xa, int T, int N, int64_t ld_xa, float scale,
                         int vocab, const int* pos, const void* places, int n_places, bool f32, cudaStream_t stream, bool pdl) {
  if (T <= 0) return nullptr;
  if (places != nullptr && (pos == nullptr || n_places < 1)) return "embed_rows32: a position table needs the positions";
  if (N % 8 || ld_xa % 8) return "embed_rows32: row widths must be multiples of 8";
  const long long ld = ld_xa;
  cudaError_t e = f32 ? launch_kernel(embed_rows32_kernel<float>, dim3(T), dim3(256), 0, stream, pdl, 1, ids,
                                      static_cast<const float*>(table), x32, static_cast<float*>(xa), N, ld, scale, vocab, pos,
                                      static_cast<const float*>(places), n_places)
                      : launch_kernel(embed_rows32_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, pdl, 1, ids,
                                      static_cast<const __nv_bfloat16*>(table), x32, static_cast<__nv_bfloat16*>(xa), N, ld, scale, vocab,
                                      pos, static_cast<const __nv_bfloat16*>(places), n_places);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

const char* post_norm_rows(const PostNormArgs& a, cudaStream_t stream, bool pdl) {
  if (a.T <= 0) return nullptr;
  if (a.N % 8 || a.n_true <= 0 || a.n_true > a.N) return "post_norm_rows: bad row width";
  const int threads = a.N <= 256 * 8 * kMaxVec ? 256 : 1024;
  if (a.N > threads * 8 * kMaxVec) return "post_norm_rows: rows of more than 32768 columns are not supported";
  cudaError_t e = a.f32 ? launch_kernel(post_norm_kernel<float>, dim3(a.T), dim3(threads), 0, stream, pdl, 1, a)
                        : launch_kernel(post_norm_kernel<__nv_bfloat16>, dim3(a.T), dim3(threads), 0, stream, pdl, 1, a);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
