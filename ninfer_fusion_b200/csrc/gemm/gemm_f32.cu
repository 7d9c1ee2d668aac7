// 32-bit GEMM for models that run entirely in fp32 (no TF32): 64 x 64 output tiles, 16-wide K slices double-buffered
// in shared memory, a 4 x 4 register tile per thread.  It exists for exactness, not for the roofline.
#include "gemm_f32.h"

#include "gemm.h"

namespace nfb {

namespace {

constexpr int kTile = 64, kSlice = 16, kThreads = 256, kPad = 4;

__device__ __forceinline__ float act_f32(float z, int mode, const float* prm) {
  switch (mode) {
    case kActGeluTanh: return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    case kActGeluErf: return 0.5f * z * (1.f + erff(z * 0.7071067811865476f));
    case kActXielu: return z > 0.f ? (prm[0] * z + 0.5f) * z : prm[1] * (expm1f(z) - z) + 0.5f * z;
    case kActRelu2: return z > 0.f ? z * z : 0.f;
    case kActSoftcap: return prm[0] * tanhf(z * prm[1]);
    default: return z;
  }
}

__global__ void __launch_bounds__(kThreads) gemm_f32_kernel(const GemmF32Args p) {
  __shared__ __align__(16) float xs[2][kSlice][kTile + kPad];
  __shared__ __align__(16) float ws[2][kSlice][kTile + kPad];
  const int n0 = blockIdx.x * kTile, t0 = blockIdx.y * kTile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;   // each thread stages four k-values of one row
  float acc[4][4] = {};
  float rx[4], rw[4];
  auto fetch = [&](int k0) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      rx[j] = (t0 + lr < p.T && k < p.K) ? p.x[(t0 + lr) * p.ldx + k] : 0.f;
      rw[j] = (n0 + lr < p.N && k < p.K) ? p.w[(n0 + lr) * p.ldw + k] : 0.f;
    }
  };
  auto stage = [&](int b) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      xs[b][lk + j][lr] = rx[j];
      ws[b][lk + j][lr] = rw[j];
    }
  };
  fetch(0);
  stage(0);
  __syncthreads();
  int b = 0;
  for (int k0 = 0; k0 < p.K; k0 += kSlice, b ^= 1) {
    const bool more = k0 + kSlice < p.K;
    if (more) fetch(k0 + kSlice);
#pragma unroll
    for (int k = 0; k < kSlice; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[b][k][ty * 4]);
      const float4 w = *reinterpret_cast<const float4*>(&ws[b][k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, wv[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
    }
    if (more) stage(b ^ 1);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const long long t = t0 + ty * 4 + i;
    if (t >= p.T) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) break;
      const float v = act_f32(acc[i][j] + (p.bias != nullptr ? p.bias[n] : 0.f), p.act, p.act_params);
      if (p.out2 != nullptr && n >= p.out2_from) p.out2[t * p.ldo2 + n - p.out2_from] = v;
      else p.out[t * p.ldo + n] = v;
    }
  }
}

}  // namespace

const char* gemm_f32(const GemmF32Args& a) {
  if (a.T <= 0 || a.N <= 0 || a.K <= 0) return "gemm_f32: empty problem";
  if ((a.act == kActXielu || a.act == kActSoftcap) && a.act_params == nullptr) return "gemm_f32: the activation needs its two parameters";
  if (a.out == nullptr && !(a.out2 != nullptr && a.out2_from == 0)) return "gemm_f32: no output";
  const dim3 grid((a.N + kTile - 1) / kTile, (a.T + kTile - 1) / kTile);
  if (grid.y > 65535) return "gemm_f32: too many tokens";
  gemm_f32_kernel<<<grid, kThreads, 0, a.stream>>>(a);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
