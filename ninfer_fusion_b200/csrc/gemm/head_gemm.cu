// Per-head GEMM of decode-sized steps: 64 tokens x 64 columns of one head per CTA, K in slices of 64 through a cp.async
// ring.  A warp owns 16 columns for all four token tiles; tiles past the last token are skipped.
#include "head_gemm.h"

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;
constexpr int kT = 64, kN = 64, kK = 64, kStages = 3, kThreads = 128, kLd = kK + 8;

__global__ void __launch_bounds__(kThreads) head_gemm_kernel(const HeadGemmArgs p) {
  extern __shared__ __align__(16) bf16 smem[];   // [kStages][kT + kN][kLd]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n0 = blockIdx.x * kN, h = blockIdx.y, t0 = blockIdx.z * kT;
  const int n_tok = min(kT, p.T - t0);
  if (p.max_tokens > 0) {     // (written before the step's first kernel: no need to wait)
    const int seq = p.token_seq[t0];
    if (seq == p.token_seq[t0 + n_tok - 1] && p.cu_seqlens[seq + 1] - p.cu_seqlens[seq] >= p.max_tokens) {
      pdl_launch_next();
      pdl_wait_prior();
      return;
    }
  }
  const int n_slices = (p.K + kK - 1) / kK;
  const bf16* w = static_cast<const bf16*>(p.w) + (static_cast<long long>(h) * p.N + n0) * p.K;
  const bf16* x = static_cast<const bf16*>(p.x) + t0 * p.ldx + static_cast<long long>(h) * p.x_step;
  const uint32_t base = smem_u32(smem);
  auto load_w = [&](int s) {
    const uint32_t dst = base + ((s % kStages) * (kT + kN) + kT) * kLd * 2;
    for (int i = tid; i < kN * (kK / 8); i += kThreads) {
      const int r = i / (kK / 8), c = (i % (kK / 8)) * 8;
      const bool ok = n0 + r < p.N && s * kK + c < p.K;
      cp_async16(dst + (r * kLd + c) * 2, ok ? w + static_cast<long long>(r) * p.K + s * kK + c : w, ok);
    }
  };
  auto load_x = [&](int s) {
    const uint32_t dst = base + (s % kStages) * (kT + kN) * kLd * 2;
    for (int i = tid; i < kT * (kK / 8); i += kThreads) {
      const int r = i / (kK / 8), c = (i % (kK / 8)) * 8;
      const bool ok = r < n_tok && s * kK + c < p.K;
      cp_async16(dst + (r * kLd + c) * 2, ok ? x + r * p.ldx + s * kK + c : x, ok);
    }
  };
  pdl_launch_next();
  // the weights do not depend on the kernel before
#pragma unroll
  for (int s = 0; s < kStages - 1; ++s)
    if (s < n_slices) load_w(s);
  pdl_wait_prior();
#pragma unroll
  for (int s = 0; s < kStages - 1; ++s) {
    if (s < n_slices) load_x(s);
    cp_async_commit();
  }
  float acc[kT / 16][2][4];
#pragma unroll
  for (int m = 0; m < kT / 16; ++m)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][n][e] = 0.f;
  for (int s = 0; s < n_slices; ++s) {
    cp_async_wait<kStages - 2>();
    __syncthreads();
    if (s + kStages - 1 < n_slices) {
      load_w(s + kStages - 1);
      load_x(s + kStages - 1);
    }
    cp_async_commit();
    const uint32_t xs = base + (s % kStages) * (kT + kN) * kLd * 2, wsm = xs + kT * kLd * 2;
#pragma unroll
    for (int kk = 0; kk < kK; kk += 16) {
      uint32_t b[4];
      ldsm_x4(wsm + ((warp * 16 + (lane & 7) + (lane >> 4) * 8) * kLd + kk + ((lane >> 3) & 1) * 8) * 2, b);
#pragma unroll
      for (int m = 0; m < kT / 16; ++m) {
        if (m * 16 < n_tok) {
          uint32_t a[4];
          ldsm_x4(xs + ((m * 16 + (lane & 15)) * kLd + kk + (lane >> 4) * 8) * 2, a);
          mma_bf16_16816(acc[m][0], a, b[0], b[1]);
          mma_bf16_16816(acc[m][1], a, b[2], b[3]);
        }
      }
    }
  }
  cp_async_wait<0>();
  bf16* out = static_cast<bf16*>(p.out) + t0 * p.ldo + static_cast<long long>(h) * p.N + n0 + warp * 16;
#pragma unroll
  for (int m = 0; m < kT / 16; ++m)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = m * 16 + (lane >> 2) + r * 8, c = n * 8 + (lane & 3) * 2;
        if (t < n_tok && n0 + warp * 16 + c < p.N)
          *reinterpret_cast<uint32_t*>(out + t * p.ldo + c) = pack_bf16x2(acc[m][n][2 * r], acc[m][n][2 * r + 1]);
      }
}

}  // namespace

const char* head_gemm(const HeadGemmArgs& a) {
  if (a.T <= 0) return nullptr;
  if (a.N % 2 || a.K % 8 || a.ldx % 8 || a.x_step % 8 || a.ldo % 2 || a.H < 1 || a.H > 65535 || a.N < 1 || a.K < 8)
    return "head_gemm: misaligned rows or widths";
  const dim3 grid((a.N + kN - 1) / kN, a.H, (a.T + kT - 1) / kT);
  if (grid.z > 65535) return "head_gemm: too many tokens";
  constexpr int smem = kStages * (kT + kN) * kLd * 2;
  cudaError_t e = cudaFuncSetAttribute(head_gemm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e == cudaSuccess) e = launch_kernel(head_gemm_kernel, grid, dim3(kThreads), smem, a.stream, a.pdl, 1, a);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
