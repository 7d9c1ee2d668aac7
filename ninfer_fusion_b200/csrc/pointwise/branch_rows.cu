// x <- x + norm(y), where y is a sublayer's output: a GEMM's result, the weighted sum over a token's experts, or the mean of
// two branches that are normed first.  One CTA per row; the row and the parts of y stay in registers between the norms, so
// everything is read once.
#include "branch_rows.h"

#include "../common/launch.h"
#include "mixture.cuh"

namespace nfb {

namespace {

// Sums over the CTA (at most 16 warps); `red` alternates between the two halves of one array from call to call.
template <int NS>
__device__ __forceinline__ void block_sums(float (&v)[NS], float (*red)[16]) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    v[i] = warp_sum(v[i]);
    if (lane == 0) red[i][warp] = v[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    v[i] = 0.f;
    for (int w = 0; w < nw; ++w) v[i] += red[i][w];
  }
}

// KV: four-column pieces per thread; PAIR: two branches.
template <typename A, int KV, bool PAIR>
__global__ void __launch_bounds__(512, KV <= 4 ? 2 : 1) branch_rows_kernel(const BranchRowsArgs p) {
  __shared__ float red[2][2][16];
  const int tid = threadIdx.x, nt = blockDim.x, N = p.N;
  // the weights come ahead of the rows when there are registers for them
  constexpr bool kAhead = KV <= 2;
  float w[kAhead ? KV : 1][4], wa[PAIR && kAhead ? KV : 1][4], wb[PAIR && kAhead ? KV : 1][4];
  if constexpr (kAhead) {
#pragma unroll
    for (int i = 0; i < KV; ++i) {
      const int c = (tid + i * nt) * 4;
      if (c < N) {
        load4(p.w + c, w[i]);
        if constexpr (PAIR) {
          load4(p.w_a + c, wa[i]);
          load4(p.w_b + c, wb[i]);
        }
      }
    }
  }
  pdl_launch_next();
  pdl_wait_prior();
  const long long t = blockIdx.x;
  const float inv_n = 1.f / static_cast<float>(p.n_true);
  float x[KV][4], y[KV][4], s1[1] = {0.f};
  if constexpr (PAIR) {
    float v[KV][4], s[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < KV; ++i) {
      const int c = (tid + i * nt) * 4;
      if (c < N) {
        load4(p.a + t * N + c, y[i]);
        load4(p.b + t * N + c, v[i]);
        load4(p.x + t * N + c, x[i]);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[0] = fmaf(y[i][e], y[i][e], s[0]);
          s[1] = fmaf(v[i][e], v[i][e], s[1]);
        }
      }
    }
    block_sums<2>(s, red[1]);
    const float ia = 0.5f / sqrtf(s[0] * inv_n + p.eps), ib = 0.5f / sqrtf(s[1] * inv_n + p.eps);
#pragma unroll
    for (int i = 0; i < KV; ++i) {
      const int c = (tid + i * nt) * 4, k = kAhead ? i : 0;
      if (c < N) {
        if constexpr (!kAhead) {
          load4(p.w_a + c, wa[0]);
          load4(p.w_b + c, wb[0]);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          y[i][e] = y[i][e] * ia * wa[k][e] + v[i][e] * ib * wb[k][e];
          s1[0] = fmaf(y[i][e], y[i][e], s1[0]);
        }
      }
    }
  } else {
    const float g = mixture_gate(p.y, t);
#pragma unroll
    for (int i = 0; i < KV; ++i) {
      const int c = (tid + i * nt) * 4;
      if (c < N) {
        load4(p.x + t * N + c, x[i]);
        mixture4<A>(p.y, t, c, N, g, y[i]);
#pragma unroll
        for (int e = 0; e < 4; ++e) s1[0] = fmaf(y[i][e], y[i][e], s1[0]);
      }
    }
  }
  block_sums<1>(s1, red[0]);
  const float inv = 1.f / sqrtf(s1[0] * inv_n + p.eps);
  float s2[1] = {0.f};
#pragma unroll
  for (int i = 0; i < KV; ++i) {
    const int c = (tid + i * nt) * 4, k = kAhead ? i : 0;
    if (c < N) {
      if constexpr (!kAhead) load4(p.w + c, w[0]);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        x[i][e] = fmaf(y[i][e] * inv, w[k][e], x[i][e]);
        s2[0] = fmaf(x[i][e], x[i][e], s2[0]);
      }
      store4(p.x + t * N + c, x[i]);
    }
  }
  float f = 1.f;
  if (p.w_final != nullptr) {
    block_sums<1>(s2, red[1]);
    f = 1.f / sqrtf(s2[0] * inv_n + p.eps);
  }
#pragma unroll
  for (int i = 0; i < KV; ++i) {
    const int c = (tid + i * nt) * 4;
    if (c < N) {
      if (p.w_final != nullptr) {
        float u[4];
        load4(p.w_final + c, u);
#pragma unroll
        for (int e = 0; e < 4; ++e) x[i][e] = x[i][e] * f * u[e];
      }
      store4(static_cast<A*>(p.out) + t * p.ld_out + c, x[i]);
    }
  }
}

template <typename A, bool PAIR>
cudaError_t pick_width(const BranchRowsArgs& a, cudaStream_t stream, bool pdl) {
  const int pieces = a.N / 4;
  auto threads = [&](int kv) { return dim3(((pieces + kv - 1) / kv + 31) / 32 * 32); };
  if (a.T >= 512 && pieces > 256) {       // many rows: small CTAs, several of them per SM between each other's barriers
    if (pieces <= 512) return launch_kernel(branch_rows_kernel<A, 2, PAIR>, dim3(a.T), threads(2), 0, stream, pdl, 1, a);
    if (pieces <= 1024) return launch_kernel(branch_rows_kernel<A, 4, PAIR>, dim3(a.T), threads(4), 0, stream, pdl, 1, a);
  }
  if (pieces <= 512) return launch_kernel(branch_rows_kernel<A, 1, PAIR>, dim3(a.T), threads(1), 0, stream, pdl, 1, a);
  if (pieces <= 1024) return launch_kernel(branch_rows_kernel<A, 2, PAIR>, dim3(a.T), threads(2), 0, stream, pdl, 1, a);
  if (pieces <= 2048) return launch_kernel(branch_rows_kernel<A, 4, PAIR>, dim3(a.T), threads(4), 0, stream, pdl, 1, a);
  return launch_kernel(branch_rows_kernel<A, 8, PAIR>, dim3(a.T), threads(8), 0, stream, pdl, 1, a);
}

}  // namespace

const char* branch_rows(const BranchRowsArgs& a, cudaStream_t stream, bool pdl) {
  if (a.T <= 0) return nullptr;
  if (a.N % 8 || a.ld_out % 8 || a.n_true <= 0 || a.n_true > a.N || a.N > 16384) return "branch_rows: bad row width (up to 16384 columns)";
  if (a.x == nullptr || a.w == nullptr || a.out == nullptr) return "branch_rows: missing rows or weights";
  const bool pair = a.a != nullptr;
  if (pair && (a.b == nullptr || a.w_a == nullptr || a.w_b == nullptr)) return "branch_rows: two branches need two rows and two weights";
  if (!pair) {
    if (a.y.delta == nullptr && a.y.choice == nullptr) return "branch_rows: no sublayer output";
    if (const char* err = bad_mixture(a.y)) return err;
  }
  cudaError_t e;
  if (pair) e = a.f32 ? pick_width<float, true>(a, stream, pdl) : pick_width<__nv_bfloat16, true>(a, stream, pdl);
  else e = a.f32 ? pick_width<float, false>(a, stream, pdl) : pick_width<__nv_bfloat16, false>(a, stream, pdl);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
