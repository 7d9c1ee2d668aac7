// Device functions that the gated linear recurrence's kernels share.
#pragma once
#include "../common/elem.cuh"
#include "rglru.h"

namespace nfb {

const char* rglru_check(const RglruArgs& a);

// Eight channels of the convolution at token t, the i-th of its sequence in this step, at position pos; `x` is the recurrent
// branch's input of the step, `ring` the slot's earlier inputs.
template <typename A>
__device__ __forceinline__ void rglru_conv8(const RglruArgs& p, const A* x, const float* ring, int t, int i, int pos, int C, int c, float* v) {
  load8(p.conv_b + c, v);
  for (int back = p.taps - 1; back >= 0; --back) {
    if (back > pos) continue;                                   // before the start
    float in[8], w[8];
    if (back <= i) load8(x + static_cast<long long>(t - back) * p.ldp + c, in);
    else load8(ring + static_cast<long long>((pos - back) % p.taps) * C + c, in);
    load8(p.conv_w + static_cast<long long>(p.taps - 1 - back) * C + c, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = fmaf(w[j], in[j], v[j]);
  }
}

// exp(x) - 1 for x <= 0 out of the hardware 2^x, a Taylor polynomial near 0 (relative error about 1e-6)
__device__ __forceinline__ float expm1_fast(float x) {
  const float near = x * fmaf(x, fmaf(x, fmaf(x, fmaf(x, 1.f / 120.f, 1.f / 24.f), 1.f / 6.f), 0.5f), 1.f);
  return x > -0.125f ? near : ex2_fast(x * kLog2e) - 1.f;
}

// a - 1 (a itself would lose what a long memory is made of: its distance from 1) and the input sqrt(1 - a^2) i u of one token
// and channel; S <- S + (a - 1) S + input.
template <typename A>
__device__ __forceinline__ void rglru_gates(float raw_r, float raw_i, float rate, float u, float& em, float& in) {
  if constexpr (sizeof(A) == 4) {
    em = expm1f(-rate / (1.f + expf(-raw_r)));
    in = sqrtf(-em * (2.f + em)) * u / (1.f + expf(-raw_i));
  } else {
    em = expm1_fast(-rate * rcp_fast(1.f + ex2_fast(-raw_r * kLog2e)));
    const float v = -em * (2.f + em);
    in = (v > 0.f ? v * rsqrtf(v) : 0.f) * u * rcp_fast(1.f + ex2_fast(-raw_i * kLog2e));
  }
}

template <typename A>
__device__ __forceinline__ float gelu_tanh_of(float z) {
  return 0.5f * z * (1.f + tanh_of<A>(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

}  // namespace nfb
