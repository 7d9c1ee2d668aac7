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

// a - 1 (a itself would lose what a long memory is made of: its distance from 1) and the input sqrt(1 - a^2) i u of one token
// and channel; S <- S + (a - 1) S + input.
__device__ __forceinline__ void rglru_gates(float raw_r, float raw_i, float rate, float u, float& em, float& in) {
  em = expm1f(-rate / (1.f + expf(-raw_r)));
  in = sqrtf(-em * (2.f + em)) * u / (1.f + expf(-raw_i));
}

template <typename A>
__device__ __forceinline__ float gelu_tanh_of(float z) {
  return 0.5f * z * (1.f + tanh_of<A>(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

}  // namespace nfb
