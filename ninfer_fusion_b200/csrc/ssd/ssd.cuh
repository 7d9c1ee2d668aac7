// Device functions that the state-space kernels share.
#pragma once
#include "../common/elem.cuh"
#include "ssd.h"

namespace nfb {

__device__ __forceinline__ float softplus_of(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// Stores the last inputs of the sequence's tokens t0 .. t1 - 1 for `n` convolved channels from `c0` on.
template <typename A>
__device__ __forceinline__ void ssd_keep_inputs(const SsdArgs& p, float* ring, int K, int t0, int t1, int c0, int n) {
  const A* x = static_cast<const A*>(p.proj) + p.x_off + c0;
  for (int t = max(t0, t1 - p.taps); t < t1; ++t) {
    float* row = ring + static_cast<long long>(p.cache_pos[t] % p.taps) * K + c0;
    for (int c = threadIdx.x; c < n; c += blockDim.x) row[c] = elem_to_f(x[t * p.ldp + c]);
  }
}

}  // namespace nfb
