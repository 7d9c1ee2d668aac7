// Gated unit g sigmoid(slope g) (u + shift) with g = min(gate, limit), u = clamp(up, +- limit).  limit = 0: SiLU(gate) * up.
#pragma once

namespace nfb {

struct GluParams {
  float limit = 0.f, slope = 1.f, shift = 0.f;
};

#ifdef __CUDACC__
__device__ __forceinline__ float gated_unit(float g, float u, const GluParams& p) {
  if (p.limit > 0.f) {
    g = fminf(g, p.limit);
    u = fminf(fmaxf(u, -p.limit), p.limit);
    return g / (1.f + __expf(-p.slope * g)) * (u + p.shift);
  }
  return g / (1.f + __expf(-g)) * u;
}
#endif

}  // namespace nfb
