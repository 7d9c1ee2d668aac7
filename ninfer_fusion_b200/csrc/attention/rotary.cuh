// Rotary positions whose angles are reduced in 64-bit.
#pragma once

namespace nfb {

#ifdef __CUDACC__
// cos and sin of pos * freq.
__device__ __forceinline__ void rotary_angle(int pos, double freq, float& c, float& s) {
  const double turn = static_cast<double>(pos) * freq * 0.15915494309189535;   // 1 / (2 pi)
  sincospif(static_cast<float>(2.0 * (turn - rint(turn))), &s, &c);
}
#endif

}  // namespace nfb
