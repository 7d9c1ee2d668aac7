// The row step of decoders whose sublayers read the residual as it is and whose outputs are normed (plain C++ ABI).
#pragma once
#include "stream_rows.h"

namespace nfb {

//   y   = (rms(a) w_a + rms(b) w_b) / 2      two branches side by side, each normed by itself
//       | a sublayer's output in parts        (MixtureParts; a single GEMM's result is its delta)
//   x  <- x + rms(y) w
//   out = x                                   (w_final null)
//       | rms(x) w_final
// with rms(v) = v / sqrt(mean(v^2) + eps) over the first n_true columns.
struct BranchRowsArgs {
  float* x = nullptr;               // [T, N]
  const float* a = nullptr;         // [T, N] or null
  const float* b = nullptr;
  const float* w_a = nullptr;       // [N]
  const float* w_b = nullptr;
  MixtureParts y;                   // without branches
  const float* w = nullptr;         // [N]
  const float* w_final = nullptr;   // [N] or null
  void* out = nullptr;              // [T, N] in the activation type, leading dimension ld_out; may be y.h
  int64_t ld_out = 0;
  int T = 0, N = 0, n_true = 0;     // columns >= n_true are zero padding
  float eps = 0.f;
  bool f32 = false;
};
const char* branch_rows(const BranchRowsArgs& a, cudaStream_t stream, bool pdl);

}  // namespace nfb
