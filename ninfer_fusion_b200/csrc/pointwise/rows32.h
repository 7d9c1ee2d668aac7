// Row kernels of decoders whose residual stream is 32-bit (plain C++ ABI).
#pragma once
#include <cuda_runtime.h>

namespace nfb {

// x32[t] = fp32(table[ids[t]]), xa[t] = table[ids[t]]; rows of N values (N % 8 == 0).  f32: table and xa are fp32.
const char* embed_rows32(const int* ids, const void* table, float* x32, void* xa, int T, int N, int vocab, bool f32,
                         cudaStream_t stream, bool pdl);

struct PostNormArgs {
  float* x32;            // [T, N] residual stream, updated in place
  const float* delta;    // [T, N] output of the sublayer, or null
  void* xa;              // [T, N] copy of the new row in the activation type (the next GEMM's operand)
  int T, N;              // N % 8 == 0; columns >= n_true are zero padding
  int n_true;
  float alpha, eps;
  const float* gain;     // one number for all columns; null = no norm (xa is then only the copy)
  const float* final_gain;  // optional: xa = rms_norm(new row) * final_gain instead of the row itself
  bool f32;              // xa is fp32 (else bf16)
};
// y = alpha * x + delta;  x = y / sqrt(mean(y^2) + eps) * gain
const char* post_norm_rows(const PostNormArgs& a, cudaStream_t stream, bool pdl);

}  // namespace nfb
