// Row kernels of decoders whose residual stream is 32-bit (plain C++ ABI).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace nfb {

// x32[t] = scale * table[ids[t]] + places[pos[t]] in fp32 (places null: without it), xa[t] = the same in the activation type
// (leading dimension ld_xa); rows of N values (N % 8 == 0).  f32: the tables and xa are fp32.  pos must be below n_places.
const char* embed_rows32(const int* ids, const void* table, float* x32, void* xa, int T, int N, int64_t ld_xa, float scale,
                         int vocab, const int* pos, const void* places, int n_places, bool f32, cudaStream_t stream, bool pdl);

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

// The step between two sublayers of a decoder with norms before and after each of them:
//   x <- x + mult * norm(delta; w_post)                     (delta null: x stays)
//   h  = norm(x; w_next)                                    (w_next null: h = x)
//   out = h + sum_j conv_w[j] * h_(t - taps + 1 + j)        (conv_w null: out = h)
// norm: RMS norm of each of `groups` equal parts of the first n_true columns by itself, one weight per column.  The
// convolution looks back inside the sequence's tokens of this step and beyond them into conv_state, the last taps - 1
// values of h of every slot (oldest first), which it then replaces.
struct SandwichArgs {
  const float* x_in;        // [T, N]
  float* x_out;             // [T, N]; with a convolution and a delta it must differ from x_in unless every sequence has one token
  const float* delta;       // [T, N] or null
  const float* w_post;      // [N]
  const float* w_next;      // [N] or null
  void* out;                // [T, ld_out] in the activation type
  int64_t ld_out;
  int T, N, n_true, groups;
  float mult, eps;
  const float* conv_w;      // [taps, N] or null
  int taps;
  float* conv_state;        // [slots, taps - 1, N]
  const int* cu_seqlens;    // [n_seq + 1]   (convolution only)
  const int* state_slot;    // [n_seq]
  int n_seq, max_seq_tokens;
  bool write_state;
  bool f32;                 // out is fp32 (else bf16)
};
const char* sandwich_rows(const SandwichArgs& a, cudaStream_t stream, bool pdl);

}  // namespace nfb
