// Latent attention (plain C++ ABI): queries, keys and values come out of low-rank latents.  One cached row per token,
// [latent c (rank) | rotated key part (rot)], shared by all heads.  With U_k, U_v the per-head expansions of c:
//   s_h(i, j) = scale * ( q_h(i) . U_k,h c(j)  +  rotate(r_h(i)) . k_rot(j) ),   j <= i and (window > 0) i - j < window
//   a_h(i, j) = exp(s_h) / ( exp(sink_h) + sum_j exp(s_h) )                       (sink = null: without it)
//   out_h(i)  = U_v,h sum_j a_h(i, j) c(j)
// Two forms.  Absorbed: the query is taken to the latent space (q' = U_k,h^T q_h) and the sum over c is expanded
// afterwards, so a row is read once for all heads: decode and short portions.  Expanded: keys and values of all visible
// positions are made by one GEMM and attended as ordinary heads: long portions, a third of the multiply-adds at the usual
// widths.  Rotation: neighbours (2i, 2i + 1) by position * freq[i], angles in 64-bit.
// A query without rotated part (rot = 0) needs no freq.  Scores, weights and sums are fp32.  Widths are multiples of 16, zero-padded by the producer.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "rotary.cuh"

namespace nfb {

struct LatentPrepArgs {
  // [T, ldp]: query latent (q_rank; 0: none, the queries are not this kernel's) at column 0; at kv_off key / value latent (rank)
  // | key part to rotate (rot)
  const void* proj = nullptr;
  int64_t ldp = 0;
  int kv_off = 0;
  int T = 0;
  int q_rank = 0, q_rank_true = 0, rank = 0, rank_true = 0, rot = 0, rot_true = 0;
  const float* q_norm = nullptr;    // [q_rank]
  const float* kv_norm = nullptr;   // [rank]
  float eps = 0.f;
  const double* freq = nullptr;     // [rot_true / 2]
  const int* table_row = nullptr;
  const int* cache_pos = nullptr;
  const int* block_table = nullptr;
  int table_ld = 0, page_size = 0;
  void* q_latent = nullptr;         // [T, ldq]
  int64_t ldq = 0;
  void* pages = nullptr;            // [pages, page_size, rank + rot]
  bool f32 = false;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};
// Norms of both latents, rotation of the shared key part, append of the row to its page.
const char* latent_prep(const LatentPrepArgs& a);

struct LatentArgs {
  const void* q_latent = nullptr;   // [T, n_heads * rank] absorbed queries, leading dimension ldl (absorbed form)
  int64_t ldl = 0;
  const void* q = nullptr;          // [T, n_heads * (dim + rot)]: unrotated | part to rotate, leading dimension ldq
  int64_t ldq = 0;
  const void* pages = nullptr;      // [pages, page_size, rank + rot]
  const int* block_table = nullptr; // [rows, table_ld]
  int table_ld = 0;
  const int* table_row = nullptr;   // [T]
  const int* kv_len = nullptr;      // [T] position + 1
  int T = 0;
  int n_heads = 0, dim = 0, rank = 0, rot = 0, rot_true = 0, page_size = 0, window = 0;
  float scale = 1.f;
  const double* freq = nullptr;
  const float* sink = nullptr;      // [H] or null
  void* out = nullptr;              // absorbed: [T, n_heads * rank], leading dimension ldo
  int64_t ldo = 0;
  bool f32 = false;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};

// Absorbed, one CTA per (token, head), on the FP32 pipes: the 32-bit runs.
const char* latent_token_attention(const LatentArgs& a);

// Absorbed, bf16 tensor cores.  Query blocks (blk_start / blk_count: consecutive tokens of one sequence, at most
// kLatentBlock); rows of the MMA are (token, head) pairs.  Blocks of sequences that bring `max_tokens` or more tokens in
// this step are left out (cu_seqlens / token_seq tell; 0: none are).  n_splits > 1: partial sums go to part_o fp32
// [T * H, n_splits, rank] and part_ml [T * H, n_splits, 2] and are merged by a second kernel.
constexpr int kLatentBlock = 64;
struct LatentBlocks {
  const int* start = nullptr;
  const int* count = nullptr;
  int n = 0, max_count = 1;
  const int* token_seq = nullptr;   // [T]
  const int* cu_seqlens = nullptr;
  int max_tokens = 0;
};
bool latent_absorbed_supported(int rank, int rot);
const char* latent_absorbed_attention(const LatentArgs& a, const LatentBlocks& b, int split_keys, int n_splits, float* part_o,
                                      float* part_ml);

// Expanded, bf16 tensor cores, for the sequences the absorbed form leaves out.  latent_gather fills `rows`; the caller makes
// `kv` from their latents (one GEMM); then latent_expanded_attention writes out [T, n_heads * vdim] of those sequences.
struct LatentExpand {
  const int* seqs = nullptr;      // [n_seqs, 4]: block-table row, first row in `rows`, first position, positions
  int n_seqs = 0, max_len = 0;    // max_len: most positions of a sequence
  const int* seq_base = nullptr;  // [sequences of the step, 2]: first row in `rows` (-1: not expanded), its position
  void* rows = nullptr;           // [total, rank + rot]
  const void* kv = nullptr;       // [total, n_heads * (dim + vdim)]: keys of all heads, values of all heads
  int vdim = 0;
};
bool latent_expanded_supported(int dim, int rot, int vdim);
const char* latent_gather(const LatentArgs& a, const LatentExpand& x);
const char* latent_expanded_attention(const LatentArgs& a, const LatentBlocks& b, const LatentExpand& x);

#ifdef __CUDACC__
__device__ __forceinline__ int latent_first(int len, int window) { return window > 0 ? max(0, len - window) : 0; }
#endif

}  // namespace nfb
