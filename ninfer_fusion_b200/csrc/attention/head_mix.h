// Attention whose scores are shaped per head and then mixed across heads before the softmax (plain C++ ABI).
//
//   c_g(i, j)  = cap * tanh(scale * q_g(i) . k_{g / (H/G)}(j) / cap)          (cap = 0: no cap)
//   s_h(i, j)  = sum_g mix[h, g] * c_g(i, j)  -  slope[h] * (i - j)            (mix = null: the identity)
//   visible    : j <= i, i - j < window (window = 0: all of the past), floor(i / chunk) = floor(j / chunk) (chunk = 0: no chunks)
//   a_h(i, j)  = exp(s_h) / (sink_one + exp(sinks[h]) + sum_j exp(s_h))        (sinks = null: without them)
//   out_h(i)   = sigmoid(gate[i, h]) * sum_j a_h(i, j) v(j)                    (gate = null: no gate)
//
// or, with `sigmoid`, weights that stand by themselves and are mixed instead of the scores:
//   w_g(i, j)  = sigmoid(scale * q_g(i) . k(j) - log_rate[g] ln(1 + log_step[g] (i - j)) + offset[g])
//   out_h(i)   = sigmoid(gate[i, h]) * sum_j (sum_g mix[h, g] w_g(i, j)) v(j)          (log_rate, offset = null: without them)
//
// `slope` is the bias AFTER mixing: a per-head bias b_g taken off before the mix is slope[h] = sum_g mix[h, g] b_g.
// Scores, weights and sums are fp32.  K and V live in paged planes [page, kv_head, token in page, width]; widths are
// multiples of 16, zero-padded by the producer.  q, k, v and out are bf16 or (f32) fp32.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#ifdef __CUDACC__
#include "../common/elem.cuh"
#endif

namespace nfb {

struct HeadMixArgs {
  const void* q = nullptr;          // [T, n_heads * dim], leading dimension ldq
  int64_t ldq = 0;
  const void* k_pages = nullptr;    // [pages, n_kv, page_size, dim]
  const void* v_pages = nullptr;    // [pages, n_kv, page_size, vdim]
  const int* block_table = nullptr; // [rows, table_ld]
  int table_ld = 0;
  const int* table_row = nullptr;   // [T]
  const int* kv_len = nullptr;      // [T] position + 1
  int T = 0;
  int n_heads = 0, n_kv = 0, dim = 0, vdim = 0, page_size = 0, window = 0, chunk = 0;
  float scale = 1.f, softcap = 0.f, sink = 0.f;   // sink: what is added to the softmax denominator (0 or 1)
  const float* sinks = nullptr;     // [H] learned scores that only count in the denominator, or null
  const float* mix = nullptr;       // [H, H] row-major, or null
  const float* slope = nullptr;     // [H], or null
  bool sigmoid = false;
  const float* log_rate = nullptr;  // [H], or null (sigmoid weights only)
  const float* log_step = nullptr;  // [H], with log_rate
  const float* offset = nullptr;    // [H], or null (sigmoid weights only)
  const float* gate = nullptr;      // [T, *] raw gate values of head h at gate[t * ld_gate + h], or null
  int64_t ld_gate = 0;
  void* out = nullptr;              // [T, n_heads * vdim], leading dimension ldo
  int64_t ldo = 0;
  bool f32 = false;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};

// One CTA per (token, split of its visible keys); a second kernel merges the splits.  part_o: fp32
// [T, n_splits, H, vdim], part_ml: fp32 [T, n_splits, H, 2]; both unused with one split.
const char* head_mix_token_attention(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml);

// The tensor-core form of the same (bf16; head_mix_token_attention picks it by itself); leaves the splits unmerged.
bool head_mix_decode_supported(const HeadMixArgs& a);
const char* head_mix_decode(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml);

// Scores that are scaled dot products and nothing else (no cap, mix, bias, gate), bf16: grouped-query attention on the tensor
// cores (group_attention.cu).  head_mix_token_attention picks the decode form by itself; it leaves the splits unmerged.
bool group_attention_supported(const HeadMixArgs& a);
const char* group_decode(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml);
// Query blocks as in head_mix_prefill.
const char* group_prefill(const HeadMixArgs& a, const int* blk_start, const int* blk_count, int n_blocks);

#ifdef __CUDACC__
// First position that the query at position len - 1 sees.
__device__ __forceinline__ int first_visible(int len, int window, int chunk) {
  int lo = window > 0 ? max(0, len - window) : 0;
  if (chunk > 0) lo = max(lo, (len - 1) / chunk * chunk);
  return lo;
}
// Numbers of one head that turn a raw score into its sigmoid weight; `fast` keeps them scaled for 2^x.
struct SigmoidHead {
  float scale, offset, rate, step;
  __device__ __forceinline__ SigmoidHead() {}
  __device__ __forceinline__ SigmoidHead(const HeadMixArgs& p, int h, bool fast) {
    const float k = fast ? -1.4426950408889634f : 1.f;
    scale = p.scale * k;
    offset = p.offset != nullptr ? p.offset[h] * k : 0.f;
    rate = p.log_rate != nullptr ? p.log_rate[h] : 0.f;
    step = p.log_rate != nullptr ? p.log_step[h] : 0.f;
  }
  // rate * log2(1 + step * d), hardware logarithm
  __device__ __forceinline__ float bias_fast(float d) const {
    float y;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(fmaf(step, fmaxf(d, 0.f), 1.f)));
    return rate * y;
  }
  __device__ __forceinline__ float weight_fast(float s, float bias) const { return rcp_fast(1.f + ex2_fast(fmaf(scale, s, offset + bias))); }
  // library functions
  __device__ __forceinline__ float weight(float s, float d) const {
    return 1.f / (1.f + expf(rate * log1pf(step * fmaxf(d, 0.f)) - fmaf(scale, s, offset)));
  }
};
// What the sum of exp(s - m) v, with m the maximum and l the sum of exp(s - m), is multiplied with.
__device__ __forceinline__ float head_mix_finish(float m, float l, float sink, const float* sinks, int h) {
  if (!(m > -3.0e38f)) return 0.f;   // no visible key
  if (sinks != nullptr) {
    const float s = sinks[h], mx = fmaxf(fmaxf(m, s), sink > 0.f ? 0.f : m);
    const float e = expf(m - mx);
    return e / (expf(s - mx) + (sink > 0.f ? sink * expf(-mx) : 0.f) + l * e);
  }
  if (sink <= 0.f) return 1.f / l;
  const float mx = fmaxf(m, 0.f);
  const float e = expf(m - mx);
  return e / (sink * expf(-mx) + l * e);
}
#endif

// bf16 prefill: query blocks of up to 64 consecutive tokens of one sequence (blk_start / blk_count, n_blocks).
// `max_keys` bounds the visible key range of a block (host).  Mixed scores pass through `scratch` (scratch_bytes) in
// register-fragment order, as many blocks at a time as fit.
const char* head_mix_prefill(const HeadMixArgs& a, const int* blk_start, const int* blk_count, int n_blocks, int max_keys,
                             void* scratch, int64_t scratch_bytes);
// Scratch for `blocks` query blocks at a time: fp32 scores, or bf16 weights (sigmoid).
int64_t head_mix_prefill_scratch(int n_heads, int max_keys, int window, int blocks, bool sigmoid);
constexpr int kHeadMixBlock = 64;

struct QkvAppendArgs {
  const void* proj = nullptr;       // [T, ldp]: q heads at q_off, k heads at k_off, v heads at v_off
  int64_t ldp = 0;
  int q_off = 0, k_off = 0, v_off = 0;
  int T = 0, n_heads = 0, n_kv = 0;
  int dim = 0, dim_true = 0, vdim = 0;     // padded q / k width, width the norm's mean runs over, padded v width
  const float* q_norm = nullptr;    // [dim] fp32 weights, or null = no norm
  const float* k_norm = nullptr;
  float eps = 0.f;
  const int* table_row = nullptr;
  const int* cache_pos = nullptr;
  const int* block_table = nullptr;
  int table_ld = 0, page_size = 0;
  const double* freq = nullptr;     // [rot / 2] rotation of neighbours (2i, 2i + 1) of the first `rot` values of q and k heads,
  int rot = 0;                      // after the norm, by position * freq[i] (angles in 64-bit); 0: none
  bool unit = false;                // q and k are normed without weights (q_norm and k_norm null)
  void* v_first = nullptr;          // [T, n_kv * vdim] values of an earlier layer: v <- (1 - lambda) v + lambda v_first, or, without a
  int64_t ld_first = 0;             // lambda, where this layer's values are left for later ones
  const float* v_lambda = nullptr;  // one number
  void* q_out = nullptr;            // [T, n_heads * dim], leading dimension ldq
  int64_t ldq = 0;
  void* k_pages = nullptr;
  void* v_pages = nullptr;
  bool f32 = false;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};
// Per-head RMS norm and rotation of q and k, k and v rows appended to their pages.
const char* qkv_append(const QkvAppendArgs& a);

}  // namespace nfb
