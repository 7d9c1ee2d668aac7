// Gated linear memory with a forget gate per head and channel (HGRN2), plain C++ ABI.  Per sequence and head, from zero:
//   f_t = l + (1 - l) sigmoid(raw_t),   k_t = 1 - f_t = (1 - l) sigmoid(-raw_t)
//   S_t = diag(f_t) S_{t-1} + k_t v_t^T,   o_t = S_t^T silu(q_t)
//   out = o_t / rms(o_t) * norm                        (rms over the head's own columns)
// State: S fp32 [slots, H, dim, vdim].  Head widths are multiples of 16, zero-padded by the producer (padded channels
// have l = 1, so their rows stay zero); the mean of the head norm runs over vdim_true columns.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace nfb {

struct GatedArgs {
  const void* proj = nullptr;     // [T, ldp]: raw q heads of `dim` at q_off, v heads of `vdim` at v_off
  int64_t ldp = 0;
  int q_off = 0, v_off = 0;
  const float* gates = nullptr;   // fp32 [T, ldg]: raw forget gates (bias added), column h * dim + d
  int64_t ldg = 0;
  const float* lower = nullptr;   // fp32 [H * dim]
  int n_heads = 0, dim = 0, vdim = 0, vdim_true = 0;
  float eps = 0.f;
  const float* norm = nullptr;    // fp32 [vdim]
  const int* cu_seqlens = nullptr;
  const int* state_slot = nullptr;
  int T = 0, n_seq = 0;
  float* S = nullptr;
  void* out = nullptr;            // [T, H * vdim], leading dimension ldo
  int64_t ldo = 0;
  bool write_state = true;
  bool one_token = false;         // every sequence brings exactly one token
  bool f32 = false;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};

// Token by token with the state in registers: decode, short portions, and every length in 32-bit.
const char* gated_recurrent(const GatedArgs& a);

// bf16 portions: chunks of 64 tokens on the tensor cores, state carried in fp32 (bf16 hi + lo operand pairs).
constexpr int kGatedChunk = 64;
int64_t gated_chunked_workspace_bytes(int T, int n_seq, int n_heads, int dim, int vdim);
bool gated_chunked_supported(int dim, int vdim);
const char* gated_chunked(const GatedArgs& a, void* workspace, int64_t workspace_bytes);

#ifdef __CUDACC__
// Forget gate and its complement, each without cancellation.
__device__ __forceinline__ void gated_forget(float raw, float lower, float& f, float& k) {
  const float e = expf(-fabsf(raw));
  const float big = 1.f / (1.f + e), small = e / (1.f + e);   // sigmoid(|raw|), sigmoid(-|raw|)
  const float r = 1.f - lower;
  f = fmaf(r, raw >= 0.f ? big : small, lower);
  k = r * (raw >= 0.f ? small : big);
}
#endif

}  // namespace nfb
