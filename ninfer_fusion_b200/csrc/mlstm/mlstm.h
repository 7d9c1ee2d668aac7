// Matrix memory with exponential gating (mLSTM), plain C++ ABI.  Per sequence and head, from zero:
//   i = cap tanh(i_raw / cap),  f = logsigmoid(cap tanh(f_raw / cap))
//   m_t = max(f + m_{t-1}, i)
//   S_t = exp(f + m_{t-1} - m_t) S_{t-1} + exp(i - m_t) k v^T        n_t likewise with k alone
//   o_t = S_t^T q' / (max(|n_t . q'|, exp(-m_t)) + 1e-6),  q' = q * q_scale
//   out = o_t / rms(o_t) * norm * sigmoid(gate)                       (rms over the head's own columns)
// State: S fp32 [slots, H, dim, vdim], n fp32 [slots, H, dim], m fp32 [slots, H].  Head widths are multiples of 16,
// zero-padded by the producer; the mean of the head norm runs over vdim_true columns.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace nfb {

struct MlstmArgs {
  const void* proj = nullptr;     // [T, ldp]: q, k heads of `dim`, v and output-gate heads of `vdim`
  int64_t ldp = 0;
  int q_off = 0, k_off = 0, v_off = 0, g_off = 0;
  const float* gates = nullptr;   // fp32 [T, ldg]: raw input gates at i_off, raw forget gates at f_off (biases added)
  int64_t ldg = 0;
  int i_off = 0, f_off = 0;
  int n_heads = 0, dim = 0, vdim = 0, vdim_true = 0;
  float q_scale = 1.f, gate_cap = 1.f, eps = 0.f;
  const float* norm = nullptr;    // fp32 [H * vdim]
  const int* cu_seqlens = nullptr;
  const int* state_slot = nullptr;
  int T = 0, n_seq = 0;
  float* S = nullptr;
  float* n = nullptr;
  float* m = nullptr;
  void* out = nullptr;            // [T, H * vdim], leading dimension ldo
  int64_t ldo = 0;
  bool write_state = true;
  bool one_token = false;         // every sequence brings exactly one token
  bool f32 = false;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};

// Token by token with the state in registers: decode, short portions, and every length in 32-bit.
const char* mlstm_recurrent(const MlstmArgs& a);

// bf16 portions: chunks of 64 tokens on the tensor cores, state carried in fp32 (bf16 hi + lo operand pairs).
constexpr int kMlstmChunk = 64;
int64_t mlstm_chunked_workspace_bytes(int T, int n_seq, int n_heads, int dim, int vdim);
bool mlstm_chunked_supported(int dim, int vdim);
const char* mlstm_chunked(const MlstmArgs& a, void* workspace, int64_t workspace_bytes);

}  // namespace nfb
