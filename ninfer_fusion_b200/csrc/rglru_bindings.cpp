// torch.ops.nfb200.rglru_*: gated linear recurrence (layer-list decoders, models/layered.py).  Activations are bf16 or fp32; every
// op takes its element type from its tensors.
#include "binding_util.h"
#include "rglru/rglru.h"

namespace {

using namespace nfb_bind;

nfb::RglruArgs rglru_args(const Tensor& proj, int64_t blocks, const Tensor& conv_w, const Tensor& conv_b, const Tensor& cu_seqlens,
                          const Tensor& token_seq, const Tensor& cache_pos, const Tensor& state_slot, const Tensor& ring) {
  nfb::RglruArgs a;
  a.f32 = act_f32(proj, "proj");
  need_rows(proj, "proj"); need(ring, at::kFloat, "ring"); need(conv_w, at::kFloat, "conv_w");
  TORCH_CHECK(conv_w.dim() == 2 && conv_w.is_contiguous() && ring.dim() == 3 && ring.is_contiguous(), "rglru: conv_w [taps, C], ring [slots, taps, C]");
  const int64_t T = proj.size(0), C = conv_w.size(1), B = state_slot.numel();
  TORCH_CHECK(blocks > 0 && C % blocks == 0 && proj.size(1) >= 2 * C && ring.size(1) == conv_w.size(0) && ring.size(2) == C, "rglru: shapes");
  need_vec(conv_b, at::kFloat, C, "conv_b");
  need_vec(cu_seqlens, at::kInt, B + 1, "cu_seqlens"); need_vec(token_seq, at::kInt, T, "token_seq");
  need_vec(cache_pos, at::kInt, T, "cache_pos"); need_vec(state_slot, at::kInt, B, "state_slot");
  a.proj = proj.data_ptr(); a.ldp = proj.stride(0); a.T = static_cast<int>(T); a.blocks = static_cast<int>(blocks);
  a.width = static_cast<int>(C / blocks); a.taps = static_cast<int>(conv_w.size(0));
  a.conv_w = static_cast<const float*>(conv_w.data_ptr()); a.conv_b = static_cast<const float*>(conv_b.data_ptr());
  a.cu_seqlens = static_cast<const int*>(cu_seqlens.data_ptr()); a.token_seq = static_cast<const int*>(token_seq.data_ptr());
  a.cache_pos = static_cast<const int*>(cache_pos.data_ptr()); a.state_slot = static_cast<const int*>(state_slot.data_ptr());
  a.n_seq = static_cast<int>(B); a.ring = static_cast<float*>(ring.data_ptr());
  a.stream = cur_stream();
  return a;
}

void out_and_state(nfb::RglruArgs& a, const Tensor& proj, const Tensor& rate, const Tensor& S, const Tensor& out, bool write_state) {
  const int64_t C = static_cast<int64_t>(a.blocks) * a.width;
  need_vec(rate, at::kFloat, C, "rate"); need(S, at::kFloat, "S"); need(out, proj.scalar_type(), "out"); need_rows(out, "out");
  TORCH_CHECK(S.dim() == 2 && S.is_contiguous() && S.size(1) == C && out.size(0) == a.T && out.size(1) == C, "rglru: state / out shape");
  a.rate = static_cast<const float*>(rate.data_ptr()); a.S = static_cast<float*>(S.data_ptr());
  a.out = out.data_ptr(); a.ldo = out.stride(0); a.write_state = write_state;
}

void rglru_conv(const Tensor& proj, int64_t blocks, const Tensor& conv_w, const Tensor& conv_b, const Tensor& cu_seqlens,
                const Tensor& token_seq, const Tensor& cache_pos, const Tensor& state_slot, const Tensor& ring, const Tensor& u, bool pdl) {
  c10::cuda::CUDAGuard guard(proj.device());
  nfb::RglruArgs a = rglru_args(proj, blocks, conv_w, conv_b, cu_seqlens, token_seq, cache_pos, state_slot, ring);
  need_vec(u, proj.scalar_type(), static_cast<int64_t>(a.T) * a.blocks * a.width, "u");
  a.ldo = 8; a.pdl = pdl;
  chk(nfb::rglru_conv(a, u.data_ptr()));
}

void rglru_scan(const Tensor& proj, int64_t blocks, const Tensor& conv_w, const Tensor& conv_b, const Tensor& cu_seqlens,
                const Tensor& token_seq, const Tensor& cache_pos, const Tensor& state_slot, const Tensor& ring, const Tensor& u,
                const Tensor& raw, const Tensor& rate, const Tensor& S, const Tensor& out, bool write_state, bool pdl) {
  c10::cuda::CUDAGuard guard(proj.device());
  nfb::RglruArgs a = rglru_args(proj, blocks, conv_w, conv_b, cu_seqlens, token_seq, cache_pos, state_slot, ring);
  const int64_t n = static_cast<int64_t>(a.T) * a.blocks * a.width;
  need_vec(u, proj.scalar_type(), n, "u"); need_vec(raw, at::kFloat, 2 * n, "raw");
  out_and_state(a, proj, rate, S, out, write_state);
  a.pdl = pdl;
  chk(nfb::rglru_scan(a, u.data_ptr(), static_cast<const float*>(raw.data_ptr())));
}

// Convolution, gates and recurrence: one token per sequence without a workspace, portions in query blocks with one.
void rglru(const Tensor& proj, int64_t blocks, const Tensor& conv_w, const Tensor& conv_b, const Tensor& cu_seqlens,
           const Tensor& token_seq, const Tensor& cache_pos, const Tensor& state_slot, const Tensor& ring, const Tensor& gate_w,
           const Tensor& gate_b, const Tensor& rate, const Tensor& S, const Tensor& out, const Tensor& blk_start, const Tensor& blk_count,
           OptT workspace, bool write_state, bool pdl) {
  c10::cuda::CUDAGuard guard(proj.device());
  nfb::RglruArgs a = rglru_args(proj, blocks, conv_w, conv_b, cu_seqlens, token_seq, cache_pos, state_slot, ring);
  need(gate_w, at::kBFloat16, "gate_w");
  TORCH_CHECK(gate_w.is_contiguous() && gate_w.numel() == blocks * 2 * a.width * a.width, "rglru: gate_w must be [blocks, 2 width, width]");
  need_vec(gate_b, at::kFloat, blocks * 2 * a.width, "gate_b");
  a.gate_w = gate_w.data_ptr(); a.gate_b = static_cast<const float*>(gate_b.data_ptr());
  out_and_state(a, proj, rate, S, out, write_state);
  a.pdl = pdl;
  if (!(workspace.has_value() && workspace->defined())) {
    chk(nfb::rglru_decode(a));
    return;
  }
  const int64_t nb = blk_start.numel();
  need_vec(blk_start, at::kInt, nb, "blk_start"); need_vec(blk_count, at::kInt, nb, "blk_count"); need_cuda(*workspace, "workspace");
  TORCH_CHECK(workspace->is_contiguous(), "workspace must be contiguous");
  chk(nfb::rglru_chunked(a, static_cast<const int*>(blk_start.data_ptr()), static_cast<const int*>(blk_count.data_ptr()), static_cast<int>(nb),
                         workspace->data_ptr(), workspace->numel() * workspace->element_size()));
}
bool rglru_fused_supported(int64_t width) { return nfb::rglru_fused_supported(static_cast<int>(width)); }
int64_t rglru_chunked_workspace_bytes(int64_t T, int64_t n_seq, int64_t channels) {
  return nfb::rglru_chunked_workspace_bytes(static_cast<int>(T), static_cast<int>(n_seq), static_cast<int>(channels));
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("rglru_conv(Tensor proj, int blocks, Tensor conv_w, Tensor conv_b, Tensor cu_seqlens, Tensor token_seq, Tensor cache_pos, Tensor state_slot, Tensor ring, Tensor u, bool pdl) -> ()", &rglru_conv);
  m.def("rglru_scan(Tensor proj, int blocks, Tensor conv_w, Tensor conv_b, Tensor cu_seqlens, Tensor token_seq, Tensor cache_pos, Tensor state_slot, Tensor ring, Tensor u, Tensor raw, Tensor rate, Tensor S, Tensor out, bool write_state, bool pdl) -> ()", &rglru_scan);
  m.def("rglru(Tensor proj, int blocks, Tensor conv_w, Tensor conv_b, Tensor cu_seqlens, Tensor token_seq, Tensor cache_pos, Tensor state_slot, Tensor ring, Tensor gate_w, Tensor gate_b, Tensor rate, Tensor S, Tensor out, Tensor blk_start, Tensor blk_count, Tensor? workspace, bool write_state, bool pdl) -> ()", &rglru);
  m.def("rglru_fused_supported(int width) -> bool", &rglru_fused_supported);
  m.def("rglru_chunked_workspace_bytes(int T, int n_seq, int channels) -> int", &rglru_chunked_workspace_bytes);
}
