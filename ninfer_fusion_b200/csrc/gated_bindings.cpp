// torch.ops.nfb200.*: gated linear memory (layer-list decoders, models/layered.py).  Activations are bf16 or fp32; every op takes
// its element type from its tensors.
#include "binding_util.h"
#include "gated/gated.h"

namespace {

using namespace nfb_bind;

void gated_memory(const Tensor& proj, int64_t q_off, int64_t v_off, const Tensor& gates, const Tensor& lower, int64_t vdim_true,
                  double eps, const Tensor& norm, const Tensor& cu_seqlens, const Tensor& state_slot, const Tensor& S,
                  const Tensor& out, bool write_state, OptT chunk_ws, bool pdl, bool one_token) {
  nfb::GatedArgs a;
  a.f32 = act_f32(proj, "proj");
  need_rows(proj, "proj"); need_rows(out, "out"); need(out, proj.scalar_type(), "out");
  need(gates, at::kFloat, "gates"); need_rows(gates, "gates"); need(S, at::kFloat, "S");
  TORCH_CHECK(S.dim() == 4 && S.is_contiguous(), "gated memory: state must be [slots, heads, dim, vdim]");
  const int64_t T = proj.size(0), H = S.size(1), D = S.size(2), V = S.size(3), B = state_slot.numel(), cols = proj.size(1);
  TORCH_CHECK(out.size(0) == T && out.size(1) == H * V && gates.size(0) == T && gates.size(1) >= H * D, "gated memory: out / gates shape");
  TORCH_CHECK(q_off >= 0 && q_off + H * D <= cols && v_off >= 0 && v_off + H * V <= cols, "gated memory: projection columns");
  TORCH_CHECK(vdim_true > 0 && vdim_true <= V, "gated memory: value width");
  need_vec(lower, at::kFloat, H * D, "lower"); need_vec(norm, at::kFloat, V, "norm");
  need_vec(cu_seqlens, at::kInt, B + 1, "cu_seqlens"); need_vec(state_slot, at::kInt, B, "state_slot");
  a.proj = proj.data_ptr(); a.ldp = proj.stride(0); a.q_off = static_cast<int>(q_off); a.v_off = static_cast<int>(v_off);
  a.gates = static_cast<const float*>(gates.data_ptr()); a.ldg = gates.stride(0); a.lower = static_cast<const float*>(lower.data_ptr());
  a.n_heads = static_cast<int>(H); a.dim = static_cast<int>(D); a.vdim = static_cast<int>(V); a.vdim_true = static_cast<int>(vdim_true);
  a.eps = static_cast<float>(eps); a.norm = static_cast<const float*>(norm.data_ptr());
  a.cu_seqlens = static_cast<const int*>(cu_seqlens.data_ptr()); a.state_slot = static_cast<const int*>(state_slot.data_ptr());
  a.T = static_cast<int>(T); a.n_seq = static_cast<int>(B); a.S = static_cast<float*>(S.data_ptr());
  a.out = out.data_ptr(); a.ldo = out.stride(0); a.write_state = write_state;
  TORCH_CHECK(!one_token || T == B, "gated memory: one token per sequence expected");
  a.one_token = one_token;
  c10::cuda::CUDAGuard guard(proj.device());
  a.stream = cur_stream(); a.pdl = pdl;
  if (chunk_ws.has_value() && chunk_ws->defined()) {
    need_cuda(*chunk_ws, "chunk_ws");
    chk(nfb::gated_chunked(a, chunk_ws->data_ptr(), chunk_ws->numel() * chunk_ws->element_size()));
  } else {
    chk(nfb::gated_recurrent(a));
  }
}

int64_t gated_chunked_workspace_bytes(int64_t T, int64_t n_seq, int64_t n_heads, int64_t dim, int64_t vdim) {
  return nfb::gated_chunked_workspace_bytes(static_cast<int>(T), static_cast<int>(n_seq), static_cast<int>(n_heads),
                                            static_cast<int>(dim), static_cast<int>(vdim));
}
bool gated_chunked_supported(int64_t dim, int64_t vdim) {
  return nfb::gated_chunked_supported(static_cast<int>(dim), static_cast<int>(vdim));
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("gated_memory(Tensor proj, int q_off, int v_off, Tensor gates, Tensor lower, int vdim_true, float eps, Tensor norm, Tensor cu_seqlens, Tensor state_slot, Tensor S, Tensor out, bool write_state, Tensor? chunk_ws, bool pdl, bool one_token=False) -> ()", &gated_memory);
  m.def("gated_chunked_workspace_bytes(int T, int n_seq, int n_heads, int dim, int vdim) -> int", &gated_chunked_workspace_bytes);
  m.def("gated_chunked_supported(int dim, int vdim) -> bool", &gated_chunked_supported);
}
