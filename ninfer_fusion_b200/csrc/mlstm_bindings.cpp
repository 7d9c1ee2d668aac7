// torch.ops.nfb200.*: matrix memory (layer-list decoders, models/layered.py).  Activations are bf16 or fp32; every op takes its
// element type from its tensors.
#include "binding_util.h"
#include "mlstm/mlstm.h"

namespace {

using namespace nfb_bind;

void mlstm(const Tensor& proj, int64_t q_off, int64_t k_off, int64_t v_off, int64_t g_off, const Tensor& gates, int64_t i_off,
           int64_t f_off, int64_t vdim_true, double q_scale, double gate_cap, double eps, const Tensor& norm,
           const Tensor& cu_seqlens, const Tensor& state_slot, const Tensor& S, const Tensor& n, const Tensor& m,
           const Tensor& out, bool write_state, OptT chunk_ws, bool pdl, bool one_token) {
  nfb::MlstmArgs a;
  a.f32 = act_f32(proj, "proj");
  need_rows(proj, "proj"); need_rows(out, "out"); need(out, proj.scalar_type(), "out");
  need(gates, at::kFloat, "gates"); need_rows(gates, "gates");
  need(S, at::kFloat, "S"); need(n, at::kFloat, "n"); need(m, at::kFloat, "m");
  TORCH_CHECK(S.dim() == 4 && S.is_contiguous() && n.is_contiguous() && m.is_contiguous(), "mlstm: state must be contiguous");
  const int64_t T = proj.size(0), slots = S.size(0), H = S.size(1), D = S.size(2), V = S.size(3), B = state_slot.numel();
  TORCH_CHECK(n.numel() == slots * H * D && m.numel() == slots * H, "mlstm: state shapes");
  TORCH_CHECK(out.size(0) == T && out.size(1) == H * V && gates.size(0) == T, "mlstm: out / gates shape");
  const int64_t cols = proj.size(1);
  TORCH_CHECK(q_off >= 0 && q_off + H * D <= cols && k_off >= 0 && k_off + H * D <= cols && v_off >= 0 &&
              v_off + H * V <= cols && g_off >= 0 && g_off + H * V <= cols, "mlstm: projection columns");
  TORCH_CHECK(i_off >= 0 && i_off + H <= gates.size(1) && f_off >= 0 && f_off + H <= gates.size(1), "mlstm: gate columns");
  need_vec(norm, at::kFloat, H * V, "norm");
  need_vec(cu_seqlens, at::kInt, B + 1, "cu_seqlens"); need_vec(state_slot, at::kInt, B, "state_slot");
  a.proj = proj.data_ptr(); a.ldp = proj.stride(0);
  a.q_off = static_cast<int>(q_off); a.k_off = static_cast<int>(k_off); a.v_off = static_cast<int>(v_off); a.g_off = static_cast<int>(g_off);
  a.gates = static_cast<const float*>(gates.data_ptr()); a.ldg = gates.stride(0);
  a.i_off = static_cast<int>(i_off); a.f_off = static_cast<int>(f_off);
  a.n_heads = static_cast<int>(H); a.dim = static_cast<int>(D); a.vdim = static_cast<int>(V); a.vdim_true = static_cast<int>(vdim_true);
  a.q_scale = static_cast<float>(q_scale); a.gate_cap = static_cast<float>(gate_cap); a.eps = static_cast<float>(eps);
  a.norm = static_cast<const float*>(norm.data_ptr());
  a.cu_seqlens = static_cast<const int*>(cu_seqlens.data_ptr()); a.state_slot = static_cast<const int*>(state_slot.data_ptr());
  a.T = static_cast<int>(T); a.n_seq = static_cast<int>(B);
  a.S = static_cast<float*>(S.data_ptr()); a.n = static_cast<float*>(n.data_ptr()); a.m = static_cast<float*>(m.data_ptr());
  a.out = out.data_ptr(); a.ldo = out.stride(0); a.write_state = write_state;
  TORCH_CHECK(!one_token || T == B, "mlstm: one token per sequence expected");
  a.one_token = one_token;
  c10::cuda::CUDAGuard guard(proj.device());
  a.stream = cur_stream(); a.pdl = pdl;
  if (chunk_ws.has_value() && chunk_ws->defined()) {
    need_cuda(*chunk_ws, "chunk_ws");
    chk(nfb::mlstm_chunked(a, chunk_ws->data_ptr(), chunk_ws->numel() * chunk_ws->element_size()));
  } else {
    chk(nfb::mlstm_recurrent(a));
  }
}

int64_t mlstm_chunked_workspace_bytes(int64_t T, int64_t n_seq, int64_t n_heads, int64_t dim, int64_t vdim) {
  return nfb::mlstm_chunked_workspace_bytes(static_cast<int>(T), static_cast<int>(n_seq), static_cast<int>(n_heads),
                                            static_cast<int>(dim), static_cast<int>(vdim));
}
bool mlstm_chunked_supported(int64_t dim, int64_t vdim) {
  return nfb::mlstm_chunked_supported(static_cast<int>(dim), static_cast<int>(vdim));
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("mlstm(Tensor proj, int q_off, int k_off, int v_off, int g_off, Tensor gates, int i_off, int f_off, int vdim_true, float q_scale, float gate_cap, float eps, Tensor norm, Tensor cu_seqlens, Tensor state_slot, Tensor S, Tensor n, Tensor m, Tensor out, bool write_state, Tensor? chunk_ws, bool pdl, bool one_token=False) -> ()", &mlstm);
  m.def("mlstm_chunked_workspace_bytes(int T, int n_seq, int n_heads, int dim, int vdim) -> int", &mlstm_chunked_workspace_bytes);
  m.def("mlstm_chunked_supported(int dim, int vdim) -> bool", &mlstm_chunked_supported);
}
