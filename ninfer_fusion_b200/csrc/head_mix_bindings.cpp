// torch.ops.nfb200.*: head-mixing attention and matrix memory (layer-list decoders, models/layered.py).  Activations are
// bf16 or fp32; every op takes its element type from its tensors.
#include "attention/head_mix.h"
#include "binding_util.h"
#include "mlstm/mlstm.h"

namespace {

using namespace nfb_bind;

void qkv_append(const Tensor& proj, int64_t q_off, int64_t k_off, int64_t v_off, int64_t n_heads, int64_t n_kv, int64_t dim_true,
                OptT q_norm, OptT k_norm, double eps, const Tensor& table_row, const Tensor& cache_pos,
                const Tensor& block_table, const Tensor& q_out, const Tensor& k_pages, const Tensor& v_pages,
                int64_t page_size, bool pdl) {
  nfb::QkvAppendArgs a;
  a.f32 = act_f32(proj, "proj");
  const auto dt = proj.scalar_type();
  need_rows(proj, "proj"); need_rows(q_out, "q_out"); need(q_out, dt, "q_out");
  need(k_pages, dt, "k_pages"); need(v_pages, dt, "v_pages"); need(block_table, at::kInt, "block_table");
  TORCH_CHECK(k_pages.dim() == 4 && k_pages.is_contiguous() && v_pages.dim() == 4 && v_pages.is_contiguous() &&
              k_pages.size(1) == n_kv && v_pages.size(1) == n_kv && k_pages.size(2) == page_size && v_pages.size(2) == page_size,
              "qkv_append: pages must be [pages, kv heads, page size, width]");
  TORCH_CHECK(block_table.dim() == 2 && block_table.stride(1) == 1, "block_table must be [rows, pages]");
  const int64_t T = proj.size(0), dim = k_pages.size(3), vdim = v_pages.size(3);
  TORCH_CHECK(q_out.size(0) == T && q_out.size(1) == n_heads * dim, "qkv_append: q_out shape");
  TORCH_CHECK(q_off >= 0 && q_off + n_heads * dim <= proj.size(1) && k_off >= 0 && k_off + n_kv * dim <= proj.size(1) &&
              v_off >= 0 && v_off + n_kv * vdim <= proj.size(1), "qkv_append: projection columns");
  need_vec(table_row, at::kInt, T, "table_row"); need_vec(cache_pos, at::kInt, T, "cache_pos");
  if (q_norm.has_value() && q_norm->defined()) need_vec(*q_norm, at::kFloat, dim, "q_norm");
  if (k_norm.has_value() && k_norm->defined()) need_vec(*k_norm, at::kFloat, dim, "k_norm");
  a.proj = proj.data_ptr(); a.ldp = proj.stride(0);
  a.q_off = static_cast<int>(q_off); a.k_off = static_cast<int>(k_off); a.v_off = static_cast<int>(v_off);
  a.T = static_cast<int>(T); a.n_heads = static_cast<int>(n_heads); a.n_kv = static_cast<int>(n_kv);
  a.dim = static_cast<int>(dim); a.dim_true = static_cast<int>(dim_true); a.vdim = static_cast<int>(vdim);
  a.q_norm = ptr_or_null<const float>(q_norm); a.k_norm = ptr_or_null<const float>(k_norm); a.eps = static_cast<float>(eps);
  a.table_row = static_cast<const int*>(table_row.data_ptr()); a.cache_pos = static_cast<const int*>(cache_pos.data_ptr());
  a.block_table = static_cast<const int*>(block_table.data_ptr()); a.table_ld = static_cast<int>(block_table.stride(0));
  a.page_size = static_cast<int>(page_size);
  a.q_out = q_out.data_ptr(); a.ldq = q_out.stride(0); a.k_pages = k_pages.data_ptr(); a.v_pages = v_pages.data_ptr();
  c10::cuda::CUDAGuard guard(proj.device());
  a.stream = cur_stream(); a.pdl = pdl;
  chk(nfb::qkv_append(a));
}

nfb::HeadMixArgs head_mix_args(const Tensor& q, const Tensor& k_pages, const Tensor& v_pages, const Tensor& block_table,
                               const Tensor& table_row, const Tensor& kv_len, int64_t window, double scale, double softcap,
                               double sink, OptT mix, OptT slope, OptT gate, const Tensor& out, bool pdl) {
  nfb::HeadMixArgs a;
  a.f32 = act_f32(q, "q");
  const auto dt = q.scalar_type();
  need_rows(q, "q"); need_rows(out, "out"); need(out, dt, "out");
  need(k_pages, dt, "k_pages"); need(v_pages, dt, "v_pages"); need(block_table, at::kInt, "block_table");
  TORCH_CHECK(k_pages.dim() == 4 && k_pages.is_contiguous() && v_pages.dim() == 4 && v_pages.is_contiguous() &&
              k_pages.size(0) == v_pages.size(0) && k_pages.size(1) == v_pages.size(1) && k_pages.size(2) == v_pages.size(2),
              "head_mix attention: pages must be [pages, kv heads, page size, width]");
  TORCH_CHECK(block_table.dim() == 2 && block_table.stride(1) == 1, "block_table must be [rows, pages]");
  const int64_t T = q.size(0), D = k_pages.size(3), V = v_pages.size(3);
  TORCH_CHECK(q.size(1) % D == 0, "head_mix attention: q width");
  const int64_t H = q.size(1) / D;
  TORCH_CHECK(out.size(0) == T && out.size(1) == H * V, "head_mix attention: out shape");
  need_vec(table_row, at::kInt, T, "table_row"); need_vec(kv_len, at::kInt, T, "kv_len");
  if (mix.has_value() && mix->defined()) need_vec(*mix, at::kFloat, H * H, "mix");
  if (slope.has_value() && slope->defined()) need_vec(*slope, at::kFloat, H, "slope");
  if (gate.has_value() && gate->defined()) {
    need(*gate, at::kFloat, "gate"); need_rows(*gate, "gate");
    TORCH_CHECK(gate->size(0) == T && gate->size(1) >= H, "head_mix attention: gate shape");
    a.gate = static_cast<const float*>(gate->data_ptr()); a.ld_gate = gate->stride(0);
  }
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.k_pages = k_pages.data_ptr(); a.v_pages = v_pages.data_ptr();
  a.block_table = static_cast<const int*>(block_table.data_ptr()); a.table_ld = static_cast<int>(block_table.stride(0));
  a.table_row = static_cast<const int*>(table_row.data_ptr()); a.kv_len = static_cast<const int*>(kv_len.data_ptr());
  a.T = static_cast<int>(T); a.n_heads = static_cast<int>(H); a.n_kv = static_cast<int>(k_pages.size(1));
  a.dim = static_cast<int>(D); a.vdim = static_cast<int>(V); a.page_size = static_cast<int>(k_pages.size(2));
  a.window = static_cast<int>(window); a.scale = static_cast<float>(scale); a.softcap = static_cast<float>(softcap);
  a.sink = static_cast<float>(sink);
  a.mix = ptr_or_null<const float>(mix); a.slope = ptr_or_null<const float>(slope);
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  a.stream = cur_stream(); a.pdl = pdl;
  return a;
}

void head_mix_attention(const Tensor& q, const Tensor& k_pages, const Tensor& v_pages, const Tensor& block_table,
                        const Tensor& table_row, const Tensor& kv_len, int64_t window, double scale, double softcap,
                        double sink, OptT mix, OptT slope, OptT gate, const Tensor& out, int64_t split_keys,
                        int64_t n_splits, OptT part_o, OptT part_ml, bool pdl) {
  c10::cuda::CUDAGuard guard(q.device());
  const nfb::HeadMixArgs a = head_mix_args(q, k_pages, v_pages, block_table, table_row, kv_len, window, scale, softcap, sink,
                                           mix, slope, gate, out, pdl);
  if (n_splits > 1) {
    TORCH_CHECK(part_o.has_value() && part_o->defined() && part_ml.has_value() && part_ml->defined(),
                "head_mix attention: splits need their workspace");
    need_vec(*part_o, at::kFloat, n_splits * a.T * a.n_heads * a.vdim, "part_o");
    need_vec(*part_ml, at::kFloat, n_splits * a.T * a.n_heads * 2, "part_ml");
  }
  chk(nfb::head_mix_token_attention(a, static_cast<int>(split_keys), static_cast<int>(n_splits), ptr_or_null<float>(part_o),
                                    ptr_or_null<float>(part_ml)));
}

void head_mix_prefill(const Tensor& q, const Tensor& k_pages, const Tensor& v_pages, const Tensor& block_table,
                      const Tensor& table_row, const Tensor& kv_len, int64_t window, double scale, double softcap, double sink,
                      OptT mix, OptT slope, OptT gate, const Tensor& out, const Tensor& blk_start, const Tensor& blk_count,
                      int64_t max_keys, const Tensor& scratch, bool pdl) {
  c10::cuda::CUDAGuard guard(q.device());
  const nfb::HeadMixArgs a = head_mix_args(q, k_pages, v_pages, block_table, table_row, kv_len, window, scale, softcap, sink,
                                           mix, slope, gate, out, pdl);
  const int64_t nb = blk_start.numel();
  need_vec(blk_start, at::kInt, nb, "blk_start"); need_vec(blk_count, at::kInt, nb, "blk_count");
  need_cuda(scratch, "scratch");
  TORCH_CHECK(scratch.is_contiguous(), "scratch must be contiguous");
  chk(nfb::head_mix_prefill(a, static_cast<const int*>(blk_start.data_ptr()), static_cast<const int*>(blk_count.data_ptr()),
                            static_cast<int>(nb), static_cast<int>(max_keys), scratch.data_ptr(),
                            scratch.numel() * scratch.element_size()));
}

int64_t head_mix_prefill_scratch(int64_t n_heads, int64_t max_keys, int64_t window, int64_t blocks) {
  return nfb::head_mix_prefill_scratch(static_cast<int>(n_heads), static_cast<int>(max_keys), static_cast<int>(window),
                                       static_cast<int>(blocks));
}
int64_t head_mix_block_tokens() { return nfb::kHeadMixBlock; }

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
  m.def("qkv_append(Tensor proj, int q_off, int k_off, int v_off, int n_heads, int n_kv, int dim_true, Tensor? q_norm, Tensor? k_norm, float eps, Tensor table_row, Tensor cache_pos, Tensor block_table, Tensor q_out, Tensor k_pages, Tensor v_pages, int page_size, bool pdl) -> ()", &qkv_append);
  m.def("head_mix_attention(Tensor q, Tensor k_pages, Tensor v_pages, Tensor block_table, Tensor table_row, Tensor kv_len, int window, float scale, float softcap, float sink, Tensor? mix, Tensor? slope, Tensor? gate, Tensor out, int split_keys, int n_splits, Tensor? part_o, Tensor? part_ml, bool pdl) -> ()", &head_mix_attention);
  m.def("head_mix_prefill(Tensor q, Tensor k_pages, Tensor v_pages, Tensor block_table, Tensor table_row, Tensor kv_len, int window, float scale, float softcap, float sink, Tensor? mix, Tensor? slope, Tensor? gate, Tensor out, Tensor blk_start, Tensor blk_count, int max_keys, Tensor scratch, bool pdl) -> ()", &head_mix_prefill);
  m.def("head_mix_prefill_scratch(int n_heads, int max_keys, int window, int blocks) -> int", &head_mix_prefill_scratch);
  m.def("head_mix_block_tokens() -> int", &head_mix_block_tokens);
  m.def("mlstm(Tensor proj, int q_off, int k_off, int v_off, int g_off, Tensor gates, int i_off, int f_off, int vdim_true, float q_scale, float gate_cap, float eps, Tensor norm, Tensor cu_seqlens, Tensor state_slot, Tensor S, Tensor n, Tensor m, Tensor out, bool write_state, Tensor? chunk_ws, bool pdl, bool one_token=False) -> ()", &mlstm);
  m.def("mlstm_chunked_workspace_bytes(int T, int n_seq, int n_heads, int dim, int vdim) -> int", &mlstm_chunked_workspace_bytes);
  m.def("mlstm_chunked_supported(int dim, int vdim) -> bool", &mlstm_chunked_supported);
}
