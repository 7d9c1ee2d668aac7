// torch.ops.nfb200.*: query / key norm with append and attention over paged rows (layer-list decoders, models/layered.py).
// Activations are bf16 or fp32; every op takes its element type from its tensors.
#include "attention/head_mix_args.h"

namespace {

using namespace nfb_bind;

void qkv_append(const Tensor& proj, int64_t q_off, int64_t k_off, int64_t v_off, int64_t n_heads, int64_t n_kv, int64_t dim_true,
                OptT q_norm, OptT k_norm, double eps, const Tensor& table_row, const Tensor& cache_pos,
                const Tensor& block_table, const Tensor& q_out, const Tensor& k_pages, const Tensor& v_pages,
                int64_t page_size, bool pdl, OptT freq, bool unit, OptT v_first, OptT v_lambda) {
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
  if (freq.has_value() && freq->defined()) {
    need(*freq, at::kDouble, "freq");
    TORCH_CHECK(freq->is_contiguous(), "freq must be contiguous");
    a.freq = static_cast<const double*>(freq->data_ptr()); a.rot = static_cast<int>(2 * freq->numel());
  }
  TORCH_CHECK(!unit || (a.q_norm == nullptr && a.k_norm == nullptr), "qkv_append: a norm without weights has none");
  a.unit = unit;
  if (v_first.has_value() && v_first->defined()) {
    need(*v_first, dt, "v_first"); need_rows(*v_first, "v_first");
    TORCH_CHECK(v_first->size(0) >= T && v_first->size(1) >= n_kv * vdim, "qkv_append: v_first shape");
    a.v_first = v_first->data_ptr(); a.ld_first = v_first->stride(0);
  }
  if (v_lambda.has_value() && v_lambda->defined()) {
    TORCH_CHECK(a.v_first != nullptr, "qkv_append: values are mixed with those of an earlier layer");
    need_vec(*v_lambda, at::kFloat, 1, "v_lambda");
    a.v_lambda = static_cast<const float*>(v_lambda->data_ptr());
  }
  c10::cuda::CUDAGuard guard(proj.device());
  a.stream = cur_stream(); a.pdl = pdl;
  chk(nfb::qkv_append(a));
}

void head_mix_attention(const Tensor& q, const Tensor& k_pages, const Tensor& v_pages, const Tensor& block_table,
                        const Tensor& table_row, const Tensor& kv_len, int64_t window, double scale, double softcap,
                        double sink, OptT mix, OptT slope, OptT gate, const Tensor& out, int64_t split_keys,
                        int64_t n_splits, OptT part_o, OptT part_ml, bool pdl, int64_t chunk, OptT sinks, bool sigmoid,
                        OptT log_rate, OptT log_step, OptT offset) {
  c10::cuda::CUDAGuard guard(q.device());
  const nfb::HeadMixArgs a = head_mix_args(q, k_pages, v_pages, block_table, table_row, kv_len, window, scale, softcap, sink,
                                           mix, slope, gate, out, pdl, chunk, sinks, sigmoid, log_rate, log_step, offset);
  if (n_splits > 1) {
    TORCH_CHECK(part_o.has_value() && part_o->defined() && part_ml.has_value() && part_ml->defined(),
                "head_mix attention: splits need their workspace");
    need_vec(*part_o, at::kFloat, n_splits * a.T * a.n_heads * a.vdim, "part_o");
    need_vec(*part_ml, at::kFloat, n_splits * a.T * a.n_heads * 2, "part_ml");
  }
  chk(nfb::head_mix_token_attention(a, static_cast<int>(split_keys), static_cast<int>(n_splits), ptr_or_null<float>(part_o),
                                    ptr_or_null<float>(part_ml)));
}

void group_prefill(const Tensor& q, const Tensor& k_pages, const Tensor& v_pages, const Tensor& block_table,
                   const Tensor& table_row, const Tensor& kv_len, int64_t window, int64_t chunk, double scale, double sink, OptT sinks,
                   const Tensor& out, const Tensor& blk_start, const Tensor& blk_count, bool pdl) {
  c10::cuda::CUDAGuard guard(q.device());
  const nfb::HeadMixArgs a = head_mix_args(q, k_pages, v_pages, block_table, table_row, kv_len, window, scale, 0.0, sink, std::nullopt,
                                           std::nullopt, std::nullopt, out, pdl, chunk, sinks, false, std::nullopt, std::nullopt, std::nullopt);
  const int64_t nb = blk_start.numel();
  need_vec(blk_start, at::kInt, nb, "blk_start"); need_vec(blk_count, at::kInt, nb, "blk_count");
  chk(nfb::group_prefill(a, static_cast<const int*>(blk_start.data_ptr()), static_cast<const int*>(blk_count.data_ptr()),
                         static_cast<int>(nb)));
}
bool group_prefill_supported(int64_t dim, int64_t vdim) {
  nfb::HeadMixArgs a;
  a.n_heads = a.n_kv = 1; a.dim = static_cast<int>(dim); a.vdim = static_cast<int>(vdim);
  return nfb::group_attention_supported(a);
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("qkv_append(Tensor proj, int q_off, int k_off, int v_off, int n_heads, int n_kv, int dim_true, Tensor? q_norm, Tensor? k_norm, float eps, Tensor table_row, Tensor cache_pos, Tensor block_table, Tensor q_out, Tensor k_pages, Tensor v_pages, int page_size, bool pdl, Tensor? freq=None, bool unit=False, Tensor? v_first=None, Tensor? v_lambda=None) -> ()", &qkv_append);
  m.def("head_mix_attention(Tensor q, Tensor k_pages, Tensor v_pages, Tensor block_table, Tensor table_row, Tensor kv_len, int window, float scale, float softcap, float sink, Tensor? mix, Tensor? slope, Tensor? gate, Tensor out, int split_keys, int n_splits, Tensor? part_o, Tensor? part_ml, bool pdl, int chunk=0, Tensor? sinks=None, bool sigmoid=False, Tensor? log_rate=None, Tensor? log_step=None, Tensor? offset=None) -> ()", &head_mix_attention);
  m.def("group_prefill(Tensor q, Tensor k_pages, Tensor v_pages, Tensor block_table, Tensor table_row, Tensor kv_len, int window, int chunk, float scale, float sink, Tensor? sinks, Tensor out, Tensor blk_start, Tensor blk_count, bool pdl) -> ()", &group_prefill);
  m.def("group_prefill_supported(int dim, int vdim) -> bool", &group_prefill_supported);
}
