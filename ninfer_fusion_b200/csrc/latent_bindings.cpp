// torch.ops.nfb200.*: latent attention (layer-list decoders, models/layered.py).  Activations are bf16 or fp32; every op takes
// its element type from its tensors.
#include "attention/latent.h"
#include "binding_util.h"
#include "gemm/head_gemm.h"

namespace {

using namespace nfb_bind;

const double* freq_ptr(const Tensor& freq, int64_t rot_true) {
  need_vec(freq, at::kDouble, rot_true / 2, "freq");
  return static_cast<const double*>(freq.data_ptr());
}
void need_pages(const Tensor& pages, at::ScalarType dt, int64_t width) {
  need(pages, dt, "pages");
  TORCH_CHECK(pages.dim() == 4 && pages.is_contiguous() && pages.size(1) == 1 && pages.size(3) == width,
              "latent pages must be [pages, 1, page size, latent + rotated part]");
}
void need_table(const Tensor& table) {
  need(table, at::kInt, "block_table");
  TORCH_CHECK(table.dim() == 2 && table.stride(1) == 1, "block_table must be [rows, pages]");
}

void latent_prep(const Tensor& proj, int64_t q_rank_true, int64_t rank_true, int64_t rot_true, OptT q_norm,
                 const Tensor& kv_norm, double eps, const Tensor& freq, const Tensor& table_row, const Tensor& cache_pos,
                 const Tensor& block_table, OptT q_latent, const Tensor& pages, bool pdl) {
  nfb::LatentPrepArgs a;
  a.f32 = act_f32(proj, "proj");
  const int64_t T = proj.size(0);
  need_rows(proj, "proj"); need_table(block_table);
  TORCH_CHECK(pages.dim() == 4, "latent pages must be [pages, 1, page size, latent + rotated part]");
  const int64_t rank = kv_norm.numel(), rot = pages.size(3) - rank, off = proj.size(1) - rank - rot;
  TORCH_CHECK(rot >= 0 && off >= 0, "latent_prep: projection columns");
  need_pages(pages, proj.scalar_type(), rank + rot);
  a.kv_off = static_cast<int>(off);
  if (q_latent.has_value() && q_latent->defined()) {
    need_rows(*q_latent, "q_latent"); need(*q_latent, proj.scalar_type(), "q_latent");
    TORCH_CHECK(q_latent->size(0) == T && q_latent->size(1) == off && q_norm.has_value(), "latent_prep: query latent");
    need_vec(*q_norm, at::kFloat, off, "q_norm");
    a.q_rank = static_cast<int>(off); a.q_rank_true = static_cast<int>(q_rank_true);
    a.q_norm = static_cast<const float*>(q_norm->data_ptr()); a.q_latent = q_latent->data_ptr(); a.ldq = q_latent->stride(0);
  }
  need_vec(kv_norm, at::kFloat, rank, "kv_norm");
  need_vec(table_row, at::kInt, T, "table_row"); need_vec(cache_pos, at::kInt, T, "cache_pos");
  a.proj = proj.data_ptr(); a.ldp = proj.stride(0); a.T = static_cast<int>(T);
  a.rank = static_cast<int>(rank); a.rank_true = static_cast<int>(rank_true);
  a.rot = static_cast<int>(rot); a.rot_true = static_cast<int>(rot_true);
  a.kv_norm = static_cast<const float*>(kv_norm.data_ptr());
  a.eps = static_cast<float>(eps); a.freq = freq_ptr(freq, rot_true);
  a.table_row = static_cast<const int*>(table_row.data_ptr()); a.cache_pos = static_cast<const int*>(cache_pos.data_ptr());
  a.block_table = static_cast<const int*>(block_table.data_ptr()); a.table_ld = static_cast<int>(block_table.stride(0));
  a.page_size = static_cast<int>(pages.size(2));
  a.pages = pages.data_ptr();
  c10::cuda::CUDAGuard guard(proj.device());
  a.stream = cur_stream(); a.pdl = pdl;
  chk(nfb::latent_prep(a));
}

nfb::LatentArgs latent_args(const Tensor& q, const Tensor& pages, const Tensor& block_table, const Tensor& table_row,
                            const Tensor& kv_len, int64_t n_heads, int64_t rank, int64_t rot_true, double scale, const Tensor& freq,
                            OptT sink, const Tensor& out, int64_t window, bool pdl) {
  nfb::LatentArgs a;
  TORCH_CHECK(window >= 0, "latent attention: window");
  a.window = static_cast<int>(window);
  a.f32 = act_f32(q, "q");
  need_rows(q, "q"); need_rows(out, "out"); need(out, q.scalar_type(), "out"); need_table(block_table);
  const int64_t T = q.size(0), rot = pages.size(3) - rank;
  need_pages(pages, q.scalar_type(), rank + rot);
  TORCH_CHECK(n_heads > 0 && q.size(1) % n_heads == 0 && q.size(1) / n_heads >= rot && out.size(0) == T, "latent attention: shapes");
  need_vec(table_row, at::kInt, T, "table_row"); need_vec(kv_len, at::kInt, T, "kv_len");
  if (sink.has_value() && sink->defined()) need_vec(*sink, at::kFloat, n_heads, "sink");
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.pages = pages.data_ptr();
  a.block_table = static_cast<const int*>(block_table.data_ptr()); a.table_ld = static_cast<int>(block_table.stride(0));
  a.table_row = static_cast<const int*>(table_row.data_ptr()); a.kv_len = static_cast<const int*>(kv_len.data_ptr());
  a.T = static_cast<int>(T); a.n_heads = static_cast<int>(n_heads); a.rank = static_cast<int>(rank); a.rot = static_cast<int>(rot);
  a.dim = static_cast<int>(q.size(1) / n_heads - rot); a.rot_true = static_cast<int>(rot_true);
  a.page_size = static_cast<int>(pages.size(2)); a.scale = static_cast<float>(scale); a.freq = freq_ptr(freq, rot_true);
  a.sink = ptr_or_null<const float>(sink); a.out = out.data_ptr(); a.ldo = out.stride(0);
  a.stream = cur_stream(); a.pdl = pdl;
  return a;
}

void latent_token_attention(const Tensor& q_latent, const Tensor& q, const Tensor& pages, const Tensor& block_table,
                            const Tensor& table_row, const Tensor& kv_len, int64_t n_heads, int64_t rot_true, double scale,
                            const Tensor& freq, OptT sink, const Tensor& out, bool pdl, int64_t window) {
  c10::cuda::CUDAGuard guard(q.device());
  need_rows(q_latent, "q_latent"); need(q_latent, q.scalar_type(), "q_latent");
  const int64_t rank = q_latent.size(1) / n_heads;
  nfb::LatentArgs a = latent_args(q, pages, block_table, table_row, kv_len, n_heads, rank, rot_true, scale, freq, sink, out, window, pdl);
  TORCH_CHECK(q_latent.size(0) == a.T && out.size(1) == n_heads * rank, "latent attention: shapes");
  a.q_latent = q_latent.data_ptr(); a.ldl = q_latent.stride(0);
  chk(nfb::latent_token_attention(a));
}

void latent_absorbed_attention(const Tensor& q_latent, const Tensor& q, const Tensor& pages, const Tensor& block_table,
                               const Tensor& table_row, const Tensor& kv_len, int64_t n_heads, int64_t rot_true, double scale,
                               const Tensor& freq, OptT sink, const Tensor& out, const Tensor& blk_start, const Tensor& blk_count,
                               int64_t max_count, const Tensor& token_seq, const Tensor& cu_seqlens, int64_t max_tokens,
                               int64_t split_keys, int64_t n_splits, OptT part_o, OptT part_ml, bool pdl, int64_t window) {
  c10::cuda::CUDAGuard guard(q.device());
  need_rows(q_latent, "q_latent"); need(q_latent, q.scalar_type(), "q_latent");
  const int64_t rank = q_latent.size(1) / n_heads;
  nfb::LatentArgs a = latent_args(q, pages, block_table, table_row, kv_len, n_heads, rank, rot_true, scale, freq, sink, out, window, pdl);
  TORCH_CHECK(q_latent.size(0) == a.T && out.size(1) == n_heads * rank, "latent attention: shapes");
  a.q_latent = q_latent.data_ptr(); a.ldl = q_latent.stride(0);
  nfb::LatentBlocks b;
  b.n = static_cast<int>(blk_start.numel());
  need_vec(blk_start, at::kInt, b.n, "blk_start"); need_vec(blk_count, at::kInt, b.n, "blk_count");
  need_vec(token_seq, at::kInt, a.T, "token_seq"); need(cu_seqlens, at::kInt, "cu_seqlens");
  b.start = static_cast<const int*>(blk_start.data_ptr()); b.count = static_cast<const int*>(blk_count.data_ptr());
  b.max_count = static_cast<int>(max_count); b.token_seq = static_cast<const int*>(token_seq.data_ptr());
  b.cu_seqlens = static_cast<const int*>(cu_seqlens.data_ptr()); b.max_tokens = static_cast<int>(max_tokens);
  if (n_splits > 1) {
    TORCH_CHECK(part_o.has_value() && part_o->defined() && part_ml.has_value() && part_ml->defined(), "latent attention: splits need their workspace");
    need_vec(*part_o, at::kFloat, n_splits * a.T * n_heads * rank, "part_o");
    need_vec(*part_ml, at::kFloat, n_splits * a.T * n_heads * 2, "part_ml");
  }
  chk(nfb::latent_absorbed_attention(a, b, static_cast<int>(split_keys), static_cast<int>(n_splits), ptr_or_null<float>(part_o),
                                     ptr_or_null<float>(part_ml)));
}
bool latent_absorbed_supported(int64_t rank, int64_t rot) {
  return nfb::latent_absorbed_supported(static_cast<int>(rank), static_cast<int>(rot));
}

void latent_gather(const Tensor& pages, const Tensor& block_table, const Tensor& seqs, int64_t max_len, const Tensor& rows, bool pdl) {
  need(pages, at::kBFloat16, "pages"); need(rows, at::kBFloat16, "rows"); need_table(block_table);
  need_pages(pages, at::kBFloat16, pages.size(3));
  TORCH_CHECK(seqs.dim() == 2 && seqs.size(1) == 4, "seqs must be [n, 4]");
  need_vec(seqs, at::kInt, seqs.size(0) * 4, "seqs");
  TORCH_CHECK(rows.dim() == 2 && rows.is_contiguous() && rows.size(1) == pages.size(3), "latent_gather: rows shape");
  nfb::LatentArgs a;
  a.pages = pages.data_ptr(); a.rank = static_cast<int>(pages.size(3)); a.rot = 0; a.page_size = static_cast<int>(pages.size(2));
  a.block_table = static_cast<const int*>(block_table.data_ptr()); a.table_ld = static_cast<int>(block_table.stride(0));
  nfb::LatentExpand x;
  x.seqs = static_cast<const int*>(seqs.data_ptr()); x.n_seqs = static_cast<int>(seqs.size(0)); x.max_len = static_cast<int>(max_len);
  x.rows = rows.data_ptr();
  c10::cuda::CUDAGuard guard(pages.device());
  a.stream = cur_stream(); a.pdl = pdl;
  chk(nfb::latent_gather(a, x));
}

void latent_expanded_attention(const Tensor& q, const Tensor& rows, const Tensor& kv, const Tensor& kv_len,
                               int64_t n_heads, int64_t rank, int64_t rot_true, double scale, const Tensor& freq, OptT sink,
                               const Tensor& out, const Tensor& blk_start, const Tensor& blk_count, int64_t max_count,
                               const Tensor& token_seq, const Tensor& seq_base, bool pdl, int64_t window) {
  nfb::LatentArgs a;
  TORCH_CHECK(window >= 0, "latent attention: window");
  a.window = static_cast<int>(window);
  need(q, at::kBFloat16, "q"); need(rows, at::kBFloat16, "rows"); need(kv, at::kBFloat16, "kv"); need(out, at::kBFloat16, "out");
  need_rows(q, "q"); need_rows(out, "out");
  TORCH_CHECK(rows.dim() == 2 && rows.is_contiguous() && kv.dim() == 2 && kv.is_contiguous() && rows.size(0) == kv.size(0),
              "latent attention: gathered rows");
  const int64_t T = q.size(0), rot = rows.size(1) - rank;
  TORCH_CHECK(n_heads > 0 && rot >= 0 && q.size(1) % n_heads == 0 && out.size(1) % n_heads == 0 && out.size(0) == T, "latent attention: shapes");
  const int64_t dim = q.size(1) / n_heads - rot, vdim = out.size(1) / n_heads;
  TORCH_CHECK(dim > 0 && kv.size(1) == n_heads * (dim + vdim), "latent attention: expanded columns");
  need_vec(kv_len, at::kInt, T, "kv_len"); need_vec(token_seq, at::kInt, T, "token_seq");
  need(seq_base, at::kInt, "seq_base");
  TORCH_CHECK(seq_base.dim() == 2 && seq_base.size(1) == 2 && seq_base.is_contiguous(), "seq_base must be [sequences, 2]");
  if (sink.has_value() && sink->defined()) need_vec(*sink, at::kFloat, n_heads, "sink");
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.kv_len = static_cast<const int*>(kv_len.data_ptr());
  a.T = static_cast<int>(T); a.n_heads = static_cast<int>(n_heads); a.dim = static_cast<int>(dim); a.rank = static_cast<int>(rank);
  a.rot = static_cast<int>(rot); a.rot_true = static_cast<int>(rot_true); a.scale = static_cast<float>(scale);
  a.freq = freq_ptr(freq, rot_true); a.sink = ptr_or_null<const float>(sink); a.out = out.data_ptr(); a.ldo = out.stride(0);
  nfb::LatentBlocks b;
  b.n = static_cast<int>(blk_start.numel()); b.max_count = static_cast<int>(max_count);
  need_vec(blk_start, at::kInt, b.n, "blk_start"); need_vec(blk_count, at::kInt, b.n, "blk_count");
  b.start = static_cast<const int*>(blk_start.data_ptr()); b.count = static_cast<const int*>(blk_count.data_ptr());
  b.token_seq = static_cast<const int*>(token_seq.data_ptr());
  nfb::LatentExpand x;
  x.seq_base = static_cast<const int*>(seq_base.data_ptr()); x.rows = rows.data_ptr(); x.kv = kv.data_ptr(); x.vdim = static_cast<int>(vdim);
  c10::cuda::CUDAGuard guard(q.device());
  a.stream = cur_stream(); a.pdl = pdl;
  chk(nfb::latent_expanded_attention(a, b, x));
}
bool latent_expanded_supported(int64_t dim, int64_t rot, int64_t vdim) {
  return nfb::latent_expanded_supported(static_cast<int>(dim), static_cast<int>(rot), static_cast<int>(vdim));
}

void head_gemm(const Tensor& x, int64_t x_step, const Tensor& w, const Tensor& out, OptT token_seq, OptT cu_seqlens, int64_t max_tokens,
               bool pdl) {
  need(x, at::kBFloat16, "x"); need(w, at::kBFloat16, "w"); need(out, at::kBFloat16, "out");
  need_rows(x, "x"); need_rows(out, "out");
  TORCH_CHECK(w.dim() == 3 && w.is_contiguous(), "head_gemm: w must be [heads, N, K]");
  nfb::HeadGemmArgs a;
  a.T = static_cast<int>(x.size(0)); a.H = static_cast<int>(w.size(0)); a.N = static_cast<int>(w.size(1)); a.K = static_cast<int>(w.size(2));
  TORCH_CHECK(x_step >= 0 && x.size(1) >= (a.H - 1) * x_step + a.K && out.size(0) == a.T && out.size(1) == w.size(0) * w.size(1),
              "head_gemm: shapes");
  a.x = x.data_ptr(); a.ldx = x.stride(0); a.x_step = static_cast<int>(x_step); a.w = w.data_ptr();
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  if (max_tokens > 0) {
    TORCH_CHECK(token_seq.has_value() && cu_seqlens.has_value(), "head_gemm: leaving tokens out needs the sequences");
    need_vec(*token_seq, at::kInt, a.T, "token_seq"); need(*cu_seqlens, at::kInt, "cu_seqlens");
    a.token_seq = static_cast<const int*>(token_seq->data_ptr()); a.cu_seqlens = static_cast<const int*>(cu_seqlens->data_ptr());
    a.max_tokens = static_cast<int>(max_tokens);
  }
  c10::cuda::CUDAGuard guard(x.device());
  a.stream = cur_stream(); a.pdl = pdl;
  chk(nfb::head_gemm(a));
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("latent_prep(Tensor proj, int q_rank_true, int rank_true, int rot_true, Tensor? q_norm, Tensor kv_norm, float eps, Tensor freq, Tensor table_row, Tensor cache_pos, Tensor block_table, Tensor? q_latent, Tensor pages, bool pdl) -> ()", &latent_prep);
  m.def("latent_token_attention(Tensor q_latent, Tensor q, Tensor pages, Tensor block_table, Tensor table_row, Tensor kv_len, int n_heads, int rot_true, float scale, Tensor freq, Tensor? sink, Tensor out, bool pdl, int window=0) -> ()", &latent_token_attention);
  m.def("latent_absorbed_attention(Tensor q_latent, Tensor q, Tensor pages, Tensor block_table, Tensor table_row, Tensor kv_len, int n_heads, int rot_true, float scale, Tensor freq, Tensor? sink, Tensor out, Tensor blk_start, Tensor blk_count, int max_count, Tensor token_seq, Tensor cu_seqlens, int max_tokens, int split_keys, int n_splits, Tensor? part_o, Tensor? part_ml, bool pdl, int window=0) -> ()", &latent_absorbed_attention);
  m.def("latent_absorbed_supported(int rank, int rot) -> bool", &latent_absorbed_supported);
  m.def("latent_gather(Tensor pages, Tensor block_table, Tensor seqs, int max_len, Tensor rows, bool pdl) -> ()", &latent_gather);
  m.def("latent_expanded_attention(Tensor q, Tensor rows, Tensor kv, Tensor kv_len, int n_heads, int rank, int rot_true, float scale, Tensor freq, Tensor? sink, Tensor out, Tensor blk_start, Tensor blk_count, int max_count, Tensor token_seq, Tensor seq_base, bool pdl, int window=0) -> ()", &latent_expanded_attention);
  m.def("latent_expanded_supported(int dim, int rot, int vdim) -> bool", &latent_expanded_supported);
  m.def("head_gemm(Tensor x, int x_step, Tensor w, Tensor out, Tensor? token_seq, Tensor? cu_seqlens, int max_tokens, bool pdl) -> ()", &head_gemm);
}
