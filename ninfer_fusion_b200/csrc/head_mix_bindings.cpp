// torch.ops.nfb200.*: prefill of attention whose scores are mixed across heads (layer-list decoders, models/layered.py).
#include "attention/head_mix_args.h"

namespace {

using namespace nfb_bind;

void head_mix_prefill(const Tensor& q, const Tensor& k_pages, const Tensor& v_pages, const Tensor& block_table,
                      const Tensor& table_row, const Tensor& kv_len, int64_t window, double scale, double softcap, double sink,
                      OptT mix, OptT slope, OptT gate, const Tensor& out, const Tensor& blk_start, const Tensor& blk_count,
                      int64_t max_keys, const Tensor& scratch, bool pdl, bool sigmoid, OptT log_rate, OptT log_step, OptT offset) {
  c10::cuda::CUDAGuard guard(q.device());
  const nfb::HeadMixArgs a = head_mix_args(q, k_pages, v_pages, block_table, table_row, kv_len, window, scale, softcap, sink,
                                           mix, slope, gate, out, pdl, 0, std::nullopt, sigmoid, log_rate, log_step, offset);
  const int64_t nb = blk_start.numel();
  need_vec(blk_start, at::kInt, nb, "blk_start"); need_vec(blk_count, at::kInt, nb, "blk_count");
  need_cuda(scratch, "scratch");
  TORCH_CHECK(scratch.is_contiguous(), "scratch must be contiguous");
  chk(nfb::head_mix_prefill(a, static_cast<const int*>(blk_start.data_ptr()), static_cast<const int*>(blk_count.data_ptr()),
                            static_cast<int>(nb), static_cast<int>(max_keys), scratch.data_ptr(),
                            scratch.numel() * scratch.element_size()));
}

int64_t head_mix_prefill_scratch(int64_t n_heads, int64_t max_keys, int64_t window, int64_t blocks, bool sigmoid) {
  return nfb::head_mix_prefill_scratch(static_cast<int>(n_heads), static_cast<int>(max_keys), static_cast<int>(window),
                                       static_cast<int>(blocks), sigmoid);
}
int64_t head_mix_block_tokens() { return nfb::kHeadMixBlock; }

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("head_mix_prefill(Tensor q, Tensor k_pages, Tensor v_pages, Tensor block_table, Tensor table_row, Tensor kv_len, int window, float scale, float softcap, float sink, Tensor? mix, Tensor? slope, Tensor? gate, Tensor out, Tensor blk_start, Tensor blk_count, int max_keys, Tensor scratch, bool pdl, bool sigmoid=False, Tensor? log_rate=None, Tensor? log_step=None, Tensor? offset=None) -> ()", &head_mix_prefill);
  m.def("head_mix_prefill_scratch(int n_heads, int max_keys, int window, int blocks, bool sigmoid=False) -> int", &head_mix_prefill_scratch);
  m.def("head_mix_block_tokens() -> int", &head_mix_block_tokens);
}
