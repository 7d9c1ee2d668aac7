// torch.ops.nfb200.*: the GEMM and token-selection ops that every model family uses.
#include "binding_util.h"
#include "sampling/sampling.h"

namespace {

using namespace nfb_bind;

void gemm_bf16(const Tensor& x, const Tensor& w, OptT out, int64_t epi, OptT resid, OptT bias, OptT partial,
               int64_t splits, OptT status, bool pdl, int64_t act, OptT conv_w, OptT conv_state, OptT conv_slot,
               OptT conv_out, OptT prefetch, OptT out32, int64_t out32_from, OptT act_params, at::ArrayRef<double> glu) {
  need(x, at::kBFloat16, "x"); need(w, at::kBFloat16, "w");
  need_rows(x, "x"); need_rows(w, "w");
  TORCH_CHECK(x.size(1) == w.size(1), "gemm_bf16: K mismatch");
  TORCH_CHECK(act >= 0 && act <= 5 && (act == 0 || epi == nfb::kEpiStore), "gemm_bf16: activation needs the store epilogue");
  c10::cuda::CUDAGuard guard(x.device());
  nfb::GemmArgs a;
  a.w = w.data_ptr(); a.N = w.size(0); a.K = w.size(1); a.ldw = w.stride(0);
  a.x = x.data_ptr(); a.T = x.size(0); a.ldx = x.stride(0);
  const int64_t out_cols = epi == nfb::kEpiSwiglu ? a.N / 2 : a.N;
  const bool has32 = out32.has_value() && out32->defined();
  if (has32) {
    need(*out32, at::kFloat, "out32"); need_rows(*out32, "out32");
    TORCH_CHECK(out32->size(0) == a.T && out32->size(1) >= a.N - out32_from, "gemm_bf16: out32 shape");
    a.out32 = static_cast<float*>(out32->data_ptr()); a.ldo32 = out32->stride(0);
    a.out32_from = static_cast<int>(out32_from);
  }
  if (act_params.has_value() && act_params->defined()) {
    need(*act_params, at::kFloat, "act_params");
    TORCH_CHECK(act_params->numel() == 2 && act_params->is_contiguous(), "gemm_bf16: act_params shape");
    a.act_params = static_cast<const float*>(act_params->data_ptr());
  }
  if (epi != nfb::kEpiPartial && !(has32 && out32_from == 0)) {
    TORCH_CHECK(out.has_value(), "gemm_bf16: out required");
    need(*out, at::kBFloat16, "out"); need_rows(*out, "out");
    TORCH_CHECK(out->size(0) == a.T && (has32 ? out->size(1) >= out32_from : out->size(1) == out_cols), "gemm_bf16: out shape");
    a.out = out->data_ptr(); a.ldo = out->stride(0);
  }
  if (epi == nfb::kEpiResidual) {
    TORCH_CHECK(resid.has_value(), "gemm_bf16: resid required");
    need(*resid, at::kBFloat16, "resid"); need_rows(*resid, "resid");
    TORCH_CHECK(resid->size(0) == a.T && resid->size(1) == a.N, "gemm_bf16: resid shape");
    a.resid = resid->data_ptr(); a.ldr = resid->stride(0);
  }
  if (bias.has_value() && bias->defined()) {
    need(*bias, at::kFloat, "bias");
    TORCH_CHECK(bias->numel() == a.N && bias->is_contiguous(), "gemm_bf16: bias shape");
    a.bias = static_cast<const float*>(bias->data_ptr());
  }
  if (epi == nfb::kEpiPartial) {
    TORCH_CHECK(partial.has_value(), "gemm_bf16: partial workspace required");
    need(*partial, at::kFloat, "partial");
    TORCH_CHECK(partial->is_contiguous() && partial->numel() >= splits * a.T * a.N, "gemm_bf16: workspace too small");
    a.partial = static_cast<float*>(partial->data_ptr());
  }
  if (!glu.empty()) {
    TORCH_CHECK(glu.size() == 3, "gemm_bf16: glu = limit, slope, shift");
    a.glu.limit = static_cast<float>(glu[0]); a.glu.slope = static_cast<float>(glu[1]); a.glu.shift = static_cast<float>(glu[2]);
  }
  a.splits = static_cast<int>(splits); a.epi = static_cast<int>(epi); a.act = static_cast<int>(act);
  a.status = ptr_or_null<int>(status);
  a.stream = cur_stream(); a.pdl = pdl;
  fill_conv(a, conv_w, conv_state, conv_slot, conv_out);
  fill_prefetch(a, prefetch);
  chk(nfb::gemm_bf16(a));
}

int64_t gemm_pick_splits(int64_t T, int64_t N, int64_t K, int64_t epi) {
  return nfb::gemm_pick_splits(static_cast<int>(T), static_cast<int>(N), static_cast<int>(K), static_cast<int>(epi),
                               static_cast<int>(sm_count()));
}

bool logits_f32(const Tensor& logits) {
  need_cuda(logits, "logits");
  TORCH_CHECK(logits.scalar_type() == at::kBFloat16 || logits.scalar_type() == at::kFloat, "logits must be bf16 or fp32");
  return logits.scalar_type() == at::kFloat;
}

void argmax_rows(const Tensor& logits, const Tensor& out, bool pdl) {
  const bool f32 = logits_f32(logits); need_rows(logits, "logits"); need(out, at::kInt, "out");
  TORCH_CHECK(out.numel() == logits.size(0));
  c10::cuda::CUDAGuard guard(logits.device());
  chk(nfb::argmax_rows(logits.data_ptr(), logits.stride(0), static_cast<int>(logits.size(0)),
                       static_cast<int>(logits.size(1)), static_cast<int*>(out.data_ptr()), f32, cur_stream(), pdl));
}

void sample_rows(const Tensor& logits, OptT temperature, OptT top_k, OptT top_p, OptT min_p, OptT presence,
                 OptT frequency, OptT token_counts, OptT seeds, OptT positions, int64_t purpose, const Tensor& out,
                 OptT out_prob, OptT draft_ids, OptT accepted, OptT draft_dist_ids, OptT draft_dist_probs,
                 OptT out_dist_ids, OptT out_dist_probs) {
  const bool f32 = logits_f32(logits);
  need_rows(logits, "logits"); need(out, at::kInt, "out");
  c10::cuda::CUDAGuard guard(logits.device());
  nfb::SampleParams p = {};
  p.logits = logits.data_ptr(); p.logits_f32 = f32; p.ld = logits.stride(0);
  p.T = static_cast<int>(logits.size(0)); p.V = static_cast<int>(logits.size(1));
  p.temperature = ptr_or_null<const float>(temperature); p.top_k = ptr_or_null<const int>(top_k);
  p.top_p = ptr_or_null<const float>(top_p); p.min_p = ptr_or_null<const float>(min_p);
  p.presence = ptr_or_null<const float>(presence); p.frequency = ptr_or_null<const float>(frequency);
  p.token_counts = ptr_or_null<const int>(token_counts);
  p.seeds = ptr_or_null<const unsigned long long>(seeds); p.positions = ptr_or_null<const int>(positions);
  p.purpose = static_cast<unsigned int>(purpose);
  p.out = static_cast<int*>(out.data_ptr()); p.out_prob = ptr_or_null<float>(out_prob);
  if (draft_ids.has_value() && draft_ids->defined()) {
    need(*draft_ids, at::kInt, "draft_ids");
    TORCH_CHECK(draft_ids->numel() >= p.T, "draft_ids: one entry per row");
    p.draft_ids = static_cast<const int*>(draft_ids->data_ptr());
  }
  if (accepted.has_value() && accepted->defined()) {
    need(*accepted, at::kInt, "accepted");
    TORCH_CHECK(accepted->numel() >= p.T, "accepted: one entry per row");
    p.accepted = static_cast<int*>(accepted->data_ptr());
  }
  if (draft_dist_ids.has_value() && draft_dist_ids->defined()) {
    TORCH_CHECK(draft_dist_probs.has_value() && draft_dist_probs->defined() && p.draft_ids != nullptr,
                "draft distribution needs ids, probabilities and draft_ids");
    need(*draft_dist_ids, at::kInt, "draft_dist_ids"); need(*draft_dist_probs, at::kFloat, "draft_dist_probs");
    TORCH_CHECK(draft_dist_ids->is_contiguous() && draft_dist_probs->is_contiguous() && draft_dist_ids->dim() == 2 &&
                draft_dist_ids->size(0) >= p.T && draft_dist_probs->sizes() == draft_dist_ids->sizes(), "draft distribution shapes");
    p.draft_dist_ids = static_cast<const int*>(draft_dist_ids->data_ptr());
    p.draft_dist_probs = static_cast<const float*>(draft_dist_probs->data_ptr());
    p.dist_k = static_cast<int>(draft_dist_ids->size(1));
  }
  if (out_dist_ids.has_value() && out_dist_ids->defined()) {
    TORCH_CHECK(out_dist_probs.has_value() && out_dist_probs->defined(), "out_dist needs ids and probabilities");
    need(*out_dist_ids, at::kInt, "out_dist_ids"); need(*out_dist_probs, at::kFloat, "out_dist_probs");
    TORCH_CHECK(out_dist_ids->is_contiguous() && out_dist_probs->is_contiguous() && out_dist_ids->dim() == 2 &&
                out_dist_ids->size(0) >= p.T && out_dist_probs->sizes() == out_dist_ids->sizes(), "out distribution shapes");
    p.out_dist_ids = static_cast<int*>(out_dist_ids->data_ptr());
    p.out_dist_probs = static_cast<float*>(out_dist_probs->data_ptr());
    p.dist_out_k = static_cast<int>(out_dist_ids->size(1));
  }
  chk(nfb::sample_rows(p, cur_stream()));
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("gemm_bf16(Tensor x, Tensor w, Tensor? out, int epi, Tensor? resid, Tensor? bias, Tensor? partial, int splits, Tensor? status, bool pdl, int act=0, Tensor? conv_w=None, Tensor? conv_state=None, Tensor? conv_slot=None, Tensor? conv_out=None, Tensor? prefetch=None, Tensor? out32=None, int out32_from=0, Tensor? act_params=None, float[] glu=[]) -> ()", &gemm_bf16);
  m.def("gemm_pick_splits(int T, int N, int K, int epi) -> int", &gemm_pick_splits);
  m.def("argmax_rows(Tensor logits, Tensor out, bool pdl) -> ()", &argmax_rows);
  m.def("sample_rows(Tensor logits, Tensor? temperature, Tensor? top_k, Tensor? top_p, Tensor? min_p, Tensor? presence, Tensor? frequency, Tensor? token_counts, Tensor? seeds, Tensor? positions, int purpose, Tensor out, Tensor? out_prob, Tensor? draft_ids=None, Tensor? accepted=None, Tensor? draft_dist_ids=None, Tensor? draft_dist_probs=None, Tensor? out_dist_ids=None, Tensor? out_dist_probs=None) -> ()", &sample_rows);
}
