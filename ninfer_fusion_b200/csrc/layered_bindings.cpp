// torch.ops.nfb200.*: ops that all layer-list decoders (models/layered.py) share: 32-bit residual rows and the 32-bit GEMM.
// Activations are bf16 or fp32; every op takes its element type from its tensors.
#include "binding_util.h"
#include "gemm/gemm_f32.h"
#include "pointwise/rows32.h"

namespace {

using namespace nfb_bind;

void embed_rows32(const Tensor& ids, const Tensor& table, const Tensor& x32, const Tensor& xa, double scale, bool pdl, OptT pos, OptT places) {
  const bool f32 = act_f32(table, "table");
  const int64_t T = ids.numel(), N = table.size(1);
  need_vec(ids, at::kInt, T, "ids");
  need_vec(table, table.scalar_type(), table.size(0) * N, "table");
  need_vec(x32, at::kFloat, T * N, "x32");
  need(xa, table.scalar_type(), "xa"); need_rows(xa, "xa");
  TORCH_CHECK(xa.size(0) == T && xa.size(1) == N, "embed_rows32: xa shape");
  const void* at = nullptr;
  int64_t n_places = 0;
  if (places.has_value() && places->defined()) {
    TORCH_CHECK(pos.has_value() && pos->defined() && places->dim() == 2 && places->size(1) == N, "embed_rows32: position table");
    n_places = places->size(0);
    need_vec(*places, table.scalar_type(), n_places * N, "places"); need_vec(*pos, at::kInt, T, "pos");
    at = places->data_ptr();
  }
  c10::cuda::CUDAGuard guard(table.device());
  chk(nfb::embed_rows32(static_cast<const int*>(ids.data_ptr()), table.data_ptr(), static_cast<float*>(x32.data_ptr()),
                        xa.data_ptr(), static_cast<int>(T), static_cast<int>(N), xa.stride(0), static_cast<float>(scale),
                        static_cast<int>(table.size(0)), ptr_or_null<const int>(pos), at, static_cast<int>(n_places), f32,
                        cur_stream(), pdl));
}

void post_norm_rows(const Tensor& x32, OptT delta, const Tensor& xa, int64_t n_true, double alpha, double eps, OptT gain,
                    OptT final_gain, bool pdl) {
  const bool f32 = act_f32(xa, "xa");
  TORCH_CHECK(x32.dim() == 2, "x32 must be [T, N]");
  nfb::PostNormArgs a;
  a.T = static_cast<int>(x32.size(0)); a.N = static_cast<int>(x32.size(1));
  const int64_t n = x32.numel();
  need_vec(x32, at::kFloat, n, "x32");
  need_vec(xa, xa.scalar_type(), n, "xa");
  if (delta.has_value() && delta->defined()) need_vec(*delta, at::kFloat, n, "delta");
  if (gain.has_value() && gain->defined()) need_vec(*gain, at::kFloat, 1, "gain");
  if (final_gain.has_value() && final_gain->defined()) need_vec(*final_gain, at::kFloat, 1, "final_gain");
  a.x32 = static_cast<float*>(x32.data_ptr()); a.delta = ptr_or_null<const float>(delta); a.xa = xa.data_ptr();
  a.n_true = static_cast<int>(n_true); a.alpha = static_cast<float>(alpha); a.eps = static_cast<float>(eps);
  a.gain = ptr_or_null<const float>(gain); a.final_gain = ptr_or_null<const float>(final_gain); a.f32 = f32;
  c10::cuda::CUDAGuard guard(x32.device());
  chk(nfb::post_norm_rows(a, cur_stream(), pdl));
}

void gemm_f32(const Tensor& x, const Tensor& w, OptT out, OptT bias, int64_t act, OptT act_params, OptT out32, int64_t out32_from) {
  need(x, at::kFloat, "x"); need(w, at::kFloat, "w");
  need_rows(x, "x"); need_rows(w, "w");
  TORCH_CHECK(x.size(1) == w.size(1), "gemm_f32: K mismatch");
  TORCH_CHECK(act >= 0 && act <= 5, "gemm_f32: unknown activation");
  nfb::GemmF32Args a;
  a.w = static_cast<const float*>(w.data_ptr()); a.N = w.size(0); a.K = w.size(1); a.ldw = w.stride(0);
  a.x = static_cast<const float*>(x.data_ptr()); a.T = x.size(0); a.ldx = x.stride(0);
  const bool split = out32.has_value() && out32->defined();
  TORCH_CHECK(out32_from >= 0 && out32_from <= a.N, "gemm_f32: bad column split");
  if (split) {
    need(*out32, at::kFloat, "out32"); need_rows(*out32, "out32");
    TORCH_CHECK(out32->size(0) == a.T && out32->size(1) >= a.N - out32_from, "gemm_f32: out32 shape");
    a.out2 = static_cast<float*>(out32->data_ptr()); a.ldo2 = out32->stride(0); a.out2_from = static_cast<int>(out32_from);
  }
  if (!(split && out32_from == 0)) {
    TORCH_CHECK(out.has_value() && out->defined(), "gemm_f32: out required");
    need(*out, at::kFloat, "out"); need_rows(*out, "out");
    TORCH_CHECK(out->size(0) == a.T && out->size(1) >= (split ? out32_from : a.N), "gemm_f32: out shape");
    a.out = static_cast<float*>(out->data_ptr()); a.ldo = out->stride(0);
  }
  if (bias.has_value() && bias->defined()) { need_vec(*bias, at::kFloat, a.N, "bias"); a.bias = static_cast<const float*>(bias->data_ptr()); }
  a.act = static_cast<int>(act);
  if (act_params.has_value() && act_params->defined()) {
    need_vec(*act_params, at::kFloat, 2, "act_params");
    a.act_params = static_cast<const float*>(act_params->data_ptr());
  }
  c10::cuda::CUDAGuard guard(x.device());
  a.stream = cur_stream();
  chk(nfb::gemm_f32(a));
}

void sandwich_rows(const Tensor& x_in, const Tensor& x_out, OptT delta, OptT w_post, OptT w_next, const Tensor& out, int64_t n_true,
                   int64_t groups, double mult, double eps, OptT conv_w, OptT conv_state, OptT cu_seqlens, OptT state_slot,
                   int64_t max_seq_tokens, bool write_state, bool pdl) {
  nfb::SandwichArgs a = {};
  a.f32 = act_f32(out, "out");
  TORCH_CHECK(x_in.dim() == 2 && x_out.sizes() == x_in.sizes(), "sandwich_rows: x must be [T, N]");
  const int64_t T = x_in.size(0), N = x_in.size(1);
  need_vec(x_in, at::kFloat, T * N, "x_in"); need_vec(x_out, at::kFloat, T * N, "x_out");
  need_rows(out, "out");
  TORCH_CHECK(out.size(0) == T && out.size(1) == N, "sandwich_rows: out shape");
  a.x_in = static_cast<const float*>(x_in.data_ptr()); a.x_out = static_cast<float*>(x_out.data_ptr());
  if (delta.has_value() && delta->defined()) need_vec(*delta, at::kFloat, T * N, "delta");
  if (w_post.has_value() && w_post->defined()) need_vec(*w_post, at::kFloat, N, "w_post");
  if (w_next.has_value() && w_next->defined()) need_vec(*w_next, at::kFloat, N, "w_next");
  a.delta = ptr_or_null<const float>(delta); a.w_post = ptr_or_null<const float>(w_post); a.w_next = ptr_or_null<const float>(w_next);
  a.out = out.data_ptr(); a.ld_out = out.stride(0);
  a.T = static_cast<int>(T); a.N = static_cast<int>(N); a.n_true = static_cast<int>(n_true); a.groups = static_cast<int>(groups);
  a.mult = static_cast<float>(mult); a.eps = static_cast<float>(eps); a.write_state = write_state;
  if (conv_w.has_value() && conv_w->defined()) {
    need(*conv_w, at::kFloat, "conv_w");
    TORCH_CHECK(conv_w->dim() == 2 && conv_w->size(1) == N && conv_w->is_contiguous(), "sandwich_rows: conv_w must be [taps, N]");
    a.taps = static_cast<int>(conv_w->size(0)); a.conv_w = static_cast<const float*>(conv_w->data_ptr());
    TORCH_CHECK(cu_seqlens.has_value() && state_slot.has_value(), "sandwich_rows: a convolution needs the sequences");
    a.n_seq = static_cast<int>(state_slot->numel()); a.max_seq_tokens = static_cast<int>(max_seq_tokens);
    need_vec(*cu_seqlens, at::kInt, a.n_seq + 1, "cu_seqlens"); need_vec(*state_slot, at::kInt, a.n_seq, "state_slot");
    a.cu_seqlens = static_cast<const int*>(cu_seqlens->data_ptr()); a.state_slot = static_cast<const int*>(state_slot->data_ptr());
    if (a.taps > 1) {
      TORCH_CHECK(conv_state.has_value() && conv_state->defined(), "sandwich_rows: a convolution needs its state");
      need(*conv_state, at::kFloat, "conv_state");
      TORCH_CHECK(conv_state->dim() == 3 && conv_state->size(1) == a.taps - 1 && conv_state->size(2) == N && conv_state->is_contiguous(),
                  "sandwich_rows: conv_state must be [slots, taps - 1, N]");
      a.conv_state = static_cast<float*>(conv_state->data_ptr());
    }
  }
  c10::cuda::CUDAGuard guard(x_in.device());
  chk(nfb::sandwich_rows(a, cur_stream(), pdl));
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("embed_rows32(Tensor ids, Tensor table, Tensor x32, Tensor xa, float scale, bool pdl, Tensor? pos=None, Tensor? places=None) -> ()", &embed_rows32);
  m.def("post_norm_rows(Tensor x32, Tensor? delta, Tensor xa, int n_true, float alpha, float eps, Tensor? gain, Tensor? final_gain, bool pdl) -> ()", &post_norm_rows);
  m.def("gemm_f32(Tensor x, Tensor w, Tensor? out, Tensor? bias, int act=0, Tensor? act_params=None, Tensor? out32=None, int out32_from=0) -> ()", &gemm_f32);
  m.def("sandwich_rows(Tensor x_in, Tensor x_out, Tensor? delta, Tensor? w_post, Tensor? w_next, Tensor out, int n_true, int groups, float mult, float eps, Tensor? conv_w, Tensor? conv_state, Tensor? cu_seqlens, Tensor? state_slot, int max_seq_tokens, bool write_state, bool pdl) -> ()", &sandwich_rows);
}
