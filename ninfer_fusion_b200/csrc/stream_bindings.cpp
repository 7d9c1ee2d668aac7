// torch.ops.nfb200.*: row steps of decoders with several residual streams, and sums over experts (layer-list decoders,
// models/layered.py).  Activations are bf16 or fp32; every op takes its element type from its tensors.
#include "pointwise/mixture_args.h"

namespace {

using namespace nfb_bind;

// x_in: [T, S, N], or null with ids and the embedding table
void stream_rows(OptT x_in, OptT ids, OptT table, OptT x_out, OptT delta, OptT gate, OptT choice, OptT weight, OptT ret, OptT h,
                 int64_t n_experts, OptT mix, OptT w_out, const Tensor& w_in, const Tensor& w_next, const Tensor& out, int64_t n_true,
                 double eps, bool pdl) {
  nfb::StreamArgs a;
  a.f32 = act_f32(out, "out");
  need_rows(out, "out");
  const int64_t T = out.size(0), N = out.size(1), S = w_in.numel();
  need_vec(w_in, at::kFloat, S, "w_in"); need_vec(w_next, at::kFloat, N, "w_next");
  if (x_in.has_value() && x_in->defined()) {
    need_vec(*x_in, at::kFloat, T * S * N, "x_in");
    a.x_in = static_cast<const float*>(x_in->data_ptr());
  } else {
    TORCH_CHECK(ids.has_value() && table.has_value(), "stream_rows: neither streams nor an embedding table");
    need_vec(*ids, at::kInt, T, "ids"); need(*table, out.scalar_type(), "table");
    TORCH_CHECK(table->dim() == 2 && table->is_contiguous() && table->size(1) == N, "stream_rows: table shape");
    a.ids = static_cast<const int*>(ids->data_ptr()); a.table = table->data_ptr(); a.vocab = static_cast<int>(table->size(0));
  }
  if (x_out.has_value() && x_out->defined()) {
    need_vec(*x_out, at::kFloat, T * S * N, "x_out");
    a.x_out = static_cast<float*>(x_out->data_ptr());
  }
  a.y = mixture_parts(T, N, out.scalar_type(), delta, gate, choice, weight, ret, h, n_experts);
  if (mix.has_value() && mix->defined()) {
    TORCH_CHECK(w_out.has_value(), "stream_rows: w_out");
    need_vec(*mix, at::kFloat, S * S, "mix"); need_vec(*w_out, at::kFloat, S, "w_out");
    a.mix = static_cast<const float*>(mix->data_ptr()); a.w_out = static_cast<const float*>(w_out->data_ptr());
  }
  a.w_in = static_cast<const float*>(w_in.data_ptr()); a.w_next = static_cast<const float*>(w_next.data_ptr());
  a.out = out.data_ptr(); a.ld_out = out.stride(0);
  a.T = static_cast<int>(T); a.S = static_cast<int>(S); a.N = static_cast<int>(N); a.n_true = static_cast<int>(n_true);
  a.eps = static_cast<float>(eps);
  c10::cuda::CUDAGuard guard(out.device());
  chk(nfb::stream_rows(a, cur_stream(), pdl));
}

void mixture_rows(OptT delta, OptT gate, const Tensor& choice, const Tensor& weight, const Tensor& ret, const Tensor& h, int64_t n_experts,
                  const Tensor& out, bool pdl) {
  TORCH_CHECK(out.dim() == 2, "mixture_rows: out must be [T, N]");
  const int64_t T = out.size(0), N = out.size(1);
  need_vec(out, at::kFloat, T * N, "out");
  const bool f32 = act_f32(h, "h");
  const nfb::MixtureParts y = mixture_parts(T, N, h.scalar_type(), delta, gate, choice, weight, ret, h, n_experts);
  c10::cuda::CUDAGuard guard(out.device());
  chk(nfb::mixture_rows(y, static_cast<float*>(out.data_ptr()), static_cast<int>(T), static_cast<int>(N), f32, cur_stream(), pdl));
}

// x [T, 2 F] (gate | up) -> out [T, F]
void glu_rows_f32(const Tensor& x, const Tensor& out, double limit, double slope, double shift, bool pdl) {
  need(x, at::kFloat, "x"); need(out, at::kFloat, "out"); need_rows(x, "x"); need_rows(out, "out");
  TORCH_CHECK(x.size(0) == out.size(0) && x.size(1) == 2 * out.size(1), "glu_rows_f32: shapes");
  c10::cuda::CUDAGuard guard(x.device());
  chk(nfb::glu_rows_f32(static_cast<const float*>(x.data_ptr()), x.stride(0), static_cast<float*>(out.data_ptr()), out.stride(0), x.size(0),
                        static_cast<int>(out.size(1)), static_cast<float>(limit), static_cast<float>(slope), static_cast<float>(shift),
                        cur_stream(), pdl));
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("stream_rows(Tensor? x_in, Tensor? ids, Tensor? table, Tensor? x_out, Tensor? delta, Tensor? gate, Tensor? choice, Tensor? weight, Tensor? ret, Tensor? h, int n_experts, Tensor? mix, Tensor? w_out, Tensor w_in, Tensor w_next, Tensor out, int n_true, float eps, bool pdl) -> ()", &stream_rows);
  m.def("mixture_rows(Tensor? delta, Tensor? gate, Tensor choice, Tensor weight, Tensor ret, Tensor h, int n_experts, Tensor out, bool pdl) -> ()", &mixture_rows);
  m.def("glu_rows_f32(Tensor x, Tensor out, float limit, float slope, float shift, bool pdl) -> ()", &glu_rows_f32);
}
