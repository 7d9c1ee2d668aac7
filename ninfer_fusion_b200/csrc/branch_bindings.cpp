// torch.ops.nfb200.*: row steps of decoders that norm their sublayers' outputs (layer-list decoders, models/layered.py).
// Activations are bf16 or fp32; every op takes its element type from its tensors.
#include "pointwise/branch_rows.h"
#include "pointwise/mixture_args.h"

namespace {

using namespace nfb_bind;

// Two branches (branch_a, branch_b, w_a, w_b), or a sublayer's output in parts (delta ... n_experts).
void branch_rows(const Tensor& x, OptT branch_a, OptT branch_b, OptT w_a, OptT w_b, OptT delta, OptT gate, OptT choice, OptT weight, OptT ret,
                 OptT h, int64_t n_experts, const Tensor& w, OptT w_final, const Tensor& out, int64_t n_true, double eps, bool pdl) {
  nfb::BranchRowsArgs a;
  a.f32 = act_f32(out, "out");
  need_rows(out, "out");
  const int64_t T = out.size(0), N = out.size(1);
  TORCH_CHECK(x.dim() == 2 && x.size(0) == T && x.size(1) == N, "branch_rows: x must be [T, N]");
  need_vec(x, at::kFloat, T * N, "x"); need_vec(w, at::kFloat, N, "w");
  if (branch_a.has_value() && branch_a->defined()) {
    TORCH_CHECK(branch_b.has_value() && w_a.has_value() && w_b.has_value(), "branch_rows: two branches need two rows and two weights");
    need_vec(*branch_a, at::kFloat, T * N, "branch_a"); need_vec(*branch_b, at::kFloat, T * N, "branch_b");
    need_vec(*w_a, at::kFloat, N, "w_a"); need_vec(*w_b, at::kFloat, N, "w_b");
    a.a = static_cast<const float*>(branch_a->data_ptr()); a.b = static_cast<const float*>(branch_b->data_ptr());
    a.w_a = static_cast<const float*>(w_a->data_ptr()); a.w_b = static_cast<const float*>(w_b->data_ptr());
  } else {
    a.y = mixture_parts(T, N, out.scalar_type(), delta, gate, choice, weight, ret, h, n_experts);
  }
  if (w_final.has_value() && w_final->defined()) {
    need_vec(*w_final, at::kFloat, N, "w_final");
    a.w_final = static_cast<const float*>(w_final->data_ptr());
  }
  a.x = static_cast<float*>(x.data_ptr()); a.w = static_cast<const float*>(w.data_ptr());
  a.out = out.data_ptr(); a.ld_out = out.stride(0);
  a.T = static_cast<int>(T); a.N = static_cast<int>(N); a.n_true = static_cast<int>(n_true); a.eps = static_cast<float>(eps);
  c10::cuda::CUDAGuard guard(out.device());
  chk(nfb::branch_rows(a, cur_stream(), pdl));
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("branch_rows(Tensor x, Tensor? branch_a, Tensor? branch_b, Tensor? w_a, Tensor? w_b, Tensor? delta, Tensor? gate, Tensor? choice, Tensor? weight, Tensor? ret, Tensor? h, int n_experts, Tensor w, Tensor? w_final, Tensor out, int n_true, float eps, bool pdl) -> ()", &branch_rows);
}
