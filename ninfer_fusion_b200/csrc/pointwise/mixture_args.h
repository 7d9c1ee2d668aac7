// Argument checks of sublayer outputs in parts, for the bindings of the row kernels.
#pragma once
#include "binding_util.h"
#include "pointwise/stream_rows.h"

namespace nfb_bind {

inline nfb::MixtureParts mixture_parts(int64_t T, int64_t N, at::ScalarType act, OptT delta, OptT gate, OptT choice, OptT weight, OptT ret, OptT h,
                                       int64_t n_experts) {
  nfb::MixtureParts y;
  if (delta.has_value() && delta->defined()) {
    need_vec(*delta, at::kFloat, T * N, "delta");
    y.delta = static_cast<const float*>(delta->data_ptr());
  }
  if (gate.has_value() && gate->defined()) {
    need(*gate, at::kFloat, "gate"); need_rows(*gate, "gate");
    TORCH_CHECK(gate->size(0) >= T && gate->size(1) >= 1, "gate shape");
    y.gate = static_cast<const float*>(gate->data_ptr()); y.ld_gate = gate->stride(0);
  }
  if (choice.has_value() && choice->defined()) {
    TORCH_CHECK(choice->dim() == 2 && weight.has_value() && ret.has_value() && h.has_value(), "expert sum: choices need weights, rows and the input");
    const int64_t k = choice->size(1);
    need_vec(*choice, at::kInt, T * k, "choice"); need_vec(*weight, at::kFloat, T * k, "weight"); need_vec(*ret, act, T * k * N, "ret");
    need(*h, act, "h"); need_rows(*h, "h");
    TORCH_CHECK(h->size(0) >= T && h->size(1) >= N, "h shape");
    y.choice = static_cast<const int*>(choice->data_ptr()); y.weight = static_cast<const float*>(weight->data_ptr());
    y.ret = ret->data_ptr(); y.h = h->data_ptr(); y.ld_h = h->stride(0);
    y.k = static_cast<int>(k); y.n_experts = static_cast<int>(n_experts);
  }
  return y;
}

}  // namespace nfb_bind
