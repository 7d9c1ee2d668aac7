// Argument checks that the mixture-of-experts bindings share.
#pragma once
#include <ATen/ATen.h>
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/library.h>

#include "moe.h"

namespace nfb_moe_bind {

using at::Tensor;
using OptT = const std::optional<Tensor>&;

inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }
inline void chk(const char* err) { TORCH_CHECK(err == nullptr, err ? err : ""); }
inline void need(const Tensor& t, at::ScalarType dt, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == dt, name, " has the wrong dtype");
  TORCH_CHECK(t.is_contiguous() || (t.dim() == 2 && t.stride(1) == 1), name, " must have unit inner stride");
}
template <typename T>
inline T* ptr_or_null(OptT t) {
  return t.has_value() && t->defined() ? static_cast<T*>(t->data_ptr()) : nullptr;
}
inline nfb::MoeState* state_ptr(const Tensor& state) {
  TORCH_CHECK(state.is_cuda() && state.scalar_type() == at::kByte &&
                  state.numel() >= static_cast<int64_t>(sizeof(nfb::MoeState)), "bad MoE state tensor");
  return reinterpret_cast<nfb::MoeState*>(state.data_ptr());
}

}  // namespace nfb_moe_bind
