// Helpers of the torch binding files: argument checks, optional tensors, current stream.
#pragma once
#include <ATen/ATen.h>
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/library.h>

#include "gemm/gemm.h"

namespace nfb_bind {

using at::Tensor;
using OptT = const std::optional<Tensor>&;

inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }

inline void chk(const char* err) { TORCH_CHECK(err == nullptr, err ? err : ""); }

inline void need_cuda(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
}
inline void need(const Tensor& t, at::ScalarType dt, const char* name) {
  need_cuda(t, name);
  TORCH_CHECK(t.scalar_type() == dt, name, " has the wrong dtype");
}
inline void need_rows(const Tensor& t, const char* name) {
  TORCH_CHECK(t.dim() == 2 && t.stride(1) == 1, name, " must be 2-D with unit inner stride");
}
template <typename T>
inline T* ptr_or_null(OptT t) {
  return t.has_value() && t->defined() ? static_cast<T*>(t->data_ptr()) : nullptr;
}

// Activation tensors are bf16 or fp32.
inline bool act_f32(const Tensor& t, const char* name) {
  need_cuda(t, name);
  TORCH_CHECK(t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat, name, " must be bf16 or fp32");
  return t.scalar_type() == at::kFloat;
}
inline void need_vec(const Tensor& t, at::ScalarType dt, int64_t n, const char* name) {
  need(t, dt, name);
  TORCH_CHECK(t.is_contiguous() && t.numel() >= n, name, " is too small or not contiguous");
}


inline int64_t sm_count() {
  static int n = 0;
  if (n == 0) n = at::cuda::getCurrentDeviceProperties()->multiProcessorCount;
  return n;
}

// Optional L2 prefetch hint: a (contiguous) tensor the next kernel will stream; at most the first 32 MB are asked for.
inline void fill_prefetch(nfb::GemmArgs& a, OptT next) {
  if (!(next.has_value() && next->defined() && next->is_cuda() && next->is_contiguous())) return;
  a.prefetch = next->data_ptr();
  const int64_t bytes = next->numel() * next->element_size();
  a.prefetch_bytes = bytes < (32 << 20) ? bytes : (32 << 20);
}

// Optional decode conv epilogue (nfb::GemmConv): all four tensors or none.
inline void fill_conv(nfb::GemmArgs& a, OptT conv_w, OptT conv_state, OptT conv_slot, OptT conv_out) {
  if (!(conv_state.has_value() && conv_state->defined())) return;
  TORCH_CHECK(conv_w.has_value() && conv_slot.has_value() && conv_out.has_value(), "conv epilogue: all four tensors");
  need(*conv_w, at::kBFloat16, "conv_w"); need(*conv_state, at::kBFloat16, "conv_state");
  need(*conv_slot, at::kInt, "conv_slot"); need(*conv_out, at::kBFloat16, "conv_out");
  TORCH_CHECK(conv_w->dim() == 2 && conv_w->size(1) == 4 && conv_w->is_contiguous(), "conv_w must be [C, 4]");
  const int64_t C = conv_w->size(0);
  TORCH_CHECK(conv_state->dim() == 3 && conv_state->size(1) == 3 && conv_state->size(2) == C && conv_state->is_contiguous(),
              "conv_state must be [slots, 3, C]");
  TORCH_CHECK(conv_out->dim() == 2 && conv_out->size(0) == a.T && conv_out->size(1) == C && conv_out->is_contiguous(),
              "conv_out must be [T, C]");
  TORCH_CHECK(conv_slot->numel() >= a.T && conv_slot->is_contiguous(), "conv_slot must hold one slot per token");
  a.conv.w = conv_w->data_ptr(); a.conv.state = conv_state->data_ptr();
  a.conv.slot = static_cast<const int*>(conv_slot->data_ptr()); a.conv.out = conv_out->data_ptr();
  a.conv.C = static_cast<int>(C);
}

// out = epilogue(x @ w^T).  epi: 0 store(+bias), 1 residual add, 2 swiglu, 3 split-K partials.
}  // namespace nfb_bind
