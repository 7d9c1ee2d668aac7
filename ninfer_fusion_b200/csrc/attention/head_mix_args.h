// Argument checks that the bindings of the paged attention kernels share.
#pragma once
#include "attention/head_mix.h"
#include "binding_util.h"

namespace nfb_bind {

inline nfb::HeadMixArgs head_mix_args(const Tensor& q, const Tensor& k_pages, const Tensor& v_pages, const Tensor& block_table,
                               const Tensor& table_row, const Tensor& kv_len, int64_t window, double scale, double softcap,
                               double sink, OptT mix, OptT slope, OptT gate, const Tensor& out, bool pdl, int64_t chunk, OptT sinks,
                               bool sigmoid, OptT log_rate, OptT log_step, OptT offset) {
  nfb::HeadMixArgs a;
  a.f32 = act_f32(q, "q");
  const auto dt = q.scalar_type();
  need_rows(q, "q"); need_rows(out, "out"); need(out, dt, "out");
  need(k_pages, dt, "k_pages"); need(v_pages, dt, "v_pages"); need(block_table, at::kInt, "block_table");
  TORCH_CHECK(k_pages.dim() == 4 && k_pages.is_contiguous() && v_pages.dim() == 4 && v_pages.is_contiguous() &&
              k_pages.size(0) == v_pages.size(0) && k_pages.size(1) == v_pages.size(1) && k_pages.size(2) == v_pages.size(2),
              "head_mix attention: pages must be [pages, kv heads, page size, width]");
  TORCH_CHECK(block_table.dim() == 2 && block_table.stride(1) == 1, "block_table must be [rows, pages]");
  const int64_t T = q.size(0), D = k_pages.size(3), V = v_pages.size(3);
  TORCH_CHECK(q.size(1) % D == 0, "head_mix attention: q width");
  const int64_t H = q.size(1) / D;
  TORCH_CHECK(out.size(0) == T && out.size(1) == H * V, "head_mix attention: out shape");
  need_vec(table_row, at::kInt, T, "table_row"); need_vec(kv_len, at::kInt, T, "kv_len");
  if (mix.has_value() && mix->defined()) need_vec(*mix, at::kFloat, H * H, "mix");
  if (slope.has_value() && slope->defined()) need_vec(*slope, at::kFloat, H, "slope");
  if (gate.has_value() && gate->defined()) {
    need(*gate, at::kFloat, "gate"); need_rows(*gate, "gate");
    TORCH_CHECK(gate->size(0) == T && gate->size(1) >= H, "head_mix attention: gate shape");
    a.gate = static_cast<const float*>(gate->data_ptr()); a.ld_gate = gate->stride(0);
  }
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.k_pages = k_pages.data_ptr(); a.v_pages = v_pages.data_ptr();
  a.block_table = static_cast<const int*>(block_table.data_ptr()); a.table_ld = static_cast<int>(block_table.stride(0));
  a.table_row = static_cast<const int*>(table_row.data_ptr()); a.kv_len = static_cast<const int*>(kv_len.data_ptr());
  a.T = static_cast<int>(T); a.n_heads = static_cast<int>(H); a.n_kv = static_cast<int>(k_pages.size(1));
  a.dim = static_cast<int>(D); a.vdim = static_cast<int>(V); a.page_size = static_cast<int>(k_pages.size(2));
  a.window = static_cast<int>(window); a.scale = static_cast<float>(scale); a.softcap = static_cast<float>(softcap);
  a.sink = static_cast<float>(sink); a.chunk = static_cast<int>(chunk);
  if (sinks.has_value() && sinks->defined()) need_vec(*sinks, at::kFloat, H, "sinks");
  a.sinks = ptr_or_null<const float>(sinks);
  for (OptT v : {std::cref(log_rate), std::cref(log_step), std::cref(offset)})
    if (v.has_value() && v->defined()) need_vec(*v, at::kFloat, H, "numbers per head");
  a.sigmoid = sigmoid;
  a.log_rate = ptr_or_null<const float>(log_rate); a.log_step = ptr_or_null<const float>(log_step); a.offset = ptr_or_null<const float>(offset);
  TORCH_CHECK((a.log_rate == nullptr) == (a.log_step == nullptr), "head_mix attention: a logarithmic bias has two numbers per head");
  TORCH_CHECK(sigmoid || (a.log_rate == nullptr && a.offset == nullptr), "head_mix attention: logarithmic bias and offset go with sigmoid weights");
  TORCH_CHECK(!sigmoid || (softcap == 0.0 && sink == 0.0 && a.sinks == nullptr && !(slope.has_value() && slope->defined())),
              "head_mix attention: sigmoid weights have neither cap nor sink nor slope");
  a.mix = ptr_or_null<const float>(mix); a.slope = ptr_or_null<const float>(slope);
  a.out = out.data_ptr(); a.ldo = out.stride(0);
  a.stream = cur_stream(); a.pdl = pdl;
  return a;
}

}  // namespace nfb_bind
