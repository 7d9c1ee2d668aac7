// torch.ops.nfb200.*: state-space recurrence (layer-list decoders, models/layered.py).  Activations are bf16 or fp32; every op takes
// its element type from its tensors.
#include "binding_util.h"
#include "ssd/ssd.h"

namespace {

using namespace nfb_bind;

// proj [T, columns] with the convolved channels from x_off on; dt [T, >= H] raw steps.  One token per sequence: one kernel.  Else
// `u` [T, K] takes the convolved channels, and the recurrence runs in chunks (chunk_ws) or token by token.
void ssd(const Tensor& proj, int64_t x_off, const Tensor& dt, const Tensor& conv_w, const Tensor& conv_b, const Tensor& rate, const Tensor& skip,
         int64_t groups, const Tensor& cu_seqlens, const Tensor& token_seq, const Tensor& cache_pos, const Tensor& state_slot, const Tensor& ring,
         const Tensor& S, OptT u, const Tensor& out, bool write_state, OptT chunk_ws, bool pdl, bool one_token) {
  nfb::SsdArgs a;
  a.f32 = act_f32(proj, "proj");
  const auto act = proj.scalar_type();
  need_rows(proj, "proj"); need_rows(out, "out"); need(out, act, "out");
  need(S, at::kFloat, "S"); need(ring, at::kFloat, "ring");
  TORCH_CHECK(S.dim() == 4 && S.is_contiguous() && ring.dim() == 3 && ring.is_contiguous() && ring.size(0) == S.size(0),
              "ssd: S [slots, H, V, N] and ring [slots, taps, K] expected");
  const int64_t T = proj.size(0), H = S.size(1), V = S.size(2), N = S.size(3), B = state_slot.numel(), taps = ring.size(1);
  const int64_t K = H * V + 2 * groups * N;
  TORCH_CHECK(groups >= 1 && H % groups == 0, "ssd: heads must be a multiple of groups");
  TORCH_CHECK(ring.size(2) == K, "ssd: ring width");
  TORCH_CHECK(x_off >= 0 && x_off + K <= proj.size(1), "ssd: projection columns");
  TORCH_CHECK(out.size(0) == T && out.size(1) == H * V, "ssd: out shape");
  need(dt, at::kFloat, "dt"); need_rows(dt, "dt");
  TORCH_CHECK(dt.size(0) >= T && dt.size(1) >= H, "ssd: dt shape");
  need_vec(conv_w, at::kFloat, taps * K, "conv_w"); need_vec(conv_b, at::kFloat, K, "conv_b");
  need_vec(rate, at::kFloat, H, "rate"); need_vec(skip, at::kFloat, H, "skip");
  need_vec(cu_seqlens, at::kInt, B + 1, "cu_seqlens"); need_vec(state_slot, at::kInt, B, "state_slot");
  need_vec(token_seq, at::kInt, T, "token_seq"); need_vec(cache_pos, at::kInt, T, "cache_pos");
  a.proj = proj.data_ptr(); a.ldp = proj.stride(0); a.x_off = static_cast<int>(x_off);
  a.dt = static_cast<const float*>(dt.data_ptr()); a.ld_dt = dt.stride(0);
  a.T = static_cast<int>(T); a.n_heads = static_cast<int>(H); a.groups = static_cast<int>(groups); a.vdim = static_cast<int>(V);
  a.state = static_cast<int>(N); a.taps = static_cast<int>(taps);
  a.conv_w = static_cast<const float*>(conv_w.data_ptr()); a.conv_b = static_cast<const float*>(conv_b.data_ptr());
  a.rate = static_cast<const float*>(rate.data_ptr()); a.skip = static_cast<const float*>(skip.data_ptr());
  a.cu_seqlens = static_cast<const int*>(cu_seqlens.data_ptr()); a.token_seq = static_cast<const int*>(token_seq.data_ptr());
  a.cache_pos = static_cast<const int*>(cache_pos.data_ptr()); a.state_slot = static_cast<const int*>(state_slot.data_ptr());
  a.n_seq = static_cast<int>(B);
  a.ring = static_cast<float*>(ring.data_ptr()); a.S = static_cast<float*>(S.data_ptr());
  a.out = out.data_ptr(); a.ldo = out.stride(0); a.write_state = write_state;
  c10::cuda::CUDAGuard guard(proj.device());
  a.stream = cur_stream(); a.pdl = pdl;
  if (one_token) {
    TORCH_CHECK(T == B, "ssd: one token per sequence expected");
    chk(nfb::ssd_decode(a));
    return;
  }
  TORCH_CHECK(u.has_value() && u->defined(), "ssd: portions need room for the convolved channels");
  need_vec(*u, act, T * K, "u");
  a.u = u->data_ptr();
  chk(nfb::ssd_conv(a));
  if (chunk_ws.has_value() && chunk_ws->defined()) {
    need_cuda(*chunk_ws, "chunk_ws");
    chk(nfb::ssd_chunked(a, chunk_ws->data_ptr(), chunk_ws->numel() * chunk_ws->element_size()));
  } else {
    chk(nfb::ssd_recurrent(a));
  }
}

// y [T, H * vdim] in place: rms of each of `norm_groups` parts of y * silu(z), times norm
void ssd_gated_norm(const Tensor& y, const Tensor& z, const Tensor& norm, int64_t n_heads, int64_t vdim_true, int64_t norm_groups, double eps,
                    bool pdl) {
  nfb::SsdNormArgs a;
  a.f32 = act_f32(y, "y");
  need_rows(y, "y"); need_rows(z, "z"); need(z, y.scalar_type(), "z");
  const int64_t T = y.size(0), C = y.size(1);
  TORCH_CHECK(n_heads >= 1 && C % n_heads == 0 && z.size(0) >= T && z.size(1) >= C, "ssd_gated_norm: shapes");
  need_vec(norm, at::kFloat, C, "norm");
  a.y = y.data_ptr(); a.ldo = y.stride(0); a.z = z.data_ptr(); a.ldz = z.stride(0); a.norm = static_cast<const float*>(norm.data_ptr());
  a.T = static_cast<int>(T); a.n_heads = static_cast<int>(n_heads); a.vdim = static_cast<int>(C / n_heads);
  a.vdim_true = static_cast<int>(vdim_true); a.norm_groups = static_cast<int>(norm_groups); a.eps = static_cast<float>(eps);
  c10::cuda::CUDAGuard guard(y.device());
  a.stream = cur_stream(); a.pdl = pdl;
  chk(nfb::ssd_gated_norm(a));
}

int64_t ssd_chunked_workspace_bytes(int64_t T, int64_t n_seq, int64_t n_heads, int64_t state, int64_t vdim) {
  return nfb::ssd_chunked_workspace_bytes(static_cast<int>(T), static_cast<int>(n_seq), static_cast<int>(n_heads), static_cast<int>(state),
                                          static_cast<int>(vdim));
}
bool ssd_chunked_supported(int64_t state, int64_t vdim) { return nfb::ssd_chunked_supported(static_cast<int>(state), static_cast<int>(vdim)); }

}  // namespace

TORCH_LIBRARY_FRAGMENT(nfb200, m) {
  m.def("ssd(Tensor proj, int x_off, Tensor dt, Tensor conv_w, Tensor conv_b, Tensor rate, Tensor skip, int groups, Tensor cu_seqlens, Tensor token_seq, Tensor cache_pos, Tensor state_slot, Tensor ring, Tensor S, Tensor? u, Tensor out, bool write_state, Tensor? chunk_ws, bool pdl, bool one_token=False) -> ()", &ssd);
  m.def("ssd_gated_norm(Tensor y, Tensor z, Tensor norm, int n_heads, int vdim_true, int norm_groups, float eps, bool pdl) -> ()", &ssd_gated_norm);
  m.def("ssd_chunked_workspace_bytes(int T, int n_seq, int n_heads, int state, int vdim) -> int", &ssd_chunked_workspace_bytes);
  m.def("ssd_chunked_supported(int state, int vdim) -> bool", &ssd_chunked_supported);
}
