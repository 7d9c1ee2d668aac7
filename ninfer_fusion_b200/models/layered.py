"""Decoders described as a list of layers (`models/layered_config.py`): weight packing and the forward pass on the
native kernels.

A layer is a mixer (attention with plain or head-mixed scores or sigmoid weights, latent attention, matrix memory, gated
linear memory, gated linear recurrence, a selective state space, or attention and a state space side by side) and an
optional feed-forward (dense, or experts: `models/experts.py`) on a 32-bit residual stream.  A sublayer meets the stream in
one of four ways: the norm after the sum, ``x <- rms_norm(alpha x + f(x)) * gain``, norms around it,
``x <- x + mult * norm(f(norm(x)))``, with an optional causal convolution in front of every mixer, several streams that it
reads a weighted sum of and mixes, or a norm on its output only, ``x <- x + norm(f(x))``.  Layers can run several times with the same weights; cache and state
belong to layer runs.  Every size and constant is a field of the description, so a design is a mapping onto these fields
(`models/kuzanex.py`, `models/tebivik.py`, `models/tuzupel.py`, `models/ratilorn.py`) and not a model file of its own.

The engine side is the hybrid runtime's: one ragged token batch per step (`runtime/batch.py`), K / V or latent rows in the
paged cache (one geometry per run), recurrent state in per-sequence slots, preallocated buffers so that a decode step can
be captured in a CUDA graph.  Activations are bf16 (tcgen05 GEMMs, tensor-core prefill kernels) or, for exact runs, fp32.
Head widths are padded to multiples of 16 and the model width to a multiple of 8 when the weights are packed: zero rows
and columns change no product, and every norm divides by the true width.
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from .._lib import StatusWord, load_native
from .experts import ExpertWorkspace, pack_experts, pack_unit, run_experts, run_unit
from .hybrid import EPI_STORE, LaunchCounter, StepBatch
from .layered_config import (ATTENTION_KINDS, AttentionMixer, GatedMemoryMixer, GatedRecurrenceMixer, LatentAttentionMixer,
                             LayeredConfig, MatrixMemoryMixer, ParallelMixer, StateSpaceMixer, mixer_parts, pad_to)

ACTIVATIONS = {"xielu": 3, "relu2": 4}     # csrc/gemm/gemm.h GemmActivation
ACT_SOFTCAP = 5
BLOCK_TOKENS = 64          # query tokens per attention block of a step (kHeadMixBlock, kLatentBlock)
PREFILL_MIN_TOKENS = 8     # shorter portions take the token-by-token kernels
EXPAND_BYTES = 4 << 30     # keys and values of expanded latents in flight
SCORE_SCRATCH_BYTES = 1 << 30    # fp32 scores in flight between the two prefill attention kernels


# ---------------------------------------------------------------------------------------------- weight packing
def _pad2(w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    out = torch.zeros((rows, cols), dtype=w.dtype, device=w.device)
    out[: w.shape[0], : w.shape[1]] = w
    return out


def _pad_head_rows(w: torch.Tensor, heads: int, width: int, width_p: int, cols: int) -> torch.Tensor:
    out = torch.zeros((heads, width_p, cols), dtype=w.dtype, device=w.device)
    out[:, :width, : w.shape[1]] = w.reshape(heads, width, w.shape[1])
    return out.reshape(heads * width_p, cols)


def _pad_head_vec(v: torch.Tensor, heads: int, width: int, width_p: int) -> torch.Tensor:
    out = torch.zeros((heads, width_p), dtype=torch.float32, device=v.device)
    out[:, :width] = v.float().reshape(heads, width)
    return out.reshape(-1)


def _pad_head_cols(w: torch.Tensor, heads: int, width: int, width_p: int, rows: int) -> torch.Tensor:
    out = torch.zeros((rows, heads, width_p), dtype=w.dtype, device=w.device)
    out[: w.shape[0], :, :width] = w.reshape(w.shape[0], heads, width)
    return out.reshape(rows, heads * width_p)


def distance_slopes(heads: int) -> torch.Tensor:
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float64)


def check_tensor_shapes(expected, shape_of) -> None:
    """Every (name, shape) of `expected` is there; `shape_of(name)` returns None for a missing tensor."""
    for name, shape in expected:
        have = shape_of(name)
        if have is None:
            raise ValueError(f"checkpoint has no tensor '{name}'")
        if tuple(have) != shape:
            raise ValueError(f"tensor '{name}' has shape {list(have)}, the configuration asks for {list(shape)}")


def _pack_attention(w, p, m: AttentionMixer, get, n_out: int, hp: int, device):
    H, G, D, V, Dp, Vp = m.heads, m.kv_heads, m.dim, m.vdim, m.dim_p, m.vdim_p
    rows = [_pad_head_rows(get("q"), H, D, Dp, hp), _pad_head_rows(get("k"), G, D, Dp, hp), _pad_head_rows(get("v"), G, V, Vp, hp)]
    bias = torch.zeros(n_out, dtype=torch.float32, device=device)
    if m.head_gate:
        rows.append(_pad2(get("g"), H, hp))
    if m.bias:
        b = torch.cat([_pad_head_vec(get("q_bias"), H, D, Dp), _pad_head_vec(get("k_bias"), G, D, Dp),
                       _pad_head_vec(get("v_bias"), G, V, Vp)])
        bias[: b.numel()] = b
    if m.qk_norm:
        w[f"{p}/mix/q_norm"] = _pad_head_vec(get("q_norm"), 1, D, Dp)
        w[f"{p}/mix/k_norm"] = _pad_head_vec(get("k_norm"), 1, D, Dp)
    mix = get("talk").double() if m.head_mixing else torch.eye(H, dtype=torch.float64, device=device)
    if m.head_mixing:
        w[f"{p}/mix/heads"] = mix.float().contiguous()
    if m.distance_bias:
        # mixing is linear: the bias taken off before it is (mix @ slope) taken off after it
        w[f"{p}/mix/slope"] = (mix @ distance_slopes(H).to(device)).float().contiguous()
    if m.bias:
        w[f"{p}/mix/in_bias"] = bias
    if m.sigmoid:
        w[f"{p}/mix/offset"] = get("offset").float().contiguous()
    if m.log_bias:
        w[f"{p}/mix/log_rate"], w[f"{p}/mix/log_step"] = get("log_rate").float().contiguous(), get("log_step").float().contiguous()
    if m.value_mix:
        w[f"{p}/mix/v_lambda"] = get("v_lambda").float().reshape(1)
    if m.head_sink:
        w[f"{p}/mix/sink"] = get("sink").float().contiguous()
    if m.rotary is not None:
        w[f"{p}/mix/freq"] = torch.tensor(m.rotary.frequencies(), dtype=torch.float64, device=device)
    return rows


def _pack_matrix_memory(w, p, m: MatrixMemoryMixer, get, n_out: int, hp: int, device):
    H, D, V, Dp, Vp = m.heads, m.dim, m.vdim, m.dim_p, m.vdim_p
    bias = torch.zeros(n_out, dtype=torch.float32, device=device)
    bias[m.main_cols: m.main_cols + H] = get("i_bias").float()
    bias[m.main_cols + H: m.main_cols + 2 * H] = get("f_bias").float()
    w[f"{p}/mix/in_bias"] = bias
    w[f"{p}/mix/norm"] = _pad_head_vec(get("norm"), H, V, Vp)
    return [_pad_head_rows(get("q"), H, D, Dp, hp), _pad_head_rows(get("k"), H, D, Dp, hp), _pad_head_rows(get("v"), H, V, Vp, hp),
            _pad_head_rows(get("g"), H, V, Vp, hp), _pad2(get("i"), H, hp), _pad2(get("f"), H, hp)]


def _pack_gated_memory(w, p, m: GatedMemoryMixer, get, n_out: int, hp: int, device):
    H, D, V, Dp, Vp = m.heads, m.dim, m.vdim, m.dim_p, m.vdim_p
    bias = torch.zeros(n_out, dtype=torch.float32, device=device)
    bias[m.main_cols: m.main_cols + H * Dp] = _pad_head_vec(get("f_bias"), H, D, Dp)
    lower = torch.ones((H, Dp), dtype=torch.float32, device=device)       # padded channels forget nothing and take nothing in
    lower[:, :D] = get("lower").float().reshape(H, D)
    w[f"{p}/mix/in_bias"] = bias
    w[f"{p}/mix/lower"] = lower.reshape(-1)
    w[f"{p}/mix/norm"] = _pad_head_vec(get("norm"), 1, V, Vp)
    return [_pad_head_rows(get("q"), H, D, Dp, hp), _pad_head_rows(get("v"), H, V, Vp, hp), _pad_head_rows(get("f"), H, D, Dp, hp)]


def _pack_latent(w, p, m: LatentAttentionMixer, get, hp: int, dtype, device):
    H, D, R, V, Q, C = m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank
    Dp, Rp, Vp, Qp, Cp = m.dim_p, m.rot_p, m.vdim_p, m.q_rank_p, m.kv_rank_p
    direct = Q == 0                                                        # queries straight from the input
    uq = (get("q") if direct else get("uq")).reshape(H, D + R, -1)
    cols = uq.shape[2]
    q = torch.zeros((H, Dp + Rp, hp if direct else Qp), dtype=uq.dtype, device=device)
    q[:, :D, :cols] = uq[:, :D]
    q[:, Dp: Dp + R, :cols] = uq[:, D:]
    q = q.reshape(H * (Dp + Rp), -1)
    k, v = _pad_head_rows(get("uk"), H, D, Dp, Cp), _pad_head_rows(get("uv"), H, V, Vp, Cp)
    w[f"{p}/mix/ukv"] = torch.cat([k, v]).to(dtype)                        # rows: keys of all heads, values of all heads
    w[f"{p}/mix/uv"] = w[f"{p}/mix/ukv"][H * Dp:].view(H, Vp, Cp)
    w[f"{p}/mix/uk_t"] = k.reshape(H, Dp, Cp).transpose(1, 2).contiguous().to(dtype)   # takes a query to the latent space
    w[f"{p}/mix/kv_norm"] = _pad_head_vec(get("dkv_norm"), 1, C, Cp)
    w[f"{p}/mix/freq"] = torch.tensor([m.rot_base ** (-2.0 * i / R) for i in range(R // 2)], dtype=torch.float64, device=device)
    if m.sink:
        w[f"{p}/mix/sink"] = get("sink").float().contiguous()
    dkv = get("dkv")
    latent = [_pad2(dkv[:C], Cp, hp), _pad2(dkv[C:], Rp, hp)]
    if direct:
        return [q] + latent
    w[f"{p}/mix/uq"] = q.to(dtype)
    w[f"{p}/mix/q_norm"] = _pad_head_vec(get("dq_norm"), 1, Q, Qp)
    return [_pad2(get("dq"), Qp, hp)] + latent


def _pack_gated_recurrence(w, p, m: GatedRecurrenceMixer, get, hp: int, dtype, device):
    B, n, np_ = m.blocks, m.vdim, m.vdim_p

    def vec(v):
        return _pad_head_vec(v, B, n, np_)
    # of the gates: per block the rows of r, then of i; padded channels get zero rows and see nothing
    gates = torch.zeros((B, 2, np_, np_), dtype=torch.float32, device=device)
    bias = torch.zeros((B, 2, np_), dtype=torch.float32, device=device)
    for j, r in enumerate(("ra", "ri")):
        gates[:, j, :n, :n] = get(r).float()
        bias[:, j, :n] = get(f"{r}_bias").float()
    w[f"{p}/mix/gates"], w[f"{p}/mix/gate_bias"] = gates.view(B, 2 * np_, np_).to(dtype), bias.view(B, 2 * np_)
    w[f"{p}/mix/rate"] = vec(8.0 * torch.nn.functional.softplus(get("lam").double()))
    w[f"{p}/mix/conv"] = torch.stack([vec(v) for v in get("conv").t()])           # [taps, width]
    w[f"{p}/mix/conv_bias"] = vec(get("conv_bias"))
    w[f"{p}/mix/in_bias"] = torch.cat([vec(get("y_bias")), vec(get("x_bias"))])
    return [_pad_head_rows(get("y"), B, n, np_, hp), _pad_head_rows(get("x"), B, n, np_, hp)]


def _pack_state_space(w, p, m: StateSpaceMixer, get, n_out: int, hp: int, device):
    H, V, Vp, G, N, Np = m.heads, m.vdim, m.vdim_p, m.groups, m.state, m.state_p
    z, x, b, c, dt = torch.split(get("in"), [H * V, H * V, G * N, G * N, H])

    def channels(v):
        x, b, c = torch.split(v, [H * V, G * N, G * N])
        return torch.cat([_pad_head_vec(x, H, V, Vp), _pad_head_vec(b, G, N, Np), _pad_head_vec(c, G, N, Np)])
    bias = torch.zeros(n_out, dtype=torch.float32, device=device)
    bias[m.main_cols: m.main_cols + H] = get("dt_bias").float()
    w[f"{p}/mix/in_bias"] = bias
    w[f"{p}/mix/conv"] = torch.stack([channels(v) for v in get("conv").t()])           # [taps, channels]
    w[f"{p}/mix/conv_bias"] = channels(get("conv_bias"))
    w[f"{p}/mix/rate"] = torch.exp(get("a_log").double()).float().contiguous()
    w[f"{p}/mix/skip"] = get("skip").float().contiguous()
    w[f"{p}/mix/norm"] = _pad_head_vec(get("norm"), H, V, Vp)
    return [_pad_head_rows(z, H, V, Vp, hp), _pad_head_rows(x, H, V, Vp, hp), _pad_head_rows(b, G, N, Np, hp),
            _pad_head_rows(c, G, N, Np, hp), _pad2(dt, H, hp)]


def _pack_parallel(w, p, m: ParallelMixer, get, n_out: int, hp: int, dtype, device):
    rows, biases = [], []
    for side, part in (("left", m.left), ("right", m.right)):
        def of(name, side=side):
            return get(f"{side}.{name}")
        cols, q = part.main_cols + part.gate_cols, f"{p}/{side}"
        rows += _pack_rows(w, q, part, of, cols, hp, dtype, device)
        bias = w.pop(f"{q}/mix/in_bias", None)
        biases.append(torch.zeros(cols, dtype=torch.float32, device=device) if bias is None else bias)
        w[f"{q}/mix/out_proj"] = _pad_head_cols(of("o"), part.heads, part.vdim, part.vdim_p, hp).to(dtype)
        w[f"{q}/norm"] = _pad_head_vec(of("out"), 1, of("out").numel(), hp)
    w[f"{p}/mix/in_bias"] = torch.zeros(n_out, dtype=torch.float32, device=device)
    w[f"{p}/mix/in_bias"][: m.main_cols + m.gate_cols] = torch.cat(biases)
    return rows


def _pack_rows(w, p, m, get, n_out: int, hp: int, dtype, device):
    """Rows of the fused input projection of a mixer, its other weights into `w`."""
    if m.kind == "parallel":
        return _pack_parallel(w, p, m, get, n_out, hp, dtype, device)
    if m.kind in ("latent_attention", "rglru"):
        return {"latent_attention": _pack_latent, "rglru": _pack_gated_recurrence}[m.kind](w, p, m, get, hp, dtype, device)
    pack = {"attention": _pack_attention, "hgrn2": _pack_gated_memory, "ssd": _pack_state_space, "mlstm": _pack_matrix_memory}[m.kind]
    return pack(w, p, m, get, n_out, hp, device)


def pack_weights(cfg: LayeredConfig, get, dtype: torch.dtype = torch.bfloat16, device="cpu") -> Dict[str, torch.Tensor]:
    """Fused, padded weights of the forward pass.  `get(layer, name)` returns a design's tensor by its role (layer -1:
    the model's own): embed, head, final_norm, positions, loop_in, loop_step; norm1, norm1b, norm2, norm2b, conv; hc1_in, hc1_out,
    hc1_mix, hc2_...; the mixers' (see the _pack functions) and o, under "left." and "right." where there are two; up, up_bias,
    down, down_bias, act; gate, up, down; the experts' (see `pack_experts`)."""
    hp, wide, streams = cfg.hidden_p, cfg.residual == "sandwich", cfg.residual == "streams"
    w: Dict[str, torch.Tensor] = {}

    def g(layer, name):
        return get(layer, name).to(device)

    def norm(layer, name):
        if cfg.residual == "post_sum":
            return g(layer, name).float().contiguous().reshape(1)
        return _pad_head_vec(g(layer, name).float() + cfg.norm_offset, 1, cfg.hidden, hp)

    def hyper(layer, q):
        for r in ("in", "out", "mix"):
            w[f"text/layers/{layer}/hc{q}/{r}"] = g(layer, f"hc{q}_{r}").float().contiguous()
    if cfg.tie_head:
        w["text/embed"] = w["text/lm_head"] = _pad2(g(-1, "embed"), cfg.vocab_p, hp).to(dtype)
    else:
        w["text/embed"] = _pad2(g(-1, "embed"), cfg.vocab, hp).to(dtype)
        w["text/lm_head"] = _pad2(g(-1, "head"), cfg.vocab_p, hp).to(dtype)
    w["text/final_norm"] = norm(-1, "final_norm") * cfg.logit_scale        # (the head is linear)
    if cfg.learned_positions:
        w["text/places"] = _pad2(g(-1, "positions"), cfg.learned_positions, hp).to(dtype)
    if streams:
        w["text/stream_sum"] = torch.ones(cfg.streams, dtype=torch.float32, device=device)
    if cfg.logit_softcap:
        w["text/softcap"] = torch.tensor([cfg.logit_softcap, 1.0 / cfg.logit_softcap], dtype=torch.float32, device=device)
    if cfg.loop is not None:
        w["text/loop/in_proj"] = _pad_head_cols(g(-1, "loop_in"), 2, cfg.hidden, hp, hp).to(dtype)
        w["text/loop/step"] = torch.stack([_pad_head_vec(v, 1, cfg.hidden, hp) for v in g(-1, "loop_step")])
    for i, spec in enumerate(cfg.layers):
        m, p = spec.mixer, f"text/layers/{i}"

        def mix(name, i=i):
            return g(i, name)
        w[f"{p}/norm1"] = norm(i, "norm1")
        if wide:
            w[f"{p}/norm1b"] = norm(i, "norm1b")
        if streams:
            hyper(i, 1)
        if cfg.conv_taps:
            w[f"{p}/conv"] = torch.stack([_pad_head_vec(v, 1, cfg.hidden, hp) for v in g(i, "conv").t()])      # [taps, width]
        n_out = pad_to(m.main_cols + m.gate_cols, 2)
        rows = _pack_rows(w, p, m, mix, n_out, hp, dtype, device)
        w[f"{p}/mix/in_proj"] = _pad2(torch.cat(rows), n_out, hp).to(dtype)
        if m.kind != "parallel":
            w[f"{p}/mix/out_proj"] = _pad_head_cols(g(i, "o"), m.heads, m.vdim, m.vdim_p, hp).to(dtype)
        if spec.mlp is not None:
            w[f"{p}/norm2"] = norm(i, "norm2")
            if wide:
                w[f"{p}/norm2b"] = norm(i, "norm2b")
            if streams:
                hyper(i, 2)
        if spec.mlp is not None and spec.mlp.kind == "moe":
            pack_experts(w, p, spec.mlp, mix, hp, dtype)
        elif spec.mlp is not None and spec.mlp.kind == "glu":
            w[f"{p}/mlp/up"], w[f"{p}/mlp/down"] = pack_unit(mix, "", spec.mlp, hp, dtype)
        elif spec.mlp is not None:
            fp = pad_to(spec.mlp.ff, 8)
            w[f"{p}/mlp/up"] = _pad2(g(i, "up"), fp, hp).to(dtype)
            w[f"{p}/mlp/down"] = _pad2(g(i, "down"), hp, fp).to(dtype)
            if spec.mlp.bias:
                w[f"{p}/mlp/up_bias"] = _pad_head_vec(g(i, "up_bias"), 1, spec.mlp.ff, fp)
                w[f"{p}/mlp/down_bias"] = _pad_head_vec(g(i, "down_bias"), 1, cfg.hidden, hp)
            if spec.mlp.activation not in ACTIVATIONS:
                raise ValueError(f"layer {i}: unknown feed-forward activation '{spec.mlp.activation}'")
            if spec.mlp.activation == "xielu":
                a = torch.nn.functional.softplus(g(i, "act").double())
                w[f"{p}/mlp/act"] = torch.stack([a[0], 0.5 + a[1]]).float().contiguous()
    return w


# ---------------------------------------------------------------------------------------------- runtime
class LayeredWorkspace:
    """Activation buffers for up to `max_tokens` tokens; addresses are stable across steps."""

    def __init__(self, cfg: LayeredConfig, max_tokens: int, max_logit_rows: int, device, dtype: torch.dtype,
                 split_rows: int = 1024, ops=None):
        T, dev, f32 = max_tokens, device, torch.float32
        moe = [l.mlp for l in cfg.layers if l.mlp is not None and l.mlp.kind == "moe"]
        mixers = [l.mixer for l in cfg.layers]
        parts = [p for m in mixers for p in mixer_parts(m)]
        attn = [m for m in parts if m.kind == "attention"]
        latent = [m for m in mixers if m.kind == "latent_attention"]

        def rows(cols, dt=dtype):
            return torch.zeros((T, cols), dtype=dt, device=dev)

        def widest(values, default, mult=64):
            return pad_to(max(values, default=default), mult)
        self.max_tokens, self.max_logit_rows = T, max_logit_rows
        if cfg.residual == "streams":
            self.streams = torch.zeros((T, cfg.streams, cfg.hidden_p), dtype=f32, device=dev)
            self.x = self.streams[:, 0]
        else:
            self.x = rows(cfg.hidden_p, f32)       # residual stream
        self.x2 = rows(cfg.hidden_p, f32) if cfg.conv_taps else self.x     # its other copy: a convolution reads rows that its step replaces
        self.xa = rows(cfg.hidden_p)               # what the next GEMM reads, in the activation type
        self.pair = rows(2 * cfg.hidden_p) if cfg.loop is not None else None   # [x, embedding output] of a pass's entry
        self.delta = rows(cfg.hidden_p, f32)       # output of the running sublayer
        self.delta2 = rows(cfg.hidden_p, f32) if len(parts) > len(mixers) else None      # and of the other one beside it
        self.proj = rows(widest((m.main_cols for m in mixers), 64))
        self.gates = rows(widest((m.gate_cols for m in mixers), 2, 4), f32)
        self.mix = rows(widest((m.out_cols for m in mixers), 64))
        self.q = rows(max([m.heads * m.dim_p for m in attn] + [m.q_cols for m in latent], default=16))
        first = next((cfg.attention_of(r) for r in cfg.value_runs), None)
        self.v_first = rows(first.kv_heads * first.vdim_p) if first is not None else None      # values that later layers mix in
        units = [T * l.mlp.ff_p for l in cfg.layers if l.mlp is not None and l.mlp.kind == "glu"]
        self.unit_act = torch.zeros(max(units, default=0), dtype=dtype, device=dev)
        self.unit_wide = torch.zeros(2 * max(units, default=0) if dtype == f32 else 0, dtype=dtype, device=dev)
        self.act = rows(widest((l.mlp.ff for l in cfg.layers if l.mlp is not None and l.mlp.kind == "dense"), 8))
        if moe:
            self.experts = ExpertWorkspace(moe, cfg.hidden_p, T, dev, dtype, ops or load_native())
        rec = max([m.out_cols for m in mixers if m.kind == "rglru"] + [m.conv_cols for m in parts if m.kind == "ssd"], default=0)
        if rec:
            self.rec_u = torch.zeros(T * rec, dtype=dtype, device=dev)
        if latent:
            self.q_latent = rows(max(16, max(m.q_rank_p for m in latent)))
            self.q_abs = rows(max(m.heads * m.kv_rank_p for m in latent))     # absorbed queries, head by head
            self.o_latent = rows(max(m.heads * m.kv_rank_p for m in latent))  # attended latents
        # split-KV partials: (query token x split) rows of decode-sized steps
        self.split_rows = split_rows
        self.part_o = torch.empty(split_rows * max([m.out_cols for m in attn] + [m.heads * m.kv_rank_p for m in latent], default=0),
                                  dtype=f32, device=dev)
        self.part_ml = torch.empty(split_rows * max((m.heads for m in attn + latent), default=0) * 2, dtype=f32, device=dev)
        self.logits = torch.zeros((max_logit_rows, cfg.vocab_p), dtype=f32, device=dev)
        self.head_in = torch.zeros((max_logit_rows, cfg.hidden_p), dtype=dtype, device=dev)
        self.next_ids = torch.zeros((max_logit_rows,), dtype=torch.int32, device=dev)


def native_subset(cfg: LayeredConfig) -> str:
    """The parts of the stand-alone library (see `_build.PARTS`) that this configuration needs."""
    mixers = [m for l in cfg.layers for m in mixer_parts(l.mixer)]
    parts = {{"latent_attention": "latent", "hgrn2": "gated"}.get(m.kind, m.kind) for m in mixers}
    if any(m.kind == "attention" and not m.plain_scores for m in mixers):
        parts.add("head_mix")
    if any(l.mlp is not None and l.mlp.kind == "moe" for l in cfg.layers):
        parts |= {"moe", "streams"}                # (the sum over the experts belongs to the row steps)
    if cfg.residual == "streams" or any(l.mlp is not None and l.mlp.kind == "glu" for l in cfg.layers):
        parts.add("streams")
    if cfg.residual == "branch":
        parts.add("branches")
    return "+".join(sorted(parts))


class LayeredModel:
    """Forward pass of a `LayeredConfig` over the ragged step batch; the interface is `models.hybrid.HybridModel`'s."""

    def __init__(self, cfg: LayeredConfig, weights: Dict[str, torch.Tensor], device, pdl: bool = False):
        self.cfg, self.w = cfg, weights
        if cfg.residual != "branch" and any(l.mixer.kind == "parallel" for l in cfg.layers):
            raise ValueError("mixers side by side need the residual form 'branch'")
        self.device = torch.device(device)
        self._raw_ops = load_native(subset=native_subset(cfg))
        self.ops = LaunchCounter(self._raw_ops)
        self.status = StatusWord(self.device)
        self.dtype = weights["text/embed"].dtype
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("weights must be bf16 or fp32")
        self.f32 = self.dtype == torch.float32
        self.pdl = pdl
        self.comm = None
        self.k_row_scale: Dict[int, torch.Tensor] = {}
        self.l2_prefetch = True
        self.prefill_kernels = True     # False: the token-by-token kernels for every size (tests)
        self.layer_hook = None          # called as hook(layer, x[:T]) after every layer run (tests, debugging)
        self._runs = cfg.runs
        self._attn_idx = {r: i for i, r in enumerate(cfg.attn_layers)}
        self._state_idx = {r: i for i, r in enumerate(cfg.state_layers)}
        self._value_runs = cfg.value_runs
        self._scratch: Dict[str, torch.Tensor] = {}
        self._keep: List[torch.Tensor] = []

    def _grown(self, name: str, n_bytes: int) -> torch.Tensor:
        """Byte scratch of at least `n_bytes` (earlier buffers stay alive: a captured graph may point at them)."""
        cur = self._scratch.get(name)
        if cur is None or cur.numel() < n_bytes:
            cur = torch.empty(n_bytes, dtype=torch.uint8, device=self.device)
            self._keep.append(cur)
            self._scratch[name] = cur
        return cur

    # ------------------------------------------------------------------ GEMM
    def _gemm(self, x, w, bias, out=None, out32=None, out32_from=0, act=0, act_params=None, prefetch=None, epi=EPI_STORE, glu=()):
        if self.f32:
            assert epi == EPI_STORE
            self.ops.gemm_f32(x, w, out, bias, act, act_params, out32, out32_from)
            return
        T, (N, K) = x.shape[0], w.shape
        splits = int(self.ops.gemm_pick_splits(T, N, K, epi))
        if not (self.l2_prefetch and T <= 64):
            prefetch = None
        self.ops.gemm_bf16(x, w, out, epi, None, bias, None, splits, self.status.tensor, self.pdl, act, None, None, None,
                           None, prefetch, out32, out32_from, act_params, glu)

    def _in_proj(self, ws, T, p, m):
        """Fused input projection: [T, main_cols] in the activation type and [T, gate_cols] in fp32."""
        proj = ws.proj[:T, : m.main_cols]
        gates = ws.gates[:T] if m.gate_cols else None
        self._gemm(ws.xa[:T], self.w[f"{p}/mix/in_proj"], self.w.get(f"{p}/mix/in_bias"), proj, gates, m.main_cols if gates is not None else 0,
                   prefetch=self.w[f"{p}/left/mix/out_proj" if m.kind == "parallel" else f"{p}/mix/out_proj"])
        return proj, gates

    # ------------------------------------------------------------------ mixers
    def _attention(self, ws, b: StepBatch, kv, run: int, T: int, p: str, m: AttentionMixer, inputs=None, out=None):
        """`inputs`: the projection's columns and gates when it is made elsewhere; `out`: where the heads' outputs go."""
        ops, w = self.ops, self.w
        proj, gates = inputs or self._in_proj(ws, T, p, m)
        planes = kv.layers[self._attn_idx[run]]
        k_pages, v_pages = planes.typed(self.dtype)
        H, G, Dp, Vp = m.heads, m.kv_heads, m.dim_p, m.vdim_p
        q = ws.q[:T, : H * Dp]
        ops.qkv_append(proj, 0, H * Dp, (H + G) * Dp, H, G, m.dim, w.get(f"{p}/mix/q_norm"), w.get(f"{p}/mix/k_norm"),
                       self.cfg.rms_eps, b.table_row, b.cache_pos, kv.table, q, k_pages, v_pages, kv.page_size, self.pdl,
                       w.get(f"{p}/mix/freq"), m.qk_unit, ws.v_first[:T] if m.value_mix else None,
                       w[f"{p}/mix/v_lambda"] if m.value_mix and run != self._value_runs[0] else None)
        out, sinks = ws.mix[:T, : H * Vp] if out is None else out, w.get(f"{p}/mix/sink")
        weights = (m.sigmoid, w.get(f"{p}/mix/log_rate"), w.get(f"{p}/mix/log_step"), w.get(f"{p}/mix/offset"))
        shape = (m.window, m.scale, m.softcap, m.sink, w.get(f"{p}/mix/heads"), w.get(f"{p}/mix/slope"),
                 gates if m.head_gate else None, out)
        portions = not self.f32 and self.prefill_kernels and b.max_seq_tokens >= PREFILL_MIN_TOKENS
        if portions and m.plain_scores and self._raw_ops.group_prefill_supported(Dp, Vp):
            ops.group_prefill(q, k_pages, v_pages, kv.table, b.table_row, b.kv_len, m.window, m.chunk, m.scale, m.sink, sinks, out,
                              b.qblk_start, b.qblk_count, self.pdl)
            return out
        if portions and not m.plain_scores:
            one = int(ops.head_mix_prefill_scratch(H, b.max_kv_len, m.window, 1, m.sigmoid))
            nb = b.qblk_start.numel()
            scratch = self._grown("scores", max(one, min(one * nb, SCORE_SCRATCH_BYTES)))
            ops.head_mix_prefill(q, k_pages, v_pages, kv.table, b.table_row, b.kv_len, *shape, b.qblk_start, b.qblk_count,
                                 b.max_kv_len, scratch, self.pdl, *weights)
            return out
        split, n = self.pick_split(ws, T, b.max_kv_len, m.look_back, ctas=G if m.plain_scores and not self.f32 else 1)
        ops.head_mix_attention(q, k_pages, v_pages, kv.table, b.table_row, b.kv_len, *shape, split, n,
                               ws.part_o if n > 1 else None, ws.part_ml if n > 1 else None, self.pdl, m.chunk, sinks, *weights)
        return out

    @staticmethod
    def pick_split(ws, T: int, max_kv_len: int, window: int, sm_count: int = 148, ctas: int = 1) -> Tuple[int, int]:
        """Keys per split (a multiple of 32) and splits per token, each of `ctas` CTAs: two CTAs per SM when the step is small."""
        keys = min(max_kv_len, window) if window > 0 else max_kv_len
        want = max(1, min(2 * sm_count // (T * ctas), ws.split_rows // T, 64))
        split = max(64, pad_to(-(-keys // want), 32))
        return split, -(-keys // split)

    @staticmethod
    def pick_latent_split(ws, b: StepBatch, m: LatentAttentionMixer, sm_count: int = 148) -> Tuple[int, int]:
        """Keys per split (a multiple of 32) and splits per query block: about one CTA per SM when the step is small."""
        rows = min(b.max_seq_tokens, BLOCK_TOKENS) * m.heads
        ctas = b.qblk_start.numel() * max(1, -(-rows // 64))
        want = max(1, min(sm_count // ctas, ws.split_rows // b.n_tokens, 64))
        keys = min(b.max_kv_len, m.window + min(b.max_seq_tokens, BLOCK_TOKENS) - 1) if m.window else b.max_kv_len
        split = max(128, pad_to(-(-keys // want), 32))
        return split, -(-keys // split)

    def _head_gemm(self, x: torch.Tensor, x_step: int, w: torch.Tensor, out: torch.Tensor, b: StepBatch, max_tokens: int) -> None:
        """out[t, h * N + n] = sum_k w[h, n, k] x[t, h * x_step + k]; tokens of sequences with `max_tokens` or more may be left out"""
        if not self.f32:
            self.ops.head_gemm(x, x_step, w, out, b.token_seq, b.cu_seqlens, max_tokens, self.pdl)
            return
        H, N, K = w.shape
        for h in range(H):
            self._gemm(x[:, h * x_step: h * x_step + K], w[h], None, out[:, h * N: (h + 1) * N])

    @staticmethod
    def expand_tokens(m: LatentAttentionMixer) -> int:
        """Portion length from which making the keys and values of all visible positions takes fewer multiply-adds than
        attending in the latent space; 0: never."""
        wide, heads = 2 * m.kv_rank_p, m.dim_p + m.vdim_p
        return max(16, -(-m.kv_rank_p * heads // (wide - heads))) if wide > heads else 0

    def _expand_plan(self, b: StepBatch, m: LatentAttentionMixer):
        """Which sequences of the step take the expanded form: (threshold, [n, 4] of block-table row / first gathered row /
        first position / positions, first row (or -1) and its position per sequence, total rows, longest, whether the others
        are left) or None."""
        least = self.expand_tokens(m)
        if (self.f32 or not self.prefill_kernels or b.seq_host is None or not least or b.max_seq_tokens < least
                or not self._raw_ops.latent_expanded_supported(m.dim_p, m.rot_p, m.vdim_p)):
            return None
        key = (least, m.heads * (m.dim_p + m.vdim_p), m.window)
        if key not in b.plans:
            seqs, base, total = [], [], 0
            for row, n, end in b.seq_host:
                first = max(0, end - n + 1 - m.window) if m.window else 0       # what the portion's first token sees
                base += [total, first] if n >= least else [-1, 0]
                if n >= least:
                    seqs.append((row, total, first, end - first))
                    total += end - first
            plan = None
            if total * key[1] * 2 <= EXPAND_BYTES:
                host = torch.tensor(base + [v for s in seqs for v in s], dtype=torch.int32)
                dev = (host.pin_memory() if self.device.type == "cuda" else host).to(self.device, non_blocking=True)
                plan = (least, dev[len(base):].view(-1, 4), dev[: len(base)].view(-1, 2), total, max(s[3] for s in seqs),
                        2 * len(seqs) < len(base))
            b.plans[key] = plan
        return b.plans[key]

    def _latent_attention(self, ws, b: StepBatch, kv, run: int, T: int, p: str, m: LatentAttentionMixer):
        ops, w, eps = self.ops, self.w, self.cfg.rms_eps
        proj, _ = self._in_proj(ws, T, p, m)
        pages, _ = kv.layers[self._attn_idx[run]].typed(self.dtype)
        c_q = ws.q_latent[:T, : m.q_rank_p] if m.q_rank else None
        q = ws.q[:T, : m.q_cols] if m.q_rank else proj[:, : m.q_cols]
        freq, sink = w[f"{p}/mix/freq"], w.get(f"{p}/mix/sink")
        ops.latent_prep(proj, m.q_rank, m.kv_rank, m.rot_dim, w.get(f"{p}/mix/q_norm"), w[f"{p}/mix/kv_norm"], eps, freq, b.table_row,
                        b.cache_pos, kv.table, c_q, pages, self.pdl)
        if m.q_rank:
            self._gemm(c_q, w[f"{p}/mix/uq"], None, q, prefetch=w[f"{p}/mix/uk_t"])
        out = ws.mix[:T, : m.out_cols]
        plan, blocks = self._expand_plan(b, m), (b.qblk_start, b.qblk_count, min(b.max_seq_tokens, BLOCK_TOKENS))
        if plan is None or plan[-1]:
            skip = 0 if plan is None else plan[0]
            q_abs, o_latent = ws.q_abs[:T, : m.heads * m.kv_rank_p], ws.o_latent[:T, : m.heads * m.kv_rank_p]
            self._head_gemm(q, m.dim_p + m.rot_p, w[f"{p}/mix/uk_t"], q_abs, b, skip)
            args = (q_abs, q, pages, kv.table, b.table_row, b.kv_len, m.heads, m.rot_dim, m.scale, freq, sink, o_latent)
            if self.f32 or not self._raw_ops.latent_absorbed_supported(m.kv_rank_p, m.rot_p):
                ops.latent_token_attention(*args, self.pdl, m.window)
            else:
                split, n = self.pick_latent_split(ws, b, m)
                ops.latent_absorbed_attention(*args, *blocks, b.token_seq, b.cu_seqlens, skip, split, n,
                                              ws.part_o if n > 1 else None, ws.part_ml if n > 1 else None, self.pdl, m.window)
            self._head_gemm(o_latent, m.kv_rank_p, w[f"{p}/mix/uv"], out, b, skip)
        if plan is not None:
            _, seqs, base, total, longest, _ = plan
            ukv = w[f"{p}/mix/ukv"]
            rows = self._grown("latent rows", total * m.row_cols * 2)[: total * m.row_cols * 2].view(self.dtype).view(total, m.row_cols)
            wide = self._grown("latent keys", total * ukv.shape[0] * 2)[: total * ukv.shape[0] * 2].view(self.dtype).view(total, ukv.shape[0])
            ops.latent_gather(pages, kv.table, seqs, longest, rows, self.pdl)
            self._gemm(rows[:, : m.kv_rank_p], ukv, None, wide)
            ops.latent_expanded_attention(q, rows, wide, b.kv_len, m.heads, m.kv_rank_p, m.rot_dim, m.scale, freq, sink, out, *blocks,
                                          b.token_seq, base, self.pdl, m.window)
        return out

    def _chunk_workspace(self, b: StepBatch, T: int, kind: str, m) -> "torch.Tensor | None":
        """Scratch of a memory's chunked prefill kernels; None when the step takes the token-by-token kernel."""
        supported, size = getattr(self._raw_ops, f"{kind}_chunked_supported"), getattr(self._raw_ops, f"{kind}_chunked_workspace_bytes")
        if self.f32 or not self.prefill_kernels or b.max_seq_tokens < PREFILL_MIN_TOKENS or not supported(m.dim_p, m.vdim_p):
            return None
        return self._grown("chunks", int(size(T, b.n_seqs, m.heads, m.dim_p, m.vdim_p)))

    def _matrix_memory(self, ws, b: StepBatch, states, run: int, T: int, p: str, m: MatrixMemoryMixer, write_state: bool):
        proj, gates = self._in_proj(ws, T, p, m)
        S, n, mx = states.layers[self._state_idx[run]][-3:]
        H, Dp, Vp = m.heads, m.dim_p, m.vdim_p
        chunk_ws = self._chunk_workspace(b, T, "mlstm", m)
        self.ops.count += 3 if chunk_ws is not None else 0
        out = ws.mix[:T, : H * Vp]
        self.ops.mlstm(proj, 0, H * Dp, 2 * H * Dp, H * (2 * Dp + Vp), gates, 0, H, m.vdim, m.dim ** -0.5, m.gate_cap,
                       self.cfg.rms_eps, self.w[f"{p}/mix/norm"], b.cu_seqlens, b.state_slot, S, n, mx, out, write_state,
                       chunk_ws, self.pdl, b.one_token_per_seq)
        return out

    def _gated_memory(self, ws, b: StepBatch, states, run: int, T: int, p: str, m: GatedMemoryMixer, write_state: bool):
        proj, gates = self._in_proj(ws, T, p, m)
        S = states.layers[self._state_idx[run]][-1]
        chunk_ws = self._chunk_workspace(b, T, "gated", m)
        self.ops.count += 2 if chunk_ws is not None else 0
        out = ws.mix[:T, : m.out_cols]
        self.ops.gated_memory(proj, 0, m.heads * m.dim_p, gates, self.w[f"{p}/mix/lower"], m.vdim, self.cfg.rms_eps,
                              self.w[f"{p}/mix/norm"], b.cu_seqlens, b.state_slot, S, out, write_state, chunk_ws, self.pdl,
                              b.one_token_per_seq)
        return out

    def _gated_recurrence(self, ws, b: StepBatch, states, run: int, T: int, p: str, m: GatedRecurrenceMixer, write_state: bool):
        ops, w = self.ops, self.w
        proj, _ = self._in_proj(ws, T, p, m)
        ring, S = states.layers[self._state_idx[run]][-2:]
        C, n, out = m.out_cols, m.vdim_p, ws.mix[:T, : m.out_cols]
        gates, gate_bias, rate = w[f"{p}/mix/gates"], w[f"{p}/mix/gate_bias"], w[f"{p}/mix/rate"]
        step = (m.blocks, w[f"{p}/mix/conv"], w[f"{p}/mix/conv_bias"], b.cu_seqlens, b.token_seq, b.cache_pos, b.state_slot, ring)
        one = b.one_token_per_seq
        if not self.f32 and self._raw_ops.rglru_fused_supported(n) and (one or self.prefill_kernels):
            chunk_ws = None if one else self._grown("recurrence", int(self._raw_ops.rglru_chunked_workspace_bytes(T, b.n_seqs, C)))
            ops.count += 0 if one else 1
            ops.rglru(proj, *step, gates, gate_bias, rate, S, out, b.qblk_start, b.qblk_count, chunk_ws, write_state, self.pdl)
            return out
        u = ws.rec_u[: T * C].view(T, C)
        raw = self._grown("gates", 8 * T * C)[: 8 * T * C].view(torch.float32).view(T, 2 * C)
        ops.rglru_conv(proj, *step, u, self.pdl)
        for k in range(m.blocks):
            self._gemm(u[:, k * n: (k + 1) * n], gates[k], gate_bias[k], out32=raw[:, 2 * k * n: 2 * (k + 1) * n])
        ops.rglru_scan(proj, *step, u, raw, rate, S, out, write_state, self.pdl)
        return out

    def _state_space(self, ws, b: StepBatch, states, run: int, T: int, p: str, m: StateSpaceMixer, write_state: bool, inputs=None, out=None):
        """`inputs`, `out`: as in `_attention`."""
        ops, w = self.ops, self.w
        proj, gates = inputs or self._in_proj(ws, T, p, m)
        ring, S = states.layers[self._state_idx[run]][-2:]
        out = ws.mix[:T, : m.out_cols] if out is None else out
        one = b.one_token_per_seq
        u = chunk_ws = None
        if not one:
            u = ws.rec_u[: T * m.conv_cols].view(T, m.conv_cols)
            if (not self.f32 and self.prefill_kernels and b.max_seq_tokens >= PREFILL_MIN_TOKENS
                    and self._raw_ops.ssd_chunked_supported(m.state_p, m.vdim_p)):
                chunk_ws = self._grown("state space", int(self._raw_ops.ssd_chunked_workspace_bytes(T, b.n_seqs, m.heads, m.state_p, m.vdim_p)))
            ops.count += 1 if chunk_ws is None else 3
        ops.ssd(proj, m.out_cols, gates, w[f"{p}/mix/conv"], w[f"{p}/mix/conv_bias"], w[f"{p}/mix/rate"], w[f"{p}/mix/skip"], m.groups,
                b.cu_seqlens, b.token_seq, b.cache_pos, b.state_slot, ring, S, u, out, write_state, chunk_ws, self.pdl, one)
        ops.ssd_gated_norm(out, proj, w[f"{p}/mix/norm"], m.heads, m.vdim, m.norm_groups, self.cfg.rms_eps, self.pdl)
        return out

    def _parallel(self, ws, b: StepBatch, kv, states, run: int, T: int, p: str, m: ParallelMixer, write_state: bool, prefetch) -> dict:
        """ws.delta, ws.delta2 <- the outputs of both sides; returns them as `branch_rows` takes them."""
        w, cut, at = self.w, m.left.out_cols, m.left.main_cols
        proj, gates = self._in_proj(ws, T, p, m)
        left, right = ws.mix[:T, :cut], ws.mix[:T, cut: cut + m.right.out_cols]
        self._attention(ws, b, kv, run, T, f"{p}/left", m.left, (proj[:, :at], None), left)
        self._state_space(ws, b, states, run, T, f"{p}/right", m.right, write_state, (proj[:, at:], gates), right)
        self._gemm(left, w[f"{p}/left/mix/out_proj"], None, out32=ws.delta[:T], prefetch=w[f"{p}/right/mix/out_proj"])
        self._gemm(right, w[f"{p}/right/mix/out_proj"], None, out32=ws.delta2[:T], prefetch=prefetch)
        return dict(branch_a=ws.delta[:T], branch_b=ws.delta2[:T], w_a=w[f"{p}/left/norm"], w_b=w[f"{p}/right/norm"])

    def _mixer(self, ws, b: StepBatch, kv, states, run: int, T: int, p: str, m, write_state: bool) -> torch.Tensor:
        if m.kind in ATTENTION_KINDS:
            fn = self._attention if m.kind == "attention" else self._latent_attention
            return fn(ws, b, kv, run, T, p, m)
        fn = {"hgrn2": self._gated_memory, "mlstm": self._matrix_memory, "rglru": self._gated_recurrence, "ssd": self._state_space}[m.kind]
        return fn(ws, b, states, run, T, p, m, write_state)

    def _feed_forward(self, ws, T: int, p: str, spec, prefetch) -> None:
        """ws.delta <- the feed-forward of ws.xa"""
        if spec.kind == "moe":
            y = run_experts(self, ws.experts, T, p, spec, ws.xa[:T], ws.delta[:T], prefetch)
            self.ops.mixture_rows(*y.values(), ws.delta[:T], self.pdl)
            return
        w, up, down = self.w, self.w[f"{p}/mlp/up"], self.w[f"{p}/mlp/down"]
        if spec.kind == "glu":
            run_unit(self, T, spec, up, down, ws.xa[:T], ws.unit_act, ws.unit_wide, ws.delta[:T], prefetch)
            return
        act = ws.act[:T, : up.shape[0]]
        self._gemm(ws.xa[:T], up, w.get(f"{p}/mlp/up_bias"), act, act=ACTIVATIONS[spec.activation], act_params=w.get(f"{p}/mlp/act"),
                   prefetch=down)
        self._gemm(act, down, w.get(f"{p}/mlp/down_bias"), out32=ws.delta[:T], prefetch=prefetch)

    # ------------------------------------------------------------------ forward
    def forward_hidden(self, ws: LayeredWorkspace, b: StepBatch, kv, states, write_state: bool = True) -> torch.Tensor:
        """Runs all layers; returns the final-normed hidden states [T, hidden (padded)]."""
        if b.n_tokens > ws.max_tokens:
            raise ValueError(f"step of {b.n_tokens} tokens exceeds the workspace ({ws.max_tokens})")
        run = {"sandwich": self._forward_sandwich, "streams": self._forward_streams, "post_sum": self._forward_post_sum,
               "branch": self._forward_branch}[self.cfg.residual]
        return run(ws, b, kv, states, write_state)

    def _next_weights(self, run: int):
        """What the GEMM after the last one of `run` reads (an L2 hint)."""
        if run + 1 == len(self._runs):
            return self.w["text/lm_head"]
        layer, opens = self._runs[run + 1]
        return self.w["text/loop/in_proj"] if opens >= 0 else self.w[f"text/layers/{layer}/mix/in_proj"]

    def _forward_post_sum(self, ws, b: StepBatch, kv, states, write_state: bool) -> torch.Tensor:
        cfg, ops, w, T = self.cfg, self.ops, self.w, b.n_tokens
        x, xa, delta = ws.x[:T], ws.xa[:T], ws.delta[:T]
        ops.embed_rows32(b.ids, w["text/embed"], x, xa, cfg.embed_scale, self.pdl)
        for run, (layer, _) in enumerate(self._runs):
            spec, p = cfg.layers[layer], f"text/layers/{layer}"
            mix = self._mixer(ws, b, kv, states, run, T, p, spec.mixer, write_state)
            last, nxt = w["text/final_norm"] if run + 1 == len(self._runs) else None, self._next_weights(run)
            self._gemm(mix, w[f"{p}/mix/out_proj"], None, out32=delta, prefetch=w.get(f"{p}/mlp/up", nxt))
            ops.post_norm_rows(x, delta, xa, cfg.hidden, cfg.residual_alpha, cfg.rms_eps, w[f"{p}/norm1"],
                               last if spec.mlp is None else None, self.pdl)
            if spec.mlp is not None:
                self._feed_forward(ws, T, p, spec.mlp, nxt)
                ops.post_norm_rows(x, delta, xa, cfg.hidden, cfg.residual_alpha, cfg.rms_eps, w[f"{p}/norm2"], last, self.pdl)
            if self.layer_hook is not None:
                self.layer_hook(run, x[:, : cfg.hidden])
        return xa

    def _forward_sandwich(self, ws, b: StepBatch, kv, states, write_state: bool) -> torch.Tensor:
        """The residual update of a sublayer waits for the row step in front of the next one (`sandwich_rows`)."""
        cfg, ops, w, T, hp = self.cfg, self.ops, self.w, b.n_tokens, self.cfg.hidden_p
        x, other, xa, delta = ws.x[:T], ws.x2[:T], ws.xa[:T], ws.delta[:T]
        post = None                   # weights of the norm of the sublayer output that waits in `delta`

        def rows(w_next, out, conv_run=-1, layer=0):
            nonlocal x, other, post
            conv = (None, None, None, None)
            if conv_run >= 0 and cfg.conv_taps:
                state = states.layers[self._state_idx[conv_run]][0] if cfg.conv_taps > 1 else None
                conv = (w[f"text/layers/{layer}/conv"], state, b.cu_seqlens, b.state_slot)
            dst = other if conv[0] is not None and post is not None and b.max_seq_tokens > 1 else x
            ops.sandwich_rows(x, dst, None if post is None else delta, post, w_next, out, cfg.hidden, cfg.norm_groups, cfg.residual_mult,
                              cfg.rms_eps, *conv, b.max_seq_tokens, write_state, self.pdl)
            if dst is other:
                x, other = other, x
            post = None
        ops.embed_rows32(b.ids, w["text/embed"], x, ws.pair[:T, hp:] if cfg.loop is not None else xa, cfg.embed_scale, self.pdl)
        for run, (layer, opens) in enumerate(self._runs):
            spec, p = cfg.layers[layer], f"text/layers/{layer}"
            if opens >= 0:
                rows(None, ws.pair[:T, :hp])
                self._gemm(ws.pair[:T], w["text/loop/in_proj"], w["text/loop/step"][opens], out32=x, prefetch=w[f"{p}/mix/in_proj"])
            rows(w[f"{p}/norm1"], xa, run, layer)
            mix = self._mixer(ws, b, kv, states, run, T, p, spec.mixer, write_state)
            nxt = self._next_weights(run)
            self._gemm(mix, w[f"{p}/mix/out_proj"], None, out32=delta, prefetch=w.get(f"{p}/mlp/up", nxt))
            post = w[f"{p}/norm1b"]
            if spec.mlp is not None:
                rows(w[f"{p}/norm2"], xa)
                self._feed_forward(ws, T, p, spec.mlp, nxt)
                post = w[f"{p}/norm2b"]
            if self.layer_hook is not None:
                rows(None, xa)
                self.layer_hook(run, x[:, : cfg.hidden])
        rows(w["text/final_norm"], xa)
        return xa

    def _forward_streams(self, ws, b: StepBatch, kv, states, write_state: bool) -> torch.Tensor:
        """The update of the streams by a sublayer waits for the row step in front of the next one (`stream_rows`); until the
        first update every stream is the embedding row itself."""
        cfg, ops, w, T = self.cfg, self.ops, self.w, b.n_tokens
        xa, delta, X = ws.xa[:T], ws.delta[:T], ws.streams[:T]
        source, y, update = None, None, (None, None)     # streams, output of the sublayer that waits and its (mix, out)

        def rows(w_in, w_next):
            nonlocal source, y, update
            parts = (None, None, None, None, None, None, 0) if y is None else tuple(y.values())
            ops.stream_rows(source, b.ids, w["text/embed"], None if y is None else X, *parts, *update, w_in, w_next, xa, cfg.hidden,
                            cfg.rms_eps, self.pdl)
            if y is not None:
                source, y, update = X, None, (None, None)
        for run, (layer, _) in enumerate(self._runs):
            spec, p = cfg.layers[layer], f"text/layers/{layer}"
            rows(w[f"{p}/hc1/in"], w[f"{p}/norm1"])
            mix, nxt = self._mixer(ws, b, kv, states, run, T, p, spec.mixer, write_state), self._next_weights(run)
            self._gemm(mix, w[f"{p}/mix/out_proj"], None, out32=delta, prefetch=w.get(f"{p}/mlp/router", w.get(f"{p}/mlp/up", nxt)))
            y, update = self._plain_sum(delta), (w[f"{p}/hc1/mix"], w[f"{p}/hc1/out"])
            if spec.mlp is not None:
                rows(w[f"{p}/hc2/in"], w[f"{p}/norm2"])
                if spec.mlp.kind == "moe":
                    y = run_experts(self, ws.experts, T, p, spec.mlp, xa, delta, nxt)
                else:
                    self._feed_forward(ws, T, p, spec.mlp, nxt)
                    y = self._plain_sum(delta)
                update = (w[f"{p}/hc2/mix"], w[f"{p}/hc2/out"])
            if self.layer_hook is not None:
                rows(w["text/stream_sum"], w["text/final_norm"])
                self.layer_hook(run, X.sum(dim=1)[:, : cfg.hidden])
        rows(w["text/stream_sum"], w["text/final_norm"])
        return xa

    def _forward_branch(self, ws, b: StepBatch, kv, states, write_state: bool) -> torch.Tensor:
        """A sublayer reads the residual itself; the row step behind it norms its output, adds it and makes the next input."""
        cfg, ops, w, T = self.cfg, self.ops, self.w, b.n_tokens
        x, xa, delta = ws.x[:T], ws.xa[:T], ws.delta[:T]
        no_branches = dict(branch_a=None, branch_b=None, w_a=None, w_b=None)

        def rows(y, branches, norm, last):
            ops.branch_rows(x, *(branches or no_branches).values(), *(y or self._plain_sum(None)).values(), norm,
                            w["text/final_norm"] if last else None, xa, cfg.hidden, cfg.rms_eps, self.pdl)
        ops.embed_rows32(b.ids, w["text/embed"], x, xa, cfg.embed_scale, self.pdl, b.cache_pos, w.get("text/places"))
        for run, (layer, _) in enumerate(self._runs):
            spec, p, last = cfg.layers[layer], f"text/layers/{layer}", run + 1 == len(self._runs)
            nxt = self._next_weights(run)
            after = w.get(f"{p}/mlp/router", w.get(f"{p}/mlp/up", nxt))
            if spec.mixer.kind == "parallel":
                y, pair = None, self._parallel(ws, b, kv, states, run, T, p, spec.mixer, write_state, after)
            else:
                mix = self._mixer(ws, b, kv, states, run, T, p, spec.mixer, write_state)
                self._gemm(mix, w[f"{p}/mix/out_proj"], None, out32=delta, prefetch=after)
                y, pair = self._plain_sum(delta), None
            rows(y, pair, w[f"{p}/norm1"], last and spec.mlp is None)
            if spec.mlp is not None:
                if spec.mlp.kind == "moe":
                    y = run_experts(self, ws.experts, T, p, spec.mlp, xa, delta, nxt)
                else:
                    self._feed_forward(ws, T, p, spec.mlp, nxt)
                    y = self._plain_sum(delta)
                rows(y, None, w[f"{p}/norm2"], last)
            if self.layer_hook is not None:
                self.layer_hook(run, x[:, : cfg.hidden])
        return xa

    @staticmethod
    def _plain_sum(delta) -> dict:
        return dict(delta=delta, gate=None, choice=None, weight=None, ret=None, h=None, n_experts=0)

    def head(self, ws: LayeredWorkspace, head_in: torch.Tensor) -> torch.Tensor:
        """fp32 logits [rows, vocab] of final-normed hidden states (at most `max_logit_rows`)."""
        out = ws.logits[: head_in.shape[0]]
        act = ACT_SOFTCAP if self.cfg.logit_softcap else 0
        self._gemm(head_in, self.w["text/lm_head"], None, out32=out, act=act, act_params=self.w.get("text/softcap"))
        return out[:, : self.cfg.vocab]

    def logits(self, ws: LayeredWorkspace, b: StepBatch, hidden: torch.Tensor) -> torch.Tensor:
        R = b.logit_rows.numel()
        if R == hidden.shape[0]:
            return self.head(ws, hidden)       # decode: every row is a logit row, in order
        head_in = ws.head_in[:R]
        torch.index_select(hidden, 0, b.logit_rows.long(), out=head_in)
        return self.head(ws, head_in)

    def forward_greedy(self, ws: LayeredWorkspace, b: StepBatch, kv, states) -> torch.Tensor:
        """One step ending in arg-max token ids for `b.logit_rows` (int32 [R], ws.next_ids)."""
        start = self.ops.count
        hidden = self.forward_hidden(ws, b, kv, states)
        if b.logit_rows.numel() == 0:
            return ws.next_ids[:0]
        lg = self.logits(ws, b, hidden)
        out = ws.next_ids[: lg.shape[0]]
        self.ops.argmax_rows(lg, out, self.pdl)
        self.ops.launches_last_forward = self.ops.count - start
        return out
