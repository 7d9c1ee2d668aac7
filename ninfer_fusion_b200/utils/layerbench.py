"""Layer-list designs beside the closest other model of equal size: model throughput and per-kernel roofline fractions.

`python bench.py --compare kuzanex-1b` prints one JSON line: prefill and decode tokens/s of the two models through the
same generator (random weights, bf16), and for every kernel of the design its time, what bounds it, and the same for
the other model's kernel of the like kind at equal size.  Kuzanex (head-mixing attention, matrix memory) stands beside the
hybrid decoder, Tebivik (latent attention, gated memory) beside Kuzanex, Tuzupel (streams, experts, plain and latent attention,
gated recurrence) and Ratilorn (head-mixing sigmoid attention, state space beside attention, experts) beside the hybrid decoder
with experts and Kuzanex's kernels.  Kernels are timed cold (L2 flushed before every launch) with CUDA
events; the roofline of a kernel is the slower of its algorithmic bytes at the measured copy bandwidth and its
algorithmic multiply-adds at the measured bf16 GEMM rate.
"""
from __future__ import annotations

from dataclasses import replace
from typing import Dict, List

import torch

from ..models import kuzanex
from ..models.architectures import LAYERED_REGISTRY, random_layered_weights
from ..models.config import ModelConfig
from ..models.weights import random_weights
from ..runtime.generator import Generator
from ..models.layered import SCORE_SCRATCH_BYTES
from .opbench import L2Flusher, measured_peaks, time_op


def equal_size_hybrid(cfg) -> ModelConfig:
    """The hybrid decoder with the same width, depth, 3 : 1 pattern, query width, state size and feed-forward weights."""
    att = cfg.layers[cfg.attn_layers[0]].mixer
    mem = cfg.layers[cfg.state_layers[0]].mixer
    ff = cfg.layers[0].mlp.ff
    v_heads = max(1, mem.heads * mem.dim * mem.vdim // (128 * 128))
    inter = max(128, round(2 * ff / 3 / 128) * 128)          # three matrices instead of two
    heads = max(1, att.heads * att.dim // 256)
    return ModelConfig(name=f"hybrid-like-{cfg.name}", n_layers=cfg.n_layers, hidden=cfg.hidden, vocab=cfg.vocab, n_q_heads=heads,
                       n_kv_heads=max(1, att.kv_heads * att.dim // 256), head_dim=256, rot_dim=64, rope_theta=1e7,
                       gdn_qk_heads=max(1, v_heads // 2), gdn_v_heads=v_heads, ffn_inter=inter, mtp_layers=0)


def _throughput(cfg, weights, batch: int, prompt: int, steps: int) -> Dict[str, float]:
    """Prefill of `batch` prompts and `steps` decode rounds (device-side graph loop)."""
    gen = Generator(cfg, weights, "cuda:0", max_batch=batch, max_context=prompt + 2 * steps + 64, page_size=64,
                    prefill_chunk=4096, use_graph=True, pdl=True)
    g = torch.Generator().manual_seed(7)
    prompts = [torch.randint(0, cfg.vocab, (prompt,), generator=g).tolist() for _ in range(batch)]
    ms = []
    for _ in range(4):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        gen.prefill(prompts)
        e1.record()
        torch.cuda.synchronize()
        ms.append(e0.elapsed_time(e1))
    graph, finish = gen.decode_device_loop(4 + steps)
    for _ in range(4):
        graph.replay()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(steps):
        graph.replay()
    e1.record()
    torch.cuda.synchronize()
    finish()
    gen.model.status.check("after the comparison run")
    dec = e0.elapsed_time(e1) / steps
    pre = sorted(ms[1:])[1]
    return {"prefill_ms": round(pre, 3), "prefill_tok_s": round(batch * prompt / pre * 1e3), "decode_ms": round(dec, 4),
            "decode_tok_s": round(batch / dec * 1e3), "launches_per_round": int(gen.model.ops.launches_last_forward)}


class _Kernels:
    """Times closures cold and puts them against their roofline."""

    def __init__(self, iters: int, only: str = "", names: "Dict[str, str] | None" = None):
        self.only = only
        self.names = names or {}       # model label of a row -> label to report, "" leaves the row out
        self.flush, self.iters, self.rows = L2Flusher(), iters, []
        self.bw, self.fl, self.how = measured_peaks()

    def add(self, what: str, model: str, fn, n_bytes: float, macs: float = 0.0) -> None:
        model = self.names.get(model, model)
        if not model or self.only not in f"{model}: {what}":
            return
        med, _ = time_op(fn, iters=self.iters, flush=self.flush)
        t_b, t_f = n_bytes / self.bw, 2.0 * macs / self.fl
        self.rows.append({"kernel": what, "model": model, "us": round(med * 1e6, 1), "bound": "bytes" if t_b >= t_f else "math",
                          "roofline_us": round(max(t_b, t_f) * 1e6, 2), "fraction": round(max(t_b, t_f) / med, 3)})


def _rand(*shape, dtype=torch.bfloat16, s=1.0):
    return (torch.randn(shape, device="cuda") * s).to(dtype)


def _ints(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda") if not torch.is_tensor(x) else x.int().cuda()


def _tokens(batch: int, new: int, total: int):
    """Row, visible keys, cu_seqlens, query blocks of `batch` sequences that bring their last `new` of `total` tokens."""
    row = torch.arange(batch).repeat_interleave(new)
    kv = torch.arange(total - new + 1, total + 1).repeat(batch)
    return _ints(row), _ints(kv), _ints(torch.arange(batch + 1) * new)


def _blocks(batch: int, new: int, block: int):
    start = [b * new + o for b in range(batch) for o in range(0, new, block)]
    count = [min(block, new - o) for _ in range(batch) for o in range(0, new, block)]
    return _ints(start), _ints(count)


def _pairs(new: int, total: int, window: int) -> int:
    """Visible (query, key) pairs of one sequence's portion."""
    return sum(min(p + 1, window) if window else p + 1 for p in range(total - new, total))


def _gemm_rows(k: _Kernels, ops, status, cfg, hyb, T: int, tag: str) -> None:
    att, mem = cfg.layers[cfg.attn_layers[0]].mixer, cfg.layers[cfg.state_layers[0]].mixer
    h, ff = cfg.hidden_p, cfg.layers[0].mlp.ff

    def run(model, what, N, K, epi=0, act=0, out32_from=None, bias=False):
        x, w = _rand(T, K), _rand(N, K, s=0.02)
        out_cols = N // 2 if epi == 2 else N
        out = torch.empty((T, out_cols), dtype=torch.bfloat16, device="cuda")
        o32 = None if out32_from is None else torch.empty((T, N - out32_from + 2), device="cuda")[:, : (N - out32_from + 1) // 2 * 2]
        b = torch.zeros(N, device="cuda") if bias else None
        prm = torch.tensor([0.8, 1.3], device="cuda") if act else None
        resid = out if epi == 1 else None
        splits = int(ops.gemm_pick_splits(T, N, K, epi))
        n_out = T * out_cols * 2 if out32_from is None else T * (out32_from * 2 + (N - out32_from) * 4)
        k.add(f"{what} {tag}", model, lambda: ops.gemm_bf16(x, w, None if out32_from == 0 else out, epi, resid, b, None, splits, status,
                                                            False, act, None, None, None, None, None, o32, out32_from or 0, prm),
              N * K * 2 + T * K * 2 + n_out, T * N * K)
    run("design", "input projection (memory)", mem.main_cols + mem.gate_cols, h, out32_from=mem.main_cols, bias=True)
    run("hybrid", "input projection (memory)", hyb.gdn_in_dim, h)
    run("design", "input projection (attention)", att.main_cols + att.gate_cols, h, out32_from=att.main_cols, bias=True)
    run("hybrid", "input projection (attention)", hyb.attn_in_dim, h)
    run("design", "output projection", h, mem.out_cols, out32_from=0)
    run("hybrid", "output projection", h, hyb.gdn_v_dim, epi=1)
    run("design", "feed-forward up", ff, h, act=3, bias=True)
    run("hybrid", "feed-forward up", 2 * hyb.ffn_inter, h, epi=2)
    run("design", "feed-forward down", h, ff, out32_from=0, bias=True)
    run("hybrid", "feed-forward down", h, hyb.ffn_inter, epi=1)
    # residual rows
    x32, d32, xa = torch.randn(T, h, device="cuda"), torch.randn(T, h, device="cuda"), _rand(T, h)
    gain = torch.ones(1, device="cuda")
    k.add(f"residual rows {tag}", "design", lambda: ops.post_norm_rows(x32, d32, xa, cfg.hidden, 2.0, 1e-6, gain, None, False), T * h * 14)
    xb, nb, nw = _rand(T, h), _rand(T, h), _rand(h)
    k.add(f"residual rows {tag}", "hybrid", lambda: ops.add_rmsnorm(None, 0, None, xb, None, nw, nb, T, h, 1e-6, True, False), T * h * 4)


def _attention_rows(k: _Kernels, ops, model, ws, cfg, hyb, batch: int, new: int, total: int, tag: str) -> None:
    m = cfg.layers[cfg.attn_layers[0]].mixer
    H, G, D, V, P = m.heads, m.kv_heads, m.dim_p, m.vdim_p, 64
    T, per = batch * new, (total + P - 1) // P
    row, kv, cu = _tokens(batch, new, total)
    pos = (kv - 1).int()
    table = torch.randperm(batch * per, device="cuda").int().view(batch, per)
    kp, vp = _rand(batch * per, G, P, D), _rand(batch * per, G, P, V)
    q, out, gate = _rand(T, H * D), _rand(T, H * V), torch.randn(T, H, device="cuda")
    mix, slope = torch.eye(H, device="cuda") + 0.1, torch.rand(H, device="cuda") * 0.01
    seen = min(total, m.window) if m.window else total
    io = T * H * (D + V) * 2
    macs = batch * _pairs(new, total, m.window) * H * (D + V)
    args = (q, kp, vp, table, row, kv, m.window, m.scale, m.softcap, m.sink, mix, slope, gate, out)
    if new > 1:
        bs, bc = _blocks(batch, new, int(ops.head_mix_block_tokens()))
        one = int(ops.head_mix_prefill_scratch(H, total, m.window, 1))
        scratch = torch.empty(max(one, min(one * bs.numel(), SCORE_SCRATCH_BYTES)), dtype=torch.uint8, device="cuda")
        k.add(f"attention {tag}", "design", lambda: ops.head_mix_prefill(*args, bs, bc, total, scratch, False),
              batch * min(total, seen + new) * G * (D + V) * 2 + io, macs)
    else:
        split, n = model.pick_split(ws, T, total, m.window)
        po, ml = torch.empty(T * n * H * V, device="cuda"), torch.empty(T * n * H * 2, device="cuda")
        k.add(f"attention {tag}", "design", lambda: ops.head_mix_attention(*args, split, n, po, ml, False),
              batch * seen * G * (D + V) * 2 + io, macs)
    proj = _rand(T, m.main_cols)
    qn = torch.ones(D, device="cuda")
    k.add(f"norm + append {tag}", "design", lambda: ops.qkv_append(proj, 0, H * D, (H + G) * D, H, G, m.dim, qn, qn, 1e-6, row, pos, table,
                                                                   q, kp, vp, P, False), T * m.main_cols * 4)
    # the hybrid's: bf16 rows, the same number of visible keys (decode) or the same prompt (prefill, all of the past)
    Hh, Gh, Dh = hyb.n_q_heads, hyb.n_kv_heads, 256
    tot = total if new > 1 else seen
    row, kv, cu = _tokens(batch, new, tot)
    pos = (kv - 1).int()
    ph = (tot + P - 1) // P
    table2 = torch.randperm(batch * ph, device="cuda").int().view(batch, ph)
    kh, vh = (torch.randint(0, 120, (batch * ph, Gh, P, 2 * Dh), dtype=torch.uint8, device="cuda") for _ in range(2))
    qh, oh, gh = _rand(T, Hh * Dh), _rand(T, Hh * Dh), _rand(T, Hh * Dh)
    if new > 1:
        bs2, bc2 = _blocks(batch, new, int(ops.prefill_attn_block_tokens(Hh, Gh)))
        k.add(f"attention {tag}", "hybrid", lambda: ops.paged_attention_prefill(qh, Hh, Gh, Dh, row, kv, bs2, bc2, table2, kh, vh, None, None, P, 0, Dh,
                                                                                Dh ** -0.5, gh, oh, False, 0, None),
              batch * tot * Gh * Dh * 4 + T * Hh * Dh * 6, batch * _pairs(new, tot, 0) * Hh * 2 * Dh)
    else:
        from ..models.hybrid import pick_attention_split
        sp, ns = pick_attention_split(tot, T * Gh)
        po2, ml2 = torch.empty(T * ns * Hh * Dh, device="cuda"), torch.empty(T * ns * Hh * 2, device="cuda")
        k.add(f"attention {tag}", "hybrid", lambda: ops.paged_attention(qh, Hh, Gh, Dh, row, kv, table2, kh, vh, None, None, P, 0, Dh, Dh ** -0.5, sp, ns,
                                                                        po2, ml2, gh, oh, None, None, 0, False),
              batch * tot * Gh * Dh * 4 + T * Hh * Dh * 6, batch * tot * Hh * 2 * Dh)
    ld = hyb.attn_in_dim
    projh, inv, w = _rand(T, ld), torch.rand(32, device="cuda"), _rand(Dh)
    k.add(f"norm + append {tag}", "hybrid",
          lambda: ops.attn_prep(projh, 0, Hh * Dh, 2 * Hh * Dh + Gh * Dh, Hh, Gh, Dh, w, w, 1e-6, True, 64, inv, 1.0, pos, row, pos, table2,
                                qh, kh, vh, None, None, P, 0, Dh, False, False, None, None), T * (Hh + 2 * Gh) * Dh * 4)


def _memory_rows(k: _Kernels, ops, cfg, hyb, batch: int, new: int, tag: str) -> None:
    m = cfg.layers[cfg.state_layers[0]].mixer
    H, D, V, T = m.heads, m.dim_p, m.vdim_p, batch * new
    cu, slot = _ints(torch.arange(batch + 1) * new), _ints(torch.arange(batch))
    proj, gates = _rand(T, m.main_cols, s=0.5), torch.randn(T, 2 * H, device="cuda")
    S, n, mm = torch.zeros((batch, H, D, V), device="cuda"), torch.zeros((batch, H, D), device="cuda"), torch.zeros((batch, H), device="cuda")
    norm, out = torch.ones(H * V, device="cuda"), _rand(T, H * V)
    ws = None if new == 1 else torch.empty(int(ops.mlstm_chunked_workspace_bytes(T, batch, H, D, V)), dtype=torch.uint8, device="cuda")
    # multiply-adds of the recurrence itself: state update and read-out, two per state element and token
    k.add(f"recurrence {tag}", "design", lambda: ops.mlstm(proj, 0, H * D, 2 * H * D, H * (2 * D + V), gates, 0, H, m.vdim, D ** -0.5, m.gate_cap, 1e-6,
                                                           norm, cu, slot, S, n, mm, out, True, ws, False, new == 1),
          2 * S.numel() * 4 + proj.numel() * 2 + out.numel() * 2, 2.0 * T * H * D * V)
    d, hk, hv = 128, hyb.gdn_qk_heads, hyb.gdn_v_heads
    qk, vd = hk * d, hv * d
    C = 2 * qk + vd
    conv, projh = _rand(T, C, s=0.5), _rand(T, C + vd + 2 * hv, s=0.5)
    ssm, A, nw, oh = torch.zeros((batch, hv, d, d), device="cuda"), torch.zeros(hv, device="cuda"), _rand(d), _rand(T, vd)
    ws2 = None if new == 1 else torch.empty(int(ops.gdn_chunked_workspace_bytes(T, batch, hv)), dtype=torch.uint8, device="cuda")
    k.add(f"recurrence {tag}", "hybrid", lambda: ops.gdn_recurrent(conv, 0, qk, 2 * qk, projh, C, C + vd, C + vd + hv, hk, hv, A, A, nw, 1e-6, cu, slot,
                                                                   ssm, True, oh, False, None, None, ws2),
          2 * ssm.numel() * 4 + conv.numel() * 2 + 2 * T * vd * 2, 2.0 * T * hv * d * d)


def equal_size_kuzanex(cfg):
    """Kuzanex with the width, the layer runs, the heads, the state size and the feed-forwards of a latent / gated-memory
    configuration; every key is visible."""
    lat = next(l.mixer for l in cfg.layers if l.mixer.kind == "latent_attention")
    mem = next(l.mixer for l in cfg.layers if l.mixer.kind == "hgrn2")
    dim = min(256, 2 * mem.dim)
    attn = dict(heads=lat.heads, kv_heads=max(1, lat.heads // 4), dim=lat.dim, vdim=lat.vdim, scale=lat.dim ** -0.5, softcap=50.0,
                mask={"size": 1 << 20})
    memory = dict(heads=max(1, mem.heads * mem.dim * mem.vdim // (dim * dim)), dim=dim, vdim=dim, gate_cap=15.0)
    pattern = "".join("a" if cfg.mixer_of(r).kind == "latent_attention" else "m" for r in range(len(cfg.runs)))
    return replace(kuzanex._design(f"kuzanex-like-{cfg.name}", cfg.hidden, cfg.vocab, pattern, attn, memory, cfg.layers[0].mlp.ff), max_context=cfg.max_context)


def _latent_design_rows(k: _Kernels, model, ws, cfg, batch: int, new: int, total: int, tag: str) -> None:
    """Kernels of a latent / gated-memory design: GEMMs, row steps, attention in the form the step takes, recurrence."""
    ops, status, w = model._raw_ops, model.status.tensor, model.w
    at, mt = (next(i for i, l in enumerate(cfg.layers) if l.mixer.kind == kind) for kind in ("latent_attention", "hgrn2"))
    m, g = cfg.layers[at].mixer, cfg.layers[mt].mixer
    T, h, P = batch * new, cfg.hidden_p, 64
    pa, pm = f"text/layers/{at}", f"text/layers/{mt}"

    def gemm(what, weight, x=None, out32_from=None, act=0, bias=None):
        N, K = weight.shape
        rows = T if x is None else x.shape[0]
        x = _rand(rows, K) if x is None else x
        out = torch.empty((rows, N), dtype=torch.bfloat16, device="cuda")
        o32 = None if out32_from is None else torch.empty((rows, N - out32_from), device="cuda")
        splits = int(ops.gemm_pick_splits(rows, N, K, 0))
        n_out = rows * N * 2 if out32_from is None else rows * (out32_from * 2 + (N - out32_from) * 4)
        k.add(f"{what} {tag}", "design", lambda: ops.gemm_bf16(x, weight, None if out32_from == 0 else out, 0, None, bias, None, splits, status,
                                                               False, act, None, None, None, None, None, o32, out32_from or 0),
              N * K * 2 + rows * K * 2 + n_out, rows * N * K)
    gemm("input projection (memory)", w[f"{pm}/mix/in_proj"], out32_from=g.main_cols, bias=w[f"{pm}/mix/in_bias"])
    gemm("input projection (attention)", w[f"{pa}/mix/in_proj"])
    gemm("query projection", w[f"{pa}/mix/uq"])
    gemm("output projection", w[f"{pm}/mix/out_proj"], out32_from=0)
    gemm("feed-forward up", w[f"{pm}/mlp/up"], act=4, bias=w[f"{pm}/mlp/up_bias"])
    gemm("feed-forward down", w[f"{pm}/mlp/down"], out32_from=0, bias=w[f"{pm}/mlp/down_bias"])
    if cfg.loop is not None:
        gemm("loop entry", w["text/loop/in_proj"], out32_from=0)
    # row steps: in front of a feed-forward (the like of the post-sum norm), and with the convolution
    x32, x2, d32, xa = torch.randn(T, h, device="cuda"), torch.empty(T, h, device="cuda"), torch.randn(T, h, device="cuda"), _rand(T, h)
    slots, cu = _ints(torch.arange(batch)), _ints(torch.arange(batch + 1) * new)
    hist = torch.zeros((batch, cfg.conv_taps - 1, h), device="cuda")
    common = (w[f"{pm}/norm1b"], w[f"{pm}/norm2"], xa, cfg.hidden, cfg.norm_groups, cfg.residual_mult, 1e-6)
    k.add(f"residual rows {tag}", "design", lambda: ops.sandwich_rows(x32, x32, d32, *common, None, None, None, None, new, True, False), T * h * 14)
    dst = x2 if new > 1 else x32
    k.add(f"residual rows + convolution {tag}", "design",
          lambda: ops.sandwich_rows(x32, dst, d32, *common, w[f"{pm}/conv"], hist, cu, slots, new, True, False),
          T * h * 14 + 2 * hist.numel() * 4)
    # latent attention
    H, R, C, V, D = m.heads, m.rot_p, m.kv_rank_p, m.vdim_p, m.dim_p
    per = (total + P - 1) // P
    row, kv, _ = _tokens(batch, new, total)
    pos = (kv - 1).int()
    table = torch.randperm(batch * per, device="cuda").int().view(batch, per)
    pages = _rand(batch * per, 1, P, C + R)
    proj, lat, q = _rand(T, m.main_cols), _rand(T, m.q_rank_p), _rand(T, m.q_cols)
    freq, sink = w[f"{pa}/mix/freq"], w[f"{pa}/mix/sink"]
    k.add(f"norm + append {tag}", "design", lambda: ops.latent_prep(proj, m.q_rank, m.kv_rank, m.rot_dim, w[f"{pa}/mix/q_norm"], w[f"{pa}/mix/kv_norm"],
                                                                   1e-6, freq, row, pos, table, lat, pages, False), T * m.main_cols * 4)
    start, count = _blocks(batch, new, 64)
    blocks = (start, count, min(new, 64))
    pairs = batch * _pairs(new, total, 0)
    if new == 1:
        from ..runtime.batch import SeqChunk, StepBuffers
        step = StepBuffers(batch, batch, "cpu", attn_block_tokens=64).build([SeqChunk(i, i, total - 1, [0]) for i in range(batch)])
        split, n = model.pick_latent_split(ws, step, m)
        q_abs, o_lat, out = _rand(T, H * C), _rand(T, H * C), _rand(T, H * V)
        po, ml = torch.empty(T * n * H * C, device="cuda"), torch.empty(T * n * H * 2, device="cuda")
        k.add(f"attention {tag}", "design", lambda: ops.latent_absorbed_attention(q_abs, q, pages, table, row, kv, H, m.rot_dim, m.scale, freq, sink, o_lat,
                                                                                *blocks, row, cu, 0, split, n, po, ml, False),
              batch * total * (C + R) * 2 + T * H * (2 * C + R) * 2, pairs * H * (2 * C + R))
        uk, uv = w[f"{pa}/mix/uk_t"], w[f"{pa}/mix/uv"]
        k.add(f"per-head GEMM, queries {tag}", "design", lambda: ops.head_gemm(q, D + R, uk, q_abs, None, None, 0, False),
              uk.numel() * 2 + T * H * (D + C) * 2, T * uk.numel())
        k.add(f"per-head GEMM, values {tag}", "design", lambda: ops.head_gemm(o_lat, C, uv, out, None, None, 0, False),
              uv.numel() * 2 + T * H * (V + C) * 2, T * uv.numel())
    else:
        rows = _rand(batch * total, C + R)
        seqs = _ints([[i, i * total, 0, total] for i in range(batch)])
        ukv = w[f"{pa}/mix/ukv"]
        wide, out, base = _rand(batch * total, ukv.shape[0]), _rand(T, H * V), _ints([[i * total, 0] for i in range(batch)])
        k.add(f"gather {tag}", "design", lambda: ops.latent_gather(pages, table, seqs, total, rows, False), rows.numel() * 4)
        gemm("expansion", ukv, x=rows[:, :C])
        k.add(f"attention {tag}", "design", lambda: ops.latent_expanded_attention(q, rows, wide, kv, H, C, m.rot_dim, m.scale, freq, sink, out, *blocks, row,
                                                                                base, False),
              wide.numel() * 2 + batch * total * R * 2 + T * H * (D + R + V) * 2, pairs * H * (D + R + V))
    # gated memory
    projm, gates = _rand(T, g.main_cols, s=0.5), torch.randn(T, g.gate_cols, device="cuda") + 3
    S, out = torch.zeros((batch, g.heads, g.dim_p, g.vdim_p), device="cuda"), _rand(T, g.out_cols)
    cws = None if new == 1 else torch.empty(int(ops.gated_chunked_workspace_bytes(T, batch, g.heads, g.dim_p, g.vdim_p)), dtype=torch.uint8, device="cuda")
    k.add(f"recurrence {tag}", "design", lambda: ops.gated_memory(projm, 0, g.heads * g.dim_p, gates, w[f"{pm}/mix/lower"], g.vdim, 1e-6, w[f"{pm}/mix/norm"], cu,
                                                                 slots, S, out, True, cws, False, new == 1),
          2 * S.numel() * 4 + projm.numel() * 2 + gates.numel() * 4 + out.numel() * 2, 2.0 * T * g.heads * g.dim_p * g.vdim_p)


def _kernels(cfg, other, weights, iters: int, only: str) -> List[dict]:
    from ..models.layered import LayeredModel, LayeredWorkspace
    latent = any(l.mixer.kind == "latent_attention" for l in cfg.layers)
    model = LayeredModel(cfg, weights, "cuda:0")
    ws = LayeredWorkspace(cfg, 64, 64, "cuda:0", torch.bfloat16)
    ops = model._raw_ops
    base, hyb = (other, equal_size_hybrid(other)) if latent else (cfg, other)
    k = _Kernels(iters, only, {"design": "kuzanex", "hybrid": ""} if latent else None)
    for T, tag in ((32, "decode x32"), (2048, "prefill 2048")):
        _gemm_rows(k, ops, model.status.tensor, base, hyb, T, tag)
    for batch, new, tag in ((32, 1, "decode x32"), (1, 2048, "prefill 2048")):
        _attention_rows(k, ops, model, ws, base, hyb, batch, new, 2048, tag)
    for batch, new, tag in ((32, 1, "decode x32"), (1, 2048, "prefill 2048")):
        _memory_rows(k, ops, base, hyb, batch, new, tag)
    if latent:
        k.names = {}
        for batch, new, tag in ((32, 1, "decode x32"), (1, 2048, "prefill 2048")):
            _latent_design_rows(k, model, ws, cfg, batch, new, 2048, tag)
    model.status.check("after the kernel timings")
    return k.rows


def compare(name: str, layers: int = 0, iters: int = 10, throughput: bool = True, only: str = "") -> Dict[str, object]:
    cfg = LAYERED_REGISTRY[name]
    if layers:
        cfg = cfg.shrink(layers)
    streams, branch = cfg.residual == "streams", cfg.residual == "branch"
    latent = not streams and any(l.mixer.kind == "latent_attention" for l in cfg.layers)
    if streams or branch:
        from . import branchbench, streambench
        other, label = (branchbench if branch else streambench).equal_size_expert_hybrid(cfg), "hybrid"
    else:
        other, label = (equal_size_kuzanex(cfg), "kuzanex") if latent else (equal_size_hybrid(cfg), "hybrid")
    res: Dict[str, object] = {"comparison": cfg.name, "design_params": cfg.param_count(), f"{label}_params": other.param_count(), "dtype": "bf16",
                              "data": "synthetic", "l2": "flushed before every kernel"}
    weights = random_layered_weights(cfg, "cuda:0")
    if streams or branch:
        rows = (branchbench.branch_kernels if branch else streambench.stream_kernels)(cfg, other, weights, iters, only)
    else:
        rows = _kernels(cfg, other, weights, iters, only)
    pair: Dict[str, dict] = {}
    for r in rows:
        pair.setdefault(r["kernel"], {})[r["model"]] = r
    res["kernels"] = rows
    likes = {n: next(v for m, v in p.items() if m != "design") for n, p in pair.items() if len(p) == 2 and "design" in p}
    res[f"farther_than_{label}"] = {n: round(like["fraction"] / max(1e-4, pair[n]["design"]["fraction"]), 2) for n, like in likes.items()}
    if throughput:
        res["throughput"] = {}
        w2 = random_layered_weights(other, "cuda:0") if latent else random_weights(other, "cuda:0", seed=0)
        for batch, prompt in ((1, 2048), (8, 1024), (32, 1024)):
            res["throughput"][f"{batch} x {prompt}"] = {"design": _throughput(cfg, weights, batch, prompt, 32),
                                                        label: _throughput(other, w2, batch, prompt, 32)}
    return res


def main(argv=None) -> int:
    import argparse
    import json
    ap = argparse.ArgumentParser(description="kernel timings of a layer-list geometry beside the hybrid's")
    ap.add_argument("model", choices=sorted(LAYERED_REGISTRY))
    ap.add_argument("--layers", type=int, default=4)
    ap.add_argument("--iters", type=int, default=10)
    ap.add_argument("--only", default="", help="only kernels whose 'design: name' or 'hybrid: name' contains this")
    args = ap.parse_args(argv)
    for r in compare(args.model, args.layers, args.iters, False, args.only)["kernels"]:
        print(json.dumps(r))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
