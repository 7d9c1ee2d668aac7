"""Layer-list designs beside the hybrid decoder of equal size: model throughput and per-kernel roofline fractions.

`python bench.py --compare kuzanex-1b` prints one JSON line: prefill and decode tokens/s of the two models through the
same generator (random weights, bf16), and for every kernel of the design its time, what bounds it, and the same for
the hybrid's kernel of the like kind at equal size.  Kernels are timed cold (L2 flushed before every launch) with CUDA
events; the roofline of a kernel is the slower of its algorithmic bytes at the measured copy bandwidth and its
algorithmic multiply-adds at the measured bf16 GEMM rate.
"""
from __future__ import annotations

from typing import Dict, List

import torch

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

    def __init__(self, iters: int, only: str = ""):
        self.only = only
        self.flush, self.iters, self.rows = L2Flusher(), iters, []
        self.bw, self.fl, self.how = measured_peaks()

    def add(self, what: str, model: str, fn, n_bytes: float, macs: float = 0.0) -> None:
        if self.only not in f"{model}: {what}":
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


def compare(name: str, layers: int = 0, iters: int = 10, throughput: bool = True, only: str = "") -> Dict[str, object]:
    cfg = LAYERED_REGISTRY[name]
    if layers:
        cfg = cfg.shrink(layers)
    hyb = equal_size_hybrid(cfg)
    res: Dict[str, object] = {"comparison": cfg.name, "design_params": cfg.param_count(), "hybrid_params": hyb.param_count(), "dtype": "bf16",
                              "data": "synthetic", "l2": "flushed before every kernel"}
    weights = random_layered_weights(cfg, "cuda:0")
    from ..models.layered import LayeredModel, LayeredWorkspace
    model = LayeredModel(cfg, weights, "cuda:0")
    ws = LayeredWorkspace(cfg, 64, 64, "cuda:0", torch.bfloat16)
    ops = model._raw_ops
    k = _Kernels(iters, only)
    for T, tag in ((32, "decode x32"), (2048, "prefill 2048")):
        _gemm_rows(k, ops, model.status.tensor, cfg, hyb, T, tag)
    _attention_rows(k, ops, model, ws, cfg, hyb, 32, 1, 2048, "decode x32")
    _attention_rows(k, ops, model, ws, cfg, hyb, 1, 2048, 2048, "prefill 2048")
    _memory_rows(k, ops, cfg, hyb, 32, 1, "decode x32")
    _memory_rows(k, ops, cfg, hyb, 1, 2048, "prefill 2048")
    model.status.check("after the kernel timings")
    del model, ws
    rows: List[dict] = k.rows
    pair: Dict[str, dict] = {}
    for r in rows:
        pair.setdefault(r["kernel"], {})[r["model"]] = r
    res["kernels"] = rows
    res["farther_than_hybrid"] = {n: round(p["hybrid"]["fraction"] / p["design"]["fraction"], 2) for n, p in pair.items() if len(p) == 2}
    if throughput:
        res["throughput"] = {}
        w2 = random_weights(hyb, "cuda:0", seed=0)
        for batch, prompt in ((1, 2048), (8, 1024), (32, 1024)):
            res["throughput"][f"{batch} x {prompt}"] = {"design": _throughput(cfg, weights, batch, prompt, 32),
                                                        "hybrid": _throughput(hyb, w2, batch, prompt, 32)}
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
