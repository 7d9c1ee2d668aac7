"""Kernel timings of the designs that norm their sublayers' outputs and run attention and a state space side by side (Ratilorn)
beside the closest other kernels at equal size: Kuzanex (attention mixed across heads, row steps) and the hybrid decoder with
sparse experts (grouped-query attention, projections, gated units, expert block, recurrence).  `utils/layerbench.py` drives it
and says how times and rooflines are taken."""
from __future__ import annotations

import torch

from ..models.config import ModelConfig, MoEConfig
from .layerbench import _blocks, _ints, _Kernels, _pairs, _rand, _tokens


def equal_size_expert_hybrid(cfg) -> ModelConfig:
    """The hybrid decoder with the same width, depth, query and key / value width, channels of recurrent state and experts."""
    par = next(l.mixer for l in cfg.layers if l.mixer.kind == "parallel")
    att, rec = par.left, par.right
    f = next(l.mlp for l in cfg.layers if l.mlp is not None and l.mlp.kind == "moe")
    v_heads = max(2, rec.heads * rec.vdim // 128 // 2 * 2)
    return ModelConfig(name=f"hybrid-like-{cfg.name}", n_layers=cfg.n_layers, hidden=cfg.hidden, vocab=cfg.vocab,
                       n_q_heads=max(1, att.heads * att.dim // 256), n_kv_heads=max(1, att.kv_heads * att.dim // 256), head_dim=256, rot_dim=64,
                       rope_theta=1e7, gdn_qk_heads=v_heads // 2, gdn_v_heads=v_heads, ffn_inter=0, mtp_layers=0,
                       moe=MoEConfig(n_experts=f.experts, top_k=f.top, expert_inter=f.expert.ff_p, shared_inter=f.shared.ff_p))


def _first(cfg, test) -> int:
    return next(i for i, l in enumerate(cfg.layers) if test(l))


def _gemms(k: _Kernels, model, cfg, hyb, T: int, tag: str) -> None:
    ops, w, status, h = model._raw_ops, model.w, model.status.tensor, cfg.hidden_p
    par, att = _first(cfg, lambda l: l.mixer.kind == "parallel"), _first(cfg, lambda l: l.mixer.kind == "attention")
    moe, dense = _first(cfg, lambda l: l.mlp.kind == "moe"), _first(cfg, lambda l: l.mlp.kind == "glu")
    m, f, d = cfg.layers[par].mixer, cfg.layers[moe].mlp, cfg.layers[dense].mlp

    def gemm(who, what, weight, epi=0, out32_from=None, bias=None):
        N, K = weight.shape
        x, cols = _rand(T, K), N // 2 if epi == 2 else N
        out = None if out32_from == 0 else torch.empty((T, cols), dtype=torch.bfloat16, device="cuda")
        o32 = None if out32_from is None else torch.empty((T, N - out32_from), device="cuda")
        splits = int(ops.gemm_pick_splits(T, N, K, epi))
        n_out = T * cols * 2 if out32_from is None else T * (out32_from * 2 + (N - out32_from) * 4)
        k.add(f"{what} {tag}", who, lambda: ops.gemm_bf16(x, weight, out, epi, out if epi == 1 else None, bias, None, splits, status, False, 0,
                                                          out32=o32, out32_from=out32_from or 0), N * K * 2 + T * K * 2 + n_out, T * N * K)

    def like(what, N, K, epi=0):
        gemm("hybrid", what, _rand(N, K, s=0.02), epi)
    p, q = f"text/layers/{par}", f"text/layers/{att}"
    gemm("design", "input projection (both mixers)", w[f"{p}/mix/in_proj"], out32_from=m.main_cols, bias=w[f"{p}/mix/in_bias"])
    like("input projection (both mixers)", hyb.gdn_in_dim, h)
    gemm("design", "input projection (attention)", w[f"{q}/mix/in_proj"], bias=w[f"{q}/mix/in_bias"])
    like("input projection (attention)", hyb.attn_in_dim, h)
    gemm("design", "output projection (attention)", w[f"{p}/left/mix/out_proj"], out32_from=0)
    like("output projection (attention)", h, hyb.n_q_heads * hyb.head_dim, 1)
    gemm("design", "output projection (state space)", w[f"{p}/right/mix/out_proj"], out32_from=0)
    like("output projection (state space)", h, hyb.gdn_v_dim, 1)
    gemm("design", "dense up", w[f"text/layers/{dense}/mlp/up"], 2)
    like("dense up", 2 * d.ff_p, h, 2)
    gemm("design", "dense down", w[f"text/layers/{dense}/mlp/down"], out32_from=0)
    like("dense down", h, d.ff_p, 1)
    gemm("design", "router", w[f"text/layers/{moe}/mlp/router"], out32_from=0)
    like("router", (f.experts + 8) // 8 * 8, h)
    gemm("design", "shared expert up", w[f"text/layers/{moe}/mlp/shared_up"], 2)
    like("shared expert up", 2 * f.shared.ff_p, h, 2)
    gemm("design", "shared expert down", w[f"text/layers/{moe}/mlp/shared_down"], out32_from=0)
    like("shared expert down", h, f.shared.ff_p)


def _rows(k: _Kernels, model, cfg, T: int, tag: str) -> None:
    """The three forms of the row step beside the norm after the sum, each with the bytes it moves."""
    ops, h = model._raw_ops, cfg.hidden_p
    f = cfg.layers[_first(cfg, lambda l: l.mlp.kind == "moe")].mlp
    x, a, b, xa, w = torch.randn(T, h, device="cuda"), torch.randn(T, h, device="cuda"), torch.randn(T, h, device="cuda"), _rand(T, h), torch.ones(h, device="cuda")
    tail = (w, None, xa, cfg.hidden, 1e-6, False)
    none4, none7 = (None,) * 4, (None,) * 6 + (0,)
    k.add(f"residual rows {tag}", "design", lambda: ops.branch_rows(x, *none4, a, *none7[1:], *tail), T * h * 14)
    gain = torch.ones(1, device="cuda")
    k.add(f"residual rows {tag}", "kuzanex", lambda: ops.post_norm_rows(x, a, xa, cfg.hidden, 2.0, 1e-6, gain, None, False), T * h * 14)
    k.add(f"residual rows, two branches {tag}", "design", lambda: ops.branch_rows(x, a, b, w, w, *none7, *tail), T * h * 18)
    k.add(f"residual rows, two branches {tag}", "kuzanex", lambda: ops.post_norm_rows(x, a, xa, cfg.hidden, 2.0, 1e-6, gain, None, False), T * h * 14)
    choice = torch.randint(0, f.experts, (T, f.top), device="cuda").int()
    weight, ret = torch.rand(T, f.top, device="cuda"), _rand(T * f.top, h)
    k.add(f"residual rows with the expert sum {tag}", "design", lambda: ops.branch_rows(x, *none4, a, None, choice, weight, ret, xa, f.experts, *tail),
          T * h * (14 + 2 * f.top))
    k.add(f"residual rows with the expert sum {tag}", "kuzanex", lambda: ops.post_norm_rows(x, a, xa, cfg.hidden, 2.0, 1e-6, gain, None, False), T * h * 14)


def _expert_block(k: _Kernels, model, ws, cfg, hyb, T: int, tag: str) -> None:
    """The whole feed-forward, row step included: what lies between two mixers' kernels."""
    from ..models.experts import run_experts
    from ..models.moe import MoeBlock
    ops, w, h = model._raw_ops, model.w, cfg.hidden_p
    at = _first(cfg, lambda l: l.mlp.kind == "moe")
    f, p, status = cfg.layers[at].mlp, f"text/layers/{at}", model.status.tensor
    E, kk, ff, sf = f.experts, f.top, f.expert.ff_p, f.shared.ff_p
    x, xo, delta, X = _rand(T, h), _rand(T, h), torch.empty(T, h, device="cuda"), torch.randn(T, h, device="cuda")
    used = int(torch.unique(run_experts(model, ws.experts, T, p, f, x, delta)["choice"]).numel())
    rows, weights = T * kk, (used * ff + sf) * 3 * h * 2

    def design():
        y = run_experts(model, ws.experts, T, p, f, x, delta)
        ops.branch_rows(X, None, None, None, None, *y.values(), w[f"{p}/norm2"], None, xo, cfg.hidden, 1e-6, False)      # (the next run routes the same rows)
    k.add(f"expert block {tag}", "design", design, weights + T * h * 14 + 2 * rows * h * 2, (rows * ff + T * sf) * 3 * h)
    block = MoeBlock(hyb, "cuda:0", T)
    hw = {f"l/moe/{n}": t for n, t in (("router", _rand(E + 1, h, s=0.02)), ("experts_gate_up", w[f"{p}/mlp/up"]), ("experts_down", w[f"{p}/mlp/down"]),
                                       ("shared_gate_up", w[f"{p}/mlp/shared_up"]), ("shared_down", w[f"{p}/mlp/shared_down"]))}

    class Host:                       # what MoeBlock.forward takes of its model
        pass
    host, hws = Host(), Host()
    host.ops, host.w, host.status = ops, hw, model.status
    host._gemm = lambda a, b, o, epi=0: ops.gemm_bf16(a, b, o, epi, None, None, None, int(ops.gemm_pick_splits(a.shape[0], *b.shape, epi)), status, False)
    hws.x, hws.normed = _rand(T, h), _rand(T, h)
    norm, normed = _rand(h), _rand(T, h)
    block.forward(host, hws, T, "l", norm, normed)
    used_h = int(torch.unique(block.ids[:T]).numel())
    hws.normed = _rand(T, h)
    k.add(f"expert block {tag}", "hybrid", lambda: block.forward(host, hws, T, "l", norm, normed), (used_h * ff + sf) * 3 * h * 2 + T * h * 8 + 2 * T * kk * h * 2,
          (T * kk * ff + T * sf) * 3 * h)
    e = ws.experts
    run_experts(model, e, T, p, f, x, delta)
    ids, pos, wts = (t[: T * kk].view(T, kk) for t in (e.ids, e.pos, e.weights))
    logits = e.logits[:T, : f.router_cols]
    k.add(f"routing {tag}", "design", lambda: ops.moe_route_scored(logits, E, 0, kk, w[f"{p}/mlp/correction"], 1.0, e.hist, ids, wts, pos, False, True, True,
                                                                   f.groups, f.keep), T * (E * 4 + kk * 12))
    lb, sg = _rand(T, (E + 8) // 8 * 8), torch.empty(T, device="cuda")
    k.add(f"routing {tag}", "hybrid", lambda: ops.moe_route(lb, E, kk, True, True, e.hist, ids, wts, pos, sg), T * (E * 2 + kk * 12))
    e.hist.zero_()


def _attention(k: _Kernels, model, ws, cfg, hyb, batch: int, new: int, total: int, tag: str) -> None:
    ops, P = model._raw_ops, 64
    T, per = batch * new, (total + P - 1) // P
    row, kv, _ = _tokens(batch, new, total)
    pos = (kv - 1).int()
    table = torch.randperm(batch * per, device="cuda").int().view(batch, per)
    # weights by sigmoid, mixed across heads, beside soft-capped scores that are mixed (Kuzanex, every key visible)
    m = cfg.layers[_first(cfg, lambda l: l.mixer.kind == "attention")].mixer
    H, G, D, V = m.heads, m.kv_heads, m.dim_p, m.vdim_p
    kp, vp = _rand(batch * per, G, P, D), _rand(batch * per, G, P, V)
    q, out, gate = _rand(T, H * D, s=0.3), _rand(T, H * V), torch.randn(T, H, device="cuda")
    mix, slope = torch.eye(H, device="cuda") + 0.1, torch.rand(H, device="cuda") * 0.01
    extra = (True, *(torch.rand(H, device="cuda") for _ in range(3)))
    macs, n_bytes = batch * _pairs(new, total, 0) * H * (D + V), batch * total * G * (D + V) * 2 + T * H * (D + V) * 2
    args = (q, kp, vp, table, row, kv)
    forms = (("design", (0, m.scale, 0.0, 0.0, mix, None, None, out), extra), ("kuzanex", (0, m.scale, 50.0, 1.0, mix, slope, gate, out), (False, None, None, None)))
    for who, shape, tail in forms:
        if new > 1:
            blocks = _blocks(batch, new, 64)
            one = int(ops.head_mix_prefill_scratch(H, total, 0, 1, tail[0]))
            scratch = torch.empty(max(one, min(one * blocks[0].numel(), 1 << 30)), dtype=torch.uint8, device="cuda")
            k.add(f"head-mixing attention {tag}", who, lambda: ops.head_mix_prefill(*args, *shape, *blocks, total, scratch, False, *tail), n_bytes, macs)
        else:
            split, n = model.pick_split(ws, T, total, 0)
            po, ml = torch.empty(T * n * H * V, device="cuda"), torch.empty(T * n * H * 2, device="cuda")
            k.add(f"head-mixing attention {tag}", who, lambda: ops.head_mix_attention(*args, *shape, split, n, po, ml, False, 0, None, *tail), n_bytes, macs)
    proj, qn = _rand(T, m.main_cols), torch.ones(D, device="cuda")
    first, lam = _rand(T, G * V), torch.tensor([0.3], device="cuda")
    append = (proj, 0, H * D, (H + G) * D, H, G, m.dim)
    k.add(f"norm + value mix + append {tag}", "design", lambda: ops.qkv_append(*append, None, None, 1e-6, row, pos, table, q, kp, vp, P, False, None, True, first,
                                                                               lam), T * (m.main_cols * 4 + G * V * 2))
    k.add(f"norm + value mix + append {tag}", "kuzanex", lambda: ops.qkv_append(*append, qn, qn, 1e-6, row, pos, table, q, kp, vp, P, False),
          T * m.main_cols * 4)
    # softmax attention of the left side beside the hybrid's
    m = cfg.layers[_first(cfg, lambda l: l.mixer.kind == "parallel")].mixer.left
    H, G, D, V = m.heads, m.kv_heads, m.dim_p, m.vdim_p
    kp, vp = _rand(batch * per, G, P, D), _rand(batch * per, G, P, V)
    q, out = _rand(T, H * D), _rand(T, H * V)
    macs, n_bytes = batch * _pairs(new, total, 0) * H * (D + V), batch * total * G * (D + V) * 2 + T * H * (D + V) * 2
    args = (q, kp, vp, table, row, kv)
    if new > 1:
        blocks = _blocks(batch, new, 64)
        k.add(f"attention {tag}", "design", lambda: ops.group_prefill(*args, 0, 0, m.scale, 0.0, None, out, *blocks, False), n_bytes, macs)
    else:
        split, n = model.pick_split(ws, T, total, 0, ctas=G)
        po, ml = torch.empty(T * n * H * V, device="cuda"), torch.empty(T * n * H * 2, device="cuda")
        k.add(f"attention {tag}", "design", lambda: ops.head_mix_attention(*args, 0, m.scale, 0.0, 0.0, None, None, None, out, split, n, po, ml, False),
              n_bytes, macs)
    Hh, Gh, Dh = hyb.n_q_heads, hyb.n_kv_heads, 256
    kh, vh = (torch.randint(0, 120, (batch * per, Gh, P, 2 * Dh), dtype=torch.uint8, device="cuda") for _ in range(2))
    qh, oh, gh = _rand(T, Hh * Dh), _rand(T, Hh * Dh), _rand(T, Hh * Dh)
    hb, hm = batch * total * Gh * Dh * 4 + T * Hh * Dh * 6, batch * _pairs(new, total, 0) * Hh * 2 * Dh
    if new > 1:
        bs, bc = _blocks(batch, new, int(ops.prefill_attn_block_tokens(Hh, Gh)))
        k.add(f"attention {tag}", "hybrid", lambda: ops.paged_attention_prefill(qh, Hh, Gh, Dh, row, kv, bs, bc, table, kh, vh, None, None, P, 0, Dh, Dh ** -0.5,
                                                                                gh, oh, False, 0, None), hb, hm)
    else:
        from ..models.hybrid import pick_attention_split
        sp, ns = pick_attention_split(total, T * Gh)
        po2, ml2 = torch.empty(T * ns * Hh * Dh, device="cuda"), torch.empty(T * ns * Hh * 2, device="cuda")
        k.add(f"attention {tag}", "hybrid", lambda: ops.paged_attention(qh, Hh, Gh, Dh, row, kv, table, kh, vh, None, None, P, 0, Dh, Dh ** -0.5, sp, ns, po2, ml2,
                                                                        gh, oh, None, None, 0, False), hb, hm)


def _recurrence(k: _Kernels, model, cfg, hyb, batch: int, new: int, tag: str) -> None:
    """Convolution, recurrence, gate and norm together: what lies between the two projections."""
    ops, w = model._raw_ops, model.w
    at = _first(cfg, lambda l: l.mixer.kind == "parallel")
    m, p = cfg.layers[at].mixer.right, f"text/layers/{at}/right/mix"
    T, H, V, N, C = batch * new, m.heads, m.vdim_p, m.state_p, m.out_cols
    cu, slot = _ints(torch.arange(batch + 1) * new), _ints(torch.arange(batch))
    seq, pos = _ints(torch.arange(batch).repeat_interleave(new)), _ints(torch.arange(100, 100 + new).repeat(batch))
    proj, dt, out = _rand(T, m.main_cols), torch.randn(T, H, device="cuda") - 3, _rand(T, C)
    ring, S = torch.zeros((batch, m.taps, m.conv_cols), device="cuda"), torch.zeros((batch, H, V, N), device="cuda")
    u = torch.empty(T * m.conv_cols, dtype=torch.bfloat16, device="cuda")
    cws = None if new == 1 else torch.empty(int(ops.ssd_chunked_workspace_bytes(T, batch, H, N, V)), dtype=torch.uint8, device="cuda")
    state = (proj, C, dt, w[f"{p}/conv"], w[f"{p}/conv_bias"], w[f"{p}/rate"], w[f"{p}/skip"], m.groups, cu, seq, pos, slot, ring, S, u, out, True, cws, False,
             new == 1)

    def design():
        ops.ssd(*state)
        ops.ssd_gated_norm(out, proj, w[f"{p}/norm"], H, m.vdim, m.norm_groups, 1e-6, False)
    k.add(f"convolution + recurrence + norm {tag}", "design", design, 2 * S.numel() * 4 + ring.numel() * 4 + proj.numel() * 2 + out.numel() * 2, 2.0 * T * H * V * N)
    d, hk, hv = 128, hyb.gdn_qk_heads, hyb.gdn_v_heads
    qk, vd = hk * d, hv * d
    n = 2 * qk + vd
    projh = _rand(T, n + vd + 2 * hv, s=0.5)
    conv, cw, cst = _rand(T, n, s=0.5), _rand(n, 4), torch.zeros((batch, 3, n), dtype=torch.bfloat16, device="cuda")
    ssm, A, nw, oh = torch.zeros((batch, hv, d, d), device="cuda"), torch.zeros(hv, device="cuda"), _rand(d), _rand(T, vd)
    ws2 = None if new == 1 else torch.empty(int(ops.gdn_chunked_workspace_bytes(T, batch, hv)), dtype=torch.uint8, device="cuda")

    def hybrid():
        ops.causal_conv1d_silu(projh, 0, n, cw, cu, seq, slot, cst, conv, True, new == 1, False)
        ops.gdn_recurrent(conv, 0, qk, 2 * qk, projh, n, n + vd, n + vd + hv, hk, hv, A, A, nw, 1e-6, cu, slot, ssm, True, oh, False, None, None, ws2)
    k.add(f"convolution + recurrence + norm {tag}", "hybrid", hybrid, 2 * ssm.numel() * 4 + 2 * cst.numel() * 2 + projh.numel() * 2 + T * vd * 2, 2.0 * T * hv * d * d)


def branch_kernels(cfg, hyb, weights, iters: int, only: str, phases=(("decode x32", 32, 1), ("prefill 2048", 1, 2048))):
    from ..models.layered import LayeredModel, LayeredWorkspace
    model = LayeredModel(cfg, weights, "cuda:0")
    ws = LayeredWorkspace(cfg, 2048, 64, "cuda:0", torch.bfloat16)
    k = _Kernels(iters, only)
    for tag, batch, new in phases:
        T = batch * new
        _gemms(k, model, cfg, hyb, T, tag)
        _rows(k, model, cfg, T, tag)
        _expert_block(k, model, ws, cfg, hyb, T, tag)
        _attention(k, model, ws, cfg, hyb, batch, new, 2048, tag)
        _recurrence(k, model, cfg, hyb, batch, new, tag)
    model.status.check("after the kernel timings")
    return k.rows
