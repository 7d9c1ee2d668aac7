"""Kernel timings of the designs with residual streams and experts (Tuzupel) beside the closest other kernels at equal size:
the hybrid decoder with sparse experts (attention, projections, rows, expert block, recurrence) and Tebivik (latent attention).
`utils/layerbench.py` drives it and says how times and rooflines are taken."""
from __future__ import annotations

import torch

from ..models.config import ModelConfig, MoEConfig
from .layerbench import _blocks, _ints, _Kernels, _pairs, _rand, _tokens


def equal_size_expert_hybrid(cfg) -> ModelConfig:
    """The hybrid decoder with the same width, depth, query and key / value width, channels of recurrent state and experts."""
    att = next(l.mixer for l in cfg.layers if l.mixer.kind == "attention")
    rec = next(l.mixer for l in cfg.layers if l.mixer.kind == "rglru")
    f = next(l.mlp for l in cfg.layers if l.mlp is not None)
    v_heads = max(2, rec.width // 128 // 2 * 2)
    return ModelConfig(name=f"hybrid-like-{cfg.name}", n_layers=cfg.n_layers, hidden=cfg.hidden, vocab=cfg.vocab,
                       n_q_heads=max(1, att.heads * att.dim // 256), n_kv_heads=max(1, att.kv_heads * att.dim // 256), head_dim=256, rot_dim=64,
                       rope_theta=1e7, gdn_qk_heads=v_heads // 2, gdn_v_heads=v_heads, ffn_inter=0, mtp_layers=0,
                       moe=MoEConfig(n_experts=f.experts, top_k=f.top, expert_inter=f.expert.ff_p, shared_inter=f.shared.ff_p))


def _layers(cfg):
    return {kind: next(i for i, l in enumerate(cfg.layers) if l.mixer.kind == kind) for kind in ("attention", "latent_attention", "rglru")}


def _gemms(k: _Kernels, model, cfg, hyb, T: int, tag: str) -> None:
    ops, w, at, status = model._raw_ops, model.w, _layers(cfg), model.status.tensor
    f = cfg.layers[0].mlp

    def gemm(who, what, weight, epi=0, out32=False, bias=None, glu=()):
        N, K = weight.shape
        x, cols = _rand(T, K), N // 2 if epi == 2 else N
        out = torch.empty((T, cols), dtype=torch.float32 if out32 else torch.bfloat16, device="cuda")
        resid = out if epi == 1 else None
        splits = int(ops.gemm_pick_splits(T, N, K, epi))
        k.add(f"{what} {tag}", who, lambda: ops.gemm_bf16(x, weight, None if out32 else out, epi, resid, bias, None, splits, status, False, 0,
                                                          out32=out if out32 else None, glu=list(glu)),
              N * K * 2 + T * K * 2 + out.numel() * out.element_size(), T * N * K)

    def like(what, N, K, epi=0):
        gemm("hybrid", what, _rand(N, K, s=0.02), epi)
    h = cfg.hidden_p
    for kind, name, cols in (("rglru", "recurrence", hyb.gdn_in_dim), ("attention", "attention", hyb.attn_in_dim),
                             ("latent_attention", "latent attention", hyb.attn_in_dim)):
        p = f"text/layers/{at[kind]}/mix"
        gemm("design", f"input projection ({name})", w[f"{p}/in_proj"], bias=w.get(f"{p}/in_bias"))
        like(f"input projection ({name})", cols, h)
    gemm("design", "output projection", w[f"text/layers/{at['attention']}/mix/out_proj"], out32=True)
    like("output projection", h, hyb.n_q_heads * hyb.head_dim, 1)
    gemm("design", "router", w["text/layers/0/mlp/router"], out32=True)
    like("router", (f.experts + 8) // 8 * 8, h)
    gemm("design", "shared expert up", w["text/layers/0/mlp/shared_up"], 2, glu=(f.shared.limit, f.shared.slope, f.shared.shift))
    like("shared expert up", 2 * f.shared.ff_p, h, 2)
    gemm("design", "shared expert down", w["text/layers/0/mlp/shared_down"], out32=True)
    like("shared expert down", h, f.shared.ff_p)


def _rows(k: _Kernels, model, cfg, T: int, tag: str) -> None:
    ops, w, h, S = model._raw_ops, model.w, cfg.hidden_p, cfg.streams
    f, p = cfg.layers[0].mlp, "text/layers/0"
    X, delta, xa = torch.randn(T, S, h, device="cuda"), torch.randn(T, h, device="cuda"), _rand(T, h)
    update = (w[f"{p}/hc1/mix"], w[f"{p}/hc1/out"], w[f"{p}/hc2/in"], w[f"{p}/norm2"], xa, cfg.hidden, 1e-6, False)
    none = (None,) * 5 + (0,)
    k.add(f"residual rows {tag}", "design", lambda: ops.stream_rows(X, None, None, X, delta, *none, *update), T * h * (8 * S + 6))
    xb, nb, nw = _rand(T, h), _rand(T, h), _rand(h)
    k.add(f"residual rows {tag}", "hybrid", lambda: ops.add_rmsnorm(None, 0, None, xb, None, nw, nb, T, h, 1e-6, True, False), T * h * 4)
    choice = torch.randint(0, f.choices, (T, f.top), device="cuda").int()
    weight, ret, gate = torch.rand(T, f.top, device="cuda"), _rand(T * f.top, h), torch.randn(T, f.router_cols, device="cuda")
    parts = (delta, gate[:, f.choices: f.choices + 1], choice, weight, ret, xa, f.experts)
    k.add(f"residual rows with the expert sum {tag}", "design", lambda: ops.stream_rows(X, None, None, X, *parts, *update),
          T * h * (8 * S + 6 + 2 * f.top + 2))


def _expert_block(k: _Kernels, model, ws, cfg, hyb, T: int, tag: str) -> None:
    """The whole feed-forward, row step included: what lies between two mixers' kernels."""
    from ..models.experts import glu, run_experts
    from ..models.hybrid import Workspace
    from ..models.moe import MoeBlock
    ops, w, h, S = model._raw_ops, model.w, cfg.hidden_p, cfg.streams
    f, p, status = cfg.layers[0].mlp, "text/layers/0", model.status.tensor
    E, kk, ff, sf = f.experts, f.top, f.expert.ff_p, f.shared.ff_p
    x, delta, X = _rand(T, h), torch.empty(T, h, device="cuda"), torch.randn(T, S, h, device="cuda")
    # experts whose weights the step reads, rows that they see
    chosen = run_experts(model, ws.experts, T, p, f, x, delta)["choice"].flatten()
    used, rows = int(torch.unique(chosen[chosen < E]).numel()), int((chosen < E).sum())
    weights = (used * ff + sf) * 3 * h * 2
    macs = (rows * ff + T * sf) * 3 * h

    def design():
        y = run_experts(model, ws.experts, T, p, f, x, delta)
        ops.stream_rows(X, None, None, X, *y.values(), w[f"{p}/hc2/mix"], w[f"{p}/hc2/out"], w[f"{p}/hc1/in"], w[f"{p}/norm1"], x, cfg.hidden,
                        1e-6, False)
    k.add(f"expert block {tag}", "design", design, weights + T * h * (8 * S + 4) + 2 * rows * h * 2, macs)
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
    k.add(f"expert block {tag}", "hybrid", lambda: block.forward(host, hws, T, "l", norm, normed), (used_h * ff + sf) * 3 * h * 2 + T * h * 8 + 2 * T * kk * h * 2, (T * kk * ff + T * sf) * 3 * h)
    # the grouped GEMMs alone, on the tables that a run leaves (both models take the same kernel; the unit differs)
    e = ws.experts
    run_experts(model, e, T, p, f, x, delta)
    tile = int(ops.moe_tile_tokens(T * kk / f.choices))
    n, cap = min(e.n_tiles, E + (T * f.slots + tile - 1) // tile), T * f.slots
    act, back = e.act[: cap * ff].view(cap, ff), (e.base, e.off["ret"], e.off["ret_flag"], status)
    for who, unit in (("design", glu(f.expert)), ("hybrid", [])):
        k.add(f"experts up {tag}", who, lambda: ops.moe_gemm(e.rows[:cap], w[f"{p}/mlp/up"], 0, tile, n, e.tiles, e.state, act, 1, None, *back, unit),
              used * 2 * ff * h * 2 + rows * (h + ff) * 2, rows * 2 * ff * h)
    k.add(f"experts down {tag}", "design", lambda: ops.moe_gemm(act, w[f"{p}/mlp/down"], 1, tile, n, e.tiles, e.state, None, 1, e.meta, *back),
          used * ff * h * 2 + rows * (h + ff) * 2, rows * ff * h)
    ids, pos, wts = (t[: T * kk].view(T, kk) for t in (e.ids, e.pos, e.weights))
    logits = e.logits[:T, : f.router_cols]
    k.add(f"routing {tag}", "design", lambda: ops.moe_route_scored(logits, E, f.identity, kk, w[f"{p}/mlp/correction"], f.scale, e.hist, ids, wts, pos, False),
          T * (f.choices * 4 + kk * 12))
    lb, sg = _rand(T, (E + 8) // 8 * 8), torch.empty(T, device="cuda")
    k.add(f"routing {tag}", "hybrid", lambda: ops.moe_route(lb, E, kk, True, True, e.hist, ids, wts, pos, sg), T * (E * 2 + kk * 12))
    e.hist.zero_()


def _attention(k: _Kernels, model, ws, cfg, hyb, batch: int, new: int, total: int, tag: str) -> None:
    ops, at = model._raw_ops, _layers(cfg)["attention"]
    m, p = cfg.layers[at].mixer, f"text/layers/{at}/mix"
    H, G, D, V, P = m.heads, m.kv_heads, m.dim_p, m.vdim_p, 64
    T, per = batch * new, (total + P - 1) // P
    row, kv, _ = _tokens(batch, new, total)
    pos = (kv - 1).int()
    table = torch.randperm(batch * per, device="cuda").int().view(batch, per)
    kp, vp = _rand(batch * per, G, P, D), _rand(batch * per, G, P, V)
    q, out, sinks = _rand(T, H * D), _rand(T, H * V), model.w[f"{p}/sink"]
    io = T * H * (D + V) * 2
    assert m.chunk >= total                        # every key is visible, as to the hybrid's queries
    macs, n_bytes = batch * _pairs(new, total, 0) * H * (D + V), batch * total * G * (D + V) * 2 + io
    args = (q, kp, vp, table, row, kv)
    if new > 1:
        blocks = _blocks(batch, new, 64)
        k.add(f"attention {tag}", "design", lambda: ops.group_prefill(*args, 0, m.chunk, m.scale, 0.0, sinks, out, *blocks, False), n_bytes, macs)
    else:
        split, n = model.pick_split(ws, T, total, m.look_back, ctas=G)
        po, ml = torch.empty(T * n * H * V, device="cuda"), torch.empty(T * n * H * 2, device="cuda")
        k.add(f"attention {tag}", "design", lambda: ops.head_mix_attention(*args, 0, m.scale, 0.0, 0.0, None, None, None, out, split, n, po, ml, False, m.chunk,
                                                                           sinks), n_bytes, macs)
    proj, qn, freq = _rand(T, m.main_cols), torch.ones(D, device="cuda"), model.w[f"{p}/freq"]
    k.add(f"norm + rotation + append {tag}", "design", lambda: ops.qkv_append(proj, 0, H * D, (H + G) * D, H, G, m.dim, qn, qn, 1e-6, row, pos, table, q, kp, vp,
                                                                              P, False, freq), T * m.main_cols * 4)
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
    projh, inv, w = _rand(T, hyb.attn_in_dim), torch.rand(32, device="cuda"), _rand(Dh)
    k.add(f"norm + rotation + append {tag}", "hybrid",
          lambda: ops.attn_prep(projh, 0, Hh * Dh, 2 * Hh * Dh + Gh * Dh, Hh, Gh, Dh, w, w, 1e-6, True, 64, inv, 1.0, pos, row, pos, table, qh, kh, vh, None, None,
                                P, 0, Dh, False, False, None, None), T * (Hh + 2 * Gh) * Dh * 4)


def _latent(k: _Kernels, model, ws, cfg, batch: int, new: int, total: int, tag: str) -> None:
    """In the window, beside the same attention with a rotated part of 64, a sink and no window over as many keys (Tebivik's)."""
    ops, at = model._raw_ops, _layers(cfg)["latent_attention"]
    m, w, p = cfg.layers[at].mixer, model.w, f"text/layers/{at}/mix"
    H, C, V, D, P = m.heads, m.kv_rank_p, m.vdim_p, m.dim_p, 64
    T, seen = batch * new, min(total, m.window) if m.window else total
    for who, R, window, length in (("design", 0, m.window, total), ("tebivik", 64, 0, total if new > 1 else seen)):
        per = (length + P - 1) // P
        row, kv, cu = _tokens(batch, new, length)
        pos = (kv - 1).int()
        table = torch.randperm(batch * per, device="cuda").int().view(batch, per)
        pages = _rand(batch * per, 1, P, C + R)
        q, freq = _rand(T, H * (D + R)), torch.rand(R // 2, dtype=torch.float64, device="cuda")
        sink = torch.ones(H, device="cuda") if R else None
        kvn, qn = torch.ones(C, device="cuda"), torch.ones(768, device="cuda")
        lat, proj = (_rand(T, 768), _rand(T, 768 + C + R)) if R else (None, _rand(T, m.main_cols))
        n_prep = T * ((768 + C + R) if R else C) * 4
        k.add(f"latent norm + append {tag}", who, lambda: ops.latent_prep(proj, 768, m.kv_rank, R, qn if R else None, kvn, 1e-6, freq, row, pos, table, lat, pages,
                                                                         False), n_prep)
        start, count = _blocks(batch, new, 64)
        blocks = (start, count, min(new, 64))
        pairs = batch * _pairs(new, length, window)
        if new == 1:
            keys = min(length, window) if window else length
            ctas = start.numel() * max(1, -(-H // 64))
            want = max(1, min(148 // ctas, ws.split_rows // T, 64))
            split = max(128, -(-(-(-keys // want)) // 32) * 32)
            n = -(-keys // split)
            q_abs, o_lat = _rand(T, H * C), _rand(T, H * C)
            po, ml = torch.empty(T * n * H * C, device="cuda"), torch.empty(T * n * H * 2, device="cuda")
            k.add(f"latent attention {tag}", who, lambda: ops.latent_absorbed_attention(q_abs, q, pages, table, row, kv, H, R, m.scale, freq, sink, o_lat, *blocks,
                                                                                      row, cu, 0, split, n, po, ml, False, window),
                  batch * keys * (C + R) * 2 + T * H * (2 * C + R) * 2, pairs * H * (2 * C + R))
        else:
            rows = _rand(batch * length, C + R)
            wide, out = _rand(batch * length, H * (D + V)), _rand(T, H * V)
            base = _ints([[i * length, 0] for i in range(batch)])
            k.add(f"latent attention {tag}", who, lambda: ops.latent_expanded_attention(q, rows, wide, kv, H, C, R, m.scale, freq, sink, out, *blocks, row, base,
                                                                                      False, window),
                  wide.numel() * 2 + rows.shape[0] * R * 2 + T * H * (D + R + V) * 2, pairs * H * (D + R + V))


def _recurrence(k: _Kernels, model, cfg, hyb, batch: int, new: int, tag: str) -> None:
    ops, at = model._raw_ops, _layers(cfg)["rglru"]
    m, w, p = cfg.layers[at].mixer, model.w, f"text/layers/{at}/mix"
    T, C = batch * new, m.out_cols
    cu, slot = _ints(torch.arange(batch + 1) * new), _ints(torch.arange(batch))
    seq, pos = _ints(torch.arange(batch).repeat_interleave(new)), _ints(torch.arange(100, 100 + new).repeat(batch))
    proj, out = _rand(T, m.main_cols), _rand(T, C)
    ring, S = torch.zeros((batch, m.taps, C), device="cuda"), torch.zeros((batch, C), device="cuda")
    blocks = _blocks(batch, new, 64)
    cws = None if new == 1 else torch.empty(int(ops.rglru_chunked_workspace_bytes(T, batch, C)), dtype=torch.uint8, device="cuda")
    gates = w[f"{p}/gates"]
    k.add(f"recurrence {tag}", "design", lambda: ops.rglru(proj, m.blocks, w[f"{p}/conv"], w[f"{p}/conv_bias"], cu, seq, pos, slot, ring, gates,
                                                           w[f"{p}/gate_bias"], w[f"{p}/rate"], S, out, *blocks, cws, True, False),
          gates.numel() * 2 + proj.numel() * 2 + out.numel() * 2 + (2 * S.numel() + ring.numel()) * 4, T * gates.numel())
    d, hk, hv = 128, hyb.gdn_qk_heads, hyb.gdn_v_heads
    qk, vd = hk * d, hv * d
    n = 2 * qk + vd
    conv, projh = _rand(T, n, s=0.5), _rand(T, n + vd + 2 * hv, s=0.5)
    ssm, A, nw, oh = torch.zeros((batch, hv, d, d), device="cuda"), torch.zeros(hv, device="cuda"), _rand(d), _rand(T, vd)
    ws2 = None if new == 1 else torch.empty(int(ops.gdn_chunked_workspace_bytes(T, batch, hv)), dtype=torch.uint8, device="cuda")
    k.add(f"recurrence {tag}", "hybrid", lambda: ops.gdn_recurrent(conv, 0, qk, 2 * qk, projh, n, n + vd, n + vd + hv, hk, hv, A, A, nw, 1e-6, cu, slot, ssm, True,
                                                                   oh, False, None, None, ws2),
          2 * ssm.numel() * 4 + conv.numel() * 2 + 2 * T * vd * 2, 2.0 * T * hv * d * d)


def stream_kernels(cfg, hyb, weights, iters: int, only: str, phases=(("decode x32", 32, 1), ("prefill 2048", 1, 2048))):
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
        _latent(k, model, ws, cfg, batch, new, 2048, tag)
        _recurrence(k, model, cfg, hyb, batch, new, tag)
    model.status.check("after the kernel timings")
    return k.rows
