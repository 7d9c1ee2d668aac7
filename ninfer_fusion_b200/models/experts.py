"""Mixture-of-experts feed-forward of the layer-list decoders (`models/layered_config.ExpertMlp`) on one GPU: packing, buffers
and the launch sequence on the kernels of `csrc/moe`.

    router GEMM (fp32 logits) -> scored routing (softmax or sigmoid, in groups or not) -> plan (tile table) -> push (rows sorted by expert) -> grouped GEMM with the
    bounded gated unit -> grouped GEMM whose epilogue puts every row in its token's place; the shared expert is a dense pair
    of GEMMs

The sum over a token's experts is left to the row step that follows (`MixtureParts` of `csrc/pointwise/stream_rows.h`): identity
experts only have a weight there.  In 32-bit runs the same tables feed an fp32 grouped GEMM."""
from __future__ import annotations

from typing import Dict, Sequence

import torch

from .layered_config import ExpertMlp, GatedUnit, pad_to

SWIGLU, RETURN = 0, 1          # csrc/moe/moe.h MoeGemmEpilogue
EPI_SWIGLU = 2                 # csrc/gemm/gemm.h
F32_TILE = 64                  # rows per tile of the fp32 grouped GEMM


def _pad(w: torch.Tensor, rows: int, cols: int, dtype) -> torch.Tensor:
    out = torch.zeros((rows, cols), dtype=dtype, device=w.device)
    out[: w.shape[0], : w.shape[1]] = w
    return out


def pack_unit(get, prefix: str, u: GatedUnit, hp: int, dtype):
    """[gate; up] and down of one unit, the unit's width padded: zero gate and up rows give zero, whatever the shift."""
    up = torch.cat([_pad(get(f"{prefix}gate"), u.ff_p, hp, dtype), _pad(get(f"{prefix}up"), u.ff_p, hp, dtype)])
    return up, _pad(get(f"{prefix}down"), hp, u.ff_p, dtype)


def pack_experts(w: Dict[str, torch.Tensor], p: str, m: ExpertMlp, get, hp: int, dtype) -> None:
    units = [pack_unit(get, f"e{e}.", m.expert, hp, dtype) for e in range(m.experts)]
    w[f"{p}/mlp/up"], w[f"{p}/mlp/down"] = torch.stack([u for u, _ in units]), torch.stack([d for _, d in units])
    router = [get("router")]
    if m.shared is not None:
        w[f"{p}/mlp/shared_up"], w[f"{p}/mlp/shared_down"] = pack_unit(get, "shared.", m.shared, hp, dtype)
        if m.shared_gate:
            router.append(get("shared_gate"))
    w[f"{p}/mlp/router"] = _pad(torch.cat(router), m.router_cols, hp, dtype)
    w[f"{p}/mlp/correction"] = get("correction").float().contiguous()


class ExpertWorkspace:
    """Buffers for steps of up to `max_tokens` tokens, shared by all layers (their routers and sizes may differ)."""

    def __init__(self, specs: Sequence[ExpertMlp], hp: int, max_tokens: int, device, dtype: torch.dtype, ops):
        T, dev, i32 = max_tokens, device, torch.int32
        self.hp, self.f32, self.max_tokens = hp, dtype == torch.float32, T
        E = max(m.experts for m in specs)
        k = max(m.top for m in specs)
        rows = T * max(m.slots for m in specs)
        self.n_tiles = E + (rows + 15) // 16
        # one allocation stands for the buffers that ranks of an expert-parallel group would see of each other
        self.off, at = {}, 0
        for name, n_bytes in (("counts", E * 4), ("count_flag", 4), ("arrive_flag", 4), ("ret_flag", 4), ("meta", rows * 4),
                              ("rows", rows * hp * dtype.itemsize), ("ret", T * k * hp * dtype.itemsize)):
            self.off[name] = at
            at += pad_to(n_bytes, 256)
        self.buf = torch.zeros(at, dtype=torch.uint8, device=dev)
        self.base = [self.buf.data_ptr()]

        def view(name, n, dt):
            return self.buf[self.off[name]: self.off[name] + n * dt.itemsize].view(dt)
        self.rows = view("rows", rows * hp, dtype).view(rows, hp)
        self.meta, self.ret = view("meta", rows, i32), view("ret", T * k * hp, dtype)
        self.hist, self.send = (torch.zeros(E, dtype=i32, device=dev) for _ in range(2))
        self.ids, self.pos = (torch.zeros(T * k, dtype=i32, device=dev) for _ in range(2))
        self.weights = torch.zeros(T * k, dtype=torch.float32, device=dev)
        self.tiles = torch.zeros((3, self.n_tiles), dtype=i32, device=dev)
        self.state = torch.zeros(int(ops.moe_state_bytes()), dtype=torch.uint8, device=dev)
        self.logits = torch.zeros((T, max(m.router_cols for m in specs)), dtype=torch.float32, device=dev)
        wide = max(m.expert.ff_p for m in specs)
        shared = max([m.shared.ff_p for m in specs if m.shared is not None], default=0)
        self.act = torch.zeros(rows * wide, dtype=dtype, device=dev)
        self.shared_act = torch.zeros(T * shared, dtype=dtype, device=dev)
        # [gate | up] columns before the unit (32-bit runs)
        self.wide, self.shared_wide = (torch.zeros(2 * t.numel() if self.f32 else 0, dtype=dtype, device=dev) for t in (self.act, self.shared_act))


def glu(u: GatedUnit):
    return [u.limit, u.slope, u.shift]


def run_unit(model, T: int, u: GatedUnit, up, down, x: torch.Tensor, act: torch.Tensor, wide, out: torch.Tensor, prefetch=None) -> None:
    """out [T, hp] fp32 <- the unit of x [T, hp].  `act` and (32-bit runs) `wide` are flat buffers."""
    h = act[: T * u.ff_p].view(T, u.ff_p)
    if model.f32:
        both = wide[: 2 * T * u.ff_p].view(T, 2 * u.ff_p)
        model._gemm(x, up, None, both)
        model.ops.glu_rows_f32(both, h, *glu(u), model.pdl)
    else:
        model._gemm(x, up, None, h, epi=EPI_SWIGLU, glu=glu(u), prefetch=down)
    model._gemm(h, down, None, out32=out, prefetch=prefetch)


def run_experts(model, ws: ExpertWorkspace, T: int, p: str, m: ExpertMlp, x: torch.Tensor, delta: torch.Tensor, prefetch=None) -> dict:
    """Launches the block on x [T, hp]; `delta` [T, hp] fp32 receives the shared expert's output.  Returns the parts of the sum
    as the row steps take them."""
    ops, w, hp = model.ops, model.w, ws.hp
    k, E, status = m.top, m.experts, model.status.tensor
    logits = ws.logits[:T, : m.router_cols]
    model._gemm(x, w[f"{p}/mlp/router"], None, out32=logits, prefetch=w[f"{p}/mlp/up"])
    n, rows = T * k, T * m.slots
    ids, pos, weights = ws.ids[:n].view(T, k), ws.pos[:n].view(T, k), ws.weights[:n].view(T, k)
    ops.moe_route_scored(logits, E, m.identity, k, w[f"{p}/mlp/correction"], m.scale, ws.hist, ids, weights, pos, model.pdl, m.sigmoid,
                         m.renormalise, m.groups, m.keep)
    tile = F32_TILE if ws.f32 else int(model._raw_ops.moe_tile_tokens(T * k / m.choices))
    n_tiles = min(ws.n_tiles, E + (rows + tile - 1) // tile)
    ops.moe_plan(1, 0, E, tile, rows, ws.hist, ws.base, ws.off["counts"], ws.off["count_flag"], ws.send, ws.tiles, ws.state, status)
    bits = x.view(torch.bfloat16) if ws.f32 else x           # rows are copied as they are
    ops.moe_push(1, 0, E, rows, bits, ids, pos, ws.send, ws.base, ws.off["rows"], ws.off["meta"], ws.off["arrive_flag"], ws.state, status)
    ff = m.expert.ff_p
    act = ws.act[: rows * ff].view(rows, ff)
    back = (ws.base, ws.off["ret"], ws.off["ret_flag"], status)
    up, down = w[f"{p}/mlp/up"], w[f"{p}/mlp/down"]
    if ws.f32:
        wide = ws.wide[: 2 * rows * ff].view(rows, 2 * ff)
        ops.moe_gemm(ws.rows[:rows], up, SWIGLU, tile, n_tiles, ws.tiles, ws.state, wide, 1, None, *back)
        ops.glu_rows_f32(wide, act, *glu(m.expert), model.pdl)
    else:
        ops.moe_gemm(ws.rows[:rows], up, SWIGLU, tile, n_tiles, ws.tiles, ws.state, act, 1, None, *back, glu(m.expert))
    ops.moe_gemm(act, down, RETURN, tile, n_tiles, ws.tiles, ws.state, None, 1, ws.meta, *back)
    parts = dict(delta=None, gate=None, choice=ids, weight=weights, ret=ws.ret[: n * hp].view(n, hp), h=x, n_experts=E)
    if m.shared is not None:
        run_unit(model, T, m.shared, w[f"{p}/mlp/shared_up"], w[f"{p}/mlp/shared_down"], x, ws.shared_act, ws.shared_wide, delta, prefetch)
        parts.update(delta=delta, gate=logits[:, m.choices: m.choices + 1] if m.shared_gate else None)
    return parts
