"""What differs between model families when a runtime is built: the model class, the geometry of the KV cache, the
recurrent state arrays, the activation buffers and the query-block size of the step descriptors.  Everything above
(lanes, admission, frontiers, sampling, graphs) is written against the result."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence

import torch

from ..models.hybrid import HybridModel, ShardGeometry, Workspace
from ..models.layered import BLOCK_TOKENS, LayeredModel, LayeredWorkspace
from ..models.layered_config import LayeredConfig
from .kv_cache import GdnStatePool, PagedKvCache


@dataclass
class Runtime:
    model: object
    kv: PagedKvCache
    states: object
    ws: object
    block_tokens: int        # query tokens per attention block of a prefill step
    vocab_rows: int          # logits columns this rank computes
    page_lookahead: int      # cache positions mapped beyond those a step writes


def is_layered(cfg) -> bool:
    return isinstance(cfg, LayeredConfig)


def context_limit(cfg, max_context: int) -> int:
    """`max_context`, or as many positions as the model has vectors for."""
    limit = getattr(cfg, "position_limit", 0)
    return min(max_context, limit) if limit else max_context


def check_positions(cfg, end: int) -> None:
    """A sequence may not grow beyond the model's positions."""
    limit = getattr(cfg, "position_limit", 0)
    if limit and end > limit:
        raise ValueError(f"{cfg.name}: position {end - 1} is beyond the model's {limit} positions")


def kv_format_for(cfg, weights, kv_format):
    """Layer-list models keep their rows in the activation type."""
    if not is_layered(cfg):
        return kv_format
    f32 = weights["text/embed"].dtype == torch.float32
    if kv_format in ("bf16", "fp32"):
        return "fp32" if f32 else "bf16"
    raise ValueError(f"{cfg.name}: its attention reads uncoded K / V rows (bf16, or fp32 when the model runs in fp32), not '{kv_format}'")


def build_runtime(cfg, weights, device, *, rows: int, pages_per_row: int, n_pages: int, page_size: int, state_slots: int,
                  step_tokens: int, logit_rows: int, kv_format="bf16", pdl: bool = True, int8_group: int = 64,
                  shard: Optional[ShardGeometry] = None, comm=None, mixed_capacity: Optional[Sequence[int]] = None,
                  mixed_hot_tier: int = 0) -> Runtime:
    from .kv_cache import RecurrentStatePool
    kv_format = kv_format_for(cfg, weights, kv_format)
    if is_layered(cfg):
        if shard is not None or comm is not None:
            raise ValueError(f"{cfg.name}: layer-list models run on one GPU")
        model = LayeredModel(cfg, weights, device, pdl=pdl)
        kv = PagedKvCache(cfg, n_pages, page_size, rows, pages_per_row, device, formats=kv_format, geometry=cfg.kv_geometry,
                          look_back=cfg.cache_window)
        states = RecurrentStatePool([[(shape, torch.float32) for shape in layer] for layer in cfg.state_shapes()], state_slots, device)
        ws = LayeredWorkspace(cfg, step_tokens, logit_rows, device, model.dtype, ops=model._raw_ops)
        return Runtime(model, kv, states, ws, BLOCK_TOKENS, cfg.vocab, 0)
    model = HybridModel(cfg, weights, device, pdl=pdl, shard=shard)
    model.comm = comm
    g = model.g
    kv = PagedKvCache(cfg, n_pages, page_size, rows, pages_per_row, device, formats=kv_format, int8_group=int8_group,
                      n_kv_heads=g.n_kv_heads, mixed_capacity=mixed_capacity, mixed_hot_tier=mixed_hot_tier)
    states = GdnStatePool(cfg, state_slots, device, n_qk_heads=g.gdn_qk_heads, n_v_heads=g.gdn_v_heads)
    ws = Workspace(cfg, step_tokens, logit_rows, device, shard=shard, x_buffer=None if comm is None else comm.x)
    cuda = torch.device(device).type == "cuda"
    qt = int(model.ops.prefill_attn_block_tokens(g.n_q_heads, g.n_kv_heads)) if cuda else 16
    return Runtime(model, kv, states, ws, qt, g.vocab_rows, 1)
