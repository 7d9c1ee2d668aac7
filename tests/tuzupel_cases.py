"""Small Tuzupel configurations of the tests and weights that make faults visible."""
import torch

from ninfer_fusion_b200.models import tuzupel


def moe(experts, top, ff, identity=1, scale=1.3, limit=1.2, shared=(40, 0.9)):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top, "scale": scale}}
    if shared:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def rot(dims, base=1e3, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def att(H, G, D, V, chunk, r=None, scale=0.25, mlp=None):
    mixer = {"heads": H, "dim": D, "vdim": V, "scale": scale, "mask": {"size": chunk}, "kv_heads": G}
    if r:
        mixer["rot"] = r
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def lat(H, D, V, C, window, scale=0.4, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": H, "dim": D, "vdim": V, "scale": scale, "mask": {"size": window}, "kv_rank": C}, "mlp": mlp}


def rec(width, blocks, taps, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": taps}, "mlp": mlp}


def conf(width, vocab, streams, layers, cap=12.0, eps=1e-4):
    out = {"architecture": "Tuzupel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "streams": streams, "layers": layers}
    if cap:
        out["logit_softcap"] = cap
    return out


CASES = {
    "mixed": conf(96, 211, 3, [rec(112, 7, 4, moe(5, 2, 48)), att(6, 2, 32, 48, 24, rot(24, scaling=(4.0, 1.0, 4.0, 64.0)), mlp=moe(5, 2, 48)),
                               lat(3, 32, 16, 48, 20, mlp=moe(9, 3, 24, 2, 0.8, 0.7)), rec(64, 2, 4), att(4, 4, 16, 16, 33, rot(16))]),
    # widths that are no multiple of anything, one stream, one expert per token, none of them an identity, no shared one
    "odd": conf(90, 77, 1, [lat(5, 12, 20, 36, 29, mlp=moe(3, 1, 30, 0, 2.0, 3.0, None)), rec(84, 3, 3, moe(4, 2, 18, 3)),
                            att(9, 3, 20, 12, 50, rot(6, 50.0), mlp=moe(2, 4, 22, 2, 1.0, 0.3, (10, 5.0)))], 0.0, 1e-2),
    # masks as wide as a query block and a page, one block, a long convolution, no rotation
    "edges": conf(64, 128, 2, [rec(64, 1, 7, moe(6, 5, 32, 2)), att(4, 1, 32, 32, 64), lat(4, 16, 16, 32, 64, mlp=moe(6, 2, 32)),
                               att(2, 2, 64, 64, 16, rot(64, scaling=(8.0, 2.0, 3.0, 100.0)))], 30.0),
    "attention_only": conf(64, 128, 4, [att(20, 1, 32, 32, 400, rot(16, scaling=(2.0, 1.0, 4.0, 512.0))), att(4, 2, 128, 128, 57, rot(64), mlp=moe(4, 2, 16))]),
    "latent_only": conf(64, 128, 5, [lat(2, 48, 64, 128, 71), lat(20, 16, 16, 64, 1, mlp=moe(4, 2, 16)), lat(2, 16, 16, 32, 500)]),
    "recurrence_only": conf(64, 130, 9, [rec(160, 2, 1, moe(3, 2, 64, 0)), rec(48, 3, 2), rec(192, 1, 4)]),
    # heads, latents and gate blocks wider than the tensor-core kernels take; many experts
    "wide": conf(136, 96, 2, [att(2, 1, 272, 144, 37, rot(200)), lat(2, 64, 160, 528, 45, mlp=moe(70, 6, 72, 5, 4.0)), rec(544, 1, 4),
                              att(2, 2, 160, 256, 90)]),
}


def build(name, seed=0):
    """(config dict, LayeredConfig, checkpoint tensors bf16, the same as float64 arrays)."""
    c = CASES[name]
    cfg = tuzupel.parse_config(c, name)
    t = tuzupel.random_tensors(cfg, seed)
    for n in list(t):
        if n.endswith((".q.norm", ".k.norm")):
            t[n] = (t[n].float() * 1.8).to(torch.bfloat16)                # scores that single keys out
        if n.endswith("mix.sink"):
            t[n] = torch.linspace(0.0, 4.0, t[n].numel()).to(torch.bfloat16)
        if n.endswith("mix.lam"):
            t[n] = torch.linspace(-7.0, 1.0, t[n].numel())[torch.randperm(t[n].numel(), generator=torch.Generator().manual_seed(1))].to(torch.bfloat16)
        if n.endswith("mlp.correction"):
            t[n] = (t[n].float() * 10).to(torch.bfloat16)                 # choices that the scores alone would not make
        if n.endswith(("mix.ra", "mix.ri", "mlp.router")):
            t[n] = (t[n].float() * 2).to(torch.bfloat16)
    return c, cfg, t, {n: v.double().numpy() for n, v in t.items()}
