"""Small Ratilorn configurations of the tests and weights that make faults visible."""
import torch

from ninfer_fusion_b200.models import ratilorn


def heads(H, G, D, V, scale):
    return {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale}


def sig(H, G, D, V, scale=0.4, v_mix=True, mlp=None):
    return {"type": "attention", "mixer": dict(heads(H, G, D, V, scale), v_mix=v_mix), "mlp": mlp}


def ssm(H, V, N, G=1, taps=4, parts=1):
    return {"heads": H, "vdim": V, "state": N, "groups": G, "conv": taps, "norm_groups": parts}


def par(left, right, mlp=None):
    return {"type": "parallel", "mixer": {"left": heads(*left), "right": ssm(*right)}, "mlp": mlp}


def moe(experts, top, ff, groups=None, shared=40):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def dense(ff):
    return {"kind": "dense", "ff": ff}


def conf(width, vocab, layers, positions=512, scale=0.7, eps=1e-4):
    return {"architecture": "Ratilorn", "width": width, "vocab": vocab, "max_positions": positions, "norm": {"eps": eps}, "logit_scale": scale,
            "layers": layers}


CASES = {
    "mixed": conf(96, 211, [par((6, 2, 32, 48, 0.3), (4, 32, 48, 2, 4, 2), dense(72)), sig(6, 3, 32, 16, mlp=moe(9, 2, 48, (3, 2))),
                            par((4, 4, 16, 32, 0.4), (6, 16, 16, 3, 3, 2), moe(8, 3, 24, (4, 2))), sig(4, 2, 48, 32, v_mix=False, mlp=moe(6, 2, 40)),
                            sig(9, 3, 16, 16, mlp=moe(8, 2, 32, (2, 1), None))], 437),
    # widths that are no multiple of anything, layers without feed-forward, one expert per token, the last layer ends with its mixer
    "odd": conf(90, 77, [sig(3, 1, 20, 36, mlp=moe(3, 1, 30, None, None)), par((5, 5, 12, 20, 0.5), (3, 20, 24, 1, 1, 4), dense(50)),
                         par((2, 1, 24, 12, 0.4), (5, 12, 20, 5, 2, 12)), sig(5, 1, 12, 36)], 300, 1.0, 1e-2),
    "sigmoid_only": conf(64, 128, [sig(8, 2, 64, 64, 0.5), sig(2, 2, 16, 64, 1.5, mlp=dense(64))], 1024, 2.5),
    "parallel_only": conf(72, 130, [par((4, 1, 48, 32, 0.4), (2, 64, 64, 1, 4, 1), dense(64)), par((2, 2, 32, 32, 0.4), (8, 16, 128, 4, 7, 2), moe(4, 2, 16, (4, 3), 24))]),
    # many heads and experts; more key / value heads and query heads per group than one kernel takes
    "many_heads": conf(128, 96, [sig(20, 4, 16, 32), sig(68, 4, 16, 32), sig(36, 4, 16, 32, mlp=moe(70, 6, 24, (7, 3))), sig(40, 40, 16, 32, v_mix=False),
                                 par((20, 1, 32, 32, 0.3), (12, 16, 32, 2, 4, 3), moe(64, 4, 16, (32, 9), 130))]),
    # heads and states wider than the tensor-core kernels take, values in several slices, a long row
    "wide": conf(136, 96, [sig(2, 1, 272, 144), par((2, 1, 160, 272, 0.1), (2, 144, 272, 1, 4, 1), moe(5, 2, 72, (5, 2))), sig(2, 2, 160, 288, v_mix=False),
                           par((1, 1, 64, 64, 0.2), (3, 80, 192, 3, 5, 1))]),
}


def build(name, seed=0):
    """(config dict, LayeredConfig, checkpoint tensors bf16, the same as float64 arrays)."""
    c = CASES[name]
    cfg = ratilorn.parse_config(c, name)
    t = ratilorn.random_tensors(cfg, seed)
    for n in list(t):
        if n.endswith((".q.norm", ".k.norm")):
            t[n] = (t[n].float() * 1.8).to(torch.bfloat16)                # scores that single keys out
        if n.endswith("mix.pb"):
            t[n] = torch.linspace(-5.0, -1.0, t[n].numel()).to(torch.bfloat16)
        if n.endswith("mix.r1"):
            t[n] = torch.linspace(0.1, 1.5, t[n].numel()).to(torch.bfloat16)
        if n.endswith("mix.r2"):
            t[n] = torch.linspace(3.0, 0.02, t[n].numel()).to(torch.bfloat16)
        if n.endswith("mix.talk"):
            t[n] = (t[n].float() * 0.7 + 0.3 * torch.roll(torch.eye(t[n].shape[0]), 1, 0)).to(torch.bfloat16)      # no symmetry
        if n.endswith("dt_bias"):
            t[n] = torch.linspace(-7.0, 1.0, t[n].numel()).to(torch.bfloat16)
        if n.endswith("mlp.correction"):
            t[n] = (t[n].float() * 8 - 0.6).to(torch.bfloat16)            # choices that the scores alone would not make; below zero
        if n.endswith("mlp.router"):
            t[n] = (t[n].float() * 2).to(torch.bfloat16)
    return c, cfg, t, {n: v.double().numpy() for n, v in t.items()}
