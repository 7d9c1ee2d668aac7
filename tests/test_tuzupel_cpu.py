"""Tuzupel on the CPU: configuration, checkpoint reading, packing, registry, cache look-back and state, and that the tests'
weights show the faults they are meant to show."""
import json
import math

import numpy as np
import pytest
import torch

import tuzupel_cases as C
import tuzupel_oracle as K
from kuzanex_cases import err, prompt
from ninfer_fusion_b200.models import architectures as AR
from ninfer_fusion_b200.models import packages as PK
from ninfer_fusion_b200.models import tuzupel
from ninfer_fusion_b200.models.layered import LayeredModel, native_subset
from ninfer_fusion_b200.models.layered_config import Rotary, RotaryScaling
from ninfer_fusion_b200.runtime.kv_cache import PagedKvCache, RecurrentStatePool


@pytest.mark.parametrize("name", sorted(C.CASES))
def test_configuration_round_trip(name):
    c, cfg, _, _ = C.build(name)
    assert tuzupel.config_dict(cfg) == c
    assert tuzupel.parse_config(tuzupel.config_dict(cfg), name) == cfg
    assert sum(math.prod(s) for _, s in tuzupel.tensor_shapes(cfg)) == cfg.param_count()


def test_stand_alone_libraries_have_the_parts_a_model_needs():
    from ninfer_fusion_b200 import _build
    want = {"mixed": "attention+latent+moe+rglru+streams", "recurrence_only": "moe+rglru+streams", "latent_only": "latent+moe+streams"}
    for name, parts in want.items():
        assert native_subset(C.build(name)[1]) == parts
        sources = _build.subset_sources(parts)
        assert all((_build.CSRC / s).exists() for s in sources) and not any("mlstm" in s or "gated" in s for s in sources)
    everything = {s for part in _build.PARTS for s in _build.subset_sources(part)}
    cu, cpp = _build._sources()
    assert everything <= {p.relative_to(_build.CSRC).as_posix() for p in cu + cpp}


def test_configuration_errors_are_named():
    for layer, what in ((dict(C.rec(64, 2, 4), type="ring"), "unknown mixer 'ring'"), (C.rec(65, 2, 4), "equal parts"), (C.rec(64, 2, 0), "tap"),
                        (C.att(4, 3, 16, 16, 8), "multiple of kv_heads"), (C.att(4, 2, 16, 16, 0), "own key"),
                        (C.att(4, 2, 16, 16, 8, C.rot(18)), "within the head"), (C.lat(2, 16, 16, 16, 0), "own key"),
                        (C.rec(64, 2, 4, C.moe(2, 5, 16, 2)), "5 of 4 experts"), (C.rec(64, 2, 4, dict(C.moe(2, 1, 16), kind="tree")), "'tree'")):
        with pytest.raises(ValueError, match=what):
            tuzupel.parse_config(C.conf(64, 40, 2, [layer]))
    with pytest.raises(ValueError, match="stream"):
        tuzupel.parse_config(C.conf(64, 40, 0, [C.rec(64, 2, 4)]))


def test_scaled_frequencies():
    """Kept, divided and mixed ones, against the oracle; both edges of the ramp meet their neighbours."""
    for dims, base, sc in ((64, 5e4, (4.0, 1.0, 4.0, 512.0)), (24, 1e3, (8.0, 2.0, 3.0, 100.0)), (6, 50.0, None)):
        r = Rotary(base, dims, None if sc is None else RotaryScaling(*sc))
        assert np.allclose(r.frequencies(), K.frequencies(C.rot(dims, base, sc)), rtol=1e-14)
    f, plain = (np.array(Rotary(5e4, 64, s).frequencies()) for s in (RotaryScaling(4.0, 1.0, 4.0, 512.0), None))
    wave = 2 * np.pi / plain
    assert (f[wave < 128] == plain[wave < 128]).all() and np.allclose(f[wave > 512], plain[wave > 512] / 4)
    mid = (wave > 128) & (wave < 512)
    assert mid.any() and (f[mid] < plain[mid]).all() and (f[mid] > plain[mid] / 4).all()


def test_cache_look_back_and_state():
    _, cfg, _, _ = C.build("mixed")
    assert cfg.attn_layers == [1, 2, 4] and cfg.state_layers == [0, 3] and cfg.cache_window == 33
    assert cfg.kv_geometry == [(2, 32, 48), (1, 48, 0), (4, 16, 16)]
    assert cfg.state_shapes() == [[(4, 112), (112,)], [(4, 64), (64,)]]
    _, odd, _, _ = C.build("odd")                       # blocks of 28 are kept 32 wide
    assert odd.state_shapes() == [[(3, 96), (96,)]]
    free = tuzupel.parse_config(C.conf(64, 40, 2, [dict(C.lat(2, 16, 16, 16, 5), mixer={k: v for k, v in C.lat(2, 16, 16, 16, 5)["mixer"].items() if k != "mask"}),
                                                   C.att(2, 2, 16, 16, 8)]))
    assert free.cache_window == 0                       # one layer sees all of the past
    st = RecurrentStatePool([[(s, torch.float32) for s in l] for l in cfg.state_shapes()], 2, "cpu")
    a = st.alloc()
    for t in st.tensors():
        t[a].fill_(3.0)
    st.release(a)
    assert st.alloc() == a and all(not t[a].any() for t in st.tensors())


def test_pages_go_back_only_when_no_chunk_or_window_needs_them():
    _, cfg, _, _ = C.build("mixed")
    kv = PagedKvCache(cfg, 16, 8, 1, 16, "cpu", formats="fp32", geometry=cfg.kv_geometry, look_back=cfg.cache_window)
    for start in range(100):
        kv.advance(0, start, start + 1)
        seen = min(start // 24 * 24, max(0, start - 19), start // 33 * 33)        # first key that a layer looks at from here
        assert all(p >= 0 for p in kv.row_pages[0][seen // 8:]) and kv.live_pages(0) <= 6


def test_expanding_plans_gather_the_window_only():
    _, cfg, _, _ = C.build("latent_only")
    from ninfer_fusion_b200.runtime.batch import SeqChunk, StepBuffers
    b = StepBuffers(512, 4, "cpu", attn_block_tokens=64).build([SeqChunk(0, 0, 90, [0] * 128), SeqChunk(1, 1, 7, [0]), SeqChunk(2, 2, 0, [0] * 200)])
    m = cfg.layers[0].mixer
    assert m.window == 71 and LayeredModel.expand_tokens(m) <= 128

    class Fake:
        f32, prefill_kernels, device = False, True, torch.device("cpu")
        expand_tokens = staticmethod(LayeredModel.expand_tokens)
        _raw_ops = type("O", (), {"latent_expanded_supported": staticmethod(lambda *a: True)})
    _, seqs, base, total, longest, others = LayeredModel._expand_plan(Fake(), b, m)
    assert seqs.tolist() == [[0, 0, 20, 198], [2, 198, 0, 200]] and base.tolist() == [[0, 20], [-1, 0], [198, 0]]
    assert (total, longest, others) == (398, 200, True)


def test_model_folder(tmp_path):
    c, cfg, t, _ = C.build("odd")
    AR.save_folder(str(tmp_path), cfg, t)
    got, w = AR.load_folder(str(tmp_path), "cpu", torch.float32)
    assert got.layers == cfg.layers and w["text/embed"].dtype == torch.float32 and got.streams == 1
    assert json.load(open(tmp_path / "config.json"))["architecture"] == "Tuzupel"
    t2 = dict(t)
    t2["l1.mix.conv"] = t2["l1.mix.conv"][:, :2].contiguous()
    AR.save_folder(str(tmp_path / "short"), cfg, t2)
    with pytest.raises(ValueError, match="l1.mix.conv"):
        AR.load_folder(str(tmp_path / "short"), "cpu")
    del t2["l1.mix.conv"]
    AR.save_folder(str(tmp_path / "less"), cfg, t2)
    with pytest.raises(ValueError, match="no tensor 'l1.mix.conv'"):
        AR.load_folder(str(tmp_path / "less"), "cpu")


def test_packing_pads_and_computes_the_same():
    c, cfg, t, w64 = C.build("odd")
    w = {n: v.double().numpy() for n, v in tuzupel.pack(cfg, t.__getitem__, torch.float32).items()}
    g, n, N = np.random.default_rng(0), cfg.hidden, cfg.hidden_p
    x = np.zeros((4, N))
    x[:, :n] = g.normal(size=(4, n))
    h = x[:, :n]
    # latent attention: [queries, latent]
    m = cfg.layers[0].mixer
    proj = x @ w["text/layers/0/mix/in_proj"].T
    assert proj.shape[1] == m.heads * m.dim_p + m.kv_rank_p
    q = proj[:, : m.q_cols].reshape(4, m.heads, m.dim_p)
    assert np.allclose(q[..., : m.dim].reshape(4, -1), h @ w64["l0.mix.q"].T) and not q[..., m.dim:].any()
    assert np.allclose(proj[:, m.q_cols: m.q_cols + m.kv_rank], h @ w64["l0.mix.dkv"].T)
    # recurrence: blocks of 28 in 32 columns
    m = cfg.layers[1].mixer
    proj = (x @ w["text/layers/1/mix/in_proj"].T + w["text/layers/1/mix/in_bias"]).reshape(4, 2, 3, 32)
    assert np.allclose(proj[:, 1, :, :28].reshape(4, -1), h @ w64["l1.mix.x"].T + w64["l1.mix.x.b"]) and not proj[..., 28:].any()
    u = proj[:, 1]
    raw = np.einsum("tbi,bgi->tbg", u, w["text/layers/1/mix/gates"]) + w["text/layers/1/mix/gate_bias"]
    assert np.allclose(K.sigmoid(raw[..., 32: 32 + 28]).reshape(4, -1),
                       K.block_gate(u[..., :28].reshape(4, -1), w64["l1.mix.ri"], w64["l1.mix.ri.b"]))
    assert np.allclose(w["text/layers/1/mix/rate"].reshape(3, 32)[:, :28].reshape(-1), 8 * K.softplus(w64["l1.mix.lam"]))
    # experts: widths of 18 in 64 columns; padded columns stay zero although the unit adds one to `up`
    spec = cfg.layers[1].mlp
    gu = x @ w["text/layers/1/mlp/up"][2].T
    y = K.glu_clamped(gu[:, :64], gu[:, 64:], 1.2)
    assert not y[:, 18:].any()
    assert np.allclose((y @ w["text/layers/1/mlp/down"][2].T)[:, :n], K.expert(w64, "l1.mlp.e2", h, 1.2))
    z = x @ w["text/layers/1/mlp/router"].T
    assert z.shape[1] == spec.router_cols == 8 and np.allclose(z[:, :7], h @ w64["l1.mlp.router"].T)
    assert np.allclose(z[:, 7:8], h @ w64["l1.mlp.shared.sg"].T)
    # norms are stored around zero, and only the true columns get their one
    for name in ("text/layers/0/norm1", "text/final_norm"):
        key = name.replace("text/layers/0/", "l0.").replace("text/final_norm", "final.norm")
        assert np.allclose(w[name][:n], 1 + w64[key]) and not w[name][n:].any()


def test_registry_and_gate():
    for name, cfg in tuzupel.CONFIGS.items():
        assert AR.LAYERED_REGISTRY[name] is cfg and PK.construct(name) is cfg
        d = PK.describe(name)
        assert d["servable"] and d["chunked"] + d["latent"] + d["rglru"] == cfg.n_layers and not d["oracle_runtime"]
    for need in ("residual-streams", "chunked-attention", "learned-sink", "scaled-rope", "gated-recurrence", "expert-mlp", "identity-experts"):
        with pytest.raises(PK.PackageRefused, match=need):
            PK.construct("tuzupel-1b", PK.ENGINE_CAPABILITIES - {need})
    with pytest.raises(PK.PackageRefused):
        PK.construct_oracle("tuzupel-tiny")


# ---------------------------------------------------------------------------- the tests' weights show faults
def _shift(name, **kw):
    return (name, lambda old: lambda T, window=0, chunk=0: old(T, window + kw.get("window", 0) if window else 0, chunk + kw.get("chunk", 0) if chunk else 0))



FAULTS = {
    "window one short": _shift("sees", window=-1),
    "window one long": _shift("sees", window=1),
    "chunk one short": _shift("sees", chunk=-1),
    "chunks are a window": ("sees", lambda old: lambda T, window=0, chunk=0: old(T, window or chunk, 0)),
    "no sink": ("softmax_over", lambda old: lambda s, seen, sink=None: old(s, seen, None)),
    "sink counted twice": ("softmax_over", lambda old: lambda s, seen, sink=None: old(s, seen, None if sink is None else sink + np.log(2.0))),
    "sink as a score of the scale": ("softmax_over", lambda old: lambda s, seen, sink=None: old(s, seen, None if sink is None else sink * 0.25)),
    "no rotation": ("rotate", lambda old: lambda x, pos, f: x),
    "unscaled frequencies": ("frequencies", lambda old: lambda rot: old(dict(rot, scaling=None))),
    "rotation of the next position for keys": ("rotate", lambda old: lambda x, pos, f: old(x, pos + (x.shape[1] in (2, 4)), f)),
    "no convolution bias": ("causal_conv", lambda old: lambda x, w, b: old(x, w, 0 * b)),
    "convolution restarts at token 40": ("causal_conv", lambda old: lambda x, w, b: np.concatenate([old(x[:40], w, b), old(x[40:], w, b)])),
    "state lost at token 40": ("linear_recurrence", lambda old: lambda u, r, i, lam: np.concatenate([old(u[:40], r[:40], i[:40], lam), old(u[40:], r[40:], i[40:], lam)])),
    "first token takes all": ("linear_recurrence", lambda old: lambda u, r, i, lam: old(u, np.concatenate([r[:1] + 1e3, r[1:]]), i, lam)),
    "gates swapped": ("linear_recurrence", lambda old: lambda u, r, i, lam: old(u, i, r, lam)),
    "no shift in the unit": ("glu_clamped", lambda old: lambda g, u, l: old(g, u, l) - np.minimum(g, l) * K.sigmoid(1.702 * np.minimum(g, l))),
    "no limit": ("glu_clamped", lambda old: lambda g, u, l: old(g, u, 1e9)),
    "gate bounded from below too": ("glu_clamped", lambda old: lambda g, u, l: old(np.maximum(g, -l), u, l)),
    "weights renormalised": ("route", lambda old: lambda z, c, top, s, f=None: (lambda i, w: (i, w / w.sum(-1, keepdims=True) * s))(*old(z, c, top, s, f))),
    "correction in the weights": ("route", lambda old: lambda z, c, top, s, f=None: old(z + np.log(np.maximum(K.router_scores(z) + c, 1e-9)) - np.log(K.router_scores(z)), 0 * c, top, s, f)),
    "no correction": ("route", lambda old: lambda z, c, top, s, f=None: old(z, 0 * c, top, s, f)),
    "plain norm weights": ("norm_about_zero", lambda old: lambda x, w, eps: old(x, w - 1.0, eps)),
    "mix read the other way": ("stream_write", lambda old: lambda X, y, mix, w: old(X, y, mix.T, w)),
    "streams read after the update": ("stream_read", lambda old: lambda X, w: old(X, w[::-1])),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_a_planted_fault_is_far_above_the_tolerances(fault, monkeypatch):
    c, _, _, w = C.build("mixed")
    ids = prompt(90, c["vocab"], 5)
    want = K.forward(w, c, ids)
    name, plant = FAULTS[fault]
    monkeypatch.setattr(K, name, plant(getattr(K, name)))
    assert err(K.forward(w, c, ids), want) > 0.05     # fp32 runs are held to 3e-5, bf16 runs to a few per cent
