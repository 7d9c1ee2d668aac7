"""Ratilorn on the CPU: configuration, checkpoint reading, packing, registry, cache, state and positions, and that the tests'
weights show the faults they are meant to show."""
import json
import math

import numpy as np
import pytest
import torch

import ratilorn_cases as C
import ratilorn_oracle as K
from kuzanex_cases import err, prompt
from ninfer_fusion_b200.models import architectures as AR
from ninfer_fusion_b200.models import packages as PK
from ninfer_fusion_b200.models import ratilorn
from ninfer_fusion_b200.models.layered import native_subset
from ninfer_fusion_b200.runtime.family import check_positions, context_limit
from ninfer_fusion_b200.runtime.kv_cache import PagedKvCache, RecurrentStatePool


@pytest.mark.parametrize("name", sorted(C.CASES))
def test_configuration_round_trip(name):
    c, cfg, _, _ = C.build(name)
    assert ratilorn.config_dict(cfg) == c
    assert ratilorn.parse_config(ratilorn.config_dict(cfg), name) == cfg
    shapes = dict(ratilorn.tensor_shapes(cfg))
    biases = sum(math.prod(s) for n, s in shapes.items() if n.endswith((".q.b", ".k.b", ".v.b")))
    assert sum(math.prod(s) for s in shapes.values()) - biases == cfg.param_count()


def test_stand_alone_libraries_have_the_parts_a_model_needs():
    from ninfer_fusion_b200 import _build
    want = {"mixed": "attention+branches+head_mix+moe+ssd+streams", "sigmoid_only": "attention+branches+head_mix+streams",
            "parallel_only": "attention+branches+moe+ssd+streams"}
    for name, parts in want.items():
        assert native_subset(C.build(name)[1]) == parts
        sources = _build.subset_sources(parts)
        assert all((_build.CSRC / s).exists() for s in sources) and not any("mlstm" in s or "latent" in s for s in sources)


def test_configuration_errors_are_named():
    good = C.par((4, 2, 16, 16, 0.3), (4, 16, 16))
    for layer, what in ((dict(good, type="ring"), "unknown mixer 'ring'"), (C.sig(4, 3, 16, 16), "multiple of kv_heads"),
                        (C.par((4, 3, 16, 16, 0.3), (4, 16, 16)), "multiple of kv_heads"), (C.par((4, 2, 16, 16, 0.3), (4, 16, 16, 3)), "multiple of groups"),
                        (C.par((4, 2, 16, 16, 0.3), (4, 16, 16, 1, 0)), "tap"), (C.par((4, 2, 16, 16, 0.3), (4, 16, 16, 1, 4, 3)), "equal parts"),
                        (dict(good, mlp=C.moe(4, 5, 16)), "5 of 4 experts"), (dict(good, mlp=C.moe(4, 2, 16, (3, 1))), "3 groups"),
                        (dict(good, mlp=C.moe(8, 3, 16, (4, 1))), "no choice of 3"), (dict(good, mlp=dict(C.dense(8), kind="tree")), "'tree'")):
        with pytest.raises(ValueError, match=what):
            ratilorn.parse_config(C.conf(64, 40, [layer]))
    with pytest.raises(ValueError, match="max_positions"):
        ratilorn.parse_config(C.conf(64, 40, [good], 0))
    with pytest.raises(ValueError, match="same value heads"):
        ratilorn.parse_config(C.conf(64, 40, [C.sig(4, 2, 16, 16), C.sig(4, 2, 16, 32)]))
    assert ratilorn.parse_config(C.conf(64, 40, [C.sig(4, 2, 16, 16), C.sig(4, 2, 16, 32, v_mix=False)])).value_runs == [0]


def test_cache_rows_and_state_of_both_sides():
    _, cfg, _, _ = C.build("mixed")
    assert cfg.attn_layers == [0, 1, 2, 3, 4] and cfg.state_layers == [0, 2] and cfg.value_runs == [1, 4] and cfg.cache_window == 0
    assert cfg.kv_geometry == [(2, 32, 48), (3, 32, 16), (4, 16, 32), (2, 48, 32), (3, 16, 16)]
    assert cfg.state_shapes() == [[(4, 4 * 32 + 2 * 2 * 48), (4, 32, 48)], [(3, 6 * 16 + 2 * 3 * 16), (6, 16, 16)]]
    _, odd, _, _ = C.build("odd")                       # heads of 20 channels are kept 32 wide, states of 24 too
    assert odd.state_shapes() == [[(1, 3 * 32 + 2 * 32), (3, 32, 32)], [(2, 5 * 16 + 2 * 5 * 32), (5, 16, 32)]]
    st = RecurrentStatePool([[(s, torch.float32) for s in l] for l in cfg.state_shapes()], 2, "cpu")
    a = st.alloc()
    for t in st.tensors():
        t[a].fill_(3.0)
    st.release(a)
    assert st.alloc() == a and all(not t[a].any() for t in st.tensors())
    kv = PagedKvCache(cfg, 8, 8, 1, 8, "cpu", formats="fp32", geometry=cfg.kv_geometry, look_back=cfg.cache_window)
    for start in range(60):
        kv.advance(0, start, start + 1)
    assert kv.live_pages(0) == 8                        # every layer sees all of the past


def test_a_model_has_so_many_positions():
    _, cfg, _, _ = C.build("odd")
    assert cfg.position_limit == 300 and context_limit(cfg, 10 ** 6) == 300 and context_limit(cfg, 64) == 64
    check_positions(cfg, 300)
    with pytest.raises(ValueError, match="position 300 is beyond"):
        check_positions(cfg, 301)
    from ninfer_fusion_b200.models.tuzupel import TINY
    assert TINY.position_limit == 0 and context_limit(TINY, 10 ** 6) == 10 ** 6
    check_positions(TINY, 10 ** 9)


def test_model_folder(tmp_path):
    c, cfg, t, _ = C.build("odd")
    AR.save_folder(str(tmp_path), cfg, t)
    got, w = AR.load_folder(str(tmp_path), "cpu", torch.float32)
    assert got.layers == cfg.layers and got.learned_positions == 300 and w["text/places"].shape == (300, cfg.hidden_p)
    assert w["text/lm_head"] is w["text/embed"] and json.load(open(tmp_path / "config.json"))["architecture"] == "Ratilorn"
    t2 = dict(t)
    t2["l2.mix.right.conv"] = t2["l2.mix.right.conv"][:, :1].contiguous()
    AR.save_folder(str(tmp_path / "short"), cfg, t2)
    with pytest.raises(ValueError, match="l2.mix.right.conv"):
        AR.load_folder(str(tmp_path / "short"), "cpu")
    del t2["l2.mix.right.conv"]
    AR.save_folder(str(tmp_path / "less"), cfg, t2)
    with pytest.raises(ValueError, match="no tensor 'l2.mix.right.conv'"):
        AR.load_folder(str(tmp_path / "less"), "cpu")


def test_packing_pads_and_computes_the_same():
    c, cfg, t, w64 = C.build("odd")
    w = {n: v.double().numpy() for n, v in ratilorn.pack(cfg, t.__getitem__, torch.float32).items()}
    g, n, N = np.random.default_rng(0), cfg.hidden, cfg.hidden_p
    x = np.zeros((4, N))
    x[:, :n] = g.normal(size=(4, n))
    h = x[:, :n]
    # sigmoid attention: [q, k, v] with their biases
    m, p = cfg.layers[0].mixer, "l0.mix."
    proj = x @ w["text/layers/0/mix/in_proj"].T + w["text/layers/0/mix/in_bias"]
    q = proj[:, : m.heads * m.dim_p].reshape(4, m.heads, m.dim_p)
    assert np.allclose(q[..., : m.dim], K.heads_of(h, w64, p + "q", 3), rtol=1e-6, atol=1e-6) and not q[..., m.dim:].any()
    # two mixers side by side: left columns, right columns, steps
    m, p = cfg.layers[1].mixer, "l1.mix."
    proj = x @ w["text/layers/1/mix/in_proj"].T + w["text/layers/1/mix/in_bias"]
    at, r = m.left.main_cols, m.right
    v = proj[:, at - 5 * m.left.vdim_p: at].reshape(4, 5, m.left.vdim_p)
    assert np.allclose(v[..., :20], K.heads_of(h, w64, p + "left.v", 5), rtol=1e-6, atol=1e-6) and not v[..., 20:].any()
    raw = h @ w64[p + "right.in"].T
    z = proj[:, at: at + r.out_cols].reshape(4, 3, r.vdim_p)
    assert np.allclose(z[..., :20].reshape(4, -1), raw[:, :60]) and not z[..., 20:].any()
    bc = proj[:, at + 2 * r.out_cols: at + r.main_cols].reshape(4, 2, r.state_p)
    assert np.allclose(bc[..., :24].reshape(4, -1), raw[:, 120:168]) and not bc[..., 24:].any()
    assert np.allclose(proj[:, at + r.main_cols: at + r.main_cols + 3], raw[:, 168:] + w64[p + "right.dt_bias"], rtol=1e-6, atol=1e-6)
    cw = w["text/layers/1/right/mix/conv"]
    assert cw.shape == (1, r.conv_cols) and np.allclose(cw[0, :96].reshape(3, 32)[:, :20].reshape(-1), w64[p + "right.conv"][:60, 0])
    y = np.zeros((4, 3, 32))
    y[..., :20] = g.normal(size=(4, 3, 20))
    assert np.allclose((y.reshape(4, -1) @ w["text/layers/1/right/mix/out_proj"].T)[:, :n], y[..., :20].reshape(4, -1) @ w64[p + "right.o"].T)
    # feed-forwards: widths of 50 and 30 in 64 columns
    gu = x @ w["text/layers/1/mlp/up"].T
    assert np.allclose((K.silu(gu[:, :64]) * gu[:, 64:] @ w["text/layers/1/mlp/down"].T)[:, :n], K.glu(w64, "l1.mlp", h))
    gu = x @ w["text/layers/0/mlp/up"][2].T
    assert np.allclose((K.silu(gu[:, :64]) * gu[:, 64:] @ w["text/layers/0/mlp/down"][2].T)[:, :n], K.glu(w64, "l0.mlp.e2", h))
    # norms: around zero for the sublayers, plain for the two sides; the logits' factor is part of the last one
    assert np.allclose(w["text/layers/2/norm1"][:n], 1 + w64["l2.norm1"]) and not w["text/layers/2/norm1"][n:].any()
    assert np.allclose(w["text/layers/2/left/norm"][:n], w64["l2.mix.left.out"])
    _, mixed, t, _ = C.build("mixed")
    assert torch.allclose(ratilorn.pack(mixed, t.__getitem__, torch.float32)["text/final_norm"][:96], 0.7 * (1 + t["final.norm"].float()))


def test_registry_and_gate():
    for name, cfg in ratilorn.CONFIGS.items():
        assert AR.LAYERED_REGISTRY[name] is cfg and PK.construct(name) is cfg
        d = PK.describe(name)
        assert d["servable"] and d["full"] == cfg.n_layers and not d["oracle_runtime"]
    for need in ("sigmoid-attention", "log-distance-bias", "value-mixing", "state-space", "parallel-mixers", "output-norms", "learned-positions",
                 "grouped-routing", "swiglu-mlp"):
        with pytest.raises(PK.PackageRefused, match=need):
            PK.construct("ratilorn-1b", PK.ENGINE_CAPABILITIES - {need})


def test_grouped_choice():
    """Groups by the sum of their two best corrected scores; scores below zero stay choices, those outside do not become zero."""
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    s = np.array([[0.9, 0.05, 0.5, 0.55, 0.6, 0.3]])
    z = np.log(s / (1 - s))
    ids, wt = K.route(z, np.full(6, -2.0), r)
    assert sorted(ids[0].tolist()) == [2, 3] and np.allclose(sorted(wt[0]), [0.5 / 1.05, 0.55 / 1.05])
    assert K.shortfall(z, np.full(6, -2.0), r, ids).max() <= 0
    for wrong in ([[0, 1]], [[4, 5]]):
        assert K.shortfall(z, np.full(6, -2.0), r, np.array(wrong)).max() > 0
    free = {"experts": 6, "top": 2}
    assert sorted(K.route(z, np.zeros(6), free)[0][0].tolist()) == [0, 4]


# ---------------------------------------------------------------------------- the tests' weights show faults
def _cut(old, n, *args, **kw):
    """The function over the first n tokens and over the rest by themselves."""
    return old(*[a[:n] for a in args], **kw), old(*[a[n:] for a in args], **kw)


FAULTS = {
    "no positions": ("embedding", lambda old: lambda e, p, t: old(e, 0 * p, t)),
    "positions start again at token 40": ("embedding", lambda old: lambda e, p, t: np.concatenate([old(e, p, t[:40]), old(e, p, t[40:])])),
    "positions one late": ("embedding", lambda old: lambda e, p, t: old(e, p[1:], t)),
    "plain norm weights": ("norm_about_zero", lambda old: lambda x, w, eps: old(x, w - 1.0, eps)),
    "no distance bias": ("log_distance_bias", lambda old: lambda T, a, b: 0 * old(T, a, b)),
    "distances one longer": ("log_distance_bias", lambda old: lambda T, a, b: np.pad(old(T + 1, a, b)[:, 1:, :-1], 0)),
    "bias numbers swapped": ("log_distance_bias", lambda old: lambda T, a, b: old(T, b, a)),
    "no offset": ("sigmoid_weights", lambda old: lambda s, o: old(s, 0 * o)),
    "weights normalised": ("sigmoid_weights", lambda old: lambda s, o: (lambda a: a / a.sum(-1, keepdims=True))(old(s, o))),
    "own key left out": ("sigmoid_weights", lambda old: lambda s, o: old(s, o) * (1 - np.eye(s.shape[-1]))),
    "first key left out": ("sigmoid_weights", lambda old: lambda s, o: np.concatenate([0 * old(s, o)[..., :1], old(s, o)[..., 1:]], -1)),
    "heads not mixed": ("mix_heads", lambda old: lambda a, t: a),
    "mix read the other way": ("mix_heads", lambda old: lambda a, t: old(a, t.T)),
    "values not mixed": ("mix_values", lambda old: lambda v, f, l: v),
    "value shares swapped": ("mix_values", lambda old: lambda v, f, l: old(f, v, l)),
    "softmax over 40 keys": ("softmax_past", lambda old: lambda s: old(np.where(np.subtract.outer(np.arange(s.shape[1]), np.arange(s.shape[1])) < 40, s, -1e30))),
    "no convolution bias": ("causal_conv", lambda old: lambda x, w, b: old(x, w, 0 * b)),
    "taps reversed": ("causal_conv", lambda old: lambda x, w, b: old(x, w[:, ::-1], b)),
    "convolution restarts at token 40": ("causal_conv", lambda old: lambda x, w, b: np.concatenate(_cut(lambda y: old(y, w, b), 40, x))),
    "state lost at token 40": ("state_space", lambda old: lambda x, B, C, dt, A, D: (np.concatenate([y for y, _ in _cut(lambda *a: old(*a, A, D), 40, x, B, C, dt)]), None)),
    "steps not in the input": ("state_space", lambda old: lambda x, B, C, dt, A, D: old(x / dt[..., None], B, C, dt, A, 0 * D)),
    "no skip": ("state_space", lambda old: lambda x, B, C, dt, A, D: old(x, B, C, dt, A, 0 * D)),
    "B and C swapped": ("state_space", lambda old: lambda x, B, C, dt, A, D: old(x, C, B, dt, A, D)),
    "first group for all heads": ("state_space", lambda old: lambda x, B, C, dt, A, D: old(x, 0 * B + B[:, :1], 0 * C + C[:, :1], dt, A, D)),
    "norm before the gate": ("gated_group_norm", lambda old: lambda y, z, w, g, eps: K.rms(y.reshape(len(y), g, -1), eps).reshape(y.shape) * w * K.silu(z)),
    "one norm for all channels": ("gated_group_norm", lambda old: lambda y, z, w, g, eps: old(y, z, w, 1, eps)),
    "correction in the weights": ("route", lambda old: lambda z, c, r, f=None: (lambda i: (i, np.take_along_axis(K.sigmoid(z) + c, i, -1)))(old(z, c, r, f)[0])),
    "no correction": ("route", lambda old: lambda z, c, r, f=None: old(z, 0 * c, r, f)),
    "weights not divided": ("route", lambda old: lambda z, c, r, f=None: (lambda i: (i, np.take_along_axis(K.sigmoid(z), i, -1)))(old(z, c, r, f)[0])),
    "no groups": ("limited_choice", lambda old: lambda c, g: c),
    "experts outside become zero": ("limited_choice", lambda old: lambda c, g: np.where(np.isinf(old(c, g)), 0.0, old(c, g))),
    "no gate in the units": ("silu", lambda old: lambda z: z),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_a_planted_fault_is_far_above_the_tolerances(fault, monkeypatch):
    c, _, _, w = C.build("mixed")
    ids = prompt(90, c["vocab"], 5)
    want = K.forward(w, c, ids)
    name, plant = FAULTS[fault]
    monkeypatch.setattr(K, name, plant(getattr(K, name)))
    assert err(K.forward(w, c, ids), want) > 0.05     # fp32 runs are held to 3e-5, bf16 runs to a few per cent
