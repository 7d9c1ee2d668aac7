"""Tebivik on the CPU: configuration, checkpoint reading, packing, registry, layer runs and their cache and state, and
that the tests' weights show the faults they are meant to show."""
import json

import numpy as np
import pytest
import torch

import tebivik_cases as C
import tebivik_oracle as K
from kuzanex_cases import err, prompt
from ninfer_fusion_b200.models import architectures as AR
from ninfer_fusion_b200.models import packages as PK
from ninfer_fusion_b200.models import tebivik
from ninfer_fusion_b200.models.layered import LayeredModel, native_subset
from ninfer_fusion_b200.runtime.kv_cache import PagedKvCache, RecurrentStatePool


@pytest.mark.parametrize("name", sorted(C.CASES))
def test_configuration_round_trip(name):
    c, cfg, _, _ = C.build(name)
    assert tebivik.config_dict(cfg) == c
    assert tebivik.parse_config(tebivik.config_dict(cfg), name) == cfg
    assert sum(int(np.prod(s)) for _, s in tebivik.tensor_shapes(cfg)) == cfg.param_count()
    assert [r for r, _ in cfg.runs] == [i for i, _ in K.layer_order(c)]
    assert [t for _, t in cfg.runs if t >= 0] == list(range(c["loop"]["times"]))
    assert native_subset(cfg) == "+".join(sorted({{"latent_attention": "latent", "hgrn2": "gated"}[l["type"]] for l in c["layers"]}))


def test_configuration_errors_are_named():
    with pytest.raises(ValueError, match="equal parts"):
        tebivik.parse_config(C.conf(64, 40, [C.mem(1, 16, 16)], (0, 1, 1), groups=3))
    with pytest.raises(ValueError, match="loop"):
        tebivik.parse_config(C.conf(64, 40, [C.mem(1, 16, 16)], (0, 2, 1)))
    with pytest.raises(ValueError, match="unknown mixer 'ring'"):
        tebivik.parse_config(C.conf(64, 40, [dict(C.mem(1, 16, 16), type="ring")], (0, 1, 1)))
    bad = C.lat(1, 16, 8, 16, 16, 16)
    bad["mixer"]["rot"]["dims"] = 6
    with pytest.raises(ValueError, match="rotated as a whole"):
        tebivik.parse_config(C.conf(64, 40, [bad], (0, 1, 1)))


def test_every_run_has_its_own_cache_and_state():
    _, cfg, _, _ = C.build("mixed")                     # runs: memory | latent, memory | latent, memory
    assert [i for i, _ in cfg.runs] == [0, 1, 2, 1, 2] and [t for _, t in cfg.runs] == [-1, 0, -1, 1, -1]
    assert cfg.attn_layers == [1, 3] and cfg.state_layers == [0, 1, 2, 3, 4]
    assert cfg.kv_geometry == [(1, 96, 0)] * 2
    conv = (3, 96)
    assert cfg.state_shapes() == [[conv, (2, 32, 48)], [conv], [conv, (3, 16, 64)], [conv], [conv, (3, 16, 64)]]
    _, one_tap, _, _ = C.build("memory_only")           # a convolution of one tap looks back on nothing
    assert all(len(s) == 1 for s in one_tap.state_shapes())
    st = RecurrentStatePool([[(s, torch.float32) for s in l] for l in cfg.state_shapes()], 2, "cpu")
    a = st.alloc()
    for t in st.tensors():
        t[a].fill_(3.0)
    st.release(a)
    assert st.alloc() == a and all(not t[a].any() for t in st.tensors())


def test_latent_rows_are_paged_without_value_planes():
    _, cfg, _, _ = C.build("mixed")
    for fmt, dt in (("bf16", torch.bfloat16), ("fp32", torch.float32)):
        kv = PagedKvCache(cfg, 8, 16, 2, 6, "cpu", formats=fmt, geometry=cfg.kv_geometry)
        assert [tuple(p.shape) for p in kv.layers[0].typed(dt)] == [(8, 1, 16, 96), (8, 1, 16, 0)]
        assert kv.bytes_per_token() == 2 * 96 * (2 if fmt == "bf16" else 4)
    kv.ensure(0, 33)
    for l in kv.layers:
        l.typed(torch.float32)[0].normal_()
    pages = kv.detach_prefix(0, 33)
    image = kv.export_pages(pages)
    fresh = kv.import_pages(image, len(pages))
    for l in kv.layers:
        assert torch.equal(l.k_codes[fresh], l.k_codes[pages])


def test_model_folder(tmp_path):
    c, cfg, t, _ = C.build("odd")
    AR.save_folder(str(tmp_path), cfg, t)
    got, w = AR.load_folder(str(tmp_path), "cpu", torch.float32)
    assert got.layers == cfg.layers and got.loop == cfg.loop and w["text/embed"].dtype == torch.float32
    assert w["text/embed"] is w["text/lm_head"] or torch.equal(w["text/embed"], w["text/lm_head"])
    del t["l1.mix.lower"]
    AR.save_folder(str(tmp_path), cfg, t)
    with pytest.raises(ValueError, match="l1.mix.lower"):
        AR.load_folder(str(tmp_path), "cpu")
    t["l1.mix.lower"] = torch.zeros(3, dtype=torch.bfloat16)
    AR.save_folder(str(tmp_path), cfg, t)
    with pytest.raises(ValueError, match="l1.mix.lower.*shape"):
        AR.load_folder(str(tmp_path), "cpu")
    (tmp_path / "config.json").write_text(json.dumps({k: v for k, v in c.items() if k != "residual_mult"}))
    with pytest.raises(ValueError, match="residual_mult"):
        AR.read_config(str(tmp_path))


def test_packing_pads_heads_with_zeros_and_keeps_products():
    _, cfg, t, w64 = C.build("odd")
    w = tebivik.pack(cfg, t.__getitem__, torch.float32)
    g = np.random.default_rng(0)
    m = cfg.layers[0].mixer
    x = np.zeros((4, cfg.hidden_p))
    x[:, : cfg.hidden] = g.normal(size=(4, cfg.hidden))
    proj = x @ w["text/layers/0/mix/in_proj"].double().numpy().T
    h = x[:, : cfg.hidden]
    assert np.allclose(proj[:, : m.q_rank], h @ w64["l0.mix.dq"].T) and not proj[:, m.q_rank: m.q_rank_p].any()
    kv = h @ w64["l0.mix.dkv"].T
    at = m.q_rank_p
    assert np.allclose(proj[:, at: at + m.kv_rank], kv[:, : m.kv_rank])
    assert np.allclose(proj[:, at + m.kv_rank_p: at + m.kv_rank_p + m.rot_dim], kv[:, m.kv_rank:])
    # a query against a key, absorbed and expanded
    c = np.zeros(m.kv_rank_p)
    c[: m.kv_rank] = g.normal(size=m.kv_rank)
    cq = np.zeros(m.q_rank_p)
    cq[: m.q_rank] = g.normal(size=m.q_rank)
    q = (w["text/layers/0/mix/uq"].double().numpy() @ cq).reshape(m.heads, m.dim_p + m.rot_p)
    ref = (w64["l0.mix.uq"] @ cq[: m.q_rank]).reshape(m.heads, -1)
    k = (w64["l0.mix.uk"] @ c[: m.kv_rank]).reshape(m.heads, m.dim)
    want = (ref[:, : m.dim] * k).sum(1)
    absorbed = np.einsum("hcd,hd->hc", w["text/layers/0/mix/uk_t"].double().numpy(), q[:, : m.dim_p]) @ c
    keys = (w["text/layers/0/mix/ukv"].double().numpy()[: m.heads * m.dim_p] @ c).reshape(m.heads, m.dim_p)
    assert np.allclose(absorbed, want) and np.allclose((keys * q[:, : m.dim_p]).sum(1), want)
    assert np.allclose(q[:, m.dim_p: m.dim_p + m.rot_dim], ref[:, m.dim:])
    lower = w["text/layers/1/mix/lower"].reshape(cfg.layers[1].mixer.heads, -1)
    assert (lower[:, cfg.layers[1].mixer.dim:] == 1).all()        # padded channels neither forget nor take in
    # the loop's input projection reads [x, x0] with both halves padded
    pair = np.concatenate([x, 2 * x], axis=1)
    assert np.allclose((pair @ w["text/loop/in_proj"].double().numpy().T)[:, : cfg.hidden], np.concatenate([h, 2 * h], 1) @ w64["loop.in"].T)


def test_registry_and_gate():
    for name, cfg in tebivik.CONFIGS.items():
        assert AR.LAYERED_REGISTRY[name] is cfg and PK.construct(name) is cfg
        d = PK.describe(name)
        assert d["servable"] and d["hgrn2"] + d["latent"] == cfg.n_layers and not d["oracle_runtime"]
    for need in ("latent-attention", "gated-memory", "layer-loop", "sandwich-norms"):
        with pytest.raises(PK.PackageRefused, match=need):
            PK.construct("tebivik-tiny", PK.ENGINE_CAPABILITIES - {need})
    with pytest.raises(PK.PackageRefused):
        PK.construct_oracle("tebivik-tiny")


def test_shrinking_keeps_what_is_left_of_the_loop():
    cfg = tebivik.T1B
    assert cfg.shrink(14).loop == tebivik.LoopSpec(12, 14, 2) and cfg.shrink(4).loop is None
    assert len(cfg.shrink(14).runs) == 16


def test_expanding_pays_from_a_portion_length_on():
    m = tebivik.T1B.layers[1].mixer if tebivik.T1B.layers[1].mixer.kind == "latent_attention" else tebivik.T1B.layers[3].mixer
    n = LayeredModel.expand_tokens(m)
    L = 5000

    def absorbed(t):
        return t * L * (2 * m.kv_rank + m.rot_dim)

    def expanded(t):
        return t * L * (m.dim + m.rot_dim + m.vdim) + L * m.kv_rank * (m.dim + m.vdim)
    assert expanded(n) <= absorbed(n) and expanded(n - 1) > absorbed(n - 1)
    _, cfg, _, _ = C.build("plain")
    assert LayeredModel.expand_tokens(cfg.layers[1].mixer) == 32


# ---------------------------------------------------------------------------- the tests' weights show faults
FAULTS = {
    "no sink": ("sink_softmax", lambda old: lambda s, sink: old(s, np.full_like(sink, -1e9))),
    "sink counted three times": ("sink_softmax", lambda old: lambda s, sink: old(s, sink + np.log(3.0))),
    "rotation in halves": ("rotate", lambda old: lambda x, pos, base: old(np.concatenate([x[..., 0::2], x[..., 1::2]], -1), pos, base)),
    "rotation by the next position": ("rotate", lambda old: lambda x, pos, base: old(x, pos + (x.ndim == 3), base)),
    "no convolution": ("causal_conv", lambda old: lambda h, w: np.zeros_like(h)),
    "convolution restarts at token 40": ("causal_conv", lambda old: lambda h, w: np.concatenate([old(h[:40], w), old(h[40:], w)])),
    "one norm for the row": ("group_norm", lambda old: lambda x, w, g, eps: old(x, w, 1, eps)),
    "no lower bound": ("forget_gate", lambda old: lambda raw, lower: old(raw, 0 * lower)),
    "state lost at token 40": ("hgrn_recurrence", lambda old: lambda *x: np.concatenate([old(*(y[:40] for y in x)), old(*(y[40:] for y in x))])),
    "no step vector": ("enter_pass", lambda old: lambda w, x, x0, t: old(dict(w, **{"loop.step": 0 * w["loop.step"]}), x, x0, t)),
    "embedding not fed back": ("enter_pass", lambda old: lambda w, x, x0, t: old(w, x, x, t)),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_a_planted_fault_is_far_above_the_tolerances(fault, monkeypatch):
    c, _, _, w = C.build("mixed")
    ids = prompt(90, c["vocab"], 5)
    want = K.forward(w, c, ids)
    name, plant = FAULTS[fault]
    monkeypatch.setattr(K, name, plant(getattr(K, name)))
    assert err(K.forward(w, c, ids), want) > 0.05     # fp32 runs are held to 3e-5, bf16 runs to a few per cent
