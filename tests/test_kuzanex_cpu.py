"""Kuzanex on the CPU: configuration, checkpoint reading, packing, registry, windowed page accounting, state slots, the
trace replay's protocol, and that the tests' weights show the faults they are meant to show."""
import io
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import kuzanex_cases as C
import kuzanex_oracle as K
from ninfer_fusion_b200.models import architectures as AR
from ninfer_fusion_b200.models import kuzanex
from ninfer_fusion_b200.models import packages as PK
from ninfer_fusion_b200.runtime.batch import SeqChunk, StepBuffers
from ninfer_fusion_b200.runtime.kv_cache import PagedKvCache, RecurrentStatePool


@pytest.mark.parametrize("name", sorted(C.CASES))
def test_configuration_round_trip(name):
    c, cfg, _, _ = C.build(name)
    assert kuzanex.config_dict(cfg) == c
    assert kuzanex.parse_config(kuzanex.config_dict(cfg), name) == cfg
    assert sorted(cfg.attn_layers + cfg.state_layers) == list(range(cfg.n_layers))
    n = sum(int(np.prod(s)) for _, s in kuzanex.tensor_shapes(cfg))
    biases = sum(int(np.prod(s)) for k, s in kuzanex.tensor_shapes(cfg) if k.endswith(".b") and ".i." not in k and ".f." not in k)
    assert n - biases == cfg.param_count()


def test_configuration_errors_are_named():
    c = C.conf(32, 40, [C.att(4, 3, 16, 16, 4)])
    with pytest.raises(ValueError, match="multiple of kv_heads"):
        kuzanex.parse_config(c)
    c = C.conf(32, 40, [dict(C.mem(1, 16, 16), type="ring")])
    with pytest.raises(ValueError, match="unknown mixer 'ring'"):
        kuzanex.parse_config(c)


def test_model_folder(tmp_path):
    c, cfg, t, _ = C.build("odd")
    AR.save_folder(str(tmp_path), cfg, t)
    assert AR.is_model_folder(str(tmp_path)) and not AR.is_model_folder(str(tmp_path / "none"))
    got, w = AR.load_folder(str(tmp_path), "cpu", torch.float32)
    assert got.layers == cfg.layers and w["text/embed"].dtype == torch.float32
    assert torch.equal(w["text/embed"][:, : cfg.hidden], t["embed"].float()) and not w["text/embed"][:, cfg.hidden:].any()
    del t["l1.mix.f.b"]
    AR.save_folder(str(tmp_path), cfg, t)
    with pytest.raises(ValueError, match="l1.mix.f.b"):
        AR.load_folder(str(tmp_path), "cpu")
    (tmp_path / "config.json").write_text(json.dumps(dict(c, architecture="Other")))
    with pytest.raises(AR.UnknownArchitecture, match="Other"):
        AR.read_config(str(tmp_path))


def test_packing_pads_heads_with_zeros_and_keeps_products():
    _, cfg, t, w64 = C.build("odd")
    w = kuzanex.pack(cfg, t.__getitem__, torch.float32)
    m = cfg.layers[0].mixer
    h = torch.zeros(4, cfg.hidden_p, dtype=torch.float64)
    h[:, : cfg.hidden] = torch.randn(4, cfg.hidden, generator=torch.Generator().manual_seed(1)).double()
    proj = h @ w["text/layers/0/mix/in_proj"].double().t() + w["text/layers/0/mix/in_bias"].double()
    x = h[:, : cfg.hidden].numpy()
    q = (x @ w64["l0.mix.q"].T + w64["l0.mix.q.b"]).reshape(4, m.heads, m.dim)
    got = proj[:, : m.heads * m.dim_p].numpy().reshape(4, m.heads, m.dim_p)
    assert np.allclose(got[:, :, : m.dim], q, atol=1e-5) and not got[:, :, m.dim:].any()
    g = proj[:, m.main_cols: m.main_cols + m.gate_cols].numpy()
    assert np.allclose(g, x @ w64["l0.mix.g"].T, atol=1e-5)
    want = w64["l0.mix.talk"] @ K.head_slopes(m.heads)
    assert np.allclose(w["text/layers/0/mix/slope"].numpy(), want, rtol=1e-6)
    assert w["text/layers/0/mix/in_proj"].shape[0] % 2 == 0 and w["text/lm_head"].shape[0] % 8 == 0


def test_registry_and_gate():
    for name, cfg in kuzanex.CONFIGS.items():
        assert AR.LAYERED_REGISTRY[name] is cfg
        assert PK.construct(name) is cfg
        d = PK.describe(name)
        assert d["servable"] and d["mlstm"] == len(cfg.state_layers) and d["sliding"] == len(cfg.attn_layers)
    with pytest.raises(PK.PackageRefused, match="matrix-memory"):
        PK.construct("kuzanex-tiny", PK.ENGINE_CAPABILITIES - {"matrix-memory"})


def test_command_line_refuses_what_the_runtime_lacks(tmp_path):
    _, cfg, t, _ = C.build("mixed")
    AR.save_folder(str(tmp_path), cfg, t)
    for extra in (["--device", "cpu"], ["--device", "cuda", "--weights", "fp8"]):
        r = subprocess.run([sys.executable, "-m", "ninfer_fusion_b200.cli", "generate", "--model", str(tmp_path), "--prompt-ids", "1,2"] + extra,
                           capture_output=True, text=True)
        assert r.returncode != 0 and "layer-list models" in r.stderr


# ---------------------------------------------------------------------------- cache, state, step descriptors
def test_windowed_rows_give_pages_back_and_stay_within_their_bound():
    _, cfg, _, _ = C.build("mixed")
    P, W = 8, cfg.cache_window
    assert W == 70
    kv = PagedKvCache(cfg, 40, P, 2, 200, "cpu", geometry=cfg.kv_geometry, look_back=W)
    for row, steps in ((0, [50, 1, 2, 64, 1, 1, 30] + [1] * 300), (1, [1] * 120)):
        pos = 0
        for n in steps:
            kv.advance(row, pos, pos + n)
            for j in range(max(0, pos - W + 1), pos + n):      # everything a query of the step may look at is mapped
                assert kv.table_host[row, j // P] >= 0
            assert kv.live_pages(row) <= kv.pages_for(pos + n, max(steps))
            pos += n
    live = [p for r in (0, 1) for p in kv.row_pages[r] if p >= 0]
    assert len(live) == len(set(live)) == 40 - kv.pool.free_pages
    pages = kv.detach_prefix(0, pos := 449)                    # a frontier with holes before the window
    assert pages is not None and pages[0] == -1
    kv.free_row(0)
    kv.attach_prefix(pages, 0, pos)
    kv.drop_pages(pages)
    for j in range(pos - W + 1, pos):
        assert kv.table_host[0, j // P] >= 0
    kv.free_row(0)
    kv.free_row(1)
    assert kv.pool.free_pages == 40


def test_rows_have_their_layers_geometry():
    _, cfg, _, _ = C.build("mixed")
    for fmt, dt in (("bf16", torch.bfloat16), ("fp32", torch.float32)):
        kv = PagedKvCache(cfg, 3, 16, 1, 3, "cpu", formats=fmt, geometry=cfg.kv_geometry)
        assert [tuple(k.shape) for k, _ in (l.typed(dt) for l in kv.layers)] == [(3, 2, 16, 32), (3, 4, 16, 16)]
        assert [tuple(v.shape) for _, v in (l.typed(dt) for l in kv.layers)] == [(3, 2, 16, 16), (3, 4, 16, 32)]
    with pytest.raises(ValueError, match="bf16 or fp32"):
        PagedKvCache(cfg, 3, 16, 1, 3, "cpu", formats="fp8", geometry=cfg.kv_geometry)


def test_state_slots_are_cleared_copied_and_moved():
    st = RecurrentStatePool([[((2, 3), torch.float32), ((2,), torch.float32)]], 3, "cpu")
    a = st.alloc()
    for t in st.tensors():
        t[a].fill_(7.0)
    b = st.alloc()
    st.copy_slot(a, b)
    image = st.export_slot(b)
    saved = st.save()
    st.reset(b)
    assert all(not t[b].any() for t in st.tensors())
    st.load(saved)
    assert all((t[b] == 7).all() for t in st.tensors())
    st.release(a)
    assert st.alloc() == a and all(not t[a].any() for t in st.tensors())     # used again: starts from zero
    st.import_slot(image, a)
    assert all((t[a] == 7).all() for t in st.tensors())


def test_wanted_places_of_a_mixed_batch():
    b = StepBuffers(32, 4, "cpu", attn_block_tokens=4, max_logit_rows=32)
    s = b.build([SeqChunk(0, 0, 10, [1, 2, 3, 4, 5], want=[0, 4]), SeqChunk(1, 1, 3, [6], want=[]), SeqChunk(2, 2, 0, [7, 8], want=[1, 0])])
    assert s.logit_rows.tolist() == [0, 4, 7, 6] and s.max_seq_tokens == 5 and s.max_kv_len == 15
    assert s.qblk_start.tolist() == [0, 4, 5, 6] and s.qblk_count.tolist() == [4, 1, 1, 2]


def test_trace_replay_protocol(tmp_path):
    from ninfer_fusion_b200.runtime.trace_replay import replay

    class Fake:
        opened, closed = 0, []

        def open_empty(self):
            self.opened += 1
            return [self.opened, 0]

        def step(self, entries):
            rows = []
            for lane, toks, want in entries:
                rows += [[lane[0], lane[1] + w, toks[w]] for w in want]
                lane[1] += len(toks)
            return torch.tensor(rows, dtype=torch.float32).reshape(-1, 3)

        def close(self, lane):
            self.closed.append(lane[0])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}, {"id": "b", "tokens": [1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [2, 3], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [9], "want": [0]}, {"id": "a", "tokens": [8], "want": [0]}], "end": ["a", "b"]}]
    log, fake = io.StringIO(), Fake()
    replay(fake, [json.dumps(s) + "\n" for s in steps], str(tmp_path), log)
    assert log.getvalue().split("\n")[:3] == ["done 0", "done 1", "done 2"]
    assert np.fromfile(tmp_path / "0.f32", "<f4").reshape(-1, 3).tolist() == [[1, 0, 5], [1, 2, 7]]
    assert not (tmp_path / "1.f32").exists()
    assert np.fromfile(tmp_path / "2.f32", "<f4").reshape(-1, 3).tolist() == [[3, 0, 9], [1, 3, 8]]
    assert fake.closed == [2, 1, 3]


# ---------------------------------------------------------------------------- the tests' weights show faults
def _planted(name, monkeypatch):
    if name == "window one too wide":
        old = K.window_mask
        monkeypatch.setattr(K, "window_mask", lambda T, size: old(T, size + 1))
    elif name == "window one too narrow":
        old = K.window_mask
        monkeypatch.setattr(K, "window_mask", lambda T, size: old(T, max(1, size - 1)))
    elif name == "no sink":
        monkeypatch.setattr(K, "sink_softmax", lambda s, m: (lambda e: e / e.sum(-1, keepdims=True))(
            np.exp(np.where(m, s - np.where(m, s, -np.inf).max(-1, keepdims=True), -np.inf))))
    elif name == "bias after mixing":
        monkeypatch.setattr(K, "distance_bias", lambda s: s)
        old = K.mix_heads
        monkeypatch.setattr(K, "mix_heads", lambda s, t: old(s, t) - K.head_slopes(len(s))[:, None, None] *
                            (np.arange(s.shape[1])[:, None] - np.arange(s.shape[1])[None, :]))
    elif name == "mixing transposed":
        old = K.mix_heads
        monkeypatch.setattr(K, "mix_heads", lambda s, t: old(s, t.T))
    elif name == "gates not capped":
        monkeypatch.setattr(K, "mlstm_gates", lambda i, f, cap: (i, -K.softplus(-f)))
    elif name == "state lost at token 40":
        old = K.mlstm_recurrence
        monkeypatch.setattr(K, "mlstm_recurrence", lambda *x: np.concatenate([old(*(y[:40] for y in x)), old(*(y[40:] for y in x))]))


@pytest.mark.parametrize("fault", ["window one too wide", "window one too narrow", "no sink", "bias after mixing", "mixing transposed",
                                   "gates not capped", "state lost at token 40"])
def test_a_planted_fault_is_far_above_the_tolerances(fault, monkeypatch):
    c, _, _, w = C.build("mixed")
    ids = C.prompt(90, c["vocab"], 5)
    want = K.forward(w, c, ids)
    _planted(fault, monkeypatch)
    assert C.err(K.forward(w, c, ids), want) > 0.05     # fp32 runs are held to 3e-5, bf16 runs to a few per cent
