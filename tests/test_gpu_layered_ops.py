"""Kernels of the layer-list decoders, each mechanism alone against the plain float64 functions of kuzanex_oracle."""
import numpy as np
import pytest
import torch

import kuzanex_oracle as K

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def ops():
    from ninfer_fusion_b200 import load_native
    return load_native()


def rnd(seed, *shape, s=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * s).to(dtype)


def f64(t):
    return t.detach().double().cpu().numpy()


def rel(got, want):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert np.isfinite(got).all()
    return float(np.abs(got - want).max() / max(1e-30, np.abs(want).max()))


@pytest.mark.parametrize("T,N,K_", [(1, 6, 24), (3, 130, 200), (70, 64, 88), (300, 514, 136), (700, 2 * 128 + 4, 64)])
def test_gemm_fp32_columns_and_xielu(ops, T, N, K_):
    from ninfer_fusion_b200._lib import StatusWord
    st = StatusWord("cuda")
    frm = N // 4 * 2
    x, w, bias = rnd(1, T, K_, s=0.5), rnd(2, N, K_, s=0.5), rnd(3, N, s=0.3)
    prm = torch.tensor([0.8, 1.3])
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 5e-3)):
        xd, wd = x.to(dt), w.to(dt)
        z = f64(xd) @ f64(wd).T + f64(bias)
        # softplus(p) = 0.8, 1/2 + softplus(q) = 1.3
        act = np.array([np.log(np.expm1(0.8)), np.log(np.expm1(0.8))])
        for mode, want in ((0, z), (3, K.xielu(z, act))):
            out = torch.zeros((T, frm), dtype=dt, device="cuda")
            o32 = torch.zeros((T, N - frm + (N - frm) % 2), dtype=torch.float32, device="cuda")
            whole = torch.zeros((T, N), dtype=torch.float32, device="cuda")
            a = prm.cuda() if mode else None
            if dt == torch.float32:
                ops.gemm_f32(xd.cuda(), wd.cuda(), out, bias.cuda(), mode, a, o32, frm)
                ops.gemm_f32(xd.cuda(), wd.cuda(), None, bias.cuda(), mode, a, whole, 0)
            else:
                splits = int(ops.gemm_pick_splits(T, N, K_, 0))
                ops.gemm_bf16(xd.cuda(), wd.cuda(), out, 0, None, bias.cuda(), None, splits, st.tensor, False, mode, None, None, None,
                              None, None, o32, frm, a)
                ops.gemm_bf16(xd.cuda(), wd.cuda(), None, 0, None, bias.cuda(), None, splits, st.tensor, False, mode, None, None, None,
                              None, None, whole, 0, a)
            st.check()
            assert rel(f64(out), want[:, :frm]) < tol
            assert rel(f64(o32)[:, : N - frm], want[:, frm:]) < (tol if dt == torch.float32 else 1e-5)   # bf16 operands, fp32 result
            assert rel(f64(whole), want) < (tol if dt == torch.float32 else 1e-5)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n_true,T", [(8, 1), (150, 5), (2048, 3), (9000, 2)])
def test_post_sum_norm_rows(ops, dt, n_true, T):
    N, alpha, eps = (n_true + 7) // 8 * 8, 1.7, 1e-3
    x, d = torch.zeros(T, N), torch.zeros(T, N)
    x[:, :n_true], d[:, :n_true] = rnd(1, T, n_true), rnd(2, T, n_true)
    gain, fin = torch.tensor([0.7]), torch.tensor([1.9])
    want = K.scalar_norm(alpha * f64(x)[:, :n_true] + f64(d)[:, :n_true], 0.7, eps)
    for final in (None, fin):
        xd, xa = x.cuda(), torch.zeros((T, N), dtype=dt, device="cuda")
        ops.post_norm_rows(xd, d.cuda(), xa, n_true, alpha, eps, gain.cuda(), None if final is None else final.cuda(), False)
        assert rel(f64(xd)[:, :n_true], want) < 1e-6
        wa = want if final is None else K.scalar_norm(want, 1.9, eps)
        assert rel(f64(xa)[:, :n_true], wa) < (1e-6 if dt == torch.float32 else 4e-3)
        assert not xd[:, n_true:].any() and not xa[:, n_true:].any()


@pytest.mark.parametrize("dt", DTYPES)
def test_embedding_rows(ops, dt):
    table = rnd(1, 37, 40, dtype=dt).cuda()
    ids = torch.tensor([3, 36, 0, 3], dtype=torch.int32, device="cuda")
    x, xa = torch.zeros((4, 40), device="cuda"), torch.zeros((4, 40), dtype=dt, device="cuda")
    ops.embed_rows32(ids, table, x, xa, 1.0, False)
    assert torch.equal(x, table[ids.long()].float()) and torch.equal(xa, table[ids.long()])


class Paged:
    """Sequences of given lengths in a shuffled page pool; `lens[s]` tokens of sequence s are in the cache."""

    def __init__(self, lens, G, D, V, P, dt, seed=0):
        g = torch.Generator().manual_seed(seed)
        per = [(n + P - 1) // P for n in lens]
        perm = torch.randperm(sum(per) + 3, generator=g).tolist()
        self.table = torch.full((len(lens), max(per)), -1, dtype=torch.int32)
        at = 0
        for s, n in enumerate(per):
            self.table[s, :n] = torch.tensor(perm[at:at + n], dtype=torch.int32)
            at += n
        self.k = torch.full((len(perm), G, P, D), float("nan")).to(dt)    # unwritten rows must never matter
        self.v = torch.zeros((len(perm), G, P, V)).to(dt)
        self.P = P

    def write(self, s, k, v):
        for j in range(k.shape[0]):
            pg = int(self.table[s, j // self.P])
            self.k[pg, :, j % self.P] = k[j]
            self.v[pg, :, j % self.P] = v[j]


GEOMETRIES = [  # heads, kv heads, key width, value width, window, page
    (4, 4, 32, 32, 8, 16), (6, 2, 48, 80, 40, 64), (3, 1, 16, 16, 1, 8), (16, 4, 128, 128, 100, 64), (20, 5, 64, 96, 33, 32),
    (32, 8, 128, 64, 64, 64), (8, 8, 64, 48, 0, 16), (2, 1, 16, 272, 50, 64), (34, 17, 32, 32, 20, 16),
    (4, 2, 160, 128, 30, 16), (12, 1, 80, 48, 21, 64), (16, 16, 64, 64, 90, 16), (7, 7, 48, 256, 11, 32)]


@pytest.mark.parametrize("geo", GEOMETRIES)
@pytest.mark.parametrize("dt", DTYPES)
def test_head_mixing_attention(ops, geo, dt):
    """Ragged batch over shuffled pages: prompts (prefill kernels and token kernel) and single tokens, with and without
    split keys.  A few keys stand out by distance: the last one inside and the first one outside of a query's window."""
    H, G, D, V, W, P = geo
    scale, cap = 0.3, 20.0
    lens, news = [130, 70, 5, 193], [130, 2, 5, 65]         # cached length after the step, tokens the step brings
    qs, ks, vs = ([rnd(10 * s + j, n, heads, width).to(dt) for s, n in enumerate(lens)]
                  for j, (heads, width) in enumerate(((H, D), (G, D), (G, V))))
    for s, n in enumerate(lens):
        for i in range(n):                                    # align the key at the window's edge with its query
            for off in ((W - 1, W) if W else (i,)):
                if i % 7 == 3 and 0 <= i - off:
                    ks[s][i - off] = (qs[s][i][:: H // G] * 1.5).to(dt)
    pg = Paged(lens, G, D, V, P, dt)
    for s in range(len(lens)):
        pg.write(s, ks[s], vs[s])
    mix, gate_all = rnd(77, H, H, s=0.2) + torch.eye(H), [rnd(90 + s, n, H) for s, n in enumerate(lens)]
    slope = torch.from_numpy(f64(mix) @ K.head_slopes(H)).float()
    want = []
    for s, n in enumerate(lens):
        sc = K.mix_heads(K.distance_bias(K.capped_scores(f64(qs[s]), f64(ks[s]), scale, cap)), f64(mix))
        a = K.sink_softmax(sc, K.window_mask(n, W or n))
        o = np.stack([a[h] @ f64(vs[s])[:, h // (H // G)] for h in range(H)], axis=1)
        want.append((o * K.sigmoid(f64(gate_all[s]))[:, :, None]).reshape(n, H * V)[n - news[s]:])
    want = np.concatenate(want)
    q = torch.cat([qs[s][n - news[s]:].reshape(news[s], H * D) for s, n in enumerate(lens)]).cuda()
    gate = torch.cat([gate_all[s][n - news[s]:] for s, n in enumerate(lens)]).cuda()
    row = torch.cat([torch.full((news[s],), s, dtype=torch.int32) for s in range(len(lens))]).cuda()
    kv_len = torch.cat([torch.arange(n - news[s] + 1, n + 1, dtype=torch.int32) for s, n in enumerate(lens)]).cuda()
    T = q.shape[0]
    common = (pg.k.cuda(), pg.v.cuda(), pg.table.cuda(), row, kv_len, W, scale, cap, 1.0, mix.cuda(), slope.cuda(), gate)
    tol = 3e-6 if dt == torch.float32 else 8e-3
    for split, n_splits in ((max(lens), 1), (32, (min(W or max(lens), max(lens)) + 31) // 32)):
        out = torch.zeros((T, H * V), dtype=dt, device="cuda")
        po, ml = torch.empty(T * n_splits * H * V, device="cuda"), torch.empty(T * n_splits * H * 2, device="cuda")
        ops.head_mix_attention(q, *common, out, split, n_splits, po, ml, False)
        assert rel(f64(out), want) < tol
    if dt == torch.bfloat16:
        B = int(ops.head_mix_block_tokens())
        start, count, t = [], [], 0
        for n in news:
            for o in range(0, n, B):
                start.append(t + o)
                count.append(min(B, n - o))
            t += n
        bs, bc = (torch.tensor(x, dtype=torch.int32, device="cuda") for x in (start, count))
        for blocks in (len(start), 2, 1):     # scratch for all query blocks, for two, for one at a time
            scratch = torch.empty(int(ops.head_mix_prefill_scratch(H, max(lens), W, blocks)), dtype=torch.uint8, device="cuda")
            out = torch.zeros((T, H * V), dtype=dt, device="cuda")
            ops.head_mix_prefill(q, *common, out, bs, bc, max(lens), scratch, False)
            assert rel(f64(out), want) < tol


@pytest.mark.parametrize("dt", DTYPES)
def test_attention_without_options(ops, dt):
    """No cap, bias, mixing, sink, gate: plain grouped-query softmax attention."""
    H, G, D, V, n = 4, 2, 32, 48, 75
    q, k, v = rnd(1, n, H, D).to(dt), rnd(2, n, G, D).to(dt), rnd(3, n, G, V).to(dt)
    pg = Paged([n], G, D, V, 16, dt)
    pg.write(0, k, v)
    s = np.stack([0.2 * f64(q)[:, h] @ f64(k)[:, h // 2].T for h in range(H)])
    s = np.where(K.window_mask(n, n), s, -np.inf)
    a = np.exp(s - s.max(-1, keepdims=True))
    a /= a.sum(-1, keepdims=True)
    want = np.stack([a[h] @ f64(v)[:, h // 2] for h in range(H)], axis=1).reshape(n, H * V)
    args = (q.reshape(n, -1).cuda(), pg.k.cuda(), pg.v.cuda(), pg.table.cuda(), torch.zeros(n, dtype=torch.int32, device="cuda"),
            torch.arange(1, n + 1, dtype=torch.int32, device="cuda"), 0, 0.2, 0.0, 0.0, None, None, None)
    out = torch.zeros((n, H * V), dtype=dt, device="cuda")
    ops.head_mix_attention(*args, out, 128, 1, None, None, False)
    assert rel(f64(out), want) < (3e-6 if dt == torch.float32 else 8e-3)
    if dt == torch.bfloat16:
        bs, bc = (torch.tensor(x, dtype=torch.int32, device="cuda") for x in ([0, 64], [64, 11]))
        scratch = torch.empty(int(ops.head_mix_prefill_scratch(H, n, 0, 2)), dtype=torch.uint8, device="cuda")
        out.zero_()
        ops.head_mix_prefill(*args, out, bs, bc, n, scratch, False)
        assert rel(f64(out), want) < 8e-3


@pytest.mark.parametrize("dt", DTYPES)
def test_qk_norm_and_append(ops, dt):
    H, G, D, Dp, V, P, eps = 3, 1, 40, 48, 32, 8, 1e-2
    T, pos0 = 11, 5
    proj = torch.zeros(T, (H + G) * Dp + G * V)
    heads = proj[:, : (H + G) * Dp].view(T, H + G, Dp)
    heads[:, :, :D] = rnd(1, T, H + G, D)
    proj[:, (H + G) * Dp:] = rnd(2, T, G * V)
    proj = proj.to(dt)
    qn, kn = torch.zeros(Dp), torch.zeros(Dp)
    qn[:D], kn[:D] = rnd(3, D), rnd(4, D)
    table = torch.tensor([[9, 9, 9], [2, 0, 3]], dtype=torch.int32)
    kp, vp = torch.zeros((4, G, P, Dp), dtype=dt, device="cuda"), torch.zeros((4, G, P, V), dtype=dt, device="cuda")
    q = torch.zeros((T, H * Dp), dtype=dt, device="cuda")
    pos = torch.arange(pos0, pos0 + T, dtype=torch.int32, device="cuda")
    ops.qkv_append(proj.cuda(), 0, H * Dp, (H + G) * Dp, H, G, D, qn.cuda(), kn.cuda(), eps,
                   torch.ones(T, dtype=torch.int32, device="cuda"), pos, table.cuda(), q, kp, vp, P, False)
    src = f64(proj)[:, : (H + G) * Dp].reshape(T, H + G, Dp)[:, :, :D]
    tol = 1e-6 if dt == torch.float32 else 5e-3
    assert rel(f64(q).reshape(T, H, Dp)[:, :, :D], K.rms(src[:, :H], eps) * f64(qn)[:D]) < tol
    assert not q.view(T, H, Dp)[:, :, D:].any()
    for t in range(T):
        pg, r = int(table[1, (pos0 + t) // P]), (pos0 + t) % P
        assert rel(f64(kp[pg, 0, r])[:D], K.rms(src[t, H], eps) * f64(kn)[:D]) < tol
        assert torch.equal(vp[pg, 0, r].cpu(), proj[t, (H + G) * Dp:])


MEMORIES = [(1, 16, 16), (5, 48, 96), (3, 80, 48), (2, 128, 80), (2, 256, 512), (1, 512, 256), (2, 64, 640)]


def run_memory(ops, geo, dt, chunked, portions, inputs, cap, eps, slots=5):
    """Runs the op over `portions` (per step: tokens each sequence brings); returns outputs per sequence and the state."""
    H, D, V = geo
    q, k, v, gate, i, f, norm = inputs
    n_seq = len(q)
    S = torch.zeros((slots, H, D, V), device="cuda")
    n, m = torch.zeros((slots, H, D), device="cuda"), torch.zeros((slots, H), device="cuda")
    outs, at = [[] for _ in range(n_seq)], [0] * n_seq
    for step in portions:
        seqs = [s for s in range(n_seq) if step[s]]
        rows, gr, cu = [], [], [0]
        for s in seqs:
            a, b = at[s], at[s] + step[s]
            rows.append(torch.cat([x[s][a:b].reshape(b - a, -1) for x in (q, k, v, gate)], 1))
            gr.append(torch.cat([i[s][a:b], f[s][a:b]], 1))
            cu.append(cu[-1] + b - a)
            at[s] = b
        proj, gates = torch.cat(rows).to(dt).cuda(), torch.cat(gr).cuda()
        T = proj.shape[0]
        out = torch.zeros((T, H * V), dtype=dt, device="cuda")
        ws = None
        if chunked:
            ws = torch.empty(int(ops.mlstm_chunked_workspace_bytes(T, len(seqs), H, D, V)), dtype=torch.uint8, device="cuda")
            ws.fill_(0xff)      # NaN patterns: nothing may be read before it is written
        ops.mlstm(proj, 0, H * D, 2 * H * D, H * (2 * D + V), gates, 0, H, V, D ** -0.5, cap, eps, norm.cuda(),
                  torch.tensor(cu, dtype=torch.int32, device="cuda"),
                  torch.tensor([slots - 1 - s for s in seqs], dtype=torch.int32, device="cuda"), S, n, m, out, True, ws, False,
                  max(step) == 1)
        for j, s in enumerate(seqs):
            outs[s].append(f64(out[cu[j]:cu[j + 1]]))
    return [np.concatenate(o) for o in outs], (f64(S), f64(n), f64(m))


@pytest.mark.parametrize("geo", MEMORIES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("i_shift,f_shift", [(0.0, 3.0), (6.0, -2.0), (-9.0, 9.0)])
def test_matrix_memory(ops, geo, dt, i_shift, f_shift):
    """Token-by-token and chunked kernels, whole prompts and portions, against the recurrence; the gate biases move the
    running maximum, forgetting and the floor of the denominator into play."""
    H, D, V = geo
    cap, eps = 8.0, 1e-3
    lens = [150, 1, 64, 77]
    x = [[rnd(100 * j + s, n, H, w) for s, n in enumerate(lens)] for j, w in enumerate((D, D, V, V))]
    x = [[t.to(dt) for t in part] for part in x]
    i = [rnd(500 + s, n, H, s=3.0) + i_shift for s, n in enumerate(lens)]
    f = [rnd(600 + s, n, H, s=3.0) + f_shift for s, n in enumerate(lens)]
    norm = 1 + 0.3 * rnd(7, H * V)
    want = []
    for s, n in enumerate(lens):
        ig, fg = K.mlstm_gates(f64(i[s]), f64(f[s]), cap)
        o = K.rms(K.mlstm_recurrence(f64(x[0][s]) * D ** -0.5, f64(x[1][s]), f64(x[2][s]), ig, fg), eps).reshape(n, H * V)
        want.append(o * f64(norm) * K.sigmoid(f64(x[3][s]).reshape(n, H * V)))
    whole = [lens]
    cut = [[64, 0, 3, 2], [2, 1, 60, 63], [82, 0, 0, 11], [1, 0, 1, 0], [1, 0, 0, 1]]
    tol = 2e-5 if dt == torch.float32 else 1.2e-2
    states = []
    for chunked in ((False, True) if dt == torch.bfloat16 and ops.mlstm_chunked_supported(D, V) else (False,)):
        for portions in (whole, cut):
            got, st = run_memory(ops, geo, dt, chunked, portions, (*x, i, f, norm), cap, eps)
            for s in range(len(lens)):
                assert rel(got[s], want[s]) < tol, (chunked, portions is cut, s)
            states.append(st)
    for st in states[1:]:      # the carried state is 32-bit whichever kernel and cut produced it
        for a, b in zip(st, states[0]):
            assert rel(a, b) < 3e-5


@pytest.mark.parametrize("dt", DTYPES)
def test_token_selection_on_both_logit_types(ops, dt):
    lg = rnd(3, 5, 301).to(dt)
    full = torch.zeros((5, 304), dtype=dt, device="cuda")
    full[:, :301] = lg.cuda()
    full[:, 301:] = 1e9           # padding columns are not part of the vocabulary
    out = torch.zeros(5, dtype=torch.int32, device="cuda")
    ops.argmax_rows(full[:, :301], out, False)
    assert out.tolist() == lg.float().argmax(1).tolist()
    one = torch.ones(5, device="cuda")
    ops.sample_rows(full[:, :301], one, torch.ones(5, dtype=torch.int32, device="cuda"), None, None, None, None, None,
                    torch.zeros(5, dtype=torch.int64, device="cuda"), torch.zeros(5, dtype=torch.int32, device="cuda"), 0, out, None)
    assert out.tolist() == lg.float().argmax(1).tolist()
