"""Kernels of latent attention, gated linear memory and the norms around sublayers, each mechanism alone against the plain
float64 functions of tebivik_oracle."""
import numpy as np
import pytest
import torch

import tebivik_oracle as K

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


def ints(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


# ---------------------------------------------------------------------------- rows
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n_true,groups", [(150, 6), (96, 3), (150, 1), (2048, 4), (4096, 1), (5000, 8), (9216, 9), (12288, 3), (24, 24)])
def test_norms_around_a_sublayer(ops, dt, n_true, groups):
    """Whole warps per group, whole vectors per group, neither; with and without the update and the next norm."""
    T, N, mult, eps = 5, (n_true + 7) // 8 * 8, 0.35, 1e-3

    def pad(t):
        out = torch.zeros(*t.shape[:-1], N)
        out[..., :n_true] = t
        return out.cuda()
    x, d, wp, wn = rnd(1, T, n_true), rnd(2, T, n_true) * 3, rnd(3, n_true), rnd(4, n_true)
    d[:, : n_true // groups] *= 50.0                       # one group far louder than the others
    new = f64(x) + mult * K.group_norm(f64(d), f64(wp), groups, eps)
    tol = 2e-6 if dt == torch.float32 else 5e-3
    for delta in (False, True):
        for nxt in (False, True):
            xi, xo, out = pad(x), torch.zeros(T, N, device="cuda"), torch.zeros((T, 2 * N), dtype=dt, device="cuda")[:, N:]
            ops.sandwich_rows(xi, xo, pad(d) if delta else None, pad(wp) if delta else None, pad(wn) if nxt else None, out, n_true, groups,
                              mult, eps, None, None, None, None, 1, True, False)
            base = new if delta else f64(x)
            want = K.group_norm(base, f64(wn), groups, eps) if nxt else base
            assert rel(f64(out)[:, :n_true], want) < tol and not out[:, n_true:].any()
            if delta:
                assert rel(f64(xo)[:, :n_true], new) < 2e-6 and not xo[:, n_true:].any()


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7, 11])
def test_input_convolution_over_cuts_and_batches(ops, dt, taps):
    """Three sequences whose tokens come in portions of all sizes, several in one step, on shuffled slots; the history in the
    slot is the last taps - 1 normed rows and nothing else of the pool is touched."""
    n_true, N, groups, mult, eps = 100, 104, 5, 0.6, 1e-4
    lens = [61, 40, 23]
    slots, n_slots = [4, 0, 2], 6
    w_conv = torch.zeros(taps, N)
    w_conv[:, :n_true] = rnd(9, taps, n_true)
    wp, wn = torch.zeros(N), torch.zeros(N)
    wp[:n_true], wn[:n_true] = rnd(3, n_true), rnd(4, n_true)
    xs, ds, want, hist = [], [], [], []
    for s, n in enumerate(lens):
        x, d = torch.zeros(n, N), torch.zeros(n, N)
        x[:, :n_true], d[:, :n_true] = rnd(20 + s, n, n_true), rnd(30 + s, n, n_true)
        new = f64(x)[:, :n_true] + mult * K.group_norm(f64(d)[:, :n_true], f64(wp)[:n_true], groups, eps)
        h = K.group_norm(new, f64(wn)[:n_true], groups, eps)
        xs.append(x); ds.append(d); hist.append(h)
        want.append((new, h + K.causal_conv(h, f64(w_conv)[:, :n_true].T)))
    state = torch.full((n_slots, taps - 1, N), 7.0, device="cuda") if taps > 1 else None
    if taps > 1:
        for s in slots:
            state[s] = 0
    at, step = [0, 0, 0], 0
    portions = [[1, 9, 2], [30, 1, 1], [1, 1, 16], [8, 1, 1], [2, 25, 1], [16, 2, 1], [3, 1, 1]]
    tol = 3e-6 if dt == torch.float32 else 5e-3
    while any(a < n for a, n in zip(at, lens)):
        todo = [(s, min(portions[step % len(portions)][s], lens[s] - at[s])) for s in range(3)]
        todo = [(s, n) for s, n in todo if n > 0]
        x = torch.cat([xs[s][at[s]:at[s] + n] for s, n in todo]).cuda()
        d = torch.cat([ds[s][at[s]:at[s] + n] for s, n in todo]).cuda()
        cu = ints(np.cumsum([0] + [n for _, n in todo]).tolist())
        xo, out = torch.zeros_like(x), torch.zeros((x.shape[0], N), dtype=dt, device="cuda")
        ops.sandwich_rows(x, xo, d, wp.cuda(), wn.cuda(), out, n_true, groups, mult, eps, w_conv.cuda(), state, cu,
                          ints([slots[s] for s, _ in todo]), max(n for _, n in todo), True, False)
        r = 0
        for s, n in todo:
            new, o = (v[at[s]:at[s] + n] for v in want[s])
            assert rel(f64(xo)[r:r + n, :n_true], new) < 3e-6
            assert rel(f64(out)[r:r + n, :n_true], o) < tol
            at[s] += n
            r += n
            if taps > 1:
                full = np.concatenate([np.zeros((taps - 1, n_true)), hist[s][:at[s]]])[-(taps - 1):]
                assert rel(f64(state)[slots[s]][:, :n_true], full) < 3e-6
        step += 1
    if taps > 1:
        assert all((state[i] == 7).all() for i in range(n_slots) if i not in slots)


@pytest.mark.parametrize("dt", DTYPES)
def test_scaled_embedding_rows(ops, dt):
    table = rnd(1, 37, 40, dtype=dt).cuda()
    x, pair = torch.zeros((3, 40), device="cuda"), torch.zeros((3, 80), dtype=dt, device="cuda")
    ops.embed_rows32(ints([3, 36, 0]), table, x, pair[:, 40:], 0.3, False)
    want = table[[3, 36, 0]].float() * 0.3
    assert torch.equal(x, want) and torch.equal(pair[:, 40:], want.to(dt)) and not pair[:, :40].any()


def test_square_of_relu(ops):
    from ninfer_fusion_b200._lib import StatusWord
    st = StatusWord("cuda")
    for T, N, K_ in ((3, 40, 64), (300, 264, 96)):
        for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 5e-3)):
            x, w, b = rnd(1, T, K_, dtype=dt), rnd(2, N, K_, s=0.2, dtype=dt), rnd(3, N)
            want = np.maximum(f64(x) @ f64(w).T + f64(b), 0) ** 2
            out = torch.zeros((T, N), dtype=dt, device="cuda")
            if dt == torch.float32:
                ops.gemm_f32(x.cuda(), w.cuda(), out, b.cuda(), 4)
            else:
                ops.gemm_bf16(x.cuda(), w.cuda(), out, 0, None, b.cuda(), None, int(ops.gemm_pick_splits(T, N, K_, 0)), st.tensor, False, 4)
            st.check()
            assert rel(f64(out), want) < tol


@pytest.mark.parametrize("T,H,N,K_", [(1, 3, 48, 16), (32, 16, 512, 128), (70, 5, 80, 144), (130, 2, 16, 528)])
def test_per_head_gemm(ops, T, H, N, K_):
    x, w = rnd(1, T, H * (K_ + 16), dtype=torch.bfloat16), rnd(2, H, N, K_, s=K_ ** -0.5, dtype=torch.bfloat16)
    want = np.einsum("hnk,thk->thn", f64(w), f64(x).reshape(T, H, K_ + 16)[..., :K_]).reshape(T, H * N)
    out = torch.zeros((T, H * N), dtype=torch.bfloat16, device="cuda")
    ops.head_gemm(x.cuda(), K_ + 16, w.cuda(), out, None, None, 0, False)
    assert rel(f64(out), want) < 5e-3
    # token tiles of long sequences are left out, tiles that a short one shares are not
    if T == 130:
        out.fill_(3.0)
        seq, cu = ints([0] * 129 + [1]), ints([0, 129, 130])
        ops.head_gemm(x.cuda(), K_ + 16, w.cuda(), out, seq, cu, 100, False)
        assert (out[:128] == 3).all() and rel(f64(out)[128:], want[128:]) < 5e-3


# ---------------------------------------------------------------------------- latent attention
class Latent:
    """Random latent attention over a ragged batch on shuffled pages: sequences of `lens` positions that bring their last
    `news` tokens.  Keys that stand out sit next to page borders, at the start, and on the diagonal."""

    def __init__(self, H, D, R, V, C, P, dt, lens, news, sink=True, seed=0):
        self.H, self.D, self.R, self.V, self.C, self.P, self.dt = H, D, R, V, C, P, dt
        self.lens, self.news, self.scale, self.base = lens, news, 0.15, 700.0
        self.uk, self.uv = rnd(1, H, D, C, s=C ** -0.5).to(dt), rnd(2, H, V, C, s=C ** -0.5).to(dt)
        self.sink = torch.linspace(-1.0, 4.0, H) if sink else None
        self.freq = torch.tensor([self.base ** (-2.0 * i / R) for i in range(R // 2)], dtype=torch.float64)
        g = torch.Generator().manual_seed(seed)
        per = [(n + P - 1) // P for n in lens]
        perm = torch.randperm(sum(per) + 2, generator=g).tolist()
        self.table = torch.full((len(lens), max(per)), -1, dtype=torch.int32)
        self.pages = torch.full((len(perm), 1, P, C + R), float("nan")).to(dt)       # unwritten rows must never matter
        self.q, self.want, at = [], [], 0
        for s, n in enumerate(lens):
            self.table[s, :per[s]] = torch.tensor(perm[at:at + per[s]], dtype=torch.int32)
            at += per[s]
            c, kr, q = rnd(10 + s, n, C).to(dt), rnd(20 + s, n, R).to(dt), rnd(30 + s, n, H, D + R).to(dt)
            for j in {0, P - 1, P, n // 2, n - 1} & set(range(n)):
                c[j] *= 3
            rot = torch.from_numpy(K.rotate(f64(kr), np.arange(n, dtype=float), self.base)).to(dt)
            for j in range(n):
                self.pages[self.table[s, j // P], 0, j % P] = torch.cat([c[j], rot[j]])
            keys, vals = np.einsum("hdc,jc->jhd", f64(self.uk), f64(c)), np.einsum("hvc,jc->jhv", f64(self.uv), f64(c))
            qr = K.rotate(f64(q)[..., D:], np.arange(n, dtype=float), self.base)
            sc = self.scale * (np.einsum("ihd,jhd->hij", f64(q)[..., :D], keys) + np.einsum("ihr,jr->hij", qr, f64(rot)))
            a = K.sink_softmax(K.causal(sc), f64(self.sink) if sink else np.full(H, -1e9))
            self.want.append(np.einsum("hij,jhv->ihv", a, vals).reshape(n, H * V)[n - news[s]:])
            self.q.append(q[n - news[s]:].reshape(news[s], -1))
        self.want = np.concatenate(self.want)
        self.q = torch.cat(self.q).cuda()
        self.T = self.q.shape[0]
        self.row = torch.cat([torch.full((m,), s, dtype=torch.int32) for s, m in enumerate(news)]).cuda()
        self.kv_len = torch.cat([torch.arange(n - m + 1, n + 1, dtype=torch.int32) for n, m in zip(lens, news)]).cuda()
        self.cu = ints(np.cumsum([0] + news).tolist())
        start, count, t = [], [], 0
        for m in news:
            for o in range(0, m, 64):
                start.append(t + o)
                count.append(min(64, m - o))
            t += m
        self.blocks = (ints(start), ints(count), max(count))
        self.table, self.pages, self.freq = self.table.cuda(), self.pages.cuda(), self.freq.cuda()
        self.sink = None if self.sink is None else self.sink.cuda()

    def absorb(self):
        q = self.q.float().cpu().reshape(self.T, self.H, self.D + self.R)[..., : self.D]
        return torch.einsum("hdc,thd->thc", self.uk.float(), q).reshape(self.T, -1).to(self.dt).cuda()

    def expand(self, o):
        return np.einsum("hvc,thc->thv", f64(self.uv), f64(o).reshape(self.T, self.H, self.C)).reshape(self.T, -1)


LATENT = [  # heads, dim, rot, vdim, rank, page
    (1, 16, 16, 16, 16, 8), (5, 32, 16, 48, 64, 16), (16, 128, 64, 128, 512, 64), (20, 48, 32, 64, 128, 64), (40, 16, 16, 32, 272, 32),
    (3, 64, 64, 160, 144, 16), (128, 32, 32, 32, 96, 64)]
RAGGED = ([130, 70, 5, 193, 67], [130, 2, 5, 65, 1])


@pytest.mark.parametrize("geo", LATENT)
@pytest.mark.parametrize("dt", DTYPES)
def test_latent_attention(ops, geo, dt):
    H, D, R, V, C, P = geo
    x = Latent(*geo, dt, *RAGGED)
    tol = 3e-6 if dt == torch.float32 else 2e-2
    out = torch.zeros((x.T, H * C), dtype=dt, device="cuda")
    args = (x.absorb(), x.q, x.pages, x.table, x.row, x.kv_len, H, R, x.scale, x.freq, x.sink)
    ops.latent_token_attention(*args, out, False)
    assert rel(x.expand(out), x.want) < tol
    if dt == torch.float32:
        return
    for split, n in ((193, 1), (64, 4), (32, 7)):
        out.zero_()
        po, ml = torch.empty(x.T * n * H * C, device="cuda"), torch.empty(x.T * n * H * 2, device="cuda")
        ops.latent_absorbed_attention(*args, out, *x.blocks, x.row, x.cu, 0, split, n, po, ml, False)
        assert rel(x.expand(out), x.want) < tol
    # long portions (at least 60 tokens) left out here ...
    out.fill_(9.0)
    ops.latent_absorbed_attention(*args, out, *x.blocks, x.row, x.cu, 60, 193, 1, None, None, False)
    short = torch.cat([torch.full((m,), m < 60) for m in RAGGED[1]]).numpy()
    assert rel(x.expand(out)[short], x.want[short]) < tol and (out[torch.from_numpy(~short).cuda()] == 9).all()
    # ... and attended in the expanded form
    base, seqs, total = [], [], 0
    for s, (n, m) in enumerate(zip(*RAGGED)):
        base.append([total if m >= 60 else -1, 0])
        if m >= 60:
            seqs.append([s, total, 0, n])
            total += n
    rows = torch.zeros((total, C + R), dtype=dt, device="cuda")
    ops.latent_gather(x.pages, x.table, ints(seqs), max(s[3] for s in seqs), rows, False)
    c = rows[:, :C].float().cpu()
    kv = torch.cat([torch.einsum("hdc,jc->jhd", x.uk.float(), c).reshape(total, -1), torch.einsum("hvc,jc->jhv", x.uv.float(), c).reshape(total, -1)], 1)
    wide = torch.full((x.T, H * V), 9.0, dtype=dt, device="cuda")
    ops.latent_expanded_attention(x.q, rows, kv.to(dt).cuda(), x.kv_len, H, C, R, x.scale, x.freq, x.sink, wide, *x.blocks, x.row, ints(base), False)
    assert rel(f64(wide)[~short], x.want[~short]) < tol and (wide[torch.from_numpy(short).cuda()] == 9).all()


@pytest.mark.parametrize("dt", DTYPES)
def test_decoding_with_and_without_a_sink(ops, dt):
    """One token of every sequence over hundreds of keys in many splits, first tokens included."""
    lens = [1, 2, 33, 300, 700]
    for sink in (False, True):
        x = Latent(7, 32, 16, 48, 112, 64, dt, lens, [1] * 5, sink=sink)
        out = torch.zeros((x.T, 7 * 112), dtype=dt, device="cuda")
        args = (x.absorb(), x.q, x.pages, x.table, x.row, x.kv_len, 7, 16, x.scale, x.freq, x.sink)
        ops.latent_token_attention(*args, out, False)
        assert rel(x.expand(out), x.want) < (3e-6 if dt == torch.float32 else 2e-2)
        if dt == torch.bfloat16:
            for split, n in ((704, 1), (128, 6), (32, 22)):
                po, ml = torch.empty(x.T * n * 7 * 112, device="cuda"), torch.empty(x.T * n * 7 * 2, device="cuda")
                ops.latent_absorbed_attention(*args, out, *x.blocks, x.row, x.cu, 0, split, n, po, ml, False)
                assert rel(x.expand(out), x.want) < 2e-2


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("Q,C,R", [(20, 36, 6), (96, 64, 32), (768, 512, 64)])
def test_latents_are_normed_rotated_and_appended(ops, dt, Q, C, R):
    """Positions in the tens of thousands keep exact angles; rows next to the appended ones are untouched."""
    T, P, eps, base, pad = 9, 16, 1e-3, 1e4, lambda n: (n + 15) // 16 * 16
    Qp, Cp, Rp = pad(Q), pad(C), pad(R)
    dq, dkv, kr = rnd(1, T, Q).to(dt), rnd(2, T, C).to(dt), rnd(3, T, R).to(dt)
    proj = torch.zeros((T, Qp + Cp + Rp), dtype=dt)
    proj[:, :Q], proj[:, Qp:Qp + C], proj[:, Qp + Cp:Qp + Cp + R] = dq, dkv, kr
    pos = [0, 1, 15, 16, 17, 1000, 40001, 40002, 65535]
    wq, wk = torch.zeros(Qp), torch.zeros(Cp)
    wq[:Q], wk[:C] = rnd(4, Q), rnd(5, C)
    table = torch.full((1, 65536 // P), -1, dtype=torch.int32)
    used = sorted({p // P for p in pos})
    for i, b in enumerate(used):
        table[0, b] = len(used) - 1 - i
    pages = torch.full((len(used), 1, P, Cp + Rp), 5.0, dtype=dt, device="cuda")
    lat = torch.zeros((T, Qp), dtype=dt, device="cuda")
    freq = torch.tensor([base ** (-2.0 * i / R) for i in range(R // 2)], dtype=torch.float64, device="cuda")
    ops.latent_prep(proj.cuda(), Q, C, R, wq.cuda(), wk.cuda(), eps, freq, ints([0] * T), ints(pos), table.cuda(), lat, pages, False)
    tol = 2e-6 if dt == torch.float32 else 5e-3
    assert rel(f64(lat)[:, :Q], K.rms(f64(dq), eps) * f64(wq)[:Q]) < tol and not lat[:, Q:].any()
    rows = torch.stack([pages[table[0, p // P], 0, p % P] for p in pos])
    assert rel(f64(rows)[:, :C], K.rms(f64(dkv), eps) * f64(wk)[:C]) < tol and not rows[:, C:Cp].any() and not rows[:, Cp + R:].any()
    assert rel(f64(rows)[:, Cp:Cp + R], K.rotate(f64(kr), np.array(pos, dtype=float), base)) < tol
    assert int((pages == 5).all(-1).sum()) == pages.shape[0] * P - T


# ---------------------------------------------------------------------------- gated memory
MEMORY = [(2, 16, 16), (3, 48, 80), (16, 128, 128), (1, 144, 272), (2, 256, 64), (5, 32, 24)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,V", MEMORY)
def test_gated_memory(ops, H, D, V, dt):
    """Ragged batch with states from before on shuffled slots: token kernel, chunked kernels, one token per sequence.  Channels
    forget between at once (gates that underflow) and almost never."""
    pad = lambda n: (n + 15) // 16 * 16
    Dp, Vp, eps = pad(D), pad(V), 1e-4
    lens, slots, n_slots = [130, 1, 64, 17, 200], [3, 0, 5, 1, 4], 6
    T = sum(lens)
    q, v = rnd(1, T, H, D).to(dt), rnd(2, T, H, V).to(dt)
    raw = rnd(3, T, H, D, s=2.0) + torch.linspace(-12, 9, D)
    raw[5] = -200.0                                      # everything forgotten at one token
    raw[77, :, ::3] = 200.0                              # nothing taken in
    lower = torch.rand(H, D, generator=torch.Generator().manual_seed(4)) * 0.9
    lower[:, : D // 2] = 0
    S0 = rnd(5, len(lens), H, D, V)
    norm = rnd(6, V)
    proj, gates = torch.zeros((T, H * (Dp + Vp)), dtype=dt), torch.zeros(T, H, Dp)
    proj[:, : H * Dp].view(T, H, Dp)[..., :D] = q
    proj[:, H * Dp:].view(T, H, Vp)[..., :V] = v
    gates[..., :D] = raw
    low = torch.ones(H, Dp)
    low[:, :D] = lower
    nw = torch.zeros(Vp)
    nw[:V] = norm
    f, k = K.forget_gate(f64(raw), f64(lower))
    want, end, t = [], [], 0
    for s, n in enumerate(lens):
        S, sl = f64(S0[s]), slice(t, t + n)
        o = np.empty((n, H, V))
        for i in range(n):
            S = f[t + i][:, :, None] * S + k[t + i][:, :, None] * f64(v[t + i])[:, None, :]
            o[i] = np.einsum("hdv,hd->hv", S, K.silu(f64(q[t + i])))
        want.append(K.rms(o, eps) * f64(norm))
        end.append(S)
        t += n
    want = np.concatenate(want)
    cu = ints(np.cumsum([0] + lens).tolist())

    def states():
        S = torch.full((n_slots, H, Dp, Vp), 7.0, device="cuda")
        for s, slot in enumerate(slots):
            S[slot] = 0
            S[slot, :, :D, :V] = S0[s].cuda()
        return S

    def check(S, out, tol, rows=slice(None), lens_=lens):
        got = f64(out).reshape(-1, H, Vp)
        assert rel(got[..., :V], want[rows]) < tol and not got[..., V:].any()
        assert (S[2] == 7).all()
    gd, pd = gates.reshape(T, -1).cuda(), proj.cuda()
    tol = 1e-5 if dt == torch.float32 else 1e-2
    for chunked in ((False, True) if dt == torch.bfloat16 else (False,)):
        S, out = states(), torch.zeros((T, H * Vp), dtype=dt, device="cuda")
        ws = None
        if chunked:
            if not ops.gated_chunked_supported(Dp, Vp):
                continue
            ws = torch.empty(int(ops.gated_chunked_workspace_bytes(T, len(lens), H, Dp, Vp)), dtype=torch.uint8, device="cuda")
        ops.gated_memory(pd, 0, H * Dp, gd, low.reshape(-1).cuda(), V, eps, nw.cuda(), cu, ints(slots), S, out, True, ws, False, False)
        check(S, out, tol)
        for s, slot in enumerate(slots):
            assert rel(f64(S[slot])[:, :D, :V], end[s]) < (1e-5 if not chunked else 5e-5)
            assert not S[slot, :, D:].any() and not S[slot, :, :, V:].any()
        # without writing the state
        S2 = states()
        ops.gated_memory(pd, 0, H * Dp, gd, low.reshape(-1).cuda(), V, eps, nw.cuda(), cu, ints(slots), S2, out, False, ws, False, False)
        assert torch.equal(S2, states())
    # first tokens as one-token steps
    first = [int(c) for c in cu[:-1].tolist()]
    S, out = states(), torch.zeros((len(lens), H * Vp), dtype=dt, device="cuda")
    ops.gated_memory(pd[first].contiguous(), 0, H * Dp, gd[first].contiguous(), low.reshape(-1).cuda(), V, eps, nw.cuda(), ints(list(range(len(lens) + 1))),
                     ints(slots), S, out, True, None, False, True)
    check(S, out, tol, rows=first)
