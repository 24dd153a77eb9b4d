"""The mechanisms of Badolix alone, through their public entry points, against the plain NumPy form:
capped scores, values inside the keys, rotated halves, latents, products per head, causal convolutions,
the selective state space, gates before norms, sigmoid routing within groups."""
import ctypes as C

import numpy as np
import pytest

from oracle import badolix_ref as R
from tests.test_gpu_biberax_mechanisms import Paged, back, prep
from tests.test_gpu_mechanisms import BS, dt, ints, put, rms_err, rounded

pytestmark = pytest.mark.gpu


# ---------------------------------------------------------------------------- attention
class Inside(Paged):
    """Values are the first VD channels of the keys: a pool of keys only."""

    def __init__(self, hb, q, k, VD, scale, dtype, **kw):
        super().__init__(hb, q, k[:, :, :VD], k, scale, dtype, **kw)
        self.a.v_cache = None


SHAPES = [  # n, heads, kv_heads, dim, vdim (inside the keys), window, keep_first, cap
    (140, 4, 2, 64, 64, 33, 5, 6.0),
    (131, 16, 1, 112, 96, 0, 0, 0.0),
    (97, 5, 1, 40, 24, 1, 0, 2.0),
    (150, 16, 1, 576, 512, 0, 0, 0.0),
    (120, 40, 1, 288, 256, 48, 17, 9.0),
    (100, 70, 1, 168, 136, 0, 0, 3.0),
    (90, 6, 2, 304, 264, 20, 3, 0.0),
    (110, 3, 1, 728, 640, 0, 0, 0.0),
    (75, 7, 1, 9, 5, 31, 4, 1.0),
]


@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_attention_over_values_inside_the_keys(hb, cuda, shape, dtype):
    n, H, G, D, VD, window, keep, cap = shape
    rng = np.random.default_rng(n + H)
    q, k = (rounded(rng.standard_normal(s), dtype) for s in ((n, H, D), (n, G, D)))
    scale = 3.0 * D ** -0.5
    want = R.capped_attention(q, k, k[:, :, :VD], scale, R.window_mask(n, window or None, keep), cap)
    p = Inside(hb, q, k, VD, scale, dtype, window=window, keep=keep)
    p.a.softcap = cap
    for form, got in p.forms():
        assert rms_err(got, want) < (4e-3 if dtype == "bf16" else 2e-6), form


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("cap", [0.5, 5.0, 30.0, 1e4])
def test_capped_scores(hb, cuda, cap, dtype):
    """Scores far beyond the cap, around it, and (the widest) where it hardly matters; with a bias and a
    sink behind the cap."""
    n, H, G, D, VD = 120, 6, 2, 32, 40
    rng = np.random.default_rng(int(cap))
    q, k, v = (rounded(s * rng.standard_normal(z), dtype) for s, z in ((6.0, (n, H, D)), (1.0, (n, G, D)), (1.0, (n, G, VD))))
    table, sink = rounded(rng.standard_normal((H, 20)), "f32"), rounded(rng.standard_normal(H), "f32")
    d = np.maximum(np.arange(n)[:, None] - np.arange(n)[None, :], 0)
    for extra in (False, True):
        p = Paged(hb, q, v, k, 0.4, dtype, window=50, keep=7, **(dict(sink=sink, bias=table) if extra else {}))
        p.a.softcap = cap
        want = np.zeros((n, H, VD))
        seen = R.window_mask(n, 50, 7)
        for h in range(H):
            s = cap * np.tanh(0.4 * (q[:, h] @ k[:, h // 3].T) / cap)
            if extra:
                s = s + table[h][np.minimum(d, 19)]
            e = np.where(seen, np.exp(s - s.max(axis=1, keepdims=True)), 0.0)
            den = e.sum(axis=1, keepdims=True) + (np.exp(sink[h] - s.max(axis=1, keepdims=True)) if extra else 0.0)
            want[:, h] = e / den @ v[:, h // 3]
        if not extra:
            np.testing.assert_allclose(want, R.capped_attention(q, k, v, 0.4, seen, cap), atol=1e-9)
        for form, got in p.forms():
            assert rms_err(got, want) < (4e-3 if dtype == "bf16" else (2e-6 if cap < 1e3 else 2e-5)), form


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("D,VD,window,keep", [(160, 144, 24, 6), (160, 144, 16, 16), (96, 64, 17, 1), (160, 144, 0, 0)])
def test_one_key_inside_or_outside_stands_out(hb, cuda, D, VD, window, keep, dtype):
    n, H = 130, 4
    rng = np.random.default_rng(5)
    base_q, base_k = (rounded(0.2 * rng.standard_normal(s), dtype) for s in ((n, H, D), (n, 1, D)))
    for at in (0, keep - 1, keep, keep + 1, 15, 16, 47, 48, 63, 64):
        if at < 0:
            continue
        q, k = base_q.copy(), base_k.copy()
        k[at] = 0.0
        k[at, :, D - 1] = 16.0  # a channel that is no value
        q[:, :, D - 1] = 4.0
        k[at, :, :VD] = rounded(30.0 + rng.standard_normal((1, VD)), dtype)
        q[:, :, :VD] = 0.0      # what is a value does not count in the score
        want = R.capped_attention(q, k, k[:, :, :VD], 0.5, R.window_mask(n, window or None, keep), 20.0)
        p = Inside(hb, q, k, VD, 0.5, dtype, window=window, keep=keep)
        p.a.softcap = 20.0
        for form, got in p.forms():
            per_pos = np.abs(got - want).max(axis=(1, 2))
            assert per_pos.max() < (0.2 if dtype == "bf16" else 1e-4), (form, at, int(per_pos.argmax()))


# ------------------------------------------------------------------- queries and keys
@pytest.mark.parametrize("H,G,D,VD,pairs", [(6, 2, 48, 40, 16), (3, 3, 10, 7, 3), (4, 1, 128, 64, 64), (5, 1, 9, 9, 4), (2, 2, 40, 8, 12)])
@pytest.mark.parametrize("biased", [False, True])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_rotated_halves_and_kv_write(hb, cuda, H, G, D, VD, pairs, biased, dtype):
    rng = np.random.default_rng(D)
    n, nb = 37, 6
    offs = (8, (8 + H * D + 7) // 8 * 8, (8 + H * D + 7) // 8 * 8 + (G * D + 7) // 8 * 8)
    p = rounded(rng.standard_normal((n, offs[2] + G * VD + 8 - (G * VD) % 8)), dtype)
    pos = rng.integers(0, 4000, n)
    slots = rng.permutation(nb * BS)[:n]
    slots[5] = -1
    freqs, gain = R.rotation(1e4, 2 * pairs, dict(factor=4.0, original=400, fast=20.0, slow=1.0))
    bq, bk = (rounded(rng.standard_normal(s * D), "f32") for s in (H, G))
    # `halves` and the gain ride along as fields of the argument block
    old = hb.AttentionPrepArgs

    class Halves(old):
        def __init__(self, *a):
            super().__init__(*a)
            self.halves, self.rotation_gain = 1, gain

    hb.AttentionPrepArgs = Halves
    try:
        rows, kc, vc, _ = prep(hb, dtype, p, offs, H, G, D, VD, pos, slots, nb, rotation=freqs,
                               **(dict(q_bias=bq, k_bias=bk) if biased else {}))
    finally:
        hb.AttentionPrepArgs = old
    limit = 4e-3 if dtype == "bf16" else 2e-6
    q = (p[:, offs[0]:offs[0] + H * D] + (bq if biased else 0.0)).reshape(n, H, D)
    k = (p[:, offs[1]:offs[1] + G * D] + (bk if biased else 0.0)).reshape(n, G, D)
    v = p[:, offs[2]:offs[2] + G * VD].reshape(n, G, VD)
    assert rms_err(rows[:, offs[0]:offs[0] + H * D].reshape(n, H, D), R.rotate_halves(q, pos, freqs, gain)) < limit
    held = slots >= 0
    assert rms_err(kc[slots[held]], R.rotate_halves(k, pos, freqs, gain)[held]) < limit
    assert np.array_equal(vc[slots[held]], v[held])
    free = np.setdiff1d(np.arange(nb * BS), slots)
    assert (kc[free] == 50.0).all() and (vc[free] == 50.0).all()          # nothing else was written
    assert np.array_equal(rows[:, :8], p[:, :8]) and np.array_equal(rows[:, offs[2]:], p[:, offs[2]:])


@pytest.mark.parametrize("halves", [0, 1])
def test_queries_without_keys(hb, cuda, halves):
    import torch

    rng = np.random.default_rng(1)
    p = rounded(rng.standard_normal((9, 64)), "bf16")
    t, pos, slots, f = put(p, "bf16"), ints(np.arange(9) * 7), ints(np.arange(9), np.int64), np.array([1.0, 0.3, 0.05, 0.01])
    tf = torch.from_numpy(f).cuda()
    a = hb.AttentionPrepArgs(t.data_ptr(), 64, 0, 0, 0, 3, 1, 16, 16, pos.data_ptr(), slots.data_ptr(), None, None, 1)
    a.rotation, a.pairs, a.halves = tf.data_ptr(), 4, halves
    hb.check(hb.lib.hb_attention_prepare(None, C.byref(a), 9, hb.BF16))
    torch.cuda.synchronize()
    q = p[:, :48].reshape(9, 3, 16)
    if halves:
        want = R.rotate_halves(q, np.arange(9) * 7, f)
    else:
        from oracle.biberax_ref import rotate_interleaved

        want = rotate_interleaved(q, np.arange(9) * 7, f)
    assert rms_err(back(t)[:, :48].reshape(9, 3, 16), want) < 4e-3
    assert np.array_equal(back(t)[:, 48:], p[:, 48:])


@pytest.mark.parametrize("H,D,RD,rank,pairs", [(4, 16, 8, 24, 4), (3, 9, 6, 11, 3), (16, 128, 64, 512, 32), (2, 8, 16, 8, 8),
                                               (1, 24, 16, 4096, 8), (5, 32, 32, 264, 8)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_latents_and_shared_keys(hb, cuda, H, D, RD, rank, pairs, dtype):
    import torch

    rng = np.random.default_rng(rank)
    n, nb, eps, KD = 21, 3, 1e-2, rank + RD
    off_q, off_c = 8, (8 + H * (D + RD) + 7) // 8 * 8
    p = rng.standard_normal((n, (off_c + KD + 7) // 8 * 8))
    p[3] *= 1e-3  # eps decides here
    p = rounded(p, dtype)
    pos, slots = rng.integers(0, 5000, n), rng.permutation(nb * BS)[:n]
    slots[4] = -1
    norm = rounded(1 + 0.3 * rng.standard_normal(rank), "f32")
    freqs, gain = R.rotation(1e3, 2 * pairs, dict(factor=8.0, original=64, fast=9.0, slow=1.0))
    t, tn, tf = put(p, dtype), put(norm), torch.from_numpy(np.ascontiguousarray(freqs)).cuda()
    q, kc = put(np.full((n, H * KD), 50.0), dtype), put(np.full((nb * BS, KD), 50.0), dtype)
    tp, ts = ints(pos), ints(slots, np.int64)
    a = hb.LatentPrepArgs(t.data_ptr(), p.shape[1], off_q, off_c, H, D, RD, rank, q.data_ptr(), H * KD, tp.data_ptr(), ts.data_ptr(),
                          kc.data_ptr(), nb, tn.data_ptr(), eps, tf.data_ptr(), pairs, gain)
    hb.check(hb.lib.hb_latent_prepare(None, C.byref(a), n, dt(hb, dtype)))
    torch.cuda.synchronize()
    limit = 4e-3 if dtype == "bf16" else 2e-6
    got, rows = back(kc), back(t)
    held = slots >= 0
    assert rms_err(got[slots[held], :rank], R.rms_norm(p[:, off_c:off_c + rank], norm, eps)[held]) < limit
    key = R.rotate_halves(p[:, None, off_c + rank:off_c + KD], pos, freqs, gain)[:, 0]
    assert rms_err(got[slots[held], rank:], key[held]) < limit
    assert (got[np.setdiff1d(np.arange(nb * BS), slots)] == 50.0).all()
    qh = p[:, off_q:off_q + H * (D + RD)].reshape(n, H, D + RD)
    want = R.rotate_halves(qh[:, :, D:], pos, freqs, gain)
    wide = back(q).reshape(n, H, KD)
    assert rms_err(wide[:, :, rank:], want) < limit and (wide[:, :, :rank] == 50.0).all()
    placed = rows[:, off_q:off_q + H * (D + RD)].reshape(n, H, D + RD)
    assert rms_err(placed[:, :, D:], want) < limit and np.array_equal(placed[:, :, :D], qh[:, :, :D])
    assert np.array_equal(rows[:, off_c:], p[:, off_c:])


@pytest.mark.parametrize("M,N,K,heads,gap", [(1, 512, 128, 16, 0), (37, 96, 32, 4, 8), (130, 128, 512, 5, 64), (300, 40, 24, 3, 16),
                                             (9, 11, 7, 4, 3), (64, 264, 520, 2, 8), (700, 64, 64, 70, 0)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_products_per_head(hb, cuda, M, N, K, heads, gap, dtype):
    import torch

    rng = np.random.default_rng(M + N)
    x = rounded(rng.standard_normal((M, heads, K + gap)), dtype)
    w = rounded(rng.standard_normal((heads, N, K)) * K ** -0.5, dtype)
    tx, tw, ty = put(x.reshape(M, -1), dtype), put(w, dtype), put(np.full((M, heads * (N + gap)), 50.0), dtype)
    hb.check(hb.lib.hb_gemm_heads(None, ty.data_ptr(), tx.data_ptr(), tw.data_ptr(), M, N, K, heads, heads * (K + gap), K + gap,
                                  heads * (N + gap), N + gap, dt(hb, dtype)))
    torch.cuda.synchronize()
    got = back(ty).reshape(M, heads, N + gap)
    assert rms_err(got[:, :, :N], np.einsum("mhk,hnk->mhn", x[:, :, :K], w)) < (4e-3 if dtype == "bf16" else 2e-6)
    assert (got[:, :, N:] == 50.0).all()  # what lies between the heads' results stays


# ------------------------------------------------------------------------- convolutions
class Conv:
    def __init__(self, hb, channels, taps, n, dtype, slots=3, seed=0):
        rng = np.random.default_rng(seed + channels)
        self.hb, self.dtype, self.channels, self.taps, self.n = hb, dtype, channels, taps, n
        self.off, ld = 8, (channels + 16) // 8 * 8 + 8
        self.p = rounded(rng.standard_normal((n, ld)), dtype)
        self.w, self.b = rounded(rng.standard_normal((channels, taps)), "f32"), rounded(rng.standard_normal(channels), "f32")
        ld_out = (channels + 7) // 8 * 8
        self.dev = [put(self.p, dtype), put(self.w.T), put(self.b), put(np.zeros((n, ld_out)), dtype),
                    put(np.full((slots, max(1, taps - 1), channels), 9.0), dtype)]  # stale: never read at position 0
        d = [t.data_ptr() for t in self.dev]
        self.a = hb.ShortConvArgs(d[0], ld, self.off, channels, taps, d[1], d[2], d[3], ld_out, d[4], None)

    def expected(self, lo, hi):
        return R.silu(R.causal_conv(self.p[lo:hi, self.off:self.off + self.channels], self.w, self.b))

    def run(self, segs):
        """segs: (first row, rows, first position, slot)."""
        import torch

        s = ints(segs)
        self.a.segments = s.data_ptr()
        short = [i for i, g in enumerate(segs) if g[1] <= 8]
        chunks = [(i, g[0] + c, min(64, g[1] - c), c // 64) for i, g in enumerate(segs) if g[1] > 8 for c in range(0, g[1], 64)]
        lst, ch = ints(short or [0]), ints(chunks or [(0, 0, 0, 0)])
        self.hb.check(self.hb.lib.hb_short_conv(None, C.byref(self.a), lst.data_ptr(), len(short), ch.data_ptr(), len(chunks),
                                                dt(self.hb, self.dtype)))
        torch.cuda.synchronize()
        return back(self.dev[3])[:, :self.channels], back(self.dev[4])


@pytest.mark.parametrize("channels,taps", [(96, 4), (40, 3), (333, 2), (7, 4), (64, 1), (48, 7), (19, 9), (520, 33), (24, 65), (2500, 4)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_convolutions_meet_in_the_state(hb, cuda, channels, taps, dtype):
    """One sequence in portions cut anywhere (down to one token) beside another in another slot."""
    c = Conv(hb, channels, taps, 260, dtype)
    want = np.concatenate([c.expected(0, 200), c.expected(200, 260)])
    limit = 4e-3 if dtype == "bf16" else 2e-6
    at = 0
    for n in (2, 1, 9, 70, 1, 64, 3, 50):
        segs = [(at, n, at, 1)] + ([(200, 60, 0, 2)] if at == 2 else [])
        out, state = c.run(segs)
        assert rms_err(out[at:at + n], want[at:at + n]) < limit, (at, n)
        at += n
    assert at == 200 and rms_err(out[200:], want[200:]) < limit
    if taps > 1:
        held = c.p[:, c.off:c.off + channels]
        assert np.array_equal(state[1], held[max(0, 201 - taps):200]) or taps > 200
        tail = held[200:][-(taps - 1):] if taps <= 61 else np.concatenate([np.zeros((taps - 61, channels)), held[200:]])
        assert np.array_equal(state[2], tail) and (state[0] == 9.0).all()


def test_a_single_input_is_felt_for_exactly_its_taps(hb, cuda):
    for at in (0, 1, 63, 64, 65, 7, 8):
        c = Conv(hb, 16, 5, 130, "bf16")
        c.p[:, c.off:c.off + 16] = 0.0
        c.p[at, c.off:c.off + 16] = 8.0
        c.w[:], c.b[:] = 1.0 + np.arange(5), 0.0
        for t, a, kind in zip(c.dev, (c.p, c.w.T, c.b), ("bf16", "f32", "f32")):
            t.copy_(put(a, kind))
        for segs in ([(0, 130, 0, 0)], None):
            if segs:
                out, _ = c.run(segs)
            else:
                pos = 0
                for n in (60, 3, 2, 1, 64):
                    out, _ = c.run([(pos, n, pos, 1)])
                    pos += n
            felt = np.flatnonzero(np.abs(out).max(axis=1))
            assert felt.tolist() == [t for t in range(at, at + 5) if t < 130], (at, felt)
            np.testing.assert_allclose(out[at, 0], 40.0, rtol=1e-2)  # the last weight meets the token itself


# ------------------------------------------------------------------------- state space
class Space:
    """Rows [v | k | q | dt] with gaps, groups of k and q, and the recurrence over them."""

    def __init__(self, hb, heads, groups, state, vdim, n, dtype, seed=0, bias=None, a_log=None, slots=3):
        import torch

        rng = np.random.default_rng(seed + heads * state)
        self.hb, self.dtype, self.n, self.heads, self.groups, self.N, self.V = hb, dtype, n, heads, groups, state, vdim
        widths = [heads * vdim, groups * state, groups * state, heads]
        offs, at = [], 8
        for w in widths:
            offs.append(at)
            at = (at + w + 7) // 8 * 8 + 8
        self.p = rounded(rng.standard_normal((n, at)), dtype)
        self.x, self.B, self.C, self.raw = (self.p[:, o:o + w] for o, w in zip(offs, widths))
        self.bias = rounded(rng.standard_normal(heads) - 1.0 if bias is None else np.full(heads, bias), "f32")
        self.a_log = rounded(rng.standard_normal(heads) if a_log is None else np.full(heads, a_log), "f32")
        self.skip = rounded(rng.standard_normal(heads), "f32")
        self.dev = [put(self.p, dtype), put(self.bias), put(self.a_log), put(self.skip)]
        self.state = torch.full((slots, heads, state, vdim), 7.0, device="cuda")  # stale: never read at position 0
        self.o = torch.zeros((n, heads * vdim), device="cuda")
        d = [t.data_ptr() for t in self.dev]
        self.a = hb.LinearRecurrenceArgs(d[0], at, offs[2], offs[1], offs[0], 0, heads, state, vdim, 1.0, 0, None, None, None, 0, 1.0,
                                         self.state.data_ptr(), self.o.data_ptr(), heads * vdim, None, d[0] + offs[3] * self.dev[0].element_size(),
                                         at, d[1], d[2], d[3], groups)

    def expected(self, lo=0, hi=None):
        hi = self.n if hi is None else hi
        n, H = hi - lo, self.heads
        per = H // self.groups
        B, Cq = (np.repeat(z[lo:hi].reshape(n, self.groups, self.N), per, axis=1) for z in (self.B, self.C))
        y, s = R.state_space(self.x[lo:hi].reshape(n, H, self.V), B, Cq, R.softplus(self.raw[lo:hi] + self.bias), self.a_log, self.skip)
        return y.reshape(n, -1), s

    def run(self, segs, chunked):
        import torch

        s = ints(segs)
        self.a.segments = s.data_ptr()
        tokens = [i for i in range(len(segs)) if not chunked[i]]
        chunks, longs = [], []
        for i, (r0, n, _, _) in enumerate(segs):
            if chunked[i]:
                longs.append([i, len(chunks), 0, 0])
                for c in range(0, n, 64):
                    chunks.append((i, r0 + c, min(64, n - c), c // 64))
                    longs[-1][2] += 1
        lst, ch, lg = ints(tokens or [0]), ints(chunks or [(0, 0, 0, 0)]), ints(longs or [(0, 0, 0, 0)])
        cum = torch.zeros((self.n, 2 * self.heads), device="cuda")
        cs = torch.zeros((max(1, len(chunks)), self.heads, self.N, self.V), device="cuda")
        self.hb.check(self.hb.lib.hb_linear_recurrence(None, C.byref(self.a), lst.data_ptr(), len(tokens), ch.data_ptr(), len(chunks),
                                                       lg.data_ptr(), len(longs), cum.data_ptr(), cs.data_ptr(), dt(self.hb, self.dtype)))
        torch.cuda.synchronize()
        return self.o.cpu().numpy().astype(np.float64), self.state.cpu().numpy().astype(np.float64)


@pytest.mark.parametrize("heads,groups,state,vdim", [(4, 2, 32, 64), (3, 1, 16, 24), (6, 6, 128, 64), (2, 1, 40, 72), (4, 2, 12, 20),
                                                     (1, 1, 7, 9), (8, 2, 200, 136), (40, 8, 16, 8), (5, 5, 1, 1)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_state_space(hb, cuda, heads, groups, state, vdim, dtype):
    r = Space(hb, heads, groups, state, vdim, 150, dtype)
    want, last = r.expected()
    o, s = r.run([(0, 150, 0, 1)], [False])
    assert rms_err(o, want) < 3e-6 and rms_err(s[1], last) < 3e-6
    if dtype == "bf16":
        assert hb.lib.hb_linear_recurrence_chunked(C.byref(r.a), hb.BF16) == 1
        o, s = r.run([(0, 150, 0, 2)], [True])
        assert rms_err(o, want) < 6e-5 and rms_err(s[2], last) < 6e-5
        assert np.all(s[0] == 7.0)  # other slots stay as they are


def test_state_space_portions_meet_in_the_state(hb, cuda):
    r = Space(hb, 4, 2, 48, 40, 200, "bf16")
    want_a, state_a = r.expected(0, 140)
    want_b, state_b = r.expected(140, 200)
    at = 0
    for n, chunk in ((2, False), (65, True), (1, False), (9, True), (63, True)):
        segs = [(at, n, at, 0)] + ([(140, 60, 0, 2)] if at == 2 else [])
        o, s = r.run(segs, [chunk, True][:len(segs)])
        assert rms_err(o[at:at + n], want_a[at:at + n]) < 1e-4, (at, n)
        at += n
    assert at == 140 and rms_err(s[0], state_a) < 1e-4
    assert rms_err(o[140:], want_b) < 1e-4 and rms_err(s[2], state_b) < 1e-4


@pytest.mark.parametrize("bias,a_log", [(-30.0, 0.0), (30.0, 3.0), (-3.0, -6.0), (8.0, 8.0), (0.0, -20.0)])
def test_state_space_at_the_ends_of_steps_and_decays(hb, cuda, bias, a_log):
    """Steps of nothing, huge steps that forget at once, decays next to one."""
    r = Space(hb, 2, 1, 32, 32, 130, "bf16", bias=bias, a_log=a_log)
    want, last = r.expected()
    for chunked in (False, True):
        o, s = r.run([(0, 130, 0, 0)], [chunked])
        assert np.isfinite(o).all() and rms_err(o, want) < 2e-4 and rms_err(s[0], last) < 2e-4


def test_state_space_remembers_a_far_token(hb, cuda):
    """A value written once and asked for hundreds of tokens later, with nothing else in its channel."""
    n = 520
    r = Space(hb, 2, 1, 32, 32, n, "bf16", bias=-5.0, a_log=-2.0)
    r.p[:] = rounded(0.01 * r.p, "bf16")
    r.B[:, 3] = 0.0
    r.B[1, :], r.B[1, 3] = 0.0, 4.0
    r.raw[1, :] = 9.0
    r.x[1, :] = rounded(np.linspace(-8, 8, 64), "bf16")
    r.C[:, :], r.C[:, 3] = 0.0, 2.0
    r.dev[0].copy_(put(r.p, "bf16"))
    want, _ = r.expected()
    for chunked in (False, True):
        o, _ = r.run([(0, n, 0, 0)], [chunked])
        assert np.abs(o[-1] - want[-1]).max() < 1e-3 * np.abs(want[-1]).max()
        assert np.abs(want[-1]).max() > 10.0


# ------------------------------------------------------------------------- norms, routing
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("groups,size", [(5, 24), (1, 200), (1, 33), (2, 1500), (12, 128)])
@pytest.mark.parametrize("silu", [0, 1])
def test_gates_before_the_norm(hb, cuda, dtype, groups, size, silu):
    import torch

    n, width, eps = 7, groups * size, 1e-3
    rng = np.random.default_rng(groups * size)
    o, g, w = rng.standard_normal((n, width)), rounded(2 * rng.standard_normal((n, width + 3)), dtype), rng.standard_normal(width)
    o[2] *= 1e-3  # eps decides here
    out = put(np.zeros((n, width + 5)), dtype)
    do, dg, dw = put(o), put(g, dtype), put(w)
    hb.check(hb.lib.hb_gated_group_norm(None, out.data_ptr(), width + 5, do.data_ptr(), width, dg.data_ptr(), width + 3,
                                        dw.data_ptr(), n, groups, size, 2 + silu, eps, dt(hb, dtype)))
    torch.cuda.synchronize()
    z = g[:, :width]
    if silu:
        want = R.gated_norm(o, z, w, groups, eps)
    else:
        y = (o * R.sigmoid(z)).reshape(n, groups, size)
        want = R.rms_norm(y, 1.0, eps).reshape(n, width) * w
    assert rms_err(back(out)[:, :width], want) < (4e-3 if dtype == "bf16" else 2e-6)


@pytest.mark.parametrize("experts,top,groups,keep", [(16, 3, 2, 1), (12, 4, 4, 3), (6, 2, 6, 2), (40, 6, 8, 3), (9, 9, 3, 3), (64, 8, 1, 1),
                                                     (70, 5, 35, 4), (256, 8, 8, 4)])
@pytest.mark.parametrize("rows", [3, 400])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_sigmoid_routing_within_groups(hb, cuda, experts, top, groups, keep, rows, dtype):
    import torch

    rng = np.random.default_rng(experts + rows)
    width, m_pad = 72, 16
    h, router = rounded(rng.standard_normal((rows, width)), dtype), rounded(rng.standard_normal((experts, width)) * 0.3, dtype)
    tiles = min(experts, rows * top) + rows * top // m_pad
    i32 = lambda *s: torch.zeros(s, device="cuda", dtype=torch.int32)
    t = [i32(rows, top), i32(rows, top), i32(rows, top), torch.zeros((rows, top), device="cuda"), i32(experts + 1), i32(experts), i32(tiles)]
    r = hb.MoeRouting(experts, top, m_pad, tiles, *(x.data_ptr() for x in t), 0, 1, groups, keep)
    th, tr = put(h, dtype), put(router, dtype)
    hb.check(hb.lib.hb_moe_route_top(None, C.byref(r), th.data_ptr(), width, tr.data_ptr(), None, rows, width, dt(hb, dtype)))
    torch.cuda.synchronize()
    spec = dict(count=groups, keep=keep)
    chosen, weight = R.route(h, router, top, spec)
    clear = R.route_margin(h, router, top, spec) > 1e-4
    assert clear.mean() > 0.9
    ids, got = t[0].cpu().numpy(), back(t[3])
    assert np.array_equal(np.sort(ids[clear]), np.sort(chosen[clear]))
    same = (ids == chosen).all(axis=1)
    assert same.mean() > 0.9
    np.testing.assert_allclose(got[same], weight[same], rtol=2e-5)
    if keep < groups:
        assert all(len(set(row // (experts // groups))) <= keep for row in ids)


def test_routing_refusals(hb, cuda):
    import torch

    z, one = torch.zeros((3, 64), device="cuda"), torch.zeros((12, 64), device="cuda")
    i32 = lambda *s: torch.zeros(s, device="cuda", dtype=torch.int32)
    t = [i32(3, 4), i32(3, 4), i32(3, 4), torch.zeros((3, 4), device="cuda"), i32(13), i32(12), i32(20)]
    for groups, keep in ((5, 1), (4, 5), (4, 1)):
        r = hb.MoeRouting(12, 4, 16, 20, *(x.data_ptr() for x in t), 0, 1, groups, keep)
        with pytest.raises(hb.HbError, match="groups"):
            hb.check(hb.lib.hb_moe_route_top(None, C.byref(r), z.data_ptr(), 64, one.data_ptr(), None, 3, 64, hb.F32))
