"""Each mechanism of the layered models alone, against its plain NumPy form: attention over a
window and the first kept positions, linear recurrences (token by token and in chunks), residual
streams, gated norms.  Limits are relative to the root mean square of the expected values."""
import ctypes as C

import numpy as np
import pytest

from oracle import latarax_ref as R
from oracle.kernels_ref import round_bf16

pytestmark = pytest.mark.gpu
BS = 16


def rms_err(got, want):
    return float(np.sqrt(np.mean((got - want) ** 2)) / (np.sqrt(np.mean(want ** 2)) + 1e-30))


def dt(hb, name):
    return hb.F32 if name == "f32" else hb.BF16


def put(a, dtype="f32"):
    import torch

    t = torch.from_numpy(np.ascontiguousarray(a, dtype=np.float32)).cuda()
    return t.to(torch.bfloat16) if dtype == "bf16" else t


def ints(a, kind=np.int32):
    import torch

    return torch.from_numpy(np.ascontiguousarray(a, dtype=kind)).cuda()


def rounded(a, dtype):
    return round_bf16(a.astype(np.float32)).astype(np.float64) if dtype == "bf16" else a.astype(np.float32).astype(np.float64)


# ---------------------------------------------------------------------------- attention
class Paged:
    """One sequence's K/V spread over a shuffled block table of a larger pool full of junk."""

    def __init__(self, hb, q, k, v, scale, window, keep, dtype, seed=0):
        import torch

        self.hb, self.dtype = hb, dtype
        n, H, D = q.shape
        G, VD = k.shape[1], v.shape[2]
        nb = -(-n // BS)
        self.n, self.H, self.VD = n, H, VD
        table = np.random.default_rng(seed).permutation(nb + 7)[:nb]
        es = torch.bfloat16 if dtype == "bf16" else torch.float32
        self.kc = torch.full((nb + 7, G, BS, D), 50.0, device="cuda", dtype=es)
        self.vc = torch.full((nb + 7, G, BS, VD), 50.0, device="cuda", dtype=es)
        kv = put(np.concatenate([k.reshape(n, -1), v.reshape(n, -1)], 1), dtype)
        self.q = put(q.reshape(n, -1), dtype)
        self.out = torch.zeros((n, H * VD), device="cuda", dtype=es)
        self.pos, self.seg, self.table = ints(np.arange(n)), ints(np.zeros(n)), ints(table)
        slots = ints(table[np.arange(n) // BS] * BS + np.arange(n) % BS, np.int64)
        self.a = hb.SpanAttentionArgs(self.q.data_ptr(), H * D, self.out.data_ptr(), H * VD, self.kc.data_ptr(),
                                      self.vc.data_ptr(), self.table.data_ptr(), nb, nb + 7, self.seg.data_ptr(),
                                      self.pos.data_ptr(), H, G, D, VD, window, keep, scale)
        hb.check(hb.lib.hb_span_kv_write(None, C.byref(self.a), kv.data_ptr(), kv.data_ptr() + G * D * kv.element_size(),
                                         G * (D + VD), slots.data_ptr(), n, dt(hb, dtype)))
        self.keep_alive = (kv, slots)

    def run(self, tiles=None, rows=None, splits=1):
        import torch

        t = ints(tiles) if tiles is not None else None
        r = ints(rows) if rows is not None else None
        ws = torch.zeros(max(1, (len(rows) if rows is not None else 0) * self.H * splits * (self.VD + 2)), device="cuda")
        self.hb.check(self.hb.lib.hb_span_attention(None, C.byref(self.a), t.data_ptr() if t is not None else None,
                                                    len(tiles) if tiles is not None else 0,
                                                    r.data_ptr() if r is not None else None,
                                                    len(rows) if rows is not None else 0, splits, ws.data_ptr(),
                                                    dt(self.hb, self.dtype)))
        torch.cuda.synchronize()
        return self.out.float().cpu().numpy().reshape(self.n, self.H, self.VD)


ATTN = [  # n, heads, kv_heads, dim, vdim, window, keep_first
    (150, 4, 2, 64, 64, 33, 5),
    (131, 6, 1, 40, 72, 48, 16),
    (97, 2, 2, 16, 8, 1, 0),
    (90, 3, 3, 104, 320, 0, 0),
    (200, 16, 1, 128, 128, 64, 1),
    (70, 5, 1, 24, 136, 17, 40),
    (65, 20, 1, 32, 32, 20, 3),
    (80, 4, 4, 12, 20, 31, 4),
    (130, 1, 1, 256, 256, 100, 7),
]


@pytest.mark.parametrize("shape", ATTN, ids=str)
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_span_attention(hb, cuda, shape, dtype):
    n, H, G, D, VD, window, keep = shape
    rng = np.random.default_rng(n)
    q, k, v = (rounded(rng.standard_normal(s), dtype) for s in ((n, H, D), (n, G, D), (n, G, VD)))
    scale = 0.37
    want = R.attention(q, k, v, scale, R.window_mask(n, window or None, keep))
    p = Paged(hb, q, k, v, scale, window, keep, dtype)
    limit = 4e-3 if dtype == "bf16" else 2e-6
    assert rms_err(p.run(rows=np.arange(n)), want) < limit
    for splits in (2, 5):
        p.out.zero_()
        assert rms_err(p.run(rows=np.arange(n), splits=splits), want) < limit
    tp = hb.check(hb.lib.hb_span_attention_tile_positions(C.byref(p.a), dt(hb, dtype)))
    assert tp == (64 // (H // G) if dtype == "bf16" and D % 8 == 0 and VD % 8 == 0 else 0)
    if tp:
        for size in {tp, max(1, tp // 2 - 1), 2}:
            tiles = [(0, i, min(size, n - i), 0) for i in range(0, n, size)] if size <= tp else []
            if tiles:
                p.out.zero_()
                assert rms_err(p.run(tiles=tiles), want) < limit, size


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("window,keep", [(24, 6), (16, 16), (17, 1), (40, 0), (0, 0)])
def test_span_attention_edges_stand_out(hb, cuda, window, keep, dtype):
    """One key at a time points at the query so strongly that seeing it or not decides the output:
    just inside and just outside the window, the last kept token and the one after it, block edges."""
    n, H, G, D, VD = 120, 4, 2, 32, 40
    rng = np.random.default_rng(5)
    base_q, base_k, v = (rounded(0.2 * rng.standard_normal(s), dtype) for s in ((n, H, D), (n, G, D), (n, G, VD)))
    for at in (0, keep - 1, keep, keep + 1, 15, 16, 47, 48, 63, 64):
        if at < 0:
            continue
        q, k = base_q.copy(), base_k.copy()
        k[at] = 0.0
        k[at, :, 0] = 16.0
        q[:, :, 0] = 4.0
        v2 = v.copy()
        v2[at] = rounded(30.0 + rng.standard_normal((G, VD)), dtype)
        want = R.attention(q, k, v2, 0.5, R.window_mask(n, window or None, keep))
        p = Paged(hb, q, k, v2, 0.5, window, keep, dtype)
        got = {"rows": p.run(rows=np.arange(n))}
        tp = hb.lib.hb_span_attention_tile_positions(C.byref(p.a), dt(hb, dtype))
        if tp:
            got["tiles"] = p.run(tiles=[(0, i, min(tp, n - i), 0) for i in range(0, n, tp)])
        for form, g in got.items():
            per_pos = np.abs(g - want).max(axis=(1, 2))
            assert per_pos.max() < (0.2 if dtype == "bf16" else 1e-4), (form, at, int(per_pos.argmax()))


# --------------------------------------------------------------------------- recurrences
class Rec:
    """Projection rows [q | k | v | a1] (with gaps between them) and the recurrence over them."""

    def __init__(self, hb, heads, dim, vdim, n, *, low_rank, dtype, seed=0, q_scale=1.0, silu=False, tau=1.0, rank=5,
                 decay=None, bias=None, slots=3):
        import torch

        rng = np.random.default_rng(seed)
        self.hb, self.dtype, self.n, self.heads, self.dim, self.vdim = hb, dtype, n, heads, dim, vdim
        self.low_rank, self.q_scale, self.silu, self.tau = low_rank, q_scale, silu, tau
        widths = [heads * dim, heads * dim, heads * vdim, rank]
        offs, at = [], 8
        for w in widths:
            offs.append(at)
            at = (at + w + 7) // 8 * 8 + 8
        self.p = rounded(rng.standard_normal((n, at)), dtype)
        self.q, self.k, self.v, self.t = (self.p[:, o:o + w] for o, w in zip(offs, widths))
        self.a2 = rounded(rng.standard_normal((heads * dim, rank)) * 0.7, "f32")
        self.bias = rounded(rng.standard_normal(heads * dim) * 2 + 1 if bias is None else np.full(heads * dim, bias), "f32")
        self.decay = np.asarray(decay if decay is not None else rng.uniform(0.3, 1.0, heads))
        self.dev = [put(self.p, dtype), put(self.a2), put(self.bias), put(self.decay)]
        self.state = torch.full((slots, heads, dim, vdim), 7.0, device="cuda")  # stale: never read at position 0
        self.o = torch.zeros((n, heads * vdim), device="cuda")
        d = [t.data_ptr() for t in self.dev]
        self.a = hb.LinearRecurrenceArgs(d[0], at, *offs, heads, dim, vdim, q_scale, int(silu), None if low_rank else d[3],
                                         d[1], d[2], rank, tau, self.state.data_ptr(), self.o.data_ptr(), heads * vdim, None)

    def expected(self, lo=0, hi=None):
        hi = self.n if hi is None else hi
        act = R.silu if self.silu else (lambda z: z)
        n, H = hi - lo, self.heads
        q = act(self.q[lo:hi]).reshape(n, H, self.dim) * self.q_scale
        k, v = act(self.k[lo:hi]).reshape(n, H, self.dim), act(self.v[lo:hi]).reshape(n, H, self.vdim)
        if self.low_rank:
            a = (R.sigmoid(self.t[lo:hi] @ self.a2.T + self.bias) ** (1.0 / self.tau)).reshape(n, H, self.dim)
        else:
            a = np.broadcast_to(self.decay[None, :, None], (n, H, self.dim))
        o, s = R.decayed_recurrence(q, k, v, a)
        return o.reshape(n, -1), s

    def run(self, segs, chunked):
        """segs: (first row, rows, first position, slot); chunked: which of them go in chunks."""
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
        cum = torch.zeros((self.n, self.heads * self.dim), device="cuda")
        cs = torch.zeros((max(1, len(chunks)), self.heads, self.dim, self.vdim), device="cuda")
        self.hb.check(self.hb.lib.hb_linear_recurrence(None, C.byref(self.a), lst.data_ptr(), len(tokens), ch.data_ptr(),
                                                       len(chunks), lg.data_ptr(), len(longs), cum.data_ptr(), cs.data_ptr(),
                                                       dt(self.hb, self.dtype)))
        torch.cuda.synchronize()
        return self.o.cpu().numpy().astype(np.float64), self.state.cpu().numpy().astype(np.float64)


REC = [  # heads, dim, vdim, rank
    (2, 32, 64, 16), (3, 16, 24, 5), (1, 128, 128, 16), (2, 40, 72, 1), (2, 12, 20, 3), (1, 7, 9, 2), (2, 200, 136, 16), (1, 64, 300, 8),
]


@pytest.mark.parametrize("shape", REC, ids=str)
@pytest.mark.parametrize("low_rank,silu,scale,tau", [(True, False, 0.25, 4.0), (True, False, 1.0, 1.0), (False, True, 1.0, 1.0)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_recurrence(hb, cuda, shape, low_rank, silu, scale, tau, dtype):
    heads, dim, vdim, rank = shape
    r = Rec(hb, heads, dim, vdim, 150, low_rank=low_rank, dtype=dtype, q_scale=scale, silu=silu, tau=tau, rank=rank)
    want, state = r.expected()
    o, s = r.run([(0, 150, 0, 1)], [False])
    assert rms_err(o, want) < 3e-6 and rms_err(s[1], state) < 3e-6
    if dtype == "bf16":
        assert hb.lib.hb_linear_recurrence_chunked(C.byref(r.a), hb.BF16) == 1
        o, s = r.run([(0, 150, 0, 2)], [True])
        assert rms_err(o, want) < 6e-5 and rms_err(s[2], state) < 6e-5
        assert np.all(s[0] == 7.0)  # other slots stay as they are


@pytest.mark.parametrize("low_rank", [True, False])
def test_recurrence_portions_meet_in_the_state(hb, cuda, low_rank):
    """Token runs and chunk runs of one sequence, cut anywhere, beside another sequence."""
    r = Rec(hb, 2, 48, 40, 200, low_rank=low_rank, dtype="bf16", tau=2.0)
    want_a, state_a = r.expected(0, 140)
    want_b, state_b = r.expected(140, 200)
    at = 0
    for n, chunk in ((2, False), (65, True), (1, False), (9, True), (63, True)):
        segs = [(at, n, at, 0)]
        if at == 2:
            segs.append((140, 60, 0, 2))
        o, s = r.run(segs, [chunk, True][:len(segs)])
        assert rms_err(o[at:at + n], want_a[at:at + n]) < 1e-4, (at, n)
        at += n
    assert at == 140 and rms_err(s[0], state_a) < 1e-4
    assert rms_err(o[140:], want_b) < 1e-4 and rms_err(s[2], state_b) < 1e-4


@pytest.mark.parametrize("bias", [-30.0, -6.0, 12.0])
def test_recurrence_extreme_low_rank_decays(hb, cuda, bias):
    """Decays near 0 and near 1 at tau 1: no exponent of the chunked form may overflow."""
    r = Rec(hb, 2, 32, 32, 130, low_rank=True, dtype="bf16", tau=1.0, bias=bias)
    want, state = r.expected()
    for chunked in (False, True):
        o, s = r.run([(0, 130, 0, 0)], [chunked])
        assert np.isfinite(o).all() and rms_err(o, want) < 2e-4 and rms_err(s[0], state) < 2e-4


def test_recurrence_constant_decays_at_their_ends(hb, cuda):
    r = Rec(hb, 4, 16, 16, 130, low_rank=False, dtype="bf16", silu=True, decay=[0.0, 1.0, 0.999, 0.5])
    want, state = r.expected()
    for chunked in (False, True):
        o, s = r.run([(0, 130, 0, 0)], [chunked])
        assert np.isfinite(o).all() and rms_err(o, want) < 1e-4 and rms_err(s[0], state) < 1e-4


def test_recurrence_remembers_a_far_token(hb, cuda):
    """A value written once and asked for hundreds of tokens later, with nothing else in its channel."""
    n, dim = 520, 32
    r = Rec(hb, 1, dim, 32, n, low_rank=False, dtype="bf16", decay=[0.999])
    r.p[:] = rounded(0.01 * r.p, "bf16")
    r.k[:, 3] = 0.0
    r.k[1, :], r.k[1, 3] = 0.0, 4.0
    r.v[1, :] = rounded(np.linspace(-8, 8, 32), "bf16")
    r.q[:, :], r.q[:, 3] = 0.0, 2.0
    r.dev[0].copy_(put(r.p, "bf16"))
    want, _ = r.expected()
    for chunked in (False, True):
        o, _ = r.run([(0, n, 0, 0)], [chunked])
        assert np.abs(o[-1] - want[-1]).max() < 1e-3 * np.abs(want[-1]).max()
        assert np.abs(want[-1]).max() > 10.0


# ------------------------------------------------------------------- streams and gated norms
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 11])
@pytest.mark.parametrize("width", [64, 101, 1000, 13000])
def test_streams(hb, cuda, dtype, streams, width):
    import torch

    n, ld, eps = 9, (width + 7) // 8 * 8, 1e-3
    rng = np.random.default_rng(streams * width)
    f = lambda *s: rng.standard_normal(s)
    lim = 4e-3 if dtype == "bf16" else 2e-6
    vec = lambda a: a.astype(np.float32).astype(np.float64)
    table, pos_table = rounded(f(37, width), dtype), rounded(f(50, width), dtype)
    ids, pos = rng.integers(0, 37, n), rng.integers(0, 50, n)
    w_in, norm, nxt_in, nxt_norm, out = vec(f(streams)), vec(0.3 * f(width)), vec(f(streams)), vec(0.3 * f(width)), vec(f(streams))
    mix, w1, w2 = vec(f(streams, streams)), vec(f(width)), vec(f(width))
    y, y2 = vec(f(n, ld)), vec(f(n, ld))
    x = torch.zeros((n, streams, width), device="cuda")
    h = put(np.zeros((n, ld)), dtype)
    code = dt(hb, dtype)
    d = {k: put(v) for k, v in dict(w_in=w_in, norm=norm, nxt_in=nxt_in, nxt_norm=nxt_norm, out=out, mix=mix, w1=w1, w2=w2,
                                    y=y, y2=y2).items()}
    tabs, dids, dpos = (put(table, dtype), put(pos_table, dtype)), ints(ids, np.int32), ints(pos)
    get = lambda: h.float().cpu().numpy().astype(np.float64)[:, :width]
    hb.check(hb.lib.hb_streams_embed(None, x.data_ptr(), h.data_ptr(), tabs[0].data_ptr(), tabs[1].data_ptr(), dids.data_ptr(),
                                     dpos.data_ptr(), d["w_in"].data_ptr(), d["norm"].data_ptr(), n, streams, width, ld, 37, 50,
                                     eps, code))
    torch.cuda.synchronize()
    xs = np.repeat((table[ids] + pos_table[pos])[None], streams, 0)
    assert rms_err(x.cpu().numpy().transpose(1, 0, 2), xs) < 1e-6
    assert rms_err(get(), R.rms_norm_around_zero(R.streams_read(xs, w_in), norm, eps)) < lim
    for two in (False, True):
        hb.check(hb.lib.hb_streams_mix(None, x.data_ptr(), h.data_ptr(), d["y"].data_ptr(), d["y2"].data_ptr() if two else None,
                                       ld, d["mix"].data_ptr(), d["out"].data_ptr(), d["nxt_in"].data_ptr(),
                                       d["nxt_norm"].data_ptr(), d["w1"].data_ptr(), d["w2"].data_ptr(), n, streams, width, ld,
                                       eps, code))
        torch.cuda.synchronize()
        a, b = y[:, :width], y2[:, :width]
        yy = 0.5 * (R.rms_norm(a, w1, eps) + R.rms_norm(b, w2, eps)) if two else a
        xs = R.streams_write(xs, mix, out, yy)
        assert rms_err(x.cpu().numpy().transpose(1, 0, 2), xs) < 2e-6
        assert rms_err(get(), R.rms_norm_around_zero(R.streams_read(xs, nxt_in), nxt_norm, eps)) < lim
    want = ints([4, 0, 8])
    hb.check(hb.lib.hb_streams_final(None, h.data_ptr(), x.data_ptr(), want.data_ptr(), d["norm"].data_ptr(), 3, streams, width,
                                     ld, eps, code))
    torch.cuda.synchronize()
    assert rms_err(get()[:3], R.rms_norm_around_zero(xs.sum(0)[[4, 0, 8]], norm, eps)) < lim


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("groups,size", [(5, 24), (1, 200), (1, 33), (2, 1500), (12, 128)])
@pytest.mark.parametrize("silu", [0, 1])
def test_gated_group_norm(hb, cuda, dtype, groups, size, silu):
    import torch

    n, width, eps = 7, groups * size, 1e-4
    rng = np.random.default_rng(groups * size)
    o, g, w = rng.standard_normal((n, width)), rounded(2 * rng.standard_normal((n, width + 3)), dtype), rng.standard_normal(size)
    out = put(np.zeros((n, width + 5)), dtype)
    do, dg, dw = put(o), put(g, dtype), put(w)
    hb.check(hb.lib.hb_gated_group_norm(None, out.data_ptr(), width + 5, do.data_ptr(), width, dg.data_ptr(), width + 3,
                                        dw.data_ptr(), n, groups, size, silu, eps, dt(hb, dtype)))
    torch.cuda.synchronize()
    gate = g[:, :width]
    want = R.rms_norm(o.reshape(n, groups, size), w, eps).reshape(n, width) * (R.silu(gate) if silu else R.sigmoid(gate))
    assert rms_err(out.float().cpu().numpy()[:, :width], want) < (4e-3 if dtype == "bf16" else 2e-6)
