"""The mechanisms of Muzopel alone, through their public entry points, against the plain NumPy form: the
residual with normed outputs, convolved inputs and sums over depth; norms in parts; latents with rotated
neighbours and queries elsewhere; one gate per head; softmax routing with a corrected choice and identity
experts; activations without a gate."""
import ctypes as C

import numpy as np
import pytest

from oracle import muzopel_ref as R
from tests.test_gpu_badolix_mechanisms import Inside
from tests.test_gpu_biberax_mechanisms import Paged, back
from tests.test_gpu_mechanisms import BS, dt, ints, put, rms_err, rounded

pytestmark = pytest.mark.gpu
EPS = 1e-3


def tight(dtype):
    return 4e-3 if dtype == "bf16" else 2e-6


# ---------------------------------------------------------------------------- residual
class Boundary:
    """Two boundaries in a row over one sequence and its slot: the first forms a convolved input, the second
    (which reads the same residual) brings the convolution's state up to date."""

    def __init__(self, hb, width, parts, taps, n, dtype, kind="product", depth=0, slots=3, slot=1, seed=0):
        import torch

        rng = np.random.default_rng(seed + width + taps)
        self.hb, self.dtype, self.width, self.parts, self.taps, self.n, self.slot = hb, dtype, width, parts, taps, n, slot
        self.ld = (width + 7) // 8 * 8 + 8
        self.x = rng.standard_normal((n, width)).astype(np.float32).astype(np.float64)
        y = rng.standard_normal((n, self.ld)).astype(np.float32)
        y[min(3, n - 1)] *= 1e-3  # eps decides here
        self.norm = rounded(1 + 0.3 * rng.standard_normal(width), "f32")
        self.conv = rounded(0.5 * rng.standard_normal((width, taps)), "f32")
        a = self.a = hb.ResidualArgs()
        self.keep = []

        def dev(array, kind="f32"):
            t = ints(array) if kind == "i32" else put(array, kind)
            self.keep.append(t)
            return t.data_ptr()

        self.v = y[:, :width].astype(np.float64)
        if kind == "experts":  # some with a product's rows beside them, some identities
            top, places = 3, 2 * n
            ey, inp = (rounded(rng.standard_normal((r, self.ld)), dtype) for r in (places, n))
            place, weight = rng.integers(-1, places, (n, top)), rounded(rng.uniform(0.1, 1.0, (n, top)), "f32")
            place[0] = -1
            for r in range(n):
                for p, g in zip(place[r], weight[r]):
                    self.v[r] += g * (inp[r] if p < 0 else ey[p])[:width]
            a.expert_y, a.input, a.ld_input = dev(ey, dtype), dev(inp, dtype), self.ld
            a.expert_place, a.expert_weight, a.top = dev(place, "i32"), dev(weight), top
        if kind == "embedding":
            table, ids = rounded(rng.standard_normal((11, width)), dtype), rng.integers(0, 11, n)
            self.v, self.x = table[ids], np.zeros_like(self.x)
            a.embed, a.ids, a.vocab = dev(table, dtype), dev(ids, "i32"), 11
        else:
            a.y, a.x = dev(y), dev(self.x)
        a.ld_y, a.norm, a.groups, a.eps = self.ld, dev(self.norm), parts, EPS
        self.earlier, self.weights = rng.standard_normal((depth, n, width)), rng.standard_normal(depth + 1)
        if depth:
            a.earlier, a.step, a.n_earlier, a.depth = dev(self.earlier), n * width, depth, dev(self.weights)
        a.conv, a.taps = dev(self.conv.T), taps
        self.state = torch.full((slots, max(1, taps - 1), width), 7.0, device="cuda")  # stale: not read at position 0
        a.state = self.state.data_ptr()
        self.result, self.x_out = (torch.zeros((n, width), device="cuda") for _ in range(2))
        self.h = put(np.zeros((n, self.ld)), dtype)
        a.result, a.x_out, a.h, a.ld_h = self.result.data_ptr(), self.x_out.data_ptr(), self.h.data_ptr(), self.ld
        b = self.b = hb.ResidualArgs()
        b.y, b.ld_y, b.norm, b.groups, b.eps = dev(y), self.ld, a.norm, parts, EPS
        b.x, b.taps, b.past = a.x_out, taps, self.state.data_ptr()

    def expected(self, lo, hi):
        made = self.x[lo:hi] + R.parts_norm(self.v[lo:hi], self.norm, self.parts, EPS)
        x = R.depth_sum([*self.earlier[:, lo:hi], made], self.weights) if len(self.earlier) else made
        return made, x, R.with_past(x, self.conv)

    def run(self, segs, run_rows, two=False):
        """segs: (first row, rows, first position, slot), cut into runs of up to run_rows.  two: the form for
        many rows."""
        import torch

        s = ints(segs)
        runs = [(g, r0 + i, min(run_rows, n - i), 0) for g, (r0, n, _, _) in enumerate(segs) for i in range(0, n, run_rows)]
        t, scale, mixed = ints(runs), put(np.zeros((self.n, self.parts))), put(np.zeros((self.n, self.ld)))
        for args in (self.a, self.b):
            args.scale, args.mixed = (scale.data_ptr(), mixed.data_ptr()) if two else (None, None)
            args.rows = max(r0 + n for r0, n, _, _ in segs)
            self.hb.check(self.hb.lib.hb_residual_step(None, C.byref(args), t.data_ptr(), len(runs), s.data_ptr(), self.width,
                                                       dt(self.hb, self.dtype)))
        torch.cuda.synchronize()
        return back(self.result), back(self.x_out), back(self.h)[:, :self.width]


SHAPES = [  # width, parts, taps
    (64, 4, 4), (75, 5, 2), (96, 1, 3), (520, 4, 4), (2080, 1, 4), (4096, 2, 4), (1030, 2, 3), (4100, 1, 2), (9000, 1, 4),
    (1501, 1, 4), (72, 3, 1), (48, 12, 6), (264, 1, 9), (33, 33, 5), (1024, 256, 2), (24, 2, 32),
]


@pytest.mark.parametrize("kind", ["product", "experts", "embedding"])
@pytest.mark.parametrize("width,parts,taps", SHAPES)
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_residual_of_a_whole_sequence(hb, cuda, width, parts, taps, kind, dtype):
    n = 37
    b = Boundary(hb, width, parts, taps, n, dtype, kind, depth=3 if kind == "experts" else 0)
    made, x, h = b.expected(0, n)
    first = None
    for run_rows, two in ((n, False), (16, False), (5, False), (2, False), (1, False), (16, True), (8, True), (3, True), (1, True)):
        got = b.run([(0, n, 0, 1)], run_rows, two)  # (also runs shorter than the convolution)
        assert rms_err(got[0], made) < 2e-6 and rms_err(got[1], x) < 2e-6 and rms_err(got[2], h) < tight(dtype), run_rows
        first = first or got
        assert all(np.array_equal(a, c) for a, c in zip(first, got))  # how rows are cut changes no bit
    if taps > 1:
        held = np.stack([x[p] for p in sorted(range(n - taps + 1, n), key=lambda p: p % (taps - 1))])
        got = back(b.state)
        assert rms_err(got[1], held) < 2e-6 and (got[0] == 7.0).all() and (got[2] == 7.0).all()


@pytest.mark.parametrize("width,parts,taps", [(96, 4, 4), (75, 3, 2), (40, 1, 7), (2080, 2, 4), (64, 2, 1), (36, 3, 12)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_portions_meet_in_the_state(hb, cuda, width, parts, taps, dtype):
    """One sequence in portions cut anywhere (down to one token) beside another in another slot, in runs
    shorter and longer than the convolution."""
    b = Boundary(hb, width, parts, taps, 130, dtype, depth=2)
    one, other = b.expected(0, 100), b.expected(100, 130)
    for run_rows, two in ((16, False), (3, False), (4, False), (16, True), (2, True)):
        at = 0
        for n in (2, 1, 9, 1, 1, 1, 40, 3, 2, 40):
            segs = [(at, n, at, 1)] + ([(100, 30, 0, 2)] if at == 2 else [])
            got = b.run(segs, run_rows, two)
            for g, e, limit in zip(got, one, (2e-6, 2e-6, tight(dtype))):
                assert rms_err(g[at:at + n], e[at:at + n]) < limit, (at, n, run_rows)
            at += n
        assert at == 100
        for g, e, limit in zip(got, other, (2e-6, 2e-6, tight(dtype))):
            assert rms_err(g[100:], e) < limit
        if taps > 1:
            assert (back(b.state)[0] == 7.0).all()


def test_an_input_is_felt_for_exactly_its_taps(hb, cuda):
    """One row whose residual is not zero, around the edges of runs and portions."""
    taps, width, n = 4, 32, 40
    for at in (0, 1, 14, 15, 16, 17, 31):
        b = Boundary(hb, width, 2, taps, n, "bf16")
        x = np.zeros((n, width))
        x[at] = 8.0
        b.keep[[t.data_ptr() for t in b.keep].index(b.a.x)].copy_(put(x))
        b.keep[[t.data_ptr() for t in b.keep].index(b.a.norm)].zero_()
        b.keep[[t.data_ptr() for t in b.keep].index(b.a.conv)].copy_(put(np.repeat(1.0 + np.arange(taps)[:, None], width, axis=1)))
        for portions, two in (((40,), 0), ((40,), 1), ((16, 24), 0), ((16, 24), 1), ((14, 1, 1, 1, 23), 0), ((1,) * 40, 1)):
            pos, h = 0, None
            for p in portions:
                h = b.run([(pos, p, pos, 0)], 16, two)[2]
                pos += p
            felt = np.flatnonzero(np.abs(h).max(axis=1))
            assert felt.tolist() == [t for t in range(at, at + taps) if t < n], (at, portions[:2], felt)
            np.testing.assert_allclose(h[at], 8.0 * (1 + taps))  # the last weight meets the token itself
            if at + 1 < n:
                np.testing.assert_allclose(h[at + 1], 8.0 * (taps - 1))


def test_residual_refusals(hb, cuda):
    b = Boundary(hb, 60, 4, 3, 5, "f32")
    for field, value, text in (("groups", 7, "parts"), ("taps", 0, "convolution"), ("taps", 33, "taps"), ("h", None, "taps"),
                               ("norm", None, "null"), ("y", None, "output"), ("state", None, "convolution")):
        old = getattr(b.a, field)
        setattr(b.a, field, value)
        with pytest.raises(hb.HbError, match=text):
            b.run([(0, 5, 0, 0)], 5)
        setattr(b.a, field, old)


@pytest.mark.parametrize("groups,size", [(1, 200), (4, 50), (5, 15), (3, 1024), (1, 4096), (2, 1333), (64, 8), (7, 1)])
@pytest.mark.parametrize("in_f32", [0, 1])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_norms_in_parts(hb, cuda, groups, size, in_f32, dtype):
    import torch

    width, n = groups * size, 9
    rng = np.random.default_rng(width)
    x = rng.standard_normal((n, width + 12))
    x[4] *= 1e-3
    x = rounded(x, "f32" if in_f32 else dtype)
    w, rows = rounded(1 + 0.3 * rng.standard_normal(width), "f32"), np.array([4, 0, 8, 8, 1])
    tx, tw, tl = put(x, "f32" if in_f32 else dtype), put(w), ints(rows)
    for lst in (None, rows):
        out = put(np.full((n, width + 4), 50.0), dtype)
        hb.check(hb.lib.hb_parts_norm(None, out.data_ptr(), width + 4, tx.data_ptr(), width + 12, in_f32 or (dtype == "f32"),
                                      None if lst is None else tl.data_ptr(), tw.data_ptr(), n if lst is None else len(rows), groups,
                                      size, EPS, dt(hb, dtype)))
        torch.cuda.synchronize()
        got = back(out)
        src = x[:, :width] if lst is None else x[rows, :width]
        assert rms_err(got[:len(src), :width], R.parts_norm(src, w, groups, EPS)) < tight(dtype)
        assert (got[:, width:] == 50.0).all() and (got[len(src):] == 50.0).all()


# ---------------------------------------------------------------------------- attention
@pytest.mark.parametrize("n,H,D,VD", [(140, 4, 64, 64), (131, 16, 112, 96), (150, 16, 576, 512), (100, 70, 168, 136), (75, 7, 9, 5),
                                      (120, 40, 288, 256), (97, 3, 40, 24)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_one_gate_per_head(hb, cuda, n, H, D, VD, dtype):
    """Gates from closed to open, beside other numbers of the same rows; over values inside the keys and over
    values of their own."""
    rng = np.random.default_rng(n + H)
    q, k, v = (rounded(rng.standard_normal(s), dtype) for s in ((n, H, D), (n, 1, D), (n, 1, VD)))
    z = rounded(4.0 * rng.standard_normal((n, H + 5)), dtype)
    scale = 3.0 * D ** -0.5
    for inside in (True, False):
        values = k[:, :, :VD] if inside else v
        want = R.capped_attention(q, k, values, scale, R.window_mask(n, None, 0)) * R.sigmoid(z[:, :H])[:, :, None]
        p = Inside(hb, q, k, VD, scale, dtype) if inside else Paged(hb, q, v, k, scale, dtype)
        tz = put(z, dtype)
        p.a.gate, p.a.ld_gate, p.a.gate_per_head = tz.data_ptr(), H + 5, 1
        for form, got in p.forms():
            assert rms_err(got, want) < tight(dtype), (inside, form)


@pytest.mark.parametrize("H,D,RD,rank,pairs", [(4, 16, 8, 24, 4), (3, 9, 6, 11, 3), (16, 128, 64, 512, 32), (2, 8, 16, 8, 4),
                                               (1, 24, 16, 4096, 8), (5, 32, 32, 264, 16), (3, 8, 8, 40, 1), (2, 16, 5, 16, 2)])
@pytest.mark.parametrize("apart", [False, True])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_latents_with_rotated_neighbours(hb, cuda, H, D, RD, rank, pairs, apart, dtype):
    """apart: the queries lie in a matrix of their own."""
    import torch

    rng = np.random.default_rng(rank)
    n, nb, KD, Q = 21, 3, rank + RD, H * (D + RD)
    off_q, off_c = 8, (8 if apart else (8 + Q + 7) // 8 * 8)
    p = rng.standard_normal((n, (off_c + KD + 7) // 8 * 8))
    p[3] *= 1e-3  # eps decides here
    p = rounded(p, dtype)
    own = rounded(rng.standard_normal((n, (Q + 15) // 8 * 8)), dtype)
    pos, slots = rng.integers(0, 5000, n), rng.permutation(nb * BS)[:n]
    slots[4] = -1
    norm = rounded(1 + 0.3 * rng.standard_normal(rank), "f32")
    freqs, gain = R.rotation(1e3, 2 * pairs, dict(factor=8.0, original=64, fast=9.0, slow=1.0))
    t, to, tn, tf = put(p, dtype), put(own, dtype), put(norm), torch.from_numpy(np.ascontiguousarray(freqs)).cuda()
    q, kc = put(np.full((n, H * KD), 50.0), dtype), put(np.full((nb * BS, KD), 50.0), dtype)
    tp, ts = ints(pos), ints(slots, np.int64)
    a = hb.LatentPrepArgs(t.data_ptr(), p.shape[1], off_q, off_c, H, D, RD, rank, q.data_ptr(), H * KD, tp.data_ptr(), ts.data_ptr(),
                          kc.data_ptr(), nb, tn.data_ptr(), EPS, tf.data_ptr(), pairs, gain)
    a.neighbours = 1
    if apart:
        a.q_rows, a.ld_q_rows = to.data_ptr(), own.shape[1]
    hb.check(hb.lib.hb_latent_prepare(None, C.byref(a), n, dt(hb, dtype)))
    torch.cuda.synchronize()
    got, limit, held = back(kc), tight(dtype), slots >= 0
    assert rms_err(got[slots[held], :rank], R.rms_norm(p[:, off_c:off_c + rank], norm, EPS)[held]) < limit
    key = R.rotate_neighbours(p[:, None, off_c + rank:off_c + KD], pos, freqs, gain)[:, 0]
    assert rms_err(got[slots[held], rank:], key[held]) < limit
    assert (got[np.setdiff1d(np.arange(nb * BS), slots)] == 50.0).all()
    src, rows = (own[:, :Q], back(to)[:, :Q]) if apart else (p[:, off_q:off_q + Q], back(t)[:, off_q:off_q + Q])
    qh, placed = src.reshape(n, H, D + RD), rows.reshape(n, H, D + RD)
    want = R.rotate_neighbours(qh[:, :, D:], pos, freqs, gain)
    wide = back(q).reshape(n, H, KD)
    assert rms_err(wide[:, :, rank:], want) < limit and (wide[:, :, :rank] == 50.0).all()
    assert rms_err(placed[:, :, D:], want) < limit and np.array_equal(placed[:, :, :D], qh[:, :, :D])
    assert np.array_equal(back(t)[:, off_c:], p[:, off_c:])
    if apart:
        assert np.array_equal(back(to)[:, Q:], own[:, Q:]) and np.array_equal(back(t), p)


# ------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("form,limit", [(0, np.inf), (1, np.inf), (2, 30.0), (2, 0.5), (1, 0.8), (0, 1.5)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_activations_without_a_gate(hb, cuda, form, limit, dtype):
    import torch

    rng = np.random.default_rng(form)
    z = 3.0 * rng.standard_normal((19, 45))
    z[0, :8] = [-300, -90, -20, 0, 20, 90, 300, 1e4]
    z = rounded(z, dtype)
    t, out = put(z, dtype), put(np.zeros((19, 45)), dtype)
    spec = hb.GatedActSpec(1.7, 0.01, limit, 0.3, form, 1)  # (the shift belongs to the factor that is not there)
    hb.check(hb.lib.hb_gated_act(None, out.data_ptr(), t.data_ptr(), 19, 45, C.byref(spec), dt(hb, dtype)))
    torch.cuda.synchronize()
    g = np.minimum(z, limit)
    want = [lambda: g * R.sigmoid(np.maximum(1.7 * (g + 0.01 * g ** 3), -700)), lambda: R.gelu(g), lambda: limit * np.tanh(z / limit)][form]()
    assert rms_err(back(out)[1:], want[1:]) < tight(dtype)
    np.testing.assert_allclose(back(out)[0], want[0], rtol=1e-2, atol=1e-6)
    with pytest.raises(hb.HbError, match="form"):
        bad = hb.GatedActSpec(1.0, 0.0, 1.0, 0.0, 2, 0)
        hb.check(hb.lib.hb_gated_act(None, out.data_ptr(), t.data_ptr(), 19, 20, C.byref(bad), dt(hb, dtype)))


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_gated_gelu_by_the_error_function(hb, cuda, dtype):
    import torch

    gu = rounded(2.0 * np.random.default_rng(0).standard_normal((11, 60)), dtype)
    t, out, spec = put(gu, dtype), put(np.zeros((11, 30)), dtype), hb.GatedActSpec(1.0, 0.0, 1.3, 0.2, 1, 0)
    hb.check(hb.lib.hb_gated_act(None, out.data_ptr(), t.data_ptr(), 11, 30, C.byref(spec), dt(hb, dtype)))
    torch.cuda.synchronize()
    want = R.gelu(np.minimum(gu[:, :30], 1.3)) * (np.clip(gu[:, 30:], -1.3, 1.3) + 0.2)
    assert rms_err(back(out), want) < tight(dtype)


class Mixture:
    """Routing, sorted rows, two grouped products and the weighted sum into a residual."""

    def __init__(self, hb, rows, width, experts, identity, top, ff, dtype, m_pad, seed=0, favour=None):
        import torch

        rng = np.random.default_rng(seed)
        self.hb, self.dtype, self.rows, self.width, self.top, self.experts, self.m_pad = hb, dtype, rows, width, top, experts, m_pad
        O, ld, ffp = experts + identity, (width + 7) // 8 * 8, (ff + 7) // 8 * 8
        h = np.zeros((rows, ld))
        h[:, :width] = rng.standard_normal((rows, width))
        h = rounded(h, dtype)
        self.h = h[:, :width]
        self.w = {"router": rounded(1.5 * rng.standard_normal((O, width)) * width ** -0.5, dtype),
                  "correction": rounded(rng.standard_normal(O) / O, "f32")}
        if favour is not None:
            self.w["correction"][:] = np.where(np.isin(np.arange(O), favour), 2.0, -2.0)
        up, down = np.zeros((experts, ffp, ld)), np.zeros((experts, ld, ffp))
        for e in range(experts):
            self.w[f"e{e}.up"] = rounded(1.7 * rng.standard_normal((ff, width)) * width ** -0.5, dtype)
            self.w[f"e{e}.down"] = rounded(rng.standard_normal((width, ff)) * ff ** -0.5, dtype)
            up[e, :ff, :width], down[e, :width, :ff] = self.w[f"e{e}.up"], self.w[f"e{e}.down"]
        n = rows * top
        tiles = min(experts, n) + n // m_pad
        z32 = lambda *s: torch.zeros(s, device="cuda", dtype=torch.int32)
        self.ids, self.rank, self.place = z32(rows, top), z32(rows, top), z32(rows, top)
        self.weight = torch.zeros((rows, top), device="cuda")
        self.count, self.first, self.tiles = z32(experts + 1), z32(experts + 1), z32(tiles)
        th, tr, tc, tu, td = put(h, dtype), put(self.w["router"], dtype), put(self.w["correction"]), put(up, dtype), put(down, dtype)
        r = hb.MoeRouting(experts, top, m_pad, tiles, *(t.data_ptr() for t in (self.ids, self.rank, self.place, self.weight, self.count,
                                                                              self.first, self.tiles)))
        r.identity, r.softmax_all, r.correction = identity, 1, tc.data_ptr()
        x, act, y = (put(np.zeros((tiles * m_pad, w)), dtype) for w in (ld, ffp, ld))
        code = dt(hb, dtype)
        for _ in range(2):  # the second run finds the counters as the first one left them
            hb.check(hb.lib.hb_moe_route_top(None, C.byref(r), th.data_ptr(), ld, tr.data_ptr(), None, rows, width, code))
            hb.check(hb.lib.hb_moe_gather(None, C.byref(r), x.data_ptr(), th.data_ptr(), ld, rows, code))
        spec = hb.GatedActSpec(1.0, 0.0, np.inf, 0.0, 1, 1)
        gemm = lambda N, K, ldx, ldy, act: hb.GroupedGemm(experts, N, K, m_pad, tiles, max(1, tiles // 2), self.tiles.data_ptr(), ldx, ldy,
                                                          act, 0, spec)
        g = gemm(ffp, ld, ld, ffp, 1 if dtype == "bf16" else 0)
        hb.check(hb.lib.hb_gemm_grouped(None, act.data_ptr(), x.data_ptr(), tu.data_ptr(), C.byref(g), code))
        if dtype == "f32":
            hb.check(hb.lib.hb_gated_act_grouped(None, act.data_ptr(), act.data_ptr(), ffp, C.byref(g), code))
        g = gemm(ld, ffp, ffp, ld, 0)
        hb.check(hb.lib.hb_gemm_grouped(None, y.data_ptr(), act.data_ptr(), td.data_ptr(), C.byref(g), code))
        a, out = hb.ResidualArgs(), torch.zeros((rows, width), device="cuda")
        one = put(np.ones(width))
        a.expert_y, a.ld_y, a.expert_place, a.expert_weight, a.top = y.data_ptr(), ld, self.place.data_ptr(), self.weight.data_ptr(), top
        a.input, a.ld_input, a.norm, a.groups, a.taps = th.data_ptr(), ld, one.data_ptr(), 1, 1
        a.eps, a.x_out = 0.0, out.data_ptr()
        s, t = ints([(0, rows, 0, 0)]), ints([(0, i, min(16, rows - i), 0) for i in range(0, rows, 16)])
        hb.check(hb.lib.hb_residual_step(None, C.byref(a), t.data_ptr(), len(t), s.data_ptr(), width, code))
        torch.cuda.synchronize()
        self.out = back(out)

    def check(self):
        chosen, weight = R.route(self.h, self.w["router"], self.w["correction"], self.top)
        clear = R.route_margin(self.h, self.w["router"], self.w["correction"], self.top) > 1e-4
        assert clear.mean() > 0.9
        ids, place, weights, tiles = self.ids.cpu().numpy(), self.place.cpu().numpy(), back(self.weight), self.tiles.cpu().numpy()
        real = ids < self.experts
        assert (place[~real] == -1).all() and len(np.unique(place[real])) == real.sum()
        assert np.array_equal(tiles[place[real] // self.m_pad], ids[real])
        used = sum(-(-int((ids == e).sum()) // self.m_pad) for e in range(self.experts))
        assert (tiles[:used] >= 0).all() and (tiles[used:] == -1).all() and not self.count.cpu().numpy().any()
        assert np.array_equal(np.sort(ids[clear]), np.sort(chosen[clear]))
        same = (ids == chosen).all(axis=1)
        assert same.mean() > 0.9
        np.testing.assert_allclose(weights[same], weight[same], rtol=2e-5)
        mlp = dict(router=dict(top=self.top, experts=self.experts))
        want = R.rms_norm(R.moe_ffn(self.h, self.w, mlp), 1.0, 0.0)
        assert rms_err(self.out[clear], want[clear]) < (6e-3 if self.dtype == "bf16" else 4e-6)


@pytest.mark.parametrize("rows,width,experts,identity,top,ff,m_pad",
                         [(1, 64, 5, 2, 2, 40, 16), (7, 72, 3, 1, 4, 24, 16), (40, 75, 40, 24, 6, 11, 16), (300, 128, 4, 0, 1, 136, 64),
                          (530, 96, 9, 7, 2, 56, 128), (64, 520, 1, 1, 1, 264, 64), (33, 64, 70, 3, 5, 16, 32), (600, 64, 8, 8, 3, 1000, 112)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_mixture_with_identities(hb, cuda, rows, width, experts, identity, top, ff, m_pad, dtype):
    Mixture(hb, rows, width, experts, identity, top, ff, dtype, m_pad, seed=rows).check()


@pytest.mark.parametrize("favour", [(0, 1), (6, 7), (2, 6)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_the_correction_decides_the_choice_and_no_weight(hb, cuda, favour, dtype):
    """A correction that overrides every score: all rows go to two experts, to two identities, to one of each."""
    m = Mixture(hb, 150, 64, 6, 3, 2, 32, dtype, 32, seed=1, favour=favour)
    assert set(m.ids.cpu().numpy().ravel()) == set(favour)
    m.check()


def test_routing_refusals(hb, cuda):
    import torch

    z, one = torch.zeros((3, 64), device="cuda"), torch.zeros((14, 64), device="cuda")
    i32 = lambda *s: torch.zeros(s, device="cuda", dtype=torch.int32)
    t = [i32(3, 5), i32(3, 5), i32(3, 5), torch.zeros((3, 5), device="cuda"), i32(13), i32(13), i32(20)]
    for change, text in ((dict(identity=-1), "identit"), (dict(identity=2, groups=2, keep=1), "together"), (dict(identity=2, shared=1), "together"),
                         (dict(softmax_all=1, sigmoid=1), "together"), (dict(correction=one.data_ptr()), "together")):
        r = hb.MoeRouting(12, 4, 16, 20, *(x.data_ptr() for x in t))
        for k, v in change.items():
            setattr(r, k, v)
        with pytest.raises(hb.HbError, match=text):
            hb.check(hb.lib.hb_moe_route_top(None, C.byref(r), z.data_ptr(), 64, one.data_ptr(), None, 3, 64, hb.F32))


@pytest.mark.parametrize("rows,N,K,m_pad", [(64, 264, 2048, 64), (128, 72, 4096, 128), (16, 40, 512, 16), (48, 1000, 24, 16)])
def test_capped_products(hb, cuda, rows, N, K, m_pad):
    """The cap of logits in the product itself, with and without a split of K, scores far beyond the cap."""
    import torch

    rng = np.random.default_rng(N)
    x, w = rounded(rng.standard_normal((rows, K)), "bf16"), rounded(20.0 * rng.standard_normal((N, K)) * K ** -0.5, "bf16")
    tiles = rows // m_pad
    tx, tw, ty, tg = put(x, "bf16"), put(w, "bf16"), put(np.zeros((rows, N))), ints(np.zeros(tiles))
    g = hb.GroupedGemm(1, N, K, m_pad, tiles, tiles, tg.data_ptr(), K, N, 1, 1, hb.GatedActSpec(0.0, 0.0, 15.0, 0.0, 2, 1))
    hb.check(hb.lib.hb_gemm_grouped(None, ty.data_ptr(), tx.data_ptr(), tw.data_ptr(), C.byref(g), hb.BF16))
    torch.cuda.synchronize()
    assert rms_err(back(ty), 15.0 * np.tanh(x @ w.T / 15.0)) < 1e-4


def test_gelu_of_a_product_within_the_formulas_bound(hb, cuda):
    """The error function inside the product: 1.5e-7 of the distribution function, so 2e-7 of z and of 1."""
    import torch

    z = rounded(np.concatenate([np.linspace(-12, 12, 4000), [0.0, -0.0, 1e-8, -1e-8, 60.0, -60.0, 1e4, -1e4] * 12]), "bf16")
    n = len(z) // 16 * 16
    x, w = np.zeros((n, 16)), np.zeros((8, 16))
    x[:, 3], w[:, 3] = z[:n], 1.0
    tx, tw, ty, tg = put(x, "bf16"), put(w, "bf16"), put(np.zeros((n, 8))), ints(np.zeros(n // 16))
    g = hb.GroupedGemm(1, 8, 16, 16, n // 16, n // 16, tg.data_ptr(), 16, 8, 1, 1, hb.GatedActSpec(1.0, 0.0, np.inf, 0.0, 1, 1))
    hb.check(hb.lib.hb_gemm_grouped(None, ty.data_ptr(), tx.data_ptr(), tw.data_ptr(), C.byref(g), hb.BF16))
    torch.cuda.synchronize()
    got = back(ty)
    assert (np.abs(got - R.gelu(z[:n])[:, None]) <= 2e-7 * np.maximum(1.0, np.abs(z[:n]))[:, None] * 2).all()
