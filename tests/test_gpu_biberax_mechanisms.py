"""The mechanisms of Biberax alone, through their public entry points, against the plain NumPy form:
chunks, sinks, gates, a bias by distance, keys that are values times a scale; rotation and norms of
queries and keys; routing, grouped matrix products and the weighted sum of experts."""
import ctypes as C

import numpy as np
import pytest

from oracle import biberax_ref as R
from oracle.latarax_ref import window_mask
from tests.test_gpu_mechanisms import BS, dt, ints, put, rms_err, rounded

pytestmark = pytest.mark.gpu


def back(t):
    return t.float().cpu().numpy().astype(np.float64)


# ---------------------------------------------------------------------------- attention
class Paged:
    """One sequence's K/V spread over a shuffled block table of a larger pool full of junk."""

    def __init__(self, hb, q, v, k, scale, dtype, *, window=0, keep=0, chunk=0, sink=None, gate=None, bias=None,
                 key_scale=None, seed=0):
        import torch

        self.hb, self.dtype = hb, dtype
        n, H, D = q.shape
        G, VD = v.shape[1], v.shape[2]
        nb = -(-n // BS)
        self.n, self.H, self.VD = n, H, VD
        table = np.random.default_rng(seed).permutation(nb + 7)[:nb]
        slots = table[np.arange(n) // BS] * BS + np.arange(n) % BS

        def pool(a, width):
            full = np.full(((nb + 7) * BS, G, width), 50.0)
            full[slots] = a
            return put(full.reshape(nb + 7, BS, G, width).transpose(0, 2, 1, 3), dtype)

        self.q = put(q.reshape(n, -1), dtype)
        self.out = torch.zeros((n, H * VD), device="cuda", dtype=self.q.dtype)
        self.vc = pool(v, VD)
        self.kc = self.vc if key_scale is not None else pool(k, D)
        self.keep_alive = [ints(np.arange(n)), ints(np.zeros(n)), ints(table)]
        pos, seg, tab = self.keep_alive
        self.a = hb.SpanAttentionArgs(self.q.data_ptr(), H * D, self.out.data_ptr(), H * VD, self.kc.data_ptr(),
                                      None if key_scale is not None else self.vc.data_ptr(), tab.data_ptr(), nb, nb + 7,
                                      seg.data_ptr(), pos.data_ptr(), H, G, D, VD, window, keep, scale)
        self.a.chunk = chunk

        def extra(field, array, kind="f32"):
            t = put(array, kind)
            self.keep_alive.append(t)
            setattr(self.a, field, t.data_ptr())

        if sink is not None:
            extra("sink", sink)
        if bias is not None:
            extra("dist_bias", bias)
            self.a.dist_len = bias.shape[1]
        if gate is not None:
            extra("gate", gate.reshape(n, -1), dtype)
            self.a.ld_gate = H * VD
        if key_scale is not None:
            full = np.full((nb + 7) * BS, 3.0)
            full[slots] = key_scale
            extra("key_scale", full)

    def tile_positions(self):
        return self.hb.check(self.hb.lib.hb_span_attention_tile_positions(C.byref(self.a), dt(self.hb, self.dtype)))

    def run(self, tiles=None, rows=None, splits=1):
        import torch

        self.out.zero_()
        t = ints(tiles) if tiles is not None else None
        r = ints(rows) if rows is not None else None
        n_rows = len(rows) if rows is not None else 0
        ws = torch.zeros(max(1, n_rows * self.H * splits * (self.VD + 2)), device="cuda")
        self.hb.check(self.hb.lib.hb_span_attention(None, C.byref(self.a), t.data_ptr() if t is not None else None,
                                                    len(tiles) if tiles is not None else 0,
                                                    r.data_ptr() if r is not None else None, n_rows, splits, ws.data_ptr(),
                                                    dt(self.hb, self.dtype)))
        torch.cuda.synchronize()
        return back(self.out).reshape(self.n, self.H, self.VD)

    def forms(self):
        """Every way the kernels can be asked for the same rows."""
        yield "rows", self.run(rows=np.arange(self.n))
        for splits in (2, 5, 8, 12):
            yield f"{splits} splits", self.run(rows=np.arange(self.n), splits=splits)
        tp = self.tile_positions()
        for size in sorted({tp, max(1, tp // 2 - 1), min(2, tp)} if tp else ()):
            yield f"tiles of {size}", self.run(tiles=[(0, i, min(size, self.n - i), 0) for i in range(0, self.n, size)])


SHAPES = [  # n, heads, kv_heads, dim, vdim, chunk, window, keep_first, bias distances, tied
    (150, 4, 2, 64, 64, 33, 0, 0, 0, False),
    (131, 6, 1, 40, 72, 48, 0, 0, 0, False),
    (97, 2, 2, 16, 8, 1, 0, 0, 0, False),
    (90, 3, 3, 104, 320, 64, 0, 0, 40, False),
    (200, 16, 1, 128, 128, 0, 0, 0, 77, True),
    (170, 4, 2, 48, 48, 0, 0, 0, 16, True),
    (140, 2, 1, 320, 320, 0, 0, 0, 100, True),
    (80, 4, 4, 24, 24, 0, 31, 4, 1, True),
    (65, 20, 1, 32, 32, 20, 0, 0, 9, False),
    (80, 4, 4, 12, 20, 31, 0, 0, 200, False),
    (75, 5, 5, 9, 9, 0, 0, 0, 30, True),
    (130, 1, 1, 256, 256, 100, 0, 0, 0, False),
]


@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_attention_with_chunks_sinks_gates_and_biases(hb, cuda, shape, dtype):
    n, H, G, D, VD, chunk, window, keep, far, tied = shape
    rng = np.random.default_rng(n + H)
    q, v, gate = (rounded(rng.standard_normal(s), dtype) for s in ((n, H, D), (n, G, VD), (n, H, VD)))
    scales = rounded(rng.uniform(0.5, 2.0, n), "f32")
    k = v * scales[:, None, None] if tied else rounded(rng.standard_normal((n, G, D)), dtype)
    sink = rounded(3.0 * rng.standard_normal(H), "f32")
    table = rounded(2.0 * rng.standard_normal((H, far)), "f32") if far else None
    visible = R.chunk_mask(n, chunk) if chunk else window_mask(n, window or None, keep)
    d = np.maximum(np.arange(n)[:, None] - np.arange(n)[None, :], 0)
    bias = table[:, np.minimum(d, far - 1)].transpose(1, 2, 0) if far else None
    scale = 0.37 if D < 200 else 0.1
    for use_sink, use_gate in ((True, True), (False, False)):
        want = R.sink_attention(q, k, v, scale, visible, sink if use_sink else None, bias)
        if use_gate:
            want = want * R.sigmoid(gate)
        p = Paged(hb, q, v, k, scale, dtype, window=window, keep=keep, chunk=chunk, sink=sink if use_sink else None,
                  gate=gate if use_gate else None, bias=table, key_scale=scales if tied else None)
        for form, got in p.forms():
            assert rms_err(got, want) < (4e-3 if dtype == "bf16" else 2e-6), form
        assert (p.tile_positions() > 0) == (dtype == "bf16" and D % 8 == 0 and VD % 8 == 0 and H // G <= 64)


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("chunk", [24, 16, 17, 64])
def test_chunk_edges_stand_out(hb, cuda, chunk, dtype):
    """One key at a time points at the query so strongly that seeing it or not decides the output."""
    n, H, G, D, VD = 120, 4, 2, 32, 40
    rng = np.random.default_rng(5)
    base_q, base_k, v = (rounded(0.2 * rng.standard_normal(s), dtype) for s in ((n, H, D), (n, G, D), (n, G, VD)))
    for at in (0, chunk - 1, chunk, chunk + 1, 47, 48, 63, 64):
        q, k, v2 = base_q.copy(), base_k.copy(), v.copy()
        k[at] = 0.0
        k[at, :, 0] = 16.0
        q[:, :, 0] = 4.0
        v2[at] = rounded(30.0 + rng.standard_normal((G, VD)), dtype)
        want = R.sink_attention(q, k, v2, 0.5, R.chunk_mask(n, chunk), np.zeros(H))
        for form, got in Paged(hb, q, v2, k, 0.5, dtype, chunk=chunk, sink=np.zeros(H)).forms():
            per_pos = np.abs(got - want).max(axis=(1, 2))
            assert per_pos.max() < (0.2 if dtype == "bf16" else 1e-4), (form, at, int(per_pos.argmax()))


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_single_distances_stand_out(hb, cuda, dtype):
    """A bias that favours one distance by far: one off, and another value comes out."""
    n, H, G, D = 150, 4, 2, 32
    rng = np.random.default_rng(6)
    q = rounded(0.2 * rng.standard_normal((n, H, D)), dtype)
    v = rounded(rng.standard_normal((n, G, D)), dtype)
    scales = rounded(rng.uniform(0.5, 1.0, n), "f32")
    for far, at in ((20, 0), (20, 7), (20, 18), (20, 19), (65, 48), (65, 63), (65, 64), (1, 0)):
        table = np.zeros((H, far))
        table[:, at] = 12.0
        d = np.maximum(np.arange(n)[:, None] - np.arange(n)[None, :], 0)
        want = R.sink_attention(q, v * scales[:, None, None], v, 0.3, R.causal_mask(n), np.zeros(H),
                                table[:, np.minimum(d, far - 1)].transpose(1, 2, 0))
        for form, got in Paged(hb, q, v, None, 0.3, dtype, sink=np.zeros(H), bias=table, key_scale=scales).forms():
            assert np.abs(got - want).max() < (0.04 if dtype == "bf16" else 1e-4), (form, far, at)


def test_a_sink_decides_the_first_tokens(hb, cuda):
    """With a strong sink the outputs nearly vanish, with one far below they are the plain softmax."""
    n, H, G, D = 40, 2, 1, 64
    rng = np.random.default_rng(7)
    q, k, v = (rounded(rng.standard_normal(s), "bf16") for s in ((n, H, D), (n, G, D), (n, G, D)))
    for value in (60.0, -60.0, 0.0):
        sink = np.array([value, -value])
        want = R.sink_attention(q, k, v, 0.1, R.causal_mask(n), sink)
        for form, got in Paged(hb, q, v, k, 0.1, "bf16", sink=sink).forms():
            assert np.abs(got - want).max() < 0.02, (form, value)


# ------------------------------------------------------------------- queries and keys
def prep(hb, dtype, p, offs, H, G, D, VD, pos, slots, nb, **kw):
    import torch

    es = torch.bfloat16 if dtype == "bf16" else torch.float32
    rows = put(p, dtype)
    kc = torch.full((nb, G, BS, D), 50.0, device="cuda", dtype=es)
    vc = torch.full((nb, G, BS, VD), 50.0, device="cuda", dtype=es)
    ks = torch.full((nb * BS,), 50.0, device="cuda")
    t_pos, t_slots = ints(pos), ints(slots, np.int64)
    tied = kw.pop("tied", False)
    a = hb.AttentionPrepArgs(rows.data_ptr(), p.shape[1], *offs, H, G, D, VD, t_pos.data_ptr(), t_slots.data_ptr(),
                             kc.data_ptr(), vc.data_ptr(), nb)
    alive = []
    for name, value in kw.items():
        if isinstance(value, float):
            setattr(a, name, value)
            continue
        t = torch.from_numpy(np.ascontiguousarray(value)).cuda() if name == "rotation" else put(value)
        alive.append(t)
        setattr(a, name, t.data_ptr())
        if name == "rotation":
            a.pairs = len(value)
    if tied:
        a.key_scale = ks.data_ptr()
    hb.check(hb.lib.hb_attention_prepare(None, C.byref(a), len(p), dt(hb, dtype)))
    torch.cuda.synchronize()
    at = lambda pool: back(pool).transpose(0, 2, 1, 3).reshape(nb * BS, G, -1)
    return back(rows), at(kc), at(vc), back(ks)


PREP = [(6, 2, 48, 40, 16), (3, 3, 10, 7, 3), (4, 1, 128, 64, 64), (2, 2, 24, 24, 0), (5, 1, 9, 9, 4)]  # H, G, D, VD, pairs


@pytest.mark.parametrize("H,G,D,VD,pairs", PREP)
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_rotation_and_kv_write(hb, cuda, H, G, D, VD, pairs, dtype):
    rng = np.random.default_rng(D)
    n, nb = 37, 6
    offs = (8, (8 + H * D + 7) // 8 * 8, (8 + H * D + 7) // 8 * 8 + (G * D + 7) // 8 * 8)
    p = rounded(rng.standard_normal((n, offs[2] + G * VD + 8 - (G * VD) % 8)), dtype)
    pos = rng.integers(0, 4000, n)
    slots = rng.permutation(nb * BS)[:n]
    slots[5] = -1
    freqs = R.rotation_frequencies(1e4, 2 * pairs, dict(factor=4.0, low=1.0, high=8.0, original=400)) if pairs else np.zeros(0)
    rows, kc, vc, _ = prep(hb, dtype, p, offs, H, G, D, VD, pos, slots, nb, **({"rotation": freqs} if pairs else {}))
    limit = 4e-3 if dtype == "bf16" else 2e-6
    q = p[:, offs[0]:offs[0] + H * D].reshape(n, H, D)
    k = p[:, offs[1]:offs[1] + G * D].reshape(n, G, D)
    v = p[:, offs[2]:offs[2] + G * VD].reshape(n, G, VD)
    assert rms_err(rows[:, offs[0]:offs[0] + H * D].reshape(n, H, D), R.rotate_interleaved(q, pos, freqs)) < limit
    held = slots >= 0
    assert rms_err(kc[slots[held]], R.rotate_interleaved(k, pos, freqs)[held]) < limit
    assert np.array_equal(vc[slots[held]], v[held])
    free = np.setdiff1d(np.arange(nb * BS), slots)
    assert (kc[free] == 50.0).all() and (vc[free] == 50.0).all()          # nothing else was written
    assert np.array_equal(rows[:, :8], p[:, :8]) and np.array_equal(rows[:, offs[2]:], p[:, offs[2]:])


@pytest.mark.parametrize("H,G,D,VD,pairs", PREP)
@pytest.mark.parametrize("tied", [False, True])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_norms_over_whole_projections(hb, cuda, H, G, D, VD, pairs, tied, dtype):
    rng = np.random.default_rng(D + 1)
    n, nb, eps = 20, 3, 1e-2
    VD = D if tied else VD
    offs = (0, (H * D + 7) // 8 * 8, (H * D + 7) // 8 * 8 + (G * D + 7) // 8 * 8)
    p = rng.standard_normal((n, offs[2] + (G * VD + 7) // 8 * 8))
    p[3] *= 1e-3  # eps decides here
    p = rounded(p, dtype)
    bq, bk, wq, wk = (rounded(rng.standard_normal(s) * f + c, "f32") for s, f, c in
                      ((H * D, 0.5, 0), (G * D, 0.5, 0), (H * D, 0.3, 1), (G * D, 0.3, 1)))
    bq[:], bk[:] = (bq, bk) if D % 2 else (bq * 1e-3, bk * 1e-3)
    slots = np.random.default_rng(1).permutation(nb * BS)[:n]
    rows, kc, vc, ks = prep(hb, dtype, p, offs, H, G, D, VD, np.arange(n), slots, nb, q_bias=bq, k_bias=bk, q_norm=wq,
                            k_norm=wk, eps=eps, tied=tied)
    limit = 4e-3 if dtype == "bf16" else 2e-6
    k_raw = p[:, offs[1]:offs[1] + G * D] + bk
    q = R.rms_norm(p[:, :H * D] + bq, wq, eps).reshape(n, H, D)
    k = R.rms_norm(k_raw, wk, eps).reshape(n, G, D)
    got_q, got_k = rows[:, :H * D].reshape(n, H, D), kc[slots]
    if not tied:
        assert rms_err(got_q, q) < limit and rms_err(got_k, k) < limit
        assert np.array_equal(vc[slots], p[:, offs[2]:offs[2] + G * VD].reshape(n, G, VD))
        return
    assert rms_err(got_k, k_raw.reshape(n, G, D)) < limit and (vc == 50.0).all()
    assert rms_err(ks[slots], 1.0 / np.sqrt((k_raw ** 2).mean(axis=1) + eps)) < limit
    # what counts are the scores: queries times the key norm's weight meet raw keys times their scale
    for h in range(H):
        g = h // (H // G)
        assert rms_err((got_q[:, h] @ got_k[:, g].T) * ks[slots][None, :], q[:, h] @ k[:, g].T) < 2 * limit


# ------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("slope,cubic,limit,shift", [(1.0, 0.0, np.inf, 0.0), (2 * (2 / np.pi) ** 0.5, 0.044715, np.inf, 0.0),
                                                     (1.702, 0.0, 0.8, 1.0), (1.3, 0.01, 2.0, -0.5)])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_gated_activations(hb, cuda, slope, cubic, limit, shift, dtype):
    import torch

    rng = np.random.default_rng(3)
    gu = rounded(3.0 * rng.standard_normal((19, 2 * 45)), dtype)
    gu[0, :8] = [-300, -90, -20, 0, 20, 90, 300, 1e4]
    gu = rounded(gu, dtype)
    t, out = put(gu, dtype), put(np.zeros((19, 45)), dtype)
    spec = hb.GatedActSpec(slope, cubic, limit, shift)
    hb.check(hb.lib.hb_gated_act(None, out.data_ptr(), t.data_ptr(), 19, 45, C.byref(spec), dt(hb, dtype)))
    torch.cuda.synchronize()
    g, u = np.minimum(gu[:, :45], limit), np.clip(gu[:, 45:], -limit, limit)
    want = g * R.sigmoid(slope * (g + cubic * g ** 3)) * (u + shift)
    if cubic == 0.044715:
        np.testing.assert_allclose(want, R.gelu_tanh(gu[:, :45]) * gu[:, 45:], rtol=1e-9, atol=1e-9)
    assert rms_err(back(out)[1:], want[1:]) < (4e-3 if dtype == "bf16" else 2e-6)
    np.testing.assert_allclose(back(out)[0], want[0], rtol=1e-2, atol=1e-6)


class Experts:
    """A whole mixture: routing, sorted rows, two grouped products, the weighted sum."""

    def __init__(self, hb, rows, width, experts, top, ff, dtype, m_pad, limit=1.4, seed=0, skew=0.0, shared_ff=0):
        import torch

        rng = np.random.default_rng(seed)
        self.hb, self.dtype, self.rows, self.width, self.top, self.ff, self.limit = hb, dtype, rows, width, top, ff, limit
        self.ld = (width + 7) // 8 * 8
        ffp = (ff + 7) // 8 * 8
        self.h = np.zeros((rows, self.ld))
        self.h[:, :width] = rng.standard_normal((rows, width))
        self.h = rounded(self.h, dtype)
        self.router = rounded(rng.standard_normal((experts, width)) * width ** -0.5, dtype)
        self.bias = rounded(rng.standard_normal(experts) - skew * np.arange(experts), "f32")
        self.w = {}
        up = np.zeros((experts, 2 * ffp, self.ld))
        down = np.zeros((experts, self.ld, ffp))
        for e in range(experts):
            for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
                self.w[f"e{e}.{name}"] = rounded(1.5 * rng.standard_normal(shape) * shape[1] ** -0.5, dtype)
            up[e, :ff, :width] = self.w[f"e{e}.gate"]
            up[e, ffp:ffp + ff, :width] = self.w[f"e{e}.up"]
            down[e, :width, :ff] = self.w[f"e{e}.down"]
        n, picks = rows * top, top + (1 if shared_ff else 0)
        tiles = min(experts, n) + n // m_pad + (-(-rows // m_pad) if shared_ff else 0)
        sfp = (shared_ff + 7) // 8 * 8
        s_up, s_down = np.zeros((2 * sfp, self.ld)), np.zeros((self.ld, sfp))
        if shared_ff:
            for name, shape in (("gate", (shared_ff, width)), ("up", (shared_ff, width)), ("down", (width, shared_ff))):
                self.w["shared." + name] = rounded(1.5 * rng.standard_normal(shape) * shape[1] ** -0.5, dtype)
            s_up[:shared_ff, :width], s_up[sfp:sfp + shared_ff, :width] = self.w["shared.gate"], self.w["shared.up"]
            s_down[:width, :shared_ff] = self.w["shared.down"]
        wide = max(ffp, sfp)
        z32 = lambda *s: torch.zeros(s, device="cuda", dtype=torch.int32)
        self.ids, self.rank, self.place = z32(rows, picks), z32(rows, picks), z32(rows, picks)
        self.weight = torch.zeros((rows, picks), device="cuda")
        self.count, self.first, self.tiles = z32(experts + 1), z32(experts + 1), z32(tiles)
        r = hb.MoeRouting(experts, top, m_pad, tiles, *(t.data_ptr() for t in (self.ids, self.rank, self.place, self.weight,
                                                                              self.count, self.first, self.tiles)),
                          1 if shared_ff else 0)
        th, tr, tb = put(self.h, dtype), put(self.router, dtype), put(self.bias)
        tu, td, tsu, tsd = put(up, dtype), put(down, dtype), put(s_up, dtype), put(s_down, dtype)
        x = put(np.zeros((tiles * m_pad, self.ld)), dtype)
        act, y = put(np.zeros((tiles * m_pad, wide)), dtype), put(np.zeros((tiles * m_pad, self.ld)), dtype)
        self.shared_limit = 0.6
        spec, spec2 = hb.GatedActSpec(1.702, 0.0, limit, 1.0), hb.GatedActSpec(1.702, 0.0, self.shared_limit, 1.0)
        for _ in range(2):  # the second run finds the counters as the first one left them
            hb.check(hb.lib.hb_moe_route_top(None, C.byref(r), th.data_ptr(), self.ld, tr.data_ptr(), tb.data_ptr(), rows, width,
                                             dt(hb, dtype)))
            hb.check(hb.lib.hb_moe_gather(None, C.byref(r), x.data_ptr(), th.data_ptr(), self.ld, rows, dt(hb, dtype)))
        likely = max(1, tiles // 2)
        gu_gemm = hb.GroupedGemm(experts, 2 * ffp, self.ld, m_pad, tiles, likely, self.tiles.data_ptr(), self.ld, wide, 1, 0, spec,
                                 tsu.data_ptr() if shared_ff else None, 2 * sfp, self.ld if shared_ff else 0, spec2)
        down_gemm = hb.GroupedGemm(experts, self.ld, ffp, m_pad, tiles, likely, self.tiles.data_ptr(), wide, self.ld, 0, 0, spec,
                                   tsd.data_ptr() if shared_ff else None, self.ld if shared_ff else 0, sfp, spec2)
        if dtype == "bf16":
            hb.check(hb.lib.hb_gemm_grouped(None, act.data_ptr(), x.data_ptr(), tu.data_ptr(), C.byref(gu_gemm), dt(hb, dtype)))
        else:
            gu = put(np.zeros((tiles * m_pad, 2 * wide)), dtype)
            gu_gemm.gated, gu_gemm.ldy = 0, 2 * wide
            hb.check(hb.lib.hb_gemm_grouped(None, gu.data_ptr(), x.data_ptr(), tu.data_ptr(), C.byref(gu_gemm), dt(hb, dtype)))
            gu_gemm.ldy = wide
            hb.check(hb.lib.hb_gated_act_grouped(None, act.data_ptr(), gu.data_ptr(), 2 * wide, C.byref(gu_gemm), dt(hb, dtype)))
        hb.check(hb.lib.hb_gemm_grouped(None, y.data_ptr(), act.data_ptr(), td.data_ptr(), C.byref(down_gemm), dt(hb, dtype)))
        # the weighted sum goes into a plain residual stream together with a shared output and a bias
        self.x0, self.shared, self.o_bias = rng.standard_normal((rows, width)), rng.standard_normal((rows, self.ld)), \
            rng.standard_normal(width)
        self.norm = rng.uniform(0.5, 1.5, width)
        tx, ts, to, tn, one = put(self.x0), put(self.shared), put(self.o_bias), put(self.norm), put(np.ones(1))
        out = put(np.zeros((rows, self.ld)), dtype)
        m = hb.StreamMixArgs(one.data_ptr(), one.data_ptr(), one.data_ptr(), tn.data_ptr(), None, None, 0.0, to.data_ptr(),
                             y.data_ptr(), self.place.data_ptr(), self.weight.data_ptr(), picks)
        hb.check(hb.lib.hb_streams_mix_ex(None, tx.data_ptr(), out.data_ptr(), ts.data_ptr(), None, self.ld, C.byref(m), rows, 1,
                                          width, self.ld, 1e-5, dt(hb, dtype)))
        torch.cuda.synchronize()
        self.x1, self.normed = back(tx), back(out)[:, :width]
        self.experts = experts
        self.m_pad = m_pad

    def check(self):
        h = self.h[:, :self.width]
        chosen, weight = R.route(h, self.router, self.bias, self.top)
        clear = R.route_margin(h, self.router, self.bias, self.top) > 1e-4
        assert clear.mean() > 0.9
        ids, place, weights = self.ids.cpu().numpy(), self.place.cpu().numpy(), back(self.weight)
        tiles = self.tiles.cpu().numpy()
        # every place once, in a tile of its own expert
        assert len(np.unique(place)) == place.size and np.array_equal(tiles[place // self.m_pad], ids)
        used = sum(-(-int((ids == e).sum()) // self.m_pad) for e in range(self.experts + 1))
        assert (tiles[:used] >= 0).all() and (tiles[used:] == -1).all()
        if ids.shape[1] > self.top:
            assert (ids[:, self.top] == self.experts).all() and (weights[:, self.top] == 1.0).all()
        ids, weights = ids[:, :self.top], weights[:, :self.top]
        assert np.array_equal(np.sort(ids[clear]), np.sort(chosen[clear]))
        same = (ids == chosen).all(axis=1)
        np.testing.assert_allclose(weights[same], weight[same], atol=2e-5)
        assert not self.count.cpu().numpy().any()
        want = self.x0 + self.shared[:, :self.width] + self.o_bias
        for t in range(self.rows):
            for e, p in zip(chosen[t], weight[t]):
                want[t] += p * R.clamped_expert(h[t:t + 1], R.sub(self.w, f"e{e}."), self.limit)[0]
        if "shared.up" in self.w:
            want += R.clamped_expert(h, R.sub(self.w, "shared."), self.shared_limit)
        limit = 5e-3 if self.dtype == "bf16" else 2e-6
        assert rms_err(self.x1[clear], want[clear]) < limit
        assert rms_err(self.normed[clear], R.rms_norm(want, self.norm, 1e-5)[clear]) < 2 * limit


MOE = [  # rows, width, experts, top, ff, m_pad
    (1, 64, 5, 2, 40, 16), (7, 72, 3, 3, 24, 16), (40, 75, 40, 6, 11, 16), (300, 128, 4, 1, 136, 64), (530, 96, 9, 2, 56, 128),
    (64, 520, 1, 1, 264, 64), (33, 64, 70, 1, 16, 32), (600, 64, 8, 3, 1000, 112),
]


@pytest.mark.parametrize("rows,width,experts,top,ff,m_pad", MOE)
@pytest.mark.parametrize("shared", ["no", "narrower", "wider"])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_mixture_of_experts(hb, cuda, rows, width, experts, top, ff, m_pad, shared, dtype):
    """shared: one more expert that every row passes through, of another width and limit."""
    shared_ff = {"no": 0, "narrower": max(3, ff // 3), "wider": 2 * ff + 70}[shared]
    Experts(hb, rows, width, experts, top, ff, dtype, m_pad, seed=rows, shared_ff=shared_ff).check()


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_everybody_chooses_the_same_experts(hb, cuda, dtype):
    """A router bias that overrides everything: two experts get all rows, the others none."""
    e = Experts(hb, 150, 64, 6, 2, 32, dtype, 32, seed=1, skew=60.0)
    assert set(e.ids.cpu().numpy().ravel()) == {0, 1}
    e.check()


def test_equal_logits_go_to_the_lower_expert(hb, cuda):
    import torch

    z = torch.zeros((3, 64), device="cuda")
    router, bias = torch.zeros((37, 64), device="cuda"), torch.zeros(37, device="cuda")
    i32 = lambda *s: torch.zeros(s, device="cuda", dtype=torch.int32)
    t = [i32(3, 5), i32(3, 5), i32(3, 5), torch.zeros((3, 5), device="cuda"), i32(38), i32(37), i32(20)]
    r = hb.MoeRouting(37, 5, 16, 20, *(x.data_ptr() for x in t))
    hb.check(hb.lib.hb_moe_route_top(None, C.byref(r), z.data_ptr(), 64, router.data_ptr(), bias.data_ptr(), 3, 64, hb.F32))
    torch.cuda.synchronize()
    assert t[0].cpu().numpy().tolist() == [[0, 1, 2, 3, 4]] * 3
    np.testing.assert_allclose(t[3].cpu().numpy(), 0.2, rtol=1e-6)
    with pytest.raises(hb.HbError, match="bad shape"):
        bad = hb.MoeRouting(37, 5, 16, 3, *(x.data_ptr() for x in t))
        hb.check(hb.lib.hb_moe_route_top(None, C.byref(bad), z.data_ptr(), 64, router.data_ptr(), bias.data_ptr(), 3, 64, hb.F32))
