"""Host side, no GPU: the plain Biberax mechanisms against second formulations of the same formulas."""
import math

import numpy as np
import pytest

from oracle import biberax_ref as R


def test_rotation_is_a_complex_product_and_keeps_the_rest():
    rng = np.random.default_rng(0)
    x = rng.standard_normal((9, 2, 14))
    pos = np.array([0, 1, 2, 50, 51, 999, 7, 8, 9])
    f = R.rotation_frequencies(300.0, 10)
    np.testing.assert_allclose(f, 300.0 ** (-np.arange(0, 10, 2) / 10))
    y = R.rotate_interleaved(x, pos, f)
    z = (x[:, :, 0:10:2] + 1j * x[:, :, 1:10:2]) * np.exp(1j * pos[:, None, None] * f[None, None, :])
    np.testing.assert_allclose(y[:, :, 0:10:2], z.real, atol=1e-12)
    np.testing.assert_allclose(y[:, :, 1:10:2], z.imag, atol=1e-12)
    assert np.array_equal(y[:, :, 10:], x[:, :, 10:])
    # scores of rotated pairs depend on the distance only
    q, k = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))
    s = [float((R.rotate_interleaved(q, [p + 5], f) * R.rotate_interleaved(k, [p], f)).sum()) for p in (0, 17, 400)]
    np.testing.assert_allclose(s, s[0], rtol=1e-9)


def test_stretched_wavelengths():
    scaling = dict(factor=8.0, low=1.0, high=4.0, original=256)
    plain, got = R.rotation_frequencies(1e4, 64), R.rotation_frequencies(1e4, 64, scaling)
    wave = 2 * math.pi / plain
    short, long = wave < 256 / 4.0, wave > 256 / 1.0
    assert short.any() and long.any() and (~short & ~long).any()
    np.testing.assert_array_equal(got[short], plain[short])
    np.testing.assert_allclose(got[long], plain[long] / 8)
    between = ~short & ~long
    assert ((got[between] < plain[between]) & (got[between] > plain[between] / 8)).all()
    assert (np.diff(got) < 0).all()


def test_distance_buckets():
    for buckets, far in ((16, 128), (32, 100), (10, 1000), (9, 40), (2, 5), (1, 4)):
        b = [R.distance_bucket(n, buckets, far) for n in range(2 * far)]
        half = buckets // 2
        assert b[:half] == list(range(half)) and (np.diff(b) >= 0).all() and max(b) == buckets - 1
        assert all(x == buckets - 1 for x in b[far:])
        if buckets > 4:
            assert b[far // 4] < buckets - 1  # the upper half is spread out
    # powers of two: one bucket per factor of sqrt(2)
    assert [R.distance_bucket(n, 16, 128) for n in (8, 11, 12, 16, 22, 23, 32, 64, 127, 128)] == [8, 8, 9, 10, 10, 11, 12, 14, 15, 15]


def test_a_sink_is_one_more_key_without_a_value():
    rng = np.random.default_rng(1)
    n, H, G, D, V = 12, 4, 2, 6, 5
    q, k, v = rng.standard_normal((n, H, D)), rng.standard_normal((n, G, D)), rng.standard_normal((n, G, V))
    sink, bias = rng.standard_normal(H), rng.standard_normal((n, n, H))
    got = R.sink_attention(q, k, v, 0.4, R.causal_mask(n), sink, bias)
    for i in range(n):
        for h in range(H):
            s = [0.4 * q[i, h] @ k[j, h // 2] + bias[i, j, h] for j in range(i + 1)] + [sink[h]]
            p = np.exp(s) / np.exp(s).sum()
            np.testing.assert_allclose(got[i, h], sum(p[j] * v[j, h // 2] for j in range(i + 1)), atol=1e-12)
    # a zero sink adds one to the denominator
    one = R.sink_attention(q[:1], k[:1], v[:1], 0.4, R.causal_mask(1), np.zeros(H))
    e = np.exp(0.4 * q[0, 0] @ k[0, 0])
    np.testing.assert_allclose(one[0, 0], e / (1 + e) * v[0, 0])


def test_chunks_count_from_the_start():
    m = R.chunk_mask(10, 4)
    assert [[int(x) for x in np.flatnonzero(r)] for r in m] == \
        [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [4], [4, 5], [4, 5, 6], [4, 5, 6, 7], [8], [8, 9]]


def test_experts_and_routing():
    rng = np.random.default_rng(2)
    h, w, b = rng.standard_normal((30, 8)), rng.standard_normal((6, 8)), rng.standard_normal(6)
    chosen, weight = R.route(h, w, b, 3)
    z = h @ w.T + b
    for t in range(30):
        assert set(chosen[t]) == set(np.argsort(z[t])[-3:])
        np.testing.assert_allclose(weight[t], np.exp(z[t, chosen[t]]) / np.exp(z[t, chosen[t]]).sum())
    assert (R.route_margin(h, w, b, 3) >= 0).all() and np.isinf(R.route_margin(h, w, b, 6)).all()
    e = {"gate": rng.standard_normal((5, 8)) * 3, "up": rng.standard_normal((5, 8)) * 3, "down": rng.standard_normal((8, 5))}
    y = R.clamped_expert(h, e, 0.7)
    g, u = np.minimum(h @ e["gate"].T, 0.7), np.maximum(np.minimum(h @ e["up"].T, 0.7), -0.7)
    np.testing.assert_allclose(y, (g / (1 + np.exp(-1.702 * g)) * (u + 1)) @ e["down"].T)
    # everybody chosen with equal logits is the mean
    mlp = {"router": {"experts": 2, "top": 2}, "expert": {"ff": 5, "limit": 0.7}}
    both = {"router": np.zeros((2, 8)), "router.b": np.zeros(2), **{f"e{i}.{k}": v for i in (0, 1) for k, v in e.items()}}
    np.testing.assert_allclose(R.moe_ffn(h, both, mlp), y)


def test_gelu():
    z = np.linspace(-6, 6, 50)
    exact = 0.5 * z * (1 + np.array([math.erf(x / math.sqrt(2)) for x in z]))
    np.testing.assert_allclose(R.gelu_tanh(z), exact, atol=2e-3)


@pytest.mark.parametrize("change", ["prefix", "order"])
def test_the_model_is_causal_and_positions_matter(change):
    layer1 = {"type": "attention", "mixer": dict(heads=2, kv_heads=1, dim=8, vdim=6, scale=0.3, mask=dict(size=5),
                                                 rot=dict(base=50.0, dims=4)), "mlp": {"kind": "dense", "ff": 12}}
    layer2 = {"type": "attention_2", "mixer": dict(heads=2, kv_heads=2, dim=8, vdim=8, scale=0.3, bias_max=9),
              "mlp": {"kind": "moe", "router": dict(experts=3, top=2), "expert": dict(ff=6, limit=1.0)}}
    c = {"width": 16, "vocab": 20, "norm": {"eps": 1e-5}, "layers": [layer1, layer2]}
    w = R.random_weights(c, seed=3, buckets=6)
    toks = np.random.default_rng(4).integers(0, 20, 18)
    full = R.forward(c, w, toks)
    if change == "prefix":
        np.testing.assert_allclose(R.forward(c, w, toks[:11]), full[:11], atol=1e-12)
    else:
        swapped = toks.copy()
        swapped[[2, 3]] = toks[[3, 2]] if toks[2] != toks[3] else (toks[[3, 2]] + 1) % 20
        assert np.abs(R.forward(c, w, swapped)[-1] - full[-1]).max() > 1e-6
