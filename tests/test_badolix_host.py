"""Host side, no GPU: the plain Badolix mechanisms against second formulations of the same formulas."""
import math

import numpy as np
import pytest

from oracle import badolix_ref as R


def test_rotated_halves_are_a_complex_product():
    rng = np.random.default_rng(0)
    x, pos = rng.standard_normal((9, 2, 14)), np.array([0, 1, 2, 50, 51, 999, 7, 8, 9])
    f, gain = R.rotation(300.0, 10)
    assert gain == 1.0
    np.testing.assert_allclose(f, 300.0 ** (-np.arange(0, 10, 2) / 10))
    z = (x[:, :, :5] + 1j * x[:, :, 5:10]) * np.exp(1j * pos[:, None, None] * f[None, None, :])
    y = R.rotate_halves(x, pos, f, 1.5)
    np.testing.assert_allclose(y[:, :, :5], 1.5 * z.real, atol=1e-12)
    np.testing.assert_allclose(y[:, :, 5:10], 1.5 * z.imag, atol=1e-12)
    assert np.array_equal(y[:, :, 10:], x[:, :, 10:])
    np.testing.assert_allclose(R.rotation(300.0, 10, dict(factor=4.0))[0], f / 4)


def test_ramped_frequencies():
    base, dims, s = 1e4, 64, dict(factor=8.0, original=512, fast=16.0, slow=1.0)
    plain, (got, gain) = R.rotation(base, dims)[0], R.rotation(base, dims, s)
    turns = s["original"] * plain / (2 * math.pi)  # whole turns of a pair within the original length
    assert gain == pytest.approx(0.1 * math.log(8.0) + 1.0)
    # a pair's number by its turns: fast ones keep their frequency, slow ones are divided
    kept, slowed = got == plain, np.isclose(got, plain / 8)
    assert kept[turns > 16 * 1.4].all() and slowed[turns < 1 / 1.4].all()
    between = ~kept & ~slowed
    assert between.any() and (np.diff(got) < 0).all()
    share = (plain[between] - got[between]) / (plain[between] - plain[between] / 8)
    np.testing.assert_allclose(np.diff(share), np.diff(share)[0])  # linear in the pair's number
    # ends of the ramp outside the pairs
    assert np.array_equal(R.rotation(10.0, 8, dict(factor=2.0, original=1e9, fast=1.0, slow=0.5))[0], R.rotation(10.0, 8)[0])


def test_capped_attention_by_hand():
    rng = np.random.default_rng(1)
    n, H, G, D, V = 14, 4, 2, 6, 5
    q, k, v = 3 * rng.standard_normal((n, H, D)), rng.standard_normal((n, G, D)), rng.standard_normal((n, G, V))
    got = R.capped_attention(q, k, v, 0.7, R.window_mask(n, 5, 2), 2.0)
    for i in range(n):
        js = [j for j in range(i + 1) if i - j < 5 or j < 2]
        for h in range(H):
            s = np.array([2.0 * math.tanh(0.7 * q[i, h] @ k[j, h // 2] / 2.0) for j in js])
            p = np.exp(s) / np.exp(s).sum()
            np.testing.assert_allclose(got[i, h], sum(a * v[j, h // 2] for a, j in zip(p, js)), atol=1e-12)


def test_latent_attention_runs_over_the_latent_itself():
    """The heads' key matrix moved to the queries and their value matrix to the outputs."""
    rng = np.random.default_rng(2)
    n, W, m = 11, 12, dict(heads=3, dim=5, rot_dim=4, vdim=6, kv_rank=7, scale=0.4,
                           rot=dict(base=20.0, dims=4, scaling=dict(factor=4.0, original=32, fast=4.0, slow=1.0)))
    w = {"q": (27, W), "dkv": (11, W), "dkv.norm": (7,), "uk": (15, 7), "uv": (18, 7), "o": (W, 18)}
    w = {k: rng.standard_normal(s) for k, s in w.items()}
    h = rng.standard_normal((n, W))
    f, gain = R.rotation(20.0, 4, m["rot"]["scaling"])
    c = R.rms_norm((h @ w["dkv"].T)[:, :7], w["dkv.norm"], 1e-5)
    shared = R.rotate_halves((h @ w["dkv"].T)[:, None, 7:], np.arange(n), f, gain)[:, 0]
    q = (h @ w["q"].T).reshape(n, 3, 9)
    qr = R.rotate_halves(q[:, :, 5:], np.arange(n), f, gain)
    out = []
    for a in range(3):
        over = np.concatenate([q[:, a, :5] @ w["uk"][5 * a:5 * a + 5], qr[:, a]], axis=1)
        s = np.where(np.tril(np.ones((n, n))) > 0, 0.4 * over @ np.concatenate([c, shared], axis=1).T, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out.append((p / p.sum(axis=1, keepdims=True)) @ c @ w["uv"][6 * a:6 * a + 6].T)
    np.testing.assert_allclose(R.latent_mixer(h, w, m, 1e-5), np.concatenate(out, axis=1) @ w["o"].T, atol=1e-10)


def test_shared_keys_and_values():
    rng = np.random.default_rng(3)
    m = dict(heads=4, kv_heads=2, dim=6, vdim=5, scale=0.3, softcap=4.0, mask=dict(size=4, keep_first=1), rot=dict(base=9.0, dims=4))
    w = {k: rng.standard_normal(s) for k, s in (("q", (24, 8)), ("k", (12, 8)), ("v", (10, 8)), ("o", (8, 20)))}
    h, h2 = rng.standard_normal((9, 8)), rng.standard_normal((9, 8))
    y, held = R.attention_mixer(h, w, m)
    again, _ = R.attention_mixer(h, {k: w[k] for k in ("q", "o")}, m, held)
    np.testing.assert_array_equal(y, again)
    assert np.abs(R.attention_mixer(h2, w, m, held)[0] - R.attention_mixer(h2, w, m)[0]).max() > 1e-3


def test_convolution_and_state_space_as_sums():
    rng = np.random.default_rng(4)
    n, H, V, N = 13, 3, 4, 5
    x, w, b = rng.standard_normal((n, 6)), rng.standard_normal((6, 4)), rng.standard_normal(6)
    padded = np.concatenate([np.zeros((3, 6)), x])
    np.testing.assert_allclose(R.causal_conv(x, w, b), sum(padded[j:j + n] * w[:, j] for j in range(4)) + b, atol=1e-12)
    v, B, Cq = rng.standard_normal((n, H, V)), rng.standard_normal((n, H, N)), rng.standard_normal((n, H, N))
    dt, a_log, D = R.softplus(rng.standard_normal((n, H))), rng.standard_normal(H), rng.standard_normal(H)
    y, S = R.state_space(v, B, Cq, dt, a_log, D)
    total = np.cumsum(-np.exp(a_log) * dt, axis=0)
    for h in range(H):
        for i in range(n):
            want = D[h] * v[i, h] + sum(np.exp(total[i, h] - total[j, h]) * dt[j, h] * (Cq[i, h] @ B[j, h]) * v[j, h] for j in range(i + 1))
            np.testing.assert_allclose(y[i, h], want, atol=1e-10)
        np.testing.assert_allclose(S[h], sum(np.exp(total[-1, h] - total[j, h]) * dt[j, h] * np.outer(B[j, h], v[j, h]) for j in range(n)), atol=1e-10)
    np.testing.assert_allclose(R.softplus(np.array([-800.0, 0.0, 800.0])), [0.0, math.log(2), 800.0])


def test_gate_then_norm():
    rng = np.random.default_rng(5)
    y, z, w = (rng.standard_normal(s) for s in ((4, 12), (4, 12), (12,)))
    got = R.gated_norm(y, z, w, 3, 1e-2)
    for t in range(4):
        for p in range(3):
            g = np.array([y[t, i] * z[t, i] / (1 + math.exp(-z[t, i])) for i in range(4 * p, 4 * p + 4)])
            np.testing.assert_allclose(got[t, 4 * p:4 * p + 4], g / math.sqrt((g * g).mean() + 1e-2) * w[4 * p:4 * p + 4])


def test_groups_limit_the_choice():
    s = np.array([[0.9, 0.1, 0.5, 0.55, 0.89, 0.2]])
    np.testing.assert_allclose(R.group_scores(s, 3), [[1.0, 1.05, 1.09]])
    z = np.log(s / (1 - s))
    router = z.T  # a token of one channel
    chosen, weight = R.route(np.ones((1, 1)), router, 2, dict(count=3, keep=1))
    assert chosen.tolist() == [[4, 5]]  # not the best expert of all
    np.testing.assert_allclose(weight, [[0.89 / 1.09, 0.2 / 1.09]])
    assert R.route(np.ones((1, 1)), router, 2, dict(count=3, keep=3))[0].tolist() == [[0, 4]] == R.route(np.ones((1, 1)), router, 2)[0].tolist()
    assert R.route_margin(np.ones((1, 1)), router, 2, dict(count=3, keep=1))[0] == pytest.approx((1.09 - 1.05) / s.std())
    np.testing.assert_allclose(R.group_scores(s, 6), s)


@pytest.mark.parametrize("change", ["prefix", "order"])
def test_the_model_is_causal_and_positions_matter(change):
    rot = dict(base=50.0, dims=4)
    attn = dict(heads=2, kv_heads=1, dim=8, vdim=6, scale=0.3, softcap=5.0, mask=dict(size=5, keep_first=1), rot=rot)
    moe = {"kind": "moe", "router": dict(experts=4, top=2, groups=dict(count=2, keep=1)), "expert": dict(ff=6)}
    layers = [{"type": "attention", "mixer": attn, "mlp": {"kind": "dense", "ff": 12}},
              {"type": "mamba2", "mixer": dict(heads=4, vdim=4, state=6, groups=2, conv=3, norm_groups=2), "mlp": moe},
              {"type": "latent_attention", "mixer": dict(heads=2, dim=4, rot_dim=4, vdim=3, kv_rank=6, scale=0.4, rot=rot), "mlp": None},
              {"type": "attention", "mixer": dict(attn, kv_from=0), "mlp": moe}]
    c = {"width": 16, "vocab": 20, "norm": {"eps": 1e-5}, "embedding": {"scale": 0.5}, "residual_mult": 0.7, "logit_scale": 3.0, "layers": layers}
    w = R.random_weights(c, seed=3)
    toks = np.random.default_rng(4).integers(0, 20, 18)
    full = R.forward(c, w, toks)
    if change == "prefix":
        np.testing.assert_allclose(R.forward(c, w, toks[:11]), full[:11], atol=1e-12)
        np.testing.assert_allclose(R.forward(dict(c, logit_scale=6.0), w, toks), 2 * full, atol=1e-9)
    else:
        swapped = toks.copy()
        swapped[[2, 3]] = toks[[3, 2]] if toks[2] != toks[3] else (toks[[3, 2]] + 1) % 20
        assert np.abs(R.forward(c, w, swapped)[-1] - full[-1]).max() > 1e-6
