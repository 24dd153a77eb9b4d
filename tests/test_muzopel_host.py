"""Host side, no GPU: the plain Muzopel mechanisms against second formulations of the same formulas."""
import math

import numpy as np
import pytest

from oracle import muzopel_ref as R


def test_rotated_neighbours_are_a_complex_product():
    rng = np.random.default_rng(0)
    x, pos = rng.standard_normal((9, 2, 14)), np.array([0, 1, 2, 50, 51, 999, 7, 8, 9])
    f, gain = R.rotation(300.0, 10, dict(factor=4.0, original=90, fast=4.0, slow=1.0))
    z = (x[:, :, 0:10:2] + 1j * x[:, :, 1:10:2]) * gain * np.exp(1j * pos[:, None, None] * f[None, None, :])
    y = R.rotate_neighbours(x, pos, f, gain)
    np.testing.assert_allclose(y[:, :, 0:10:2], z.real, atol=1e-12)
    np.testing.assert_allclose(y[:, :, 1:10:2], z.imag, atol=1e-12)
    assert np.array_equal(y[:, :, 10:], x[:, :, 10:]) and gain == pytest.approx(1 + 0.1 * math.log(4))


def test_norm_in_parts():
    rng = np.random.default_rng(1)
    x, w = rng.standard_normal((4, 12)), rng.standard_normal(12)
    got = R.parts_norm(x, w, 3, 1e-2)
    for t in range(4):
        for i in range(12):
            part = x[t, i // 4 * 4:i // 4 * 4 + 4]
            assert got[t, i] == pytest.approx(x[t, i] / math.sqrt(sum(part ** 2) / 4 + 1e-2) * w[i])
    np.testing.assert_allclose(R.parts_norm(x, w, 1, 1e-2), R.rms_norm(x, w, 1e-2))


@pytest.mark.parametrize("taps", [1, 2, 5])
def test_inputs_with_their_past(taps):
    rng = np.random.default_rng(taps)
    x, w = rng.standard_normal((11, 6)), rng.standard_normal((6, taps))
    got = R.with_past(x, w)
    for c in range(6):
        np.testing.assert_allclose(got[:, c], x[:, c] + np.convolve(x[:, c], w[c, ::-1])[:11], atol=1e-12)


def test_depth_sums():
    rng = np.random.default_rng(2)
    xs, w = [rng.standard_normal((3, 4)) for _ in range(5)], rng.standard_normal(5)
    np.testing.assert_allclose(R.depth_sum(xs, w), np.tensordot(w, np.stack(xs), 1), atol=1e-12)
    with pytest.raises(ValueError):
        R.depth_sum(xs, w[:4])


def test_latent_attention_runs_over_the_latent_itself():
    """The heads' key matrix moved to the queries and their value matrix to the outputs, gates among them."""
    rng = np.random.default_rng(3)
    n, W, Q, m = 11, 12, 8, dict(heads=3, dim=5, rot_dim=4, vdim=6, kv_rank=7, scale=0.4,
                                 rot=dict(base=20.0, dims=4, scaling=dict(factor=4.0, original=32, fast=4.0, slow=1.0)))
    shapes = {"dq": (Q, W), "dq.norm": (Q,), "uq": (27, Q), "dkv": (11, W), "dkv.norm": (7,), "uk": (15, 7), "uv": (18, 7), "g": (3, W),
              "o": (W, 18)}
    w = {k: rng.standard_normal(s) for k, s in shapes.items()}
    h = rng.standard_normal((n, W))
    own = R.latent_mixer(h, w, m, 1e-5)
    f, gain = R.rotation(20.0, 4, m["rot"]["scaling"])
    cq = R.rms_norm(h @ w["dq"].T, w["dq.norm"], 1e-5)
    c = R.rms_norm((h @ w["dkv"].T)[:, :7], w["dkv.norm"], 1e-5)
    k_rot = R.rotate_neighbours((h @ w["dkv"].T)[:, None, 7:], np.arange(n), f, gain)[:, 0]
    for gated in (True, False):
        q = (cq if gated else h[:, :Q]) @ w["uq"].T
        out = []
        for a in range(3):
            qa = q[:, a * 9:a * 9 + 9]
            meet = qa[:, :5] @ w["uk"][a * 5:a * 5 + 5]
            turned = R.rotate_neighbours(qa[:, None, 5:], np.arange(n), f, gain)[:, 0]
            s = np.where(np.tri(n, dtype=bool), (meet @ c.T + turned @ k_rot.T) * 0.4, -np.inf)
            p = np.exp(s - s.max(axis=1, keepdims=True))
            o = (p / p.sum(axis=1, keepdims=True)) @ c @ w["uv"][a * 6:a * 6 + 6].T
            out.append(o / (1 + np.exp(-(h @ w["g"][a])))[:, None] if gated else o)
        want = np.concatenate(out, axis=1) @ w["o"].T
        if gated:
            np.testing.assert_allclose(own, want, atol=1e-10)
        else:
            other = {k: v for k, v in w.items() if k not in ("dq", "dq.norm", "uq", "g")}
            other["q"] = np.concatenate([w["uq"], np.zeros((27, W - Q))], axis=1)
            np.testing.assert_allclose(R.latent_mixer(h, other, m, 1e-5), want, atol=1e-10)


def test_routing_by_hand():
    rng = np.random.default_rng(4)
    h, router, corr = rng.standard_normal((20, 6)), rng.standard_normal((7, 6)), rng.standard_normal(7)
    chosen, weight = R.route(h, router, corr, 3)
    margin = R.route_margin(h, router, corr, 3)
    for t in range(20):
        e = [math.exp(router[i] @ h[t]) for i in range(7)]
        s = [v / sum(e) for v in e]
        order = sorted(range(7), key=lambda i: -(s[i] + corr[i]))
        assert list(chosen[t]) == order[:3]
        np.testing.assert_allclose(weight[t], [s[i] for i in order[:3]])
        assert (margin[t] > 0) == (s[order[2]] + corr[order[2]] > s[order[3]] + corr[order[3]])
    assert np.isinf(R.route_margin(h, router, corr, 7)).all()
    # identities hand the input on
    w = {"router": router, "correction": np.where(np.arange(7) >= 5, 9.0, 0.0)}
    s = R.router_scores(h, router)
    np.testing.assert_allclose(R.moe_ffn(h, w, dict(router=dict(top=2, experts=5))), h * (s[:, 5] + s[:, 6])[:, None])


def test_gelu_is_the_normal_distribution():
    z = np.linspace(-6, 6, 25)
    grid = np.linspace(-12, 6, 200001)
    density = np.exp(-grid ** 2 / 2) / math.sqrt(2 * math.pi)
    cdf = np.concatenate([[0.0], np.cumsum((density[1:] + density[:-1]) / 2 * np.diff(grid))])
    np.testing.assert_allclose(R.gelu(z), z * np.interp(z, grid, cdf), atol=1e-6)


def test_forward_is_causal():
    from tests.test_gpu_muzopel import CONFIGS

    for name in ("narrow", "odd"):
        w = R.random_weights(CONFIGS[name], seed=3)
        toks = np.random.default_rng(0).integers(0, CONFIGS[name]["vocab"], 12)
        whole, layers = R.forward(CONFIGS[name], w, toks), []
        np.testing.assert_allclose(R.forward(CONFIGS[name], w, toks[:7], layers_out=layers), whole[:7], atol=1e-9)
        assert len(layers) == len(CONFIGS[name]["layers"]) and np.abs(whole).max() <= CONFIGS[name]["logit_softcap"]


def test_steady_routers_leave_the_choice_to_the_token():
    from tests.test_gpu_muzopel import CONFIGS

    config = CONFIGS["narrow"]
    w = R.steady_routers(config, R.random_weights(config, seed=5))
    scores = []
    for toks in ([9], [4, 30, 9, 2]):
        x = R.parts_norm(w["embed"][toks], w["embed.norm"], 3, 1e-5)
        y = R.parts_norm(np.random.default_rng(len(toks)).standard_normal(x.shape), w["l0.norm1"], 3, 1e-5)
        scores.append(R.router_scores(R.with_past(x + y, w["l0.canon2"]), w["l0.mlp.router"])[toks.index(9)])
    np.testing.assert_allclose(scores[0], scores[1], atol=1e-12)
