"""Plain NumPy restatement of the Muzopel design: one function per mechanism, every formula written
out position by position or with full [n, n] score matrices, no cache, no chunks, no batches.

Test infrastructure: nothing of the product imports it and it shares no code with it.  The
arithmetic runs in the dtype of the arrays it is given (tests use float64).
"""
from __future__ import annotations

import math

import numpy as np

from .badolix_ref import capped_attention, rotation
from .kernels_ref import round_bf16
from .latarax_ref import rms_norm, sigmoid, sub, window_mask, write_model  # noqa: F401


# ------------------------------------------------------------------- norms, inputs, depth
def parts_norm(x, weight, parts, eps):
    """Every one of `parts` equal pieces of a row by its own root mean square, then the weight."""
    n, width = x.shape
    p = x.reshape(n, parts, width // parts)
    return (p / np.sqrt(np.mean(p * p, axis=2, keepdims=True) + eps)).reshape(n, width) * weight


def with_past(x, w):
    """x [n, width] plus its causal convolution per channel; the last of w's [width, taps] columns
    meets the token itself."""
    taps = w.shape[1]
    y = x.copy()
    for t in range(len(x)):
        for back in range(min(taps, t + 1)):
            y[t] = y[t] + w[:, taps - 1 - back] * x[t - back]
    return y


def depth_sum(states, weight):
    """Weighted sum over everything the layers so far have made (the embedding first)."""
    y = np.zeros_like(states[0])
    for x, c in zip(states, weight, strict=True):
        y = y + c * x
    return y


# ---------------------------------------------------------------------------- attention
def rotate_neighbours(x, positions, freqs, gain=1.0):
    """x [n, heads, dim]: channels 2i and 2i + 1 of each head are turned by position * freqs[i]."""
    y = x.copy()
    for i, f in enumerate(freqs):
        a = (np.asarray(positions) * f)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = gain * (u * np.cos(a) - v * np.sin(a))
        y[:, :, 2 * i + 1] = gain * (v * np.cos(a) + u * np.sin(a))
    return y


def turned(x, rot):
    if not rot:
        return x
    f, gain = rotation(rot["base"], rot["dims"], rot.get("scaling"))
    return rotate_neighbours(x, np.arange(len(x)), f, gain)


def latent_mixer(h, w, m, eps):
    """Keys and values of all heads grow out of one normed latent; one rotated key part is shared.
    Queries come from h, or (a matrix `dq`) from a normed latent of their own; heads may be gated."""
    n, H, D, R, V, C = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T if "dq" in w else h @ w["q"].T
    q = q.reshape(n, H, D + R)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :C], w["dkv.norm"], eps)
    k_rot = turned(down[:, None, C:], m.get("rot"))
    k = np.concatenate([(c @ w["uk"].T).reshape(n, H, D), np.repeat(k_rot, H, axis=1)], axis=2)
    q = np.concatenate([q[:, :, :D], turned(q[:, :, D:], m.get("rot"))], axis=2)
    o = capped_attention(q, k, (c @ w["uv"].T).reshape(n, H, V), m["scale"], window_mask(n, None, 0))
    if "g" in w:
        o = o * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(n, H * V) @ w["o"].T


# -------------------------------------------------------------------------- feed-forward
def gelu(z):
    return 0.5 * z * (1.0 + np.vectorize(math.erf)(z / math.sqrt(2.0)))


def expert_ffn(h, w):
    return gelu(h @ w["up"].T) @ w["down"].T


def router_scores(h, w_router):
    z = h @ w_router.T
    p = np.exp(z - z.max(axis=1, keepdims=True))
    return p / p.sum(axis=1, keepdims=True)


def route(h, w_router, correction, top):
    """The `top` of all outputs by corrected score, and their scores as they are."""
    s = router_scores(h, w_router)
    chosen = np.argsort(-(s + correction), axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def route_margin(h, w_router, correction, top):
    """How far the last chosen output lies above the first left out, in units of the spread of the
    choice scores (infinite where none is left out)."""
    c = router_scores(h, w_router) + correction
    z = np.sort(c, axis=1)[:, ::-1]
    if z.shape[1] <= top:
        return np.full(len(z), np.inf)
    return (z[:, top - 1] - z[:, top]) / max(float(c.std()), 1e-9)


def moe_ffn(h, w, mlp):
    """Router outputs past the experts hand the input on."""
    chosen, weight = route(h, w["router"], w["correction"], mlp["router"]["top"])
    y = np.zeros_like(h)
    for t in range(len(h)):
        for e, p in zip(chosen[t], weight[t]):
            y[t] += p * (h[t] if e >= mlp["router"]["experts"] else expert_ffn(h[t:t + 1], sub(w, f"e{e}."))[0])
    return y


# ------------------------------------------------------------------------------ the model
def forward(config: dict, weights: dict, tokens, layers_out: list | None = None, margins_out: list | None = None):
    """Logits [n, vocab] of one sequence from its first token.  `layers_out`: what every layer hands
    to the next one."""
    eps, parts = config["norm"]["eps"], config["norm"]["groups"]
    x = parts_norm(weights["embed"][np.asarray(tokens, dtype=np.int64)], weights["embed.norm"], parts, eps)
    states = [x]
    for i, layer in enumerate(config["layers"]):
        w, mlp = sub(weights, f"l{i}."), layer.get("mlp")
        y = latent_mixer(with_past(x, w["canon1"]), sub(w, "mix."), layer["mixer"], eps)
        x = x + parts_norm(y, w["norm1"], parts, eps)
        if mlp:
            h = with_past(x, w["canon2"])
            if margins_out is not None:
                margins_out.append(route_margin(h, w["mlp.router"], w["mlp.correction"], mlp["router"]["top"]))
            x = x + parts_norm(moe_ffn(h, sub(w, "mlp."), mlp), w["norm2"], parts, eps)
        states.append(x)
        x = depth_sum(states, w["dwa"])
        if layers_out is not None:
            layers_out.append(x.copy())
    cap = config["logit_softcap"]
    return cap * np.tanh(parts_norm(x, weights["final.norm"], parts, eps) @ weights["head"].T / cap)


def greedy_generate(config, weights, prompt, n_new):
    toks, rows = list(prompt), []
    for _ in range(n_new):
        rows.append(forward(config, weights, toks)[-1])
        toks.append(int(np.argmax(rows[-1])))
    return toks[len(prompt):], rows


# ------------------------------------------------------------------ small models for tests
def tensor_shapes(config: dict) -> dict:
    W, V, taps = config["width"], config["vocab"], config["canon"]["taps"]
    out = {"embed": (V, W), "embed.norm": (W,)}
    for i, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        t, H, C = p + "mix.", m["heads"], m["kv_rank"]
        out[p + "norm1"] = (W,)
        Q = H * (m["dim"] + m["rot_dim"])
        if layer["type"] == "latent_attention":
            R = m["q_rank"]
            out.update({t + "dq": (R, W), t + "dq.norm": (R,), t + "uq": (Q, R), t + "g": (H, W)})
        else:
            out[t + "q"] = (Q, W)
        out.update({t + "dkv": (C + m["rot_dim"], W), t + "dkv.norm": (C,), t + "uk": (H * m["dim"], C),
                    t + "uv": (H * m["vdim"], C), t + "o": (W, H * m["vdim"]),
                    p + "canon1": (W, taps), p + "dwa": (i + 2,)})
        if mlp:
            F, E = mlp["expert"]["ff"], mlp["router"]["experts"]
            n = E + mlp["router"].get("identity", 0)
            out.update({p + "norm2": (W,), p + "canon2": (W, taps), p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
            for e in range(E):
                out.update({f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    out.update({"final.norm": (W,), "head": (V, W)})
    return out


def steady_routers(config: dict, weights: dict, channels: int = 6) -> dict:
    """The same model with routers that read only the last `channels` of the width, which the embedding
    sets and no sublayer writes to (their norms' weights are zero there, and so is the convolution ahead of
    the router): rounding inside the layers then hardly moves a score, a token alone decides its experts,
    and a 16-bit run chooses those an exact one does."""
    w = {k: v.copy() for k, v in weights.items()}
    rng = np.random.default_rng(7)
    w["embed"][:, -channels:] = rng.choice([-3.0, -2.0, -1.0, 1.0, 2.0, 3.0], w["embed"][:, -channels:].shape)
    for name, a in w.items():
        if name.endswith(".router"):
            a[:, :-channels] = 0.0
            a[:, -channels:] = round_bf16((a[:, -channels:] * (a.shape[1] / channels) ** 0.5).astype(np.float32))
        elif name.endswith((".norm1", ".norm2", ".canon2")):
            a[-channels:] = 0.0
    return w


def random_weights(config: dict, seed: int = 0) -> dict:
    """float64 arrays whose values are exact in bfloat16 (what a checkpoint can hold)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        r = rng.standard_normal(shape)
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2"):
            a = 1.0 + 0.3 * r
        elif leaf == "correction":   # as large as the scores themselves
            a = r / shape[0]
        elif leaf == "dwa":          # the newest counts most, all of them count
            a = 0.3 * r + (np.arange(shape[0]) == shape[0] - 1)
        elif leaf in ("canon1", "canon2"):
            a = 0.4 * r
        elif name == "embed":
            a = r
        else:
            a = r * (1.7 if leaf in ("up", "head") else 1.0) * shape[-1] ** -0.5
        out[name] = round_bf16(a.astype(np.float32)).astype(np.float64)
    return out
