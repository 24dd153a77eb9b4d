"""Plain NumPy restatement of the Biberax design: one function per mechanism, every formula written
out position by position or with full [n, n] score matrices, no cache, no batches.

Test infrastructure: nothing of the product imports it and it shares no code with it.  The
arithmetic runs in the dtype of the arrays it is given (tests use float64).
"""
from __future__ import annotations

import math

import numpy as np

from .kernels_ref import round_bf16
from .latarax_ref import rms_norm, sigmoid, sub, write_model  # noqa: F401


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------------------- positions
def rotation_frequencies(base, dims, scaling=None):
    """Frequency of every pair of rotated channels; with `scaling` long wavelengths are stretched by
    `factor`, short ones kept, and those between original/high and original/low blended."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > original / low:
                f = f / factor
            elif wave >= original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return np.array(out)


def rotate_interleaved(x, positions, freqs):
    """x [n, heads, dim]: channels (2i, 2i + 1) of each head turned by position * freqs[i]; channels
    past the last pair stay."""
    y = x.copy()
    for i, f in enumerate(freqs):
        a = (np.asarray(positions) * f)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = u * np.cos(a) - v * np.sin(a)
        y[:, :, 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return y


def distance_bucket(n, buckets, far):
    """Bucket of distance n >= 0: exact in the lower half, logarithmic up to `far` above it."""
    half = buckets // 2
    if n < half:
        return n
    if half == 0:
        return 0
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (buckets - half)))


def distance_bias(n, table, far):
    """bias[i, j, h] for j <= i (zero elsewhere); table [buckets, heads]."""
    per = np.stack([table[distance_bucket(d, len(table), far)] for d in range(n)])
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return np.where((j <= i)[:, :, None], per[np.abs(i - j)], 0.0)


# ---------------------------------------------------------------------------- attention
def causal_mask(n):
    return np.tril(np.ones((n, n), dtype=bool))


def chunk_mask(n, size):
    i = np.arange(n)
    return causal_mask(n) & (i[:, None] // size == i[None, :] // size)


def sink_attention(q, k, v, scale, visible, sink, bias=None):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim]; the softmax of head h has one more member of
    score sink[h] (None: no such member) that carries no value."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    out = np.zeros((n, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        if bias is not None:
            s = s + bias[:, :, h]
        s = np.where(visible, s, -np.inf)
        top = s.max(axis=1, keepdims=True)
        if sink is not None:
            top = np.maximum(top, sink[h])
        p = np.exp(s - top)
        den = p.sum(axis=1, keepdims=True)
        if sink is not None:
            den = den + np.exp(sink[h] - top)
        out[:, h] = (p / den) @ v[:, h // rep]
    return out


def chunk_mixer(h, w, m):
    """Rotated queries and keys, attention inside chunks, one added to the softmax denominator."""
    n, H, G, D, V = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    f = rotation_frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling"))
    q = rotate_interleaved((h @ w["q"].T).reshape(n, H, D), np.arange(n), f)
    k = rotate_interleaved((h @ w["k"].T).reshape(n, G, D), np.arange(n), f)
    v = (h @ w["v"].T).reshape(n, G, V)
    o = sink_attention(q, k, v, m["scale"], chunk_mask(n, m["mask"]["size"]), np.zeros(H)).reshape(n, H * V)
    return (o * sigmoid(h @ w["g"].T)) @ w["o"].T


def bias_mixer(h, w, m, eps):
    """Values that are the projected keys, norms over the whole projections, a learned bias by
    distance and a learned sink."""
    n, H, G, D = len(h), m["heads"], m["kv_heads"], m["dim"]
    q = h @ w["q"].T + w["q.b"]
    k = h @ w["k"].T + w["k.b"]
    v = k.reshape(n, G, D)
    q = rms_norm(q, w["q.norm"], eps).reshape(n, H, D)
    k = rms_norm(k, w["k.norm"], eps).reshape(n, G, D)
    o = sink_attention(q, k, v, m["scale"], causal_mask(n), w["sink"], distance_bias(n, w["rel"], m["bias_max"]))
    return (o.reshape(n, H * D) * sigmoid(h @ w["g"].T)) @ w["o"].T + w["o.b"]


# -------------------------------------------------------------------------- feed-forward
def dense_ffn(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def clamped_expert(h, w, limit):
    g = np.minimum(h @ w["gate"].T, limit)
    u = np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def route(h, w_router, bias, top):
    """The `top` experts of largest logit per token and the softmax over their logits."""
    z = h @ w_router.T + bias
    chosen = np.argsort(-z, axis=1, kind="stable")[:, :top]
    c = np.take_along_axis(z, chosen, axis=1)
    e = np.exp(c - c.max(axis=1, keepdims=True))
    return chosen, e / e.sum(axis=1, keepdims=True)


def route_margin(h, w_router, bias, top):
    """How far the last chosen logit of every token lies above the first one left out, in units of
    the spread of all logits (infinite when nothing is left out)."""
    z = np.sort(h @ w_router.T + bias, axis=1)[:, ::-1]
    if z.shape[1] == top:
        return np.full(len(z), np.inf)
    return (z[:, top - 1] - z[:, top]) / max(float(z.std()), 1e-9)


def moe_ffn(h, w, mlp):
    chosen, weight = route(h, w["router"], w["router.b"], mlp["router"]["top"])
    y = np.zeros_like(h)
    for t in range(len(h)):
        for e, p in zip(chosen[t], weight[t]):
            y[t] += p * clamped_expert(h[t:t + 1], sub(w, f"e{e}."), mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        y = y + clamped_expert(h, sub(w, "shared."), mlp["shared"]["limit"])
    return y


# ------------------------------------------------------------------------------ the model
def forward(config: dict, weights: dict, tokens, layers_out: list | None = None, margins_out: list | None = None):
    """Logits [n, vocab] of one sequence from its first token."""
    eps = config["norm"]["eps"]
    x = weights["embed"][np.asarray(tokens, dtype=np.int64)]
    for i, layer in enumerate(config["layers"]):
        w = sub(weights, f"l{i}.")
        h = rms_norm(x, w["norm1"], eps)
        mix = sub(w, "mix.")
        x = x + (chunk_mixer(h, mix, layer["mixer"]) if layer["type"] == "attention" else
                 bias_mixer(h, mix, layer["mixer"], eps))
        mlp = layer.get("mlp")
        if mlp:
            h = rms_norm(x, w["norm2"], eps)
            if margins_out is not None and mlp["kind"] == "moe":
                margins_out.append(route_margin(h, w["mlp.router"], w["mlp.router.b"], mlp["router"]["top"]))
            x = x + (dense_ffn(h, sub(w, "mlp.")) if mlp["kind"] == "dense" else moe_ffn(h, sub(w, "mlp."), mlp))
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, weights["final.norm"], eps) @ weights["head"].T


def greedy_generate(config, weights, prompt, n_new):
    toks, rows = list(prompt), []
    for _ in range(n_new):
        rows.append(forward(config, weights, toks)[-1])
        toks.append(int(np.argmax(rows[-1])))
    return toks[len(prompt):], rows


# ------------------------------------------------------------------ small models for tests
def tensor_shapes(config: dict, buckets: int = 12) -> dict:
    W, V = config["width"], config["vocab"]
    out = {"embed": (V, W)}
    for i, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
        out.update({p + "norm1": (W,), p + "mix.q": (q, W), p + "mix.k": (k, W), p + "mix.g": (v, W), p + "mix.o": (W, v)})
        if layer["type"] == "attention":
            out[p + "mix.v"] = (m["kv_heads"] * m["vdim"], W)
        else:
            out.update({p + "mix.q.b": (q,), p + "mix.k.b": (k,), p + "mix.o.b": (W,), p + "mix.q.norm": (q,),
                        p + "mix.k.norm": (k,), p + "mix.rel": (buckets, m["heads"]), p + "mix.sink": (m["heads"],)})
        if not mlp:
            continue
        out[p + "norm2"] = (W,)
        parts = {"": mlp["ff"]} if mlp["kind"] == "dense" else \
            {f"e{e}.": mlp["expert"]["ff"] for e in range(mlp["router"]["experts"])}
        if mlp["kind"] == "moe":
            out.update({p + "mlp.router": (mlp["router"]["experts"], W), p + "mlp.router.b": (mlp["router"]["experts"],)})
            if mlp.get("shared"):
                parts["shared."] = mlp["shared"]["ff"]
        for name, F in parts.items():
            out.update({f"{p}mlp.{name}gate": (F, W), f"{p}mlp.{name}up": (F, W), f"{p}mlp.{name}down": (W, F)})
    out["final.norm"] = (W,)
    out["head"] = (V, W)
    return out


def steady_routers(config: dict, weights: dict, channels: int = 6) -> dict:
    """The same model with routers that read only the last `channels` of the width, which the
    embedding sets and no layer writes to: rounding inside the layers then hardly moves a logit, and a
    16-bit run chooses the experts an exact one does (close calls apart)."""
    w = {k: v.copy() for k, v in weights.items()}
    rng = np.random.default_rng(7)
    w["embed"][:, -channels:] = rng.choice([-3.0, -2.0, -1.0, 1.0, 2.0, 3.0], w["embed"][:, -channels:].shape)
    for name, a in w.items():
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith(".router"):
            a[:, :-channels] = 0.0
            a[:, -channels:] = round_bf16((a[:, -channels:] * (a.shape[1] / channels) ** 0.5).astype(np.float32))
        elif leaf in ("o", "down") or name.endswith(".o.b"):
            a[-channels:] = 0.0
    return w


def random_weights(config: dict, seed: int = 0, buckets: int = 12) -> dict:
    """float64 arrays whose values are exact in bfloat16 (what a checkpoint can hold)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config, buckets).items():
        r = rng.standard_normal(shape)
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2"):
            a = 1.0 + 0.3 * r
        elif leaf in ("b", "rel", "sink"):
            a = (0.5 if leaf == "b" else 1.5) * r
        elif name == "embed":
            a = r
        else:
            a = r * (1.7 if leaf in ("gate", "up") else 1.0) * shape[-1] ** -0.5
        out[name] = round_bf16(a.astype(np.float32)).astype(np.float64)
    return out
