"""Plain NumPy restatement of the Badolix design: one function per mechanism, every formula written
out position by position or with full [n, n] score matrices, no cache, no chunks, no batches.

Test infrastructure: nothing of the product imports it and it shares no code with it.  The
arithmetic runs in the dtype of the arrays it is given (tests use float64).
"""
from __future__ import annotations

import math

import numpy as np

from .kernels_ref import round_bf16
from .latarax_ref import rms_norm, sigmoid, silu, sub, window_mask, write_model  # noqa: F401


# ---------------------------------------------------------------------------- positions
def rotation(base, dims, scaling=None):
    """(frequency of every channel pair, factor on sines and cosines).  `scaling` with `factor` alone
    slows every frequency down by it; with `original`, `fast` and `slow` only those pairs that turn
    seldom within `original` positions (a ramp over the pair's number), and the vectors grow."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    factor = float(scaling["factor"])
    if "original" not in scaling:
        return f / factor, 1.0

    def pair_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_halves(x, positions, freqs, gain=1.0):
    """x [n, heads, dim]: channel i of each head is turned together with channel i + len(freqs) by
    position * freqs[i]; channels past the pairs stay."""
    y, P = x.copy(), len(freqs)
    for i, f in enumerate(freqs):
        a = (np.asarray(positions) * f)[:, None]
        u, v = x[:, :, i], x[:, :, i + P]
        y[:, :, i] = gain * (u * np.cos(a) - v * np.sin(a))
        y[:, :, i + P] = gain * (v * np.cos(a) + u * np.sin(a))
    return y


def turned(x, rot):
    if not rot:
        return x
    f, gain = rotation(rot["base"], rot["dims"], rot.get("scaling"))
    return rotate_halves(x, np.arange(len(x)), f, gain)


# ---------------------------------------------------------------------------- attention
def capped_attention(q, k, v, scale, visible, cap=None):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim]; scores are squeezed into (-cap, cap)."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    out = np.zeros((n, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        if cap:
            s = cap * np.tanh(s / cap)
        s = np.where(visible, s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h // rep]
    return out


def attention_mixer(h, w, m, held=None):
    """`held`: rotated keys and values of another layer.  Returns (output, (keys, values))."""
    n, H, G, D, V = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = turned((h @ w["q"].T).reshape(n, H, D), m.get("rot"))
    if held is None:
        held = turned((h @ w["k"].T).reshape(n, G, D), m.get("rot")), (h @ w["v"].T).reshape(n, G, V)
    mask = m.get("mask") or {}
    o = capped_attention(q, held[0], held[1], m["scale"], window_mask(n, mask.get("size"), mask.get("keep_first", 0)),
                         m.get("softcap"))
    return o.reshape(n, H * V) @ w["o"].T, held


def latent_mixer(h, w, m, eps):
    """Keys and values of all heads grow out of one normed latent; one rotated part is shared."""
    n, H, D, R, V, C = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w["q"].T).reshape(n, H, D + R)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :C], w["dkv.norm"], eps)
    k_rot = turned(down[:, None, C:], m.get("rot"))
    k = (c @ w["uk"].T).reshape(n, H, D)
    v = (c @ w["uv"].T).reshape(n, H, V)
    q = np.concatenate([q[:, :, :D], turned(q[:, :, D:], m.get("rot"))], axis=2)
    k = np.concatenate([k, np.repeat(k_rot, H, axis=1)], axis=2)
    return capped_attention(q, k, v, m["scale"], window_mask(n, None, 0)).reshape(n, H * V) @ w["o"].T


# ----------------------------------------------------------------- state-space recurrence
def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def causal_conv(x, w, bias):
    """x [n, channels], w [channels, taps]: the last tap meets the token itself."""
    taps = w.shape[1]
    y = np.zeros_like(x)
    for t in range(len(x)):
        for j in range(taps):
            if t - (taps - 1 - j) >= 0:
                y[t] += w[:, j] * x[t - (taps - 1 - j)]
    return y + bias


def state_space(x, B, C, dt, A_log, D):
    """x [n, heads, vdim], B and C [n, heads, state], dt [n, heads] -> y [n, heads, vdim], last state."""
    n, H, V = x.shape
    S = np.zeros((H, B.shape[2], V), dtype=x.dtype)
    y = np.zeros_like(x)
    for t in range(n):
        decay = np.exp(-np.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnv,hn->hv", S, C[t]) + D[:, None] * x[t]
    return y, S


def gated_norm(y, z, weight, parts, eps):
    """The gate first, then every part by its own root mean square."""
    n, width = y.shape
    g = (y * silu(z)).reshape(n, parts, width // parts)
    return (g / np.sqrt(np.mean(g * g, axis=2, keepdims=True) + eps)).reshape(n, width) * weight


def mamba2_mixer(h, w, m, eps):
    n, H, V, N, G = len(h), m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x = xbc[:, :inner].reshape(n, H, V)
    B = np.repeat(xbc[:, inner:inner + G * N].reshape(n, G, N), H // G, axis=1)
    C = np.repeat(xbc[:, inner + G * N:].reshape(n, G, N), H // G, axis=1)
    y, _ = state_space(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    return gated_norm(y.reshape(n, inner), z, w["norm"], m["norm_groups"], eps) @ w["o"].T


# -------------------------------------------------------------------------- feed-forward
def biased_ffn(h, w):
    return (silu(h @ w["gate"].T + w["gate.b"]) * (h @ w["up"].T + w["up.b"])) @ w["down"].T + w["down.b"]


def expert_ffn(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def group_scores(s, count):
    """Sum of the two largest scores of every group of neighbouring experts."""
    g = np.sort(s.reshape(len(s), count, -1), axis=2)[:, :, ::-1]
    return g[:, :, :2].sum(axis=2)


def route(h, w_router, top, groups=None):
    """The `top` experts of largest sigmoid score among the best groups, and their scores over the sum."""
    s = sigmoid(h @ w_router.T)
    allowed = np.ones_like(s, dtype=bool)
    if groups:
        best = np.argsort(-group_scores(s, groups["count"]), axis=1, kind="stable")[:, :groups["keep"]]
        in_group = np.zeros((len(s), groups["count"]), dtype=bool)
        np.put_along_axis(in_group, best, True, axis=1)
        allowed = np.repeat(in_group, s.shape[1] // groups["count"], axis=1)
    chosen = np.argsort(np.where(allowed, -s, np.inf), axis=1, kind="stable")[:, :top]
    c = np.take_along_axis(s, chosen, axis=1)
    return chosen, c / (c.sum(axis=1, keepdims=True) + 1e-20)


def route_margin(h, w_router, top, groups=None):
    """How far every decision of a token (the last group kept, the last expert chosen) lies above its
    first alternative, in units of the spread of the scores (infinite where nothing is left out)."""
    s = sigmoid(h @ w_router.T)
    spread = max(float(s.std()), 1e-9)
    margin = np.full(len(s), np.inf)
    if groups and groups["keep"] < groups["count"]:
        g = group_scores(s, groups["count"])
        order = np.argsort(-g, axis=1, kind="stable")
        r = np.take_along_axis(g, order, axis=1)
        margin = (r[:, groups["keep"] - 1] - r[:, groups["keep"]]) / spread
        in_group = np.zeros_like(g, dtype=bool)
        np.put_along_axis(in_group, order[:, :groups["keep"]], True, axis=1)
        s = np.where(np.repeat(in_group, s.shape[1] // groups["count"], axis=1), s, -np.inf)
    z = np.sort(s, axis=1)[:, ::-1]
    if z.shape[1] > top:
        margin = np.minimum(margin, (z[:, top - 1] - z[:, top]) / spread)
    return margin


def moe_ffn(h, w, mlp):
    chosen, weight = route(h, w["router"], mlp["router"]["top"], mlp["router"].get("groups"))
    y = np.zeros_like(h)
    for t in range(len(h)):
        for e, p in zip(chosen[t], weight[t]):
            y[t] += p * expert_ffn(h[t:t + 1], sub(w, f"e{e}."))[0]
    return y


# ------------------------------------------------------------------------------ the model
def forward(config: dict, weights: dict, tokens, layers_out: list | None = None, margins_out: list | None = None):
    """Logits [n, vocab] of one sequence from its first token."""
    eps, mult = config["norm"]["eps"], config["residual_mult"]
    x = weights["embed"][np.asarray(tokens, dtype=np.int64)] * config["embedding"]["scale"]
    held = {}
    for i, layer in enumerate(config["layers"]):
        w, m = sub(weights, f"l{i}."), layer["mixer"]
        h = rms_norm(x, w["norm1"], eps)
        mix = sub(w, "mix.")
        if layer["type"] == "latent_attention":
            y = latent_mixer(h, mix, m, eps)
        elif layer["type"] == "mamba2":
            y = mamba2_mixer(h, mix, m, eps)
        else:
            y, held[i] = attention_mixer(h, mix, m, held[m["kv_from"]] if "kv_from" in m else None)
        x = x + mult * y
        mlp = layer.get("mlp")
        if mlp:
            h = rms_norm(x, w["norm2"], eps)
            if margins_out is not None and mlp["kind"] == "moe":
                margins_out.append(route_margin(h, w["mlp.router"], mlp["router"]["top"], mlp["router"].get("groups")))
            x = x + mult * (biased_ffn(h, sub(w, "mlp.")) if mlp["kind"] == "dense" else moe_ffn(h, sub(w, "mlp."), mlp))
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, weights["final.norm"], eps) @ weights["embed"].T * config["logit_scale"]


def greedy_generate(config, weights, prompt, n_new):
    toks, rows = list(prompt), []
    for _ in range(n_new):
        rows.append(forward(config, weights, toks)[-1])
        toks.append(int(np.argmax(rows[-1])))
    return toks[len(prompt):], rows


# ------------------------------------------------------------------ small models for tests
def tensor_shapes(config: dict) -> dict:
    W, V = config["width"], config["vocab"]
    out = {"embed": (V, W)}
    for i, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        t = p + "mix."
        out[p + "norm1"] = (W,)
        if layer["type"] == "latent_attention":
            H, C = m["heads"], m["kv_rank"]
            out.update({t + "q": (H * (m["dim"] + m["rot_dim"]), W), t + "dkv": (C + m["rot_dim"], W), t + "dkv.norm": (C,),
                        t + "uk": (H * m["dim"], C), t + "uv": (H * m["vdim"], C), t + "o": (W, H * m["vdim"])})
        elif layer["type"] == "mamba2":
            H, inner, bc = m["heads"], m["heads"] * m["vdim"], 2 * m["groups"] * m["state"]
            out.update({t + "in": (2 * inner + bc + H, W), t + "conv": (inner + bc, m["conv"]), t + "conv.b": (inner + bc,),
                        t + "dt_bias": (H,), t + "A_log": (H,), t + "D": (H,), t + "norm": (inner,), t + "o": (W, inner)})
        else:
            out[t + "q"] = (m["heads"] * m["dim"], W)
            if "kv_from" not in m:
                out.update({t + "k": (m["kv_heads"] * m["dim"], W), t + "v": (m["kv_heads"] * m["vdim"], W)})
            out[t + "o"] = (W, m["heads"] * m["vdim"])
        if not mlp:
            continue
        out[p + "norm2"] = (W,)
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            out.update({p + "mlp.gate": (F, W), p + "mlp.gate.b": (F,), p + "mlp.up": (F, W), p + "mlp.up.b": (F,),
                        p + "mlp.down": (W, F), p + "mlp.down.b": (W,)})
        else:
            F = mlp["expert"]["ff"]
            out[p + "mlp.router"] = (mlp["router"]["experts"], W)
            for e in range(mlp["router"]["experts"]):
                out.update({f"{p}mlp.e{e}.gate": (F, W), f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    out["final.norm"] = (W,)
    return out


def steady_routers(config: dict, weights: dict, channels: int = 6) -> dict:
    """The same model with routers that read only the last `channels` of the width, which the
    embedding sets and no layer writes to: rounding inside the layers then hardly moves a score, and a
    16-bit run chooses the experts an exact one does (close calls apart)."""
    w = {k: v.copy() for k, v in weights.items()}
    rng = np.random.default_rng(7)
    w["embed"][:, -channels:] = rng.choice([-3.0, -2.0, -1.0, 1.0, 2.0, 3.0], w["embed"][:, -channels:].shape)
    for name, a in w.items():
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith(".router"):
            a[:, :-channels] = 0.0
            a[:, -channels:] = round_bf16((a[:, -channels:] * (a.shape[1] / channels) ** 0.5).astype(np.float32))
        elif leaf in ("o", "down") or name.endswith(".down.b"):
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
        elif leaf == "b":
            a = 0.5 * r
        elif leaf == "dt_bias":      # steps from small to about one
            a = -2.0 + 1.5 * r
        elif leaf == "A_log":
            a = 0.5 + r
        elif leaf == "D" or name == "embed":
            a = r
        else:
            a = r * (1.7 if leaf in ("gate", "up") else 1.0) * shape[-1] ** -0.5
        out[name] = round_bf16(a.astype(np.float32)).astype(np.float64)
    return out
