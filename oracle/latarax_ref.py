"""Plain NumPy restatement of the Latarax design: one function per mechanism, every formula
written out position by position or with full [n, n] score matrices, no cache, no chunks.

Test infrastructure: nothing of the product imports it and it shares no code with it.  The
arithmetic runs in the dtype of the arrays it is given (tests use float64).
"""
from __future__ import annotations

import json
import os

import numpy as np

from .kernels_ref import round_bf16
from .llama_ref import write_safetensors


# ------------------------------------------------------------------------- small pieces
def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def rms_norm_around_zero(x, weight, eps):
    """The norm whose weight is stored as its distance from one."""
    return rms_norm(x, 1.0 + weight, eps)


def gated_ffn(h, w_gate, w_up, w_down):
    return (silu(h @ w_gate.T) * (h @ w_up.T)) @ w_down.T


# ---------------------------------------------------------------------------- attention
def window_mask(n, size, keep_first):
    """visible[i, j]: j is not in the future and is either within the last `size` positions of
    i (itself included) or among the first `keep_first` of the sequence."""
    i = np.arange(n)[:, None]
    j = np.arange(n)[None, :]
    seen = j <= i
    if size is not None:
        seen &= ((i - j) < size) | (j < keep_first)
    return seen


def attention(q, k, v, scale, visible):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim]: softmax over the visible keys, query head h
    on key/value head h // (H / G).  Returns [n, H, vdim]."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    out = np.zeros((n, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        s = np.where(visible, s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h // rep]
    return out


# ----------------------------------------------------------------------- linear recurrences
def decayed_recurrence(q, k, v, decay, state=None):
    """S_t = decay_t (per key channel) * S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t, token by token.
    q, k, decay [n, heads, dim], v [n, heads, vdim].  Returns (o [n, heads, vdim], last state)."""
    n, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]), dtype=q.dtype) if state is None else state.copy()
    o = np.zeros_like(v)
    for t in range(n):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o, S


def gla_decay(h, w_a1, w_a2, bias, tau):
    """Decay of every key channel in (0, 1): sigmoid of a low-rank projection to the power 1/tau."""
    return sigmoid((h @ w_a1.T) @ w_a2.T + bias) ** (1.0 / tau)


def gla_mixer(h, w, spec, eps):
    n, H, D, V = len(h), spec["heads"], spec["dim"], spec["vdim"]
    q = (h @ w["q"].T).reshape(n, H, D) * D ** -0.5
    k = (h @ w["k"].T).reshape(n, H, D)
    v = (h @ w["v"].T).reshape(n, H, V)
    a = gla_decay(h, w["a1"], w["a2"], w["a2.b"], spec["tau"]).reshape(n, H, D)
    o, _ = decayed_recurrence(q, k, v, a)
    o = rms_norm(o, w["norm"], eps).reshape(n, H * V)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def lightning_mixer(h, w, spec, eps):
    n, H, D, V = len(h), spec["heads"], spec["dim"], spec["vdim"]
    q = silu(h @ w["q"].T).reshape(n, H, D)
    k = silu(h @ w["k"].T).reshape(n, H, D)
    v = silu(h @ w["v"].T).reshape(n, H, V)
    a = np.broadcast_to(np.asarray(spec["decay"], dtype=h.dtype)[None, :, None], (n, H, D))
    o, _ = decayed_recurrence(q, k, v, a)
    o = rms_norm(o.reshape(n, H * V), w["norm"], eps)
    return (o * sigmoid(h @ w["g"].T)) @ w["o"].T


def window_attention_mixer(h, w, spec):
    n, H, G, D, V = len(h), spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = (h @ w["q"].T).reshape(n, H, D)
    k = (h @ w["k"].T).reshape(n, G, D)
    v = (h @ w["v"].T).reshape(n, G, V)
    m = spec.get("mask") or {}
    o = attention(q, k, v, spec["scale"], window_mask(n, m.get("size"), m.get("keep_first", 0)))
    return o.reshape(n, H * V) @ w["o"].T


def parallel_mixer(h, w, spec, eps):
    left = window_attention_mixer(h, sub(w, "left."), spec["left"])
    right = lightning_mixer(h, sub(w, "right."), spec["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


# --------------------------------------------------------------------- several residual streams
def streams_read(x, w_in):
    """x [streams, n, width]: the sublayer's input before its norm."""
    return np.einsum("s,snw->nw", w_in, x)


def streams_write(x, mix, w_out, y):
    """Every stream at once from the old ones: new[t] = sum_s mix[s, t] x[s] + out[t] y."""
    return np.einsum("st,snw->tnw", mix, x) + w_out[:, None, None] * y[None]


# ------------------------------------------------------------------------------ the model
def sub(w: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config: dict, weights: dict, tokens, layers_out: list | None = None):
    """Logits [n, vocab] of one sequence from its first token."""
    eps = config["norm"]["eps"]
    tokens = np.asarray(tokens, dtype=np.int64)
    e = weights["embed"][tokens] + weights["pos"][: len(tokens)]
    x = np.repeat(e[None], config.get("streams", 1), axis=0)
    for i, layer in enumerate(config["layers"]):
        w = sub(weights, f"l{i}.")
        u = rms_norm_around_zero(streams_read(x, w["hc1.in"]), w["norm1"], eps)
        mix_w = sub(w, "mix.")
        y = gla_mixer(u, mix_w, layer["mixer"], eps) if layer["type"] == "gla" else \
            parallel_mixer(u, mix_w, layer["mixer"], eps)
        x = streams_write(x, w["hc1.mix"], w["hc1.out"], y)
        if layer.get("mlp"):
            u = rms_norm_around_zero(streams_read(x, w["hc2.in"]), w["norm2"], eps)
            y = gated_ffn(u, w["mlp.gate"], w["mlp.up"], w["mlp.down"])
            x = streams_write(x, w["hc2.mix"], w["hc2.out"], y)
        if layers_out is not None:
            layers_out.append(x.sum(axis=0))
    return rms_norm_around_zero(x.sum(axis=0), weights["final.norm"], eps) @ weights["head"].T


def greedy_generate(config, weights, prompt, n_new):
    toks = list(prompt)
    rows = []
    for _ in range(n_new):
        rows.append(forward(config, weights, toks)[-1])
        toks.append(int(np.argmax(rows[-1])))
    return toks[len(prompt):], rows


# ------------------------------------------------------------------ small models for tests
def tensor_shapes(config: dict, rank: int = 16) -> dict:
    W, V, s = config["width"], config["vocab"], config["streams"]
    out = {"embed": (V, W), "pos": (config["max_positions"], W)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        out[p + "norm1"] = (W,)
        if layer["type"] == "gla":
            H, D, VD = m["heads"], m["dim"], m["vdim"]
            out.update({p + "mix.q": (H * D, W), p + "mix.k": (H * D, W), p + "mix.v": (H * VD, W),
                        p + "mix.g": (H * VD, W), p + "mix.o": (W, H * VD), p + "mix.norm": (VD,),
                        p + "mix.a1": (rank, W), p + "mix.a2": (H * D, rank), p + "mix.a2.b": (H * D,)})
        else:
            a, r = m["left"], m["right"]
            out.update({p + "mix.left.q": (a["heads"] * a["dim"], W), p + "mix.left.k": (a["kv_heads"] * a["dim"], W),
                        p + "mix.left.v": (a["kv_heads"] * a["vdim"], W),
                        p + "mix.left.o": (W, a["heads"] * a["vdim"]), p + "mix.left.out": (W,)})
            D, VD = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            out.update({p + "mix.right.q": (D, W), p + "mix.right.k": (D, W), p + "mix.right.v": (VD, W),
                        p + "mix.right.g": (VD, W), p + "mix.right.o": (W, VD), p + "mix.right.norm": (VD,),
                        p + "mix.right.out": (W,)})
        subs = ["1"]
        if layer.get("mlp"):
            F = layer["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
            subs.append("2")
        for q in subs:
            out.update({p + f"hc{q}.in": (s,), p + f"hc{q}.out": (s,), p + f"hc{q}.mix": (s, s)})
    out["final.norm"] = (W,)
    out["head"] = (V, W)
    return out


def random_weights(config: dict, seed: int = 0, rank: int = 16) -> dict:
    """float64 arrays whose values are exact in bfloat16 (what a checkpoint can hold)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config, rank).items():
        leaf = name.split(".", 1)[1] if name[0] == "l" and "." in name else name
        r = rng.standard_normal(shape)
        if leaf in ("norm1", "norm2", "norm"):            # stored around zero
            a = 0.2 * r
        elif leaf in ("mix.norm", "mix.left.out", "mix.right.norm", "mix.right.out"):
            a = 1.0 + 0.2 * r
        elif leaf == "mix.a2.b":
            a = 1.5 + 2.0 * r
        elif leaf.endswith(".in"):
            a = 0.6 + 0.3 * r
        elif leaf.endswith(".out") and leaf.startswith("hc"):
            a = 0.8 + 0.3 * r
        elif leaf.endswith(".mix"):
            a = np.eye(shape[0]) * 0.8 + 0.15 * r
        elif name in ("embed", "pos"):
            a = r * (1.0 if name == "embed" else 0.3)
        else:
            a = r * shape[-1] ** -0.5
        out[name] = round_bf16(a.astype(np.float32)).astype(np.float64)
    return out


def write_model(path: str, config: dict, weights: dict) -> None:
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(config, f)
    write_safetensors(os.path.join(path, "model.safetensors"),
                      {k: v.astype(np.float32) for k, v in weights.items()}, "BF16")
