"""Models described layer by layer beside the Llama family (and, for a mixture of experts, its
Mixtral form) at equal width, feed-forward, depth and vocabulary.

`python bench.py --workload latarax`, `biberax`, `badolix` or `muzopel` runs it on one GPU: prefill of one long prompt and
of several shorter ones, decode at several batch sizes, random weights and tokens.  For every kind of
kernel it reports the time of a profiled step and the fraction of the roofline (the larger of bytes /
measured HBM bandwidth and FLOPs / measured bf16 throughput, over the time).
"""
from __future__ import annotations

import numpy as np

VOCAB = 32000


def gla(heads, dim, vdim, ff):
    return {"type": "gla", "mixer": dict(heads=heads, dim=dim, vdim=vdim, tau=16.0), "mlp": {"kind": "dense", "ff": ff}}


def parallel(heads, kv, dim, window, keep, rec_heads, ff):
    decay = [1.0 - 2.0 ** (-3.0 - 5.0 * i / max(1, rec_heads - 1)) for i in range(rec_heads)]
    return {"type": "parallel",
            "mixer": {"left": dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=dim ** -0.5,
                                   mask=dict(size=window, keep_first=keep)),
                      "right": dict(heads=rec_heads, dim=128, vdim=128, decay=decay)},
            "mlp": {"kind": "dense", "ff": ff}}


def biberax_layers(heads, chunk, far, dense_ff, experts, top, ff, shared, layers):
    """Chunked and distance-biased attention in turn; a dense feed-forward first, experts after it."""
    sizes = dict(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5)
    rot = dict(base=500000.0, dims=128, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192))
    mixers = [("attention", dict(sizes, mask=dict(size=chunk), rot=rot)), ("attention_2", dict(sizes, bias_max=far))]
    moe = {"kind": "moe", "expert": dict(ff=ff, limit=7.0), "router": dict(experts=experts, top=top),
           "shared": dict(ff=shared, limit=7.0)}
    return [{"type": mixers[i % 2][0], "mixer": mixers[i % 2][1], "mlp": {"kind": "dense", "ff": dense_ff} if i == 0 else moe}
            for i in range(layers)]


def badolix_layers(heads, window, keep, dense_ff, experts, top, ff, layers):
    """Latent attention, a selective state space, windowed attention and a layer that shares its keys and
    values, in turn; dense feed-forwards and experts alternate."""
    rot = dict(base=500000.0, dims=128, scaling=dict(factor=8.0))
    yarn = dict(base=10000.0, dims=64, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0))
    attn = dict(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5, softcap=30.0, rot=rot,
                mask=dict(size=window, keep_first=keep))
    latent = dict(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, rot=yarn)
    mamba = dict(heads=4 * heads, vdim=64, state=128, groups=8, conv=4, norm_groups=8)
    dense = {"kind": "dense", "ff": dense_ff}
    moe = {"kind": "moe", "expert": dict(ff=ff), "router": dict(experts=experts, top=top, groups=dict(count=4, keep=2))}
    out = []
    for i in range(0, layers, 4):
        out += [{"type": "latent_attention", "mixer": latent, "mlp": dense}, {"type": "mamba2", "mixer": mamba, "mlp": moe},
                {"type": "attention", "mixer": attn, "mlp": dense}, {"type": "attention", "mixer": dict(attn, kv_from=i + 2), "mlp": moe}]
    return out


def muzopel_layers(heads, q_rank, experts, identity, top, ff, layers):
    """Latent attention with queries from a latent and gated heads, and without, in turn; experts without
    gates in every layer."""
    latent = dict(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5)
    rot = dict(base=10000.0, dims=64)
    yarn = dict(rot, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0))
    mixers = [("latent_attention", dict(latent, q_rank=q_rank, rot=yarn)), ("latent_attention_2", dict(latent, rot=rot))]
    moe = {"kind": "moe", "expert": dict(ff=ff), "router": dict(experts=experts, identity=identity, top=top)}
    return [{"type": mixers[i % 2][0], "mixer": mixers[i % 2][1], "mlp": moe} for i in range(layers)]


def sizes(design: str) -> list[dict]:
    """Layers of about 1.3B- and 8B-parameter models (dense ones; a mixture has more)."""
    if design == "muzopel":  # beside Badolix with the same latent attention and (gated) experts in every layer
        out = []
        for small in sizes("badolix"):
            llama, bad = small["llama"], small["badolix"]
            width, layers = llama["hidden_size"], llama["num_hidden_layers"]
            mixer, f = bad["layers"][0]["mixer"], bad["layers"][1]["mlp"]
            experts, top, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
            out.append({"name": small["name"],
                        "muzopel": {"architecture": "Muzopel", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-6, "groups": 4},
                                    "canon": {"taps": 4}, "logit_softcap": 30.0,
                                    "layers": muzopel_layers(width // 128, 3 * width // 8, experts, experts // 4, top, ff, layers)},
                        "badolix": dict(bad, layers=[{"type": "latent_attention", "mixer": mixer, "mlp": f}] * layers),
                        "llama": llama})
        return out
    if design == "badolix":  # beside the designs its kernels are shared with or like
        out = []
        for small, other in zip(sizes("biberax"), sizes("latarax")):
            llama, bib = small["llama"], small["biberax"]
            width, layers, f = llama["hidden_size"], llama["num_hidden_layers"], bib["layers"][1]["mlp"]
            experts, top, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
            out.append({"name": small["name"],
                        "badolix": {"architecture": "Badolix", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-6},
                                    "embedding": {"scale": 1.0}, "residual_mult": 1.0, "logit_scale": 1.0,
                                    "layers": badolix_layers(width // 128, 1024, 16, llama["intermediate_size"], experts, top, ff, layers)},
                        "biberax": bib, "latarax": other["latarax"], "llama": llama})
        return out
    if design == "biberax":
        out = []
        for width, dense_ff, experts, top, ff, shared, layers in ((2048, 5632, 16, 4, 1408, 1408, 12),
                                                                  (4096, 14336, 8, 2, 7168, 7168, 8)):
            heads = width // 128
            llama = dict(hidden_size=width, intermediate_size=dense_ff, num_hidden_layers=layers, num_attention_heads=heads,
                         num_key_value_heads=heads // 4, vocab_size=VOCAB, rms_norm_eps=1e-6, rope_theta=500000.0)
            out.append({"name": f"width {width}, {top} of {experts} experts of {ff}, {layers} layers",
                        "biberax": {"architecture": "Biberax", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-6},
                                    "layers": biberax_layers(heads, 1024, 1024, dense_ff, experts, top, ff, shared, layers)},
                        "llama": llama,
                        "mixtral": dict(llama, intermediate_size=ff, num_local_experts=experts, num_experts_per_tok=top)})
        return out
    out = []
    for width, ff, layers in ((2048, 5632, 12), (4096, 14336, 8)):
        heads = width // 128
        pattern = [gla(heads, 64, 128, ff), parallel(heads, heads // 4, 128, 1024, 16, heads // 2, ff)]
        out.append({
            "name": f"width {width}, ff {ff}, {layers} layers",
            "latarax": {"architecture": "Latarax", "width": width, "vocab": VOCAB, "streams": 4, "max_positions": 8192,
                        "norm": {"eps": 1e-6}, "layers": [pattern[i % 2] for i in range(layers)]},
            "llama": dict(hidden_size=width, intermediate_size=ff, num_hidden_layers=layers, num_attention_heads=heads,
                          num_key_value_heads=heads // 4, vocab_size=VOCAB, rms_norm_eps=1e-6, rope_theta=500000.0)})
    return out


# ------------------------------------------------------------------------- work per kind
def keys_seen(pos: np.ndarray, window: int, keep: int) -> float:
    lo = np.maximum(0, pos - window + 1) if window else np.zeros_like(pos)
    return float(np.sum(np.minimum(keep, lo) + pos - lo + 1))


def work(shape: dict, family: str, positions: list[np.ndarray], wanted: int) -> dict:
    """{kind: (bytes, flops)} of one step; positions[i] are the positions of segment i's rows."""
    rows = float(sum(len(p) for p in positions))
    w: dict = {}

    def add(kind, nbytes, flops=0.0):
        b, f = w.get(kind, (0.0, 0.0))
        w[kind] = (b + nbytes, f + flops)

    def gemm(kind, n, k, m=rows, n_out=None, out=2):
        add(kind, 2.0 * n * k + 2.0 * m * k + out * m * (n_out or n), 2.0 * m * n * k)

    def state_space(m, H):
        inner, bc, heads = m["heads"] * m["vdim"], 2 * m["groups"] * m["state"], m["heads"]
        st = heads * m["state"] * m["vdim"]
        gemm("gemm_qkv", 2 * inner + bc + heads, H)
        add("convolution", 4.0 * rows * (inner + bc) + 4.0 * len(positions) * (m["conv"] - 1) * (inner + bc))
        add("recurrence", 8.0 * st * len(positions) + rows * (2.0 * (inner + bc + heads) + 4.0 * inner), 6.0 * st * rows)
        add("norm", rows * inner * (4.0 + 2.0 + 2.0))
        gemm("gemm_o_proj", H, inner, out=4)

    def latent(m, H):
        h, d, r, v, c = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        if m.get("q_rank"):
            gemm("gemm_qkv", m["q_rank"] + c + r + h, H)
            add("norm", 4.0 * rows * m["q_rank"])
            gemm("gemm_qkv", h * (d + r), m["q_rank"])
        else:
            gemm("gemm_qkv", h * (d + r) + c + r, H)
        add("rope_kv", 4.0 * rows * (h * r + c + r))
        for p in positions:
            n, span, seen = len(p), float(p[-1] + 1), keys_seen(p, 0, 0)
            if n == 1:  # over the latent itself
                add("attention", 2.0 * (c + r) * span + 2.0 * h * (2 * c + r), 2.0 * h * (2 * c + r) * seen)
                add("latent", 2.0 * h * (d + v + 2 * c), 2.0 * h * c * (d + v))
            else:       # keys and values of the heads grown out of the latents
                add("attention", 2.0 * h * (d + v) * span + 2.0 * r * span + 2.0 * n * h * (d + r + v), 2.0 * h * (d + r + v) * seen)
                add("latent", 2.0 * span * (c + h * (d + v)), 2.0 * span * h * c * (d + v))
        add("latent", 2.0 * h * (d + v) * c)
        gemm("gemm_o_proj", H, h * v, out=4)

    def attention(heads, kv, dim, vdim, window, keep, chunk=0, tied=False, gated=False):
        if chunk:
            seen = sum(float(np.sum(p % chunk + 1)) for p in positions)
            span = sum(float(p[-1] - p[0] // chunk * chunk + 1) for p in positions)
            add("attention", 2.0 * kv * (dim + vdim) * span + 2.0 * rows * heads * (dim + vdim * (2 if gated else 1)),
                2.0 * heads * (dim + vdim) * seen)
            return
        if tied:  # one read serves as keys and values
            seen, span = sum(keys_seen(p, 0, 0) for p in positions), sum(float(p[-1] + 1) for p in positions)
            add("attention", (2.0 * kv * dim + 4.0) * span + 2.0 * rows * heads * (dim + vdim * (2 if gated else 1)),
                2.0 * heads * (dim + vdim) * seen)
            return
        seen = sum(keys_seen(p, window, keep) for p in positions)
        # every key a segment reads is counted once per segment (decode: once per row)
        span = sum((min(p[-1] + 1, len(p) - 1 + window + min(keep, max(0, p[0] - window + 1))) if window else p[-1] + 1)
                   for p in positions)
        add("attention", 2.0 * kv * (dim + vdim) * span + 2.0 * rows * heads * (dim + vdim), 2.0 * heads * (dim + vdim) * seen)

    if family in ("llama", "mixtral"):
        H, I, hq, kv = (shape[k] for k in ("hidden_size", "intermediate_size", "num_attention_heads", "num_key_value_heads"))
        for _ in range(shape["num_hidden_layers"]):
            gemm("gemm_qkv", (hq + 2 * kv) * 128, H)
            attention(hq, kv, 128, 128, 0, 0)
            gemm("gemm_o_proj", H, hq * 128)
            E = shape.get("num_local_experts", 1)  # every expert runs on every token
            gemm("gemm_gate_up", 2 * E * I, H, n_out=E * I)
            gemm("gemm_down", H, E * I)
        gemm("gemm_lm_head", shape["vocab_size"], H, m=rows, out=4)  # this family computes every row's logits
        return w
    if family == "biberax":
        H = shape["width"]
        for layer in shape["layers"]:
            m, f = layer["mixer"], layer["mlp"]
            tied = layer["type"] == "attention_2"
            q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            kv = k if tied else k + m["kv_heads"] * m["vdim"]
            gemm("gemm_qkv", q + kv + v, H)
            add("rope_kv", 4.0 * rows * (q + kv))
            attention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], 0, 0, m.get("mask", {}).get("size", 0), tied, True)
            gemm("gemm_o_proj", H, v, out=4)
            add("norm", 2 * rows * H * 14.0)
            if f["kind"] == "dense":
                gemm("gemm_gate_up", 2 * f["ff"], H, n_out=f["ff"])
                gemm("gemm_down", H, f["ff"], out=4)
            else:  # the experts' products, the shared one among them
                S = f["shared"]["ff"]
                gemm("experts_gate_up", 2 * S, H, n_out=S)
                gemm("experts_down", H, S)
                E, top, F = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
                picks = rows * top
                active = E * (1.0 - (1.0 - top / E) ** rows)
                add("routing", 2.0 * E * H + 2.0 * rows * H * (2 + top))
                add("experts_gate_up", 4.0 * active * F * H + 2.0 * picks * (H + F), 4.0 * picks * F * H)
                add("experts_down", 2.0 * active * F * H + 2.0 * picks * (H + F), 2.0 * picks * F * H)
                add("norm", (2.0 * picks + 2.0 * rows) * H)
        add("norm", wanted * H * 6.0)
        gemm("gemm_lm_head", shape["vocab"], H, m=wanted, out=4)
        return w
    if family == "badolix":
        H = shape["width"]
        for layer in shape["layers"]:
            m, f = layer["mixer"], layer["mlp"]
            if layer["type"] == "mamba2":
                state_space(m, H)
            elif layer["type"] == "latent_attention":
                latent(m, H)
            else:
                q, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
                kv = 0 if "kv_from" in m else m["kv_heads"] * (m["dim"] + m["vdim"])
                gemm("gemm_qkv", q + kv, H)
                add("rope_kv", 4.0 * rows * (q + kv))
                attention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"], m["mask"]["keep_first"])
                gemm("gemm_o_proj", H, v, out=4)
            add("norm", 2 * rows * H * 14.0)
            if f["kind"] == "dense":
                gemm("gemm_gate_up", 2 * f["ff"], H, n_out=f["ff"])
                gemm("gemm_down", H, f["ff"], out=4)
            else:
                E, top, F = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
                picks = rows * top
                active = E * (1.0 - (1.0 - top / E) ** rows)
                add("routing", 2.0 * E * H + 2.0 * rows * H * (2 + top))
                add("experts_gate_up", 4.0 * active * F * H + 2.0 * picks * (H + F), 4.0 * picks * F * H)
                add("experts_down", 2.0 * active * F * H + 2.0 * picks * (H + F), 2.0 * picks * F * H)
                add("norm", (2.0 * picks - 2.0 * rows) * H)
        add("norm", wanted * H * 6.0)
        gemm("gemm_lm_head", shape["vocab"], H, m=wanted, out=4)
        return w
    if family == "muzopel":
        H, held = shape["width"], shape["canon"]["taps"] - 1
        # a boundary: output, residual in and out, next input, inputs of earlier tokens
        past = sum(held + min(len(p), held) for p in positions)
        add("norm", rows * H * (2.0 + 4.0 + 2.0) + 4.0 * held * H * len(positions))  # the embedding
        for i, layer in enumerate(shape["layers"]):
            f = layer["mlp"]
            latent(layer["mixer"], H)
            add("norm", rows * H * 14.0 + 4.0 * past * H)
            E, top, F = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
            O = E + f["router"]["identity"]
            picks = rows * top * E / O
            active = E * (1.0 - (1.0 - top / O) ** rows)
            add("routing", 2.0 * O * H + 2.0 * rows * H + 2.0 * (rows + picks) * H)
            add("experts_gate_up", 2.0 * active * F * H + 2.0 * picks * (H + F), 2.0 * picks * F * H)
            add("experts_down", 2.0 * active * F * H + 2.0 * picks * (H + F), 2.0 * picks * F * H)
            # the weighted outputs in place of a product's rows, and the sum over depth
            add("norm", 2.0 * (picks + (rows if picks < rows * top else 0)) * H + rows * H * 10.0 + 4.0 * past * H)
            add("norm", rows * H * 4.0 * (i + 2))
        add("norm", wanted * H * 6.0)
        gemm("gemm_lm_head", shape["vocab"], H, m=wanted, out=4)
        return w
    H, S = shape["width"], shape["streams"]
    for layer in shape["layers"]:
        m, I = layer["mixer"], layer["mlp"]["ff"]
        recs = []
        if layer["type"] == "gla":
            q, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            gemm("gemm_qkv", 2 * q + 2 * v + 16, H)
            recs.append(m)
        else:
            a, r = m["left"], m["right"]
            recs.append(r)
            q, v = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            kvw = a["kv_heads"] * (a["dim"] + a["vdim"])
            gemm("gemm_qkv", a["heads"] * a["dim"] + kvw + 2 * q + 2 * v, H)
            add("rope_kv", 4.0 * rows * kvw)
            attention(a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["mask"]["size"], a["mask"]["keep_first"])
            gemm("gemm_o_proj", H, a["heads"] * a["vdim"], out=4)
        for r in recs:
            hd, hv, st = r["heads"] * r["dim"], r["heads"] * r["vdim"], r["heads"] * r["dim"] * r["vdim"]
            # state in and out once per segment; q, k, v in, o out; the recurrence itself is 6 flops per
            # state element and token (chunked forms do more, which is not counted)
            add("recurrence", 8.0 * st * len(positions) + rows * (2.0 * (2 * hd + hv) + 4.0 * hv), 6.0 * st * rows)
            add("norm", rows * hv * (4.0 + 2.0 + 2.0))
            gemm("gemm_o_proj", H, hv, out=4)
        for two in (layer["type"] != "gla", False):
            add("norm", rows * H * (8.0 * S + (8.0 if two else 4.0) + 2.0))
        gemm("gemm_gate_up", 2 * I, H, n_out=I)
        gemm("gemm_down", H, I, out=4)
    add("norm", wanted * H * (4.0 * S + 2.0))
    gemm("gemm_lm_head", shape["vocab"], H, m=wanted, out=4)
    return w


def kinds(ms: dict, w: dict, hbm_gbs: float, tflops: float) -> dict:
    out = {}
    for kind, (nbytes, flops) in w.items():
        t = ms.get(kind, 0.0)
        if t > 0:
            ideal = max(nbytes / (hbm_gbs * 1e9), flops / (tflops * 1e12)) * 1e3
            out[kind] = {"ms": round(t, 4), "roofline": round(ideal / t, 3)}
    out["other"] = {"ms": round(sum(v for k, v in ms.items() if k not in w), 4)}
    return out


# ------------------------------------------------------------------------------ timing
def prefill(eng, prompts, rows: int, steps: int, warmup: int):
    """ms of one pass over the prompts: portions of up to `rows` tokens a step, all prompts together."""
    per = max(1, rows // len(prompts))

    def run(profile=False):
        seqs = [eng.create_kv_cache() for _ in prompts]
        total, ms, at, n = 0.0, {}, 0, len(prompts[0])
        eng.set_profiling(profile)
        while at < n:
            c = min(per, n - at)
            last = at + c == n
            eng.step([(s, p[at:at + c], [c - 1] if last else []) for s, p in zip(seqs, prompts)], logits=False)
            total += eng.last_step_ms()
            if profile:
                ms = {k: ms.get(k, 0.0) + v for k, v in eng.profile_ms().items()}
            at += c
        eng.set_profiling(False)
        for s in seqs:
            s.free()
        return total, ms

    for _ in range(warmup):
        run()
    t = min(run()[0] for _ in range(steps))
    return t, run(profile=True)[1]


def decode(eng, batch: int, ctx: int, steps: int, warmup: int, rows: int):
    rng = np.random.default_rng(1)
    seqs = [eng.create_kv_cache() for _ in range(batch)]
    for s in seqs:
        p = rng.integers(0, VOCAB, ctx)
        for at in range(0, ctx, rows):
            eng.step([(s, p[at:at + rows], [])], logits=False)
    nxt = np.zeros(batch, dtype=np.uint32)
    draw = lambda: rng.integers(0, VOCAB, batch).astype(np.uint32)  # what greedy random weights repeat is no workload
    for _ in range(warmup):
        eng.decode_batch(seqs, draw(), next_tokens=nxt)
    ms = 0.0
    for _ in range(steps):
        eng.decode_batch(seqs, draw(), next_tokens=nxt)
        ms += eng.last_step_ms()
    _, prof = eng.profile_step(seqs, draw())
    launches = eng.last_step_launches()
    prof.pop("gemm", None)
    for s in seqs:
        s.free()
    return ms / steps, prof, launches


def run(hb, hbm_gbs: float, tflops: float, steps: int, warmup: int, design: str = "latarax", only: str = "",
        batches=(1, 16, 64, 128)) -> dict:
    rows, ctx = 2048, 1536
    report = {}
    launches = 0
    for size in sizes(design):
        if only and only not in size["name"]:
            continue
        entry = report[size["name"]] = {}
        for family in [design] + [f for f in ("badolix", "biberax", "latarax", "llama", "mixtral") if f != design]:
            shape = size.get(family)
            if not shape:
                continue
            kw = dict(max_seq_len=4224, max_batch=rows, max_seqs=128, num_kv_blocks=128 * 128)
            eng = hb.Engine.create_random_config(shape, **kw) if "architecture" in shape else \
                hb.Engine.create_random(shape, **{k: v for k, v in kw.items() if k != "max_seqs"})
            res = entry[family] = {"parameters": eng.param_count()}
            rng = np.random.default_rng(0)
            for label, n, length in (("prefill 1 x 4096", 1, 4096), ("prefill 8 x 512", 8, 512)):
                prompts = rng.integers(0, VOCAB, (n, length))
                ms, prof = prefill(eng, prompts, rows, 3, 2)
                per = max(1, rows // n)
                total: dict = {}
                for at in range(0, length, per):
                    w = work(shape, family, [np.arange(at, min(at + per, length))] * n, n if at + per >= length else 0)
                    for k, (b, f) in w.items():
                        total[k] = (total.get(k, (0, 0))[0] + b, total.get(k, (0, 0))[1] + f)
                res[label] = {"tok_s": round(n * length / ms * 1e3), "ms": round(ms, 3),
                              "kinds": kinds(prof, total, hbm_gbs, tflops)}
            for batch in batches:
                ms, prof, n_launch = decode(eng, batch, ctx, steps, warmup, rows)
                launches += n_launch * steps
                w = work(shape, family, [np.arange(ctx + warmup + steps, ctx + warmup + steps + 1)] * batch, batch)
                res[f"decode batch {batch}"] = {"tok_s": round(batch / ms * 1e3), "ms": round(ms, 4), "launches": n_launch,
                                                "kinds": kinds(prof, w, hbm_gbs, tflops)}
            eng.close()
    report["gpu_launches"] = launches
    return report
