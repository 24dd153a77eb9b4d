"""Biberax through the engine: whole prompts, portions, token by token, mixed batches, reused blocks,
caller-owned block tables, long decoding, greedy generation — against the plain NumPy form of the
whole model."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

from oracle import biberax_ref as R

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=1.5, shared=None):
    out = {"kind": "moe", "expert": dict(ff=ff, limit=limit), "router": dict(experts=experts, top=top)}
    if shared:
        out["shared"] = dict(ff=shared[0], limit=shared[1])
    return out


def chunked(heads, kv, dim, vdim, scale, size, rot, mlp, scaling=None):
    r = dict(base=rot[0], dims=rot[1])
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mlp": mlp,
            "mixer": dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, mask=dict(size=size), rot=r)}


def biased(heads, kv, dim, scale, far, mlp):
    return {"type": "attention_2", "mlp": mlp,
            "mixer": dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale, bias_max=far)}


def model(width, vocab, layers, eps=1e-5):
    return {"architecture": "Biberax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # (config, rows of the bias tables)
    "narrow": (model(80, 61, [chunked(3, 1, 24, 40, 0.25, 19, (1e3, 16), moe(5, 2, 40, 1.1, (24, 0.7)), (8.0, 1.0, 4.0, 64)),
                              biased(4, 2, 16, 0.3, 90, dense(72)),
                              chunked(2, 2, 16, 24, 0.3, 32, (500.0, 16), None)]), 14),
    "odd": (model(75, 64, [biased(5, 1, 9, 0.4, 33, moe(3, 3, 11, 3.0, (13, 2.0))),
                           chunked(3, 3, 10, 7, 0.2, 7, (100.0, 6), dense(50)),
                           biased(3, 3, 15, 0.2, 300, moe(7, 1, 20, 0.9))], eps=1e-3), 9),
    "one": (model(64, 48, [chunked(1, 1, 32, 8, 0.5, 1, (10.0, 2), moe(1, 1, 16, 2.5)),
                           biased(1, 1, 8, 0.5, 7, None)]), 1),
    "wide": (model(128, 200, [chunked(8, 1, 128, 256, 0.09, 70, (1e4, 128), dense(264), (2.0, 0.5, 6.0, 100)),
                              biased(2, 1, 320, 0.05, 120, moe(4, 2, 136, 1.6, (72, 1.2))),
                              biased(8, 2, 64, 0.12, 16, moe(16, 4, 24, 1.4, (40, 1.4)))]), 20),
    # plans whose last K chunk and last feature tile are ragged
    "broad": (model(520, 1001, [biased(6, 2, 48, 0.15, 64, moe(9, 3, 296, 2.0, (1100, 1.0))),
                                chunked(6, 2, 48, 80, 0.15, 48, (2e4, 40), dense(1100))]), 33),
    "many": (model(72, 56, [biased(20, 1, 16, 0.3, 50, moe(40, 6, 16, 1.0, (32, 3.0))),
                            chunked(34, 2, 8, 16, 0.4, 40, (50.0, 4), moe(10, 9, 24, 5.0))]), 2),
}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, (config, buckets)) in enumerate(CONFIGS.items()):
        w = R.steady_routers(config, R.random_weights(config, seed=40 + i, buckets=buckets))
        path = tmp_path_factory.mktemp("biberax_" + name)
        R.write_model(str(path), config, w)
        out[name] = (config, w, str(path))
    return out


_expected = {}


def expected(models, name, tokens):
    """(logits, least router margin of every position over the layers)"""
    key = (name, tuple(int(t) for t in tokens))
    if key not in _expected:
        margins = []
        logits = R.forward(models[name][0], models[name][1], tokens, margins_out=margins)
        _expected[key] = logits, np.min(margins, axis=0) if margins else np.full(len(tokens), np.inf)
    return _expected[key]


def load(hb, path, dtype, tokens=1024, max_seqs=6, max_batch=640):
    return hb.Engine.load(path, max_seq_len=512, bf16=dtype == "bf16", force_f32=dtype == "f32", max_batch=max_batch,
                          max_seqs=max_seqs, num_kv_blocks=tokens // 16)


def prompt(models, name, n, seed):
    return np.random.default_rng(seed).integers(0, models[name][0]["vocab"], n)


def errors(got, want):
    d = got - want
    d = d - d.mean(axis=1, keepdims=True)
    return np.sqrt((d * d).mean(axis=1)) / np.sqrt(np.mean((want - want.mean(axis=1, keepdims=True)) ** 2))


LIMIT = {"f32": 3e-5, "bf16": 5e-2}


def check(got, want, dtype, where="", rows=slice(None)):
    """want: logits, or (logits, margins): in bf16 a token whose experts hang on a close call may go
    to another one, so such positions only count for the median."""
    want, margin = want if isinstance(want, tuple) else (want, np.full(len(want), np.inf))
    e = errors(got, want[rows])
    clear = margin[rows] > (0.02 if dtype == "bf16" else 0.0)
    worst = e[clear].max() if clear.any() else 0.0
    assert worst < LIMIT[dtype] and np.median(e) < 0.5 * LIMIT[dtype], (where, int(e.argmax()), float(worst), float(e.mean()))


def feed(eng, seq, tokens, sizes):
    """All logits of `tokens`, fed in portions whose sizes repeat `sizes`."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[i % len(sizes)], len(tokens) - at)
        out.append(eng.step([(seq, tokens[at:at + n], range(n))])[1])
        at += n
        i += 1
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", CONFIGS)
def test_whole_prompt(hb, cuda, models, name, dtype):
    eng = load(hb, models[name][2], dtype)
    assert eng.num_layers() == len(models[name][0]["layers"]) and eng.hidden_size() == models[name][0]["width"]
    assert eng.param_count() == sum(v.size for v in models[name][1].values())
    for n in (1, 2, 17, 301):
        toks = prompt(models, name, n, n)
        seq = eng.create_kv_cache()
        check(feed(eng, seq, toks, [n]), expected(models, name, toks), dtype, n)
        assert len(seq) == n
        seq.free()
    eng.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", CONFIGS)
def test_portions_and_single_tokens(hb, cuda, models, name, dtype):
    """The same prompt in portions of many sizes, and token by token: prefill against decoding."""
    eng = load(hb, models[name][2], dtype)
    toks = prompt(models, name, 210, 3)
    want = expected(models, name, toks)
    for sizes in ([2], [3, 61], [16], [64, 1, 2], [9, 130], [1]):
        seq = eng.create_kv_cache()
        check(feed(eng, seq, toks, sizes), want, dtype, sizes)
        seq.free()
    eng.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_decoding(hb, cuda, models, dtype):
    eng = load(hb, models["narrow"][2], dtype)
    toks = prompt(models, "narrow", 480, 8)
    want = expected(models, "narrow", toks)
    seq = eng.create_kv_cache()
    check(feed(eng, seq, toks[:30], [30]), want, dtype, rows=slice(0, 30))
    logits = np.empty((1, 61), dtype=np.float32)
    rows = []
    for t in toks[30:]:
        nxt = eng.decode_batch([seq], [t], logits=logits)
        assert nxt[0] == np.argmax(logits[0])
        rows.append(logits[0].copy())
    check(np.stack(rows), want, dtype, rows=slice(30, None))
    eng.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["narrow", "wide", "odd", "many"])
def test_mixed_batches_and_reuse(hb, cuda, models, name, dtype):
    """Unequal requests come and go: portions beside single tokens, some left out of a step, the
    pool just large enough, so that later requests get the blocks that earlier ones held."""
    rng = np.random.default_rng(11)
    lengths = [150, 5, 33, 97, 64, 16, 201, 2, 120, 80]
    reqs = [prompt(models, name, n, 100 + i) for i, n in enumerate(lengths)]
    live_cap, blocks = 4, 40
    eng = load(hb, models[name][2], dtype, tokens=blocks * 16, max_seqs=live_cap)
    waiting, live, got = list(range(len(reqs))), {}, {i: [] for i in range(len(reqs))}
    held = lambda: sum(-(-len(reqs[i]) // 16) for i in live)
    while waiting or live:
        while waiting and len(live) < live_cap and held() + -(-len(reqs[waiting[0]]) // 16) <= blocks:
            i = waiting.pop(0)
            live[i] = [eng.create_kv_cache(), 0]
        entries, plan = [], []
        for i, (seq, at) in live.items():
            if len(live) > 1 and rng.random() < 0.2:
                continue
            n = int(min(len(reqs[i]) - at, rng.choice([1, 1, 1, 2, 3, 15, 16, 31, 70, 128])))
            entries.append((seq, reqs[i][at:at + n], range(n)))
            plan.append((i, n))
        if not entries:
            continue
        logits = eng.step(entries)[1]
        at = 0
        for i, n in plan:
            got[i].append(logits[at:at + n])
            at += n
            live[i][1] += n
            if live[i][1] == len(reqs[i]):
                live.pop(i)[0].free()
    for i, toks in enumerate(reqs):
        check(np.concatenate(got[i]), expected(models, name, toks), dtype, i)
    assert eng.num_free_blocks() == blocks
    assert sum(-(-n // 16) for n in lengths) > blocks  # something was used twice
    eng.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["wide", "many"])
def test_batch_against_each_alone(hb, cuda, models, name, dtype):
    """Decoding a batch of unequal contexts gives what each gives alone."""
    eng = load(hb, models[name][2], dtype, tokens=2048)
    reqs = [prompt(models, name, n, 40 + n) for n in (3, 70, 71, 130, 220)]
    seqs = [eng.create_kv_cache() for _ in reqs]
    for s, r in zip(seqs, reqs):
        eng.step([(s, r[:-2], [])])
    logits = np.empty((len(reqs), models[name][0]["vocab"]), dtype=np.float32)
    for k in (-2, -1):
        eng.decode_batch(seqs, [r[k] for r in reqs], logits=logits)
        for i, r in enumerate(reqs):
            check(logits[i:i + 1], expected(models, name, r), dtype, (k, i), rows=slice(len(r) + k, len(r) + k + 1))
    eng.close()


def test_a_wide_batch_of_decoded_tokens(hb, cuda, models):
    """More rows than a batch tile of any expert holds, unequal contexts."""
    name = "narrow"
    eng = load(hb, models[name][2], "f32", tokens=8192, max_seqs=150)
    base = prompt(models, name, 60, 77)
    want = expected(models, name, base)
    lens = [3 + i % 50 for i in range(150)]
    seqs = [eng.create_kv_cache() for _ in lens]
    for s, n in zip(seqs, lens):
        eng.step([(s, base[:n], [])])
    logits = np.empty((150, 61), dtype=np.float32)
    eng.decode_batch(seqs, [base[n] for n in lens], logits=logits)
    assert errors(logits, want[0][lens]).max() < LIMIT["f32"]
    eng.close()


def plant_far_key(config, weights, layer, token, gain):
    """A token whose key of every head meets every query: the first channel of all queries is driven
    by the embedding's first column, and so is that token's key by its second.  Unrotated places are
    used, so the score does not turn with the distance."""
    w = {k: v.copy() for k, v in weights.items()}
    m = config["layers"][layer]["mixer"]
    p = f"l{layer}.mix."
    w["embed"][:, 0] = 3.0            # every token: the query's direction
    w["embed"][:, 1] = 0.0
    w["embed"][token, 1] = 40.0       # that token only: the key's direction
    at = m["dim"] - 1                 # a channel that is not rotated
    for name, heads, col in (("q", m["heads"], 0), ("k", m["kv_heads"], 1)):
        for h in range(heads):
            w[p + name][h * m["dim"] + at, :] = 0.0
            w[p + name][h * m["dim"] + at, col] = gain
    return w


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("size", [37, 32, 48])
def test_a_standing_out_key_at_every_edge_of_a_chunk(hb, cuda, tmp_path, size, dtype):
    """The same strong token first, last and first of the next chunk, at block edges: its presence
    shows in every position of its chunk and in none of the next, in prompts and in decoding."""
    config = model(64, 40, [chunked(4, 2, 16, 24, 1.0, size, (100.0, 8), dense(32))])
    w = plant_far_key(config, R.random_weights(config, seed=9), 0, 7, 2.5)
    R.write_model(str(tmp_path), config, w)
    eng = load(hb, str(tmp_path), dtype)
    felt = []
    for at in (0, size - 1, size, 47, 48, 63):
        toks = np.random.default_rng(at).integers(8, 40, 130)
        toks[at] = 7
        want = R.forward(config, w, toks)
        for sizes in ([130], [50, 2, 3], [70] + [1] * 60):
            seq = eng.create_kv_cache()
            check(feed(eng, seq, toks, sizes), want, dtype, (at, sizes[0]))
            seq.free()
        # the oracle itself must feel the token: with chunks one longer the logits move
        config2 = json.loads(json.dumps(config))
        config2["layers"][0]["mixer"]["mask"]["size"] = size + 1
        felt.append(errors(R.forward(config2, w, toks), want).max())
    assert min(felt) > 4 * LIMIT["bf16"], felt
    eng.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_a_standing_out_far_key_and_the_bias_edges(hb, cuda, tmp_path, dtype):
    """A single strong key far away (past the last bucket), and bias rows that differ by several
    units from bucket to bucket, so that a distance in the wrong bucket shows."""
    config = model(64, 40, [biased(4, 2, 16, 1.0, 61, dense(32))])
    w = R.random_weights(config, seed=10, buckets=11)
    w["l0.mix.rel"] = 3.0 * np.sign(w["l0.mix.rel"]) * (1 + np.arange(11) % 3)[:, None]
    w["l0.mix.sink"] = np.round(w["l0.mix.sink"]) + 9.0
    w = plant_far_key(config, w, 0, 7, 1.5)
    R.write_model(str(tmp_path), config, w)
    eng = load(hb, str(tmp_path), dtype)
    for at in (0, 1, 15, 16, 100):
        toks = np.random.default_rng(at).integers(8, 40, 250)
        toks[at] = 7
        want = R.forward(config, w, toks)
        for sizes in ([250], [90, 2, 3], [180] + [1] * 70):
            seq = eng.create_kv_cache()
            check(feed(eng, seq, toks, sizes), want, dtype, (at, sizes[0]))
            seq.free()
    # the oracle itself feels a shifted bucket edge, a missing sink and a missing far key
    config2 = json.loads(json.dumps(config))
    config2["layers"][0]["mixer"]["bias_max"] = 66
    assert errors(R.forward(config2, w, toks), want).max() > 4 * LIMIT["bf16"]
    assert errors(R.forward(config, dict(w, **{"l0.mix.sink": w["l0.mix.sink"] - 50}), toks), want).max() > 4 * LIMIT["bf16"]
    toks2 = toks.copy()
    toks2[100] = 8
    assert errors(R.forward(config, w, toks2), want)[180:].max() > 4 * LIMIT["bf16"]
    eng.close()


def greedy_margin(rows):
    top = np.sort(np.asarray(rows), axis=1)[:, -2:]
    return (top[:, 1] - top[:, 0]) / np.sqrt(np.mean(np.asarray(rows) ** 2))


def test_greedy_generation_through_the_scheduler(hb, cuda, models):
    from vllm_hb_b200 import serve

    name = "narrow"
    config, w, path = models[name]
    prompts = [prompt(models, name, n, 60 + n).tolist() for n in (5, 40, 1, 23, 90, 17)]
    want = [R.greedy_generate(config, w, p, 12) for p in prompts]
    eng = load(hb, path, "f32", tokens=400, max_seqs=3)
    got = serve.generate(eng, prompts, 12, max_live=3, step_tokens=24)
    for g, (toks, rows), p in zip(got, want, prompts):
        clear = greedy_margin(rows) > 1e-3
        first_unclear = len(clear) if clear.all() else int(np.argmin(clear))
        assert g[:first_unclear] == toks[:first_unclear], len(p)
    assert eng.num_free_blocks() == 25
    # drawing: the same seed gives the same tokens whatever else is in the batch
    one = serve.generate(eng, prompts[:1], 10, max_live=3, temperature=0.8, top_p=0.9, seed=4)
    many = serve.generate(eng, prompts, 10, max_live=3, temperature=0.8, top_p=0.9, seed=4)
    assert one[0] == many[0] and max(max(o) for o in many) < config["vocab"]
    eng.close()


def test_generate_and_replay_commands(hb, cuda, models, tmp_path):
    config, w, path = models["odd"]
    p = prompt(models, "odd", 21, 5)
    out = subprocess.run([sys.executable, str(ROOT / "bin" / "generate"), "--model", path, "--dtype", "float32", "--max-tokens",
                          "6"], input=json.dumps(p.tolist()) + "\n", capture_output=True, text=True, timeout=120)
    assert out.returncode == 0, out.stderr
    toks, rows = R.greedy_generate(config, w, p.tolist(), 6)
    if (greedy_margin(rows) > 1e-3).all():
        assert json.loads(out.stdout) == toks
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": p[:9].tolist(), "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": p[9:20].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": p[20:].tolist(), "want": [0]}], "end": ["a"]}]
    out = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", path, "--dtype", "float32", "--out", str(tmp_path),
                          "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                         text=True, timeout=120)
    assert out.returncode == 0 and out.stdout.split("\n")[:3] == ["done 0", "done 1", "done 2"], out.stderr
    want = expected(models, "odd", p)[0]
    check(np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(2, -1), want[[0, 8]], "f32")
    check(np.fromfile(tmp_path / "2.f32", dtype="<f4").reshape(1, -1), want[[20]], "f32")
    assert not (tmp_path / "1.f32").exists()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_caller_owned_tables_copies_swaps_and_truncation(hb, cuda, models, dtype):
    """Blocks are moved with all they hold (keys, values, scales of keys): a prefix shared by two
    tables, copied on write, swapped out and in, and a sequence wound back."""
    name = "narrow"
    eng = load(hb, models[name][2], dtype, tokens=640)
    toks = prompt(models, name, 70, 21)
    other = toks.copy()
    other[40:] = prompt(models, name, 30, 22)
    want, want2 = expected(models, name, toks), expected(models, name, other)
    row = np.empty(61, dtype=np.float32)
    table = [30, 5, 17, 2, 9]
    row = eng.forward_tables(toks[:40], 0, table)
    check(row[None], want, dtype, rows=slice(39, 40))
    # the second sequence shares blocks 30 and 5 and takes a copy of the half-filled 17
    eng.kv_copy_blocks([(17, 21)])
    table2 = [30, 5, 21, 3, 4]
    check(eng.forward_tables(toks[40:], 40, table)[None], want, dtype, rows=slice(69, 70))
    check(eng.forward_tables(other[40:], 40, table2)[None], want2, dtype, rows=slice(69, 70))
    # everything of the first sequence out, its blocks overwritten, back into other blocks
    eng.reserve_cpu_blocks(8)
    eng.kv_swap_blocks([(b, i) for i, b in enumerate(table)], to_cpu=True)
    eng.forward_tables(prompt(models, name, 70, 23), 0, table)
    back = [11, 12, 13, 14, 15]
    eng.kv_swap_blocks([(i, b) for i, b in enumerate(back)], to_cpu=False)
    logits = np.empty((1, 61), dtype=np.float32)
    eng.decode_batch_tables([toks[69]], [69], [back], logits=logits)
    check(logits, want, dtype, rows=slice(69, 70))
    # a sequence wound back in the middle of a block goes on differently
    seq = eng.create_kv_cache()
    feed(eng, seq, toks[:61], [61])
    eng.truncate(seq, 40)
    check(feed(eng, seq, other[40:], [7]), want2, dtype, rows=slice(40, None))
    eng.close()


def test_refusals(hb, cuda, models, tmp_path):
    config, w, path = models["narrow"]
    with pytest.raises(hb.HbError, match="f16"):
        hb.Engine.load(path, bf16=False)

    def altered(layer, **mixer):
        c = json.loads(json.dumps(config))
        c["layers"][layer]["mixer"].update(mixer)
        return c

    def fed(layer, **mlp):
        c = json.loads(json.dumps(config))
        c["layers"][layer]["mlp"].update(mlp)
        return c

    cases = [(dict(config, norm={}), "eps"), (dict(config, width=72), "shape"), (dict(config, layers=[]), "no layers"),
             (dict(config, layers=[dict(config["layers"][0], type="other")]), "unknown type"),
             (altered(0, heads=0), "sizes"), (altered(0, kv_heads=2), "sizes"), (altered(0, mask=dict(size=0)), "chunks"),
             (altered(0, rot=dict(base=10.0, dims=26)), "rotation"), (altered(0, rot=dict(base=10.0, dims=5)), "rotation"),
             (altered(1, vdim=8), "width"), (altered(1, bias_max=0), "bias_max"), (fed(0, kind="other"), "unknown kind"),
             (fed(0, router=dict(experts=5, top=6)), "experts"), (fed(0, expert=dict(ff=40)), "limit"),
             (fed(0, router=dict(experts=6, top=2)), "l0.mlp.e5")]
    for bad, text in cases:
        R.write_model(str(tmp_path), bad, w)
        with pytest.raises(hb.HbError, match=text):
            load(hb, str(tmp_path), "bf16")
    for missing in ("l1.mix.rel", "l1.mix.sink", "l0.mlp.router.b", "l1.mix.o.b", "final.norm"):
        R.write_model(str(tmp_path), config, {k: v for k, v in w.items() if k != missing})
        with pytest.raises(hb.HbError, match=missing):
            load(hb, str(tmp_path), "bf16")


def test_random_engine_and_profile(hb, cuda):
    config = CONFIGS["wide"][0]
    eng = hb.Engine.create_random_config(config, max_seq_len=128, max_batch=128, max_seqs=4)
    seqs = [eng.create_kv_cache() for _ in range(4)]
    eng.step([(s, np.arange(20) + i, []) for i, s in enumerate(seqs)])
    nxt, ms = eng.profile_step(seqs, np.arange(4))
    assert len(nxt) == 4 and min(ms[k] for k in ("routing", "experts_gate_up", "experts_down", "attention", "gemm")) > 0
    assert eng.step_bytes([20] * 4) > 0 and eng.gemm_bytes(4) > 0 and eng.last_step_launches() > 10
    eng.close()
