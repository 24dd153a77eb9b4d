"""Latarax through the engine: whole prompts, portions, token by token, mixed batches, reused
blocks and slots, greedy generation — against the plain NumPy form of the whole model."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

from oracle import latarax_ref as R

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent


def gla(heads, dim, vdim, tau, ff=None):
    return {"type": "gla", "mixer": dict(heads=heads, dim=dim, vdim=vdim, tau=tau),
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def par(heads, kv, dim, vdim, scale, mask, rh, rd, rv, decay, ff=None):
    left = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale)
    if mask:
        left["mask"] = dict(size=mask[0], keep_first=mask[1])
    return {"type": "parallel", "mixer": {"left": left, "right": dict(heads=rh, dim=rd, vdim=rv, decay=decay)},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(width, vocab, streams, layers, eps=1e-5, max_positions=512):
    return {"architecture": "Latarax", "width": width, "vocab": vocab, "streams": streams, "max_positions": max_positions,
            "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # (config, low rank of the decays)
    "narrow": (model(96, 101, 2, [gla(3, 16, 24, 4.0, 80), par(4, 1, 24, 40, 0.3, (19, 5), 2, 24, 16, [0.9, 0.995], 72),
                                  gla(2, 24, 16, 1.0)]), 16),
    "odd": (model(75, 64, 3, [par(3, 3, 12, 20, 0.2, (33, 0), 3, 10, 7, [0.5, 0.97, 1.0]), gla(1, 9, 11, 7.5, 50)], eps=1e-3), 5),
    "one": (model(64, 48, 1, [par(1, 1, 32, 8, 0.5, (1, 1), 1, 32, 32, [0.8], 64), gla(1, 32, 64, 1.0, 64)]), 1),
    "wide": (model(128, 200, 4, [par(8, 1, 128, 256, 0.09, (70, 20), 2, 128, 72, [0.6, 0.999], 264), gla(2, 136, 80, 16.0, 128),
                                 par(2, 2, 64, 320, 0.12, None, 4, 16, 16, [0.99, 0.9, 0.7, 0.1], 40)]), 8),
    # split-K plans whose last K chunk and last feature tile are ragged
    "broad": (model(520, 1001, 3, [par(6, 2, 48, 80, 0.15, (64, 16), 3, 40, 56, [0.9, 0.99, 0.5], 1100),
                                   gla(5, 40, 104, 8.0, 1100)]), 12),
    "many": (model(72, 56, 6, [gla(2, 16, 16, 2.0, 40), gla(2, 16, 16, 3.0, 40),
                               par(20, 1, 8, 16, 0.4, (40, 3), 1, 8, 8, [0.95], 40)]), 3),
}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, (config, rank)) in enumerate(CONFIGS.items()):
        w = R.random_weights(config, seed=20 + i, rank=rank)
        path = tmp_path_factory.mktemp("latarax_" + name)
        R.write_model(str(path), config, w)
        out[name] = (config, w, str(path))
    return out


_expected = {}


def expected(models, name, tokens):
    key = (name, tuple(int(t) for t in tokens))
    if key not in _expected:
        _expected[key] = R.forward(models[name][0], models[name][1], tokens)
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


def check(got, want, dtype, where=""):
    e = errors(got, want)
    assert e.max() < LIMIT[dtype] and e.mean() < 0.5 * LIMIT[dtype], (where, int(e.argmax()), float(e.max()), float(e.mean()))


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
    check(feed(eng, seq, toks[:30], [30]), want[:30], dtype)
    logits = np.empty((1, 101), dtype=np.float32)
    rows = []
    for t in toks[30:]:
        nxt = eng.decode_batch([seq], [t], logits=logits)
        assert nxt[0] == np.argmax(logits[0])
        rows.append(logits[0].copy())
    check(np.stack(rows), want[30:], dtype)
    eng.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["narrow", "wide", "odd"])
def test_mixed_batches_and_reuse(hb, cuda, models, name, dtype):
    """Unequal requests come and go: portions beside single tokens, some left out of a step, the
    pool and the state slots just large enough, so that later requests get what earlier ones held."""
    rng = np.random.default_rng(11)
    lengths = [150, 5, 33, 97, 64, 16, 201, 2, 120, 80]
    reqs = [prompt(models, name, n, 100 + i) for i, n in enumerate(lengths)]
    live_cap, blocks = 4, 40
    eng = load(hb, models[name][2], dtype, tokens=blocks * 16, max_seqs=live_cap)
    waiting, live, got = list(range(len(reqs))), {}, {i: [] for i in range(len(reqs))}
    seen_slots = set()
    held = lambda: sum(-(-len(reqs[i]) // 16) for i in live)
    steps = 0
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
                seen_slots.update(live[i][0].block_table())
                live.pop(i)[0].free()
        steps += 1
    for i, toks in enumerate(reqs):
        check(np.concatenate(got[i]), expected(models, name, toks), dtype, i)
    assert eng.num_free_blocks() == blocks and eng.num_free_state_slots() == live_cap
    assert sum(-(-n // 16) for n in lengths) > blocks  # something was used twice
    eng.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_batch_against_each_alone(hb, cuda, models, dtype):
    """Decoding a batch of unequal contexts gives what each gives alone."""
    name = "wide"
    eng = load(hb, models[name][2], dtype, tokens=2048)
    reqs = [prompt(models, name, n, 40 + n) for n in (3, 70, 71, 130, 220)]
    seqs = [eng.create_kv_cache() for _ in reqs]
    for s, r in zip(seqs, reqs):
        eng.step([(s, r[:-2], [])])
    logits = np.empty((len(reqs), models[name][0]["vocab"]), dtype=np.float32)
    for k in (-2, -1):
        eng.decode_batch(seqs, [r[k] for r in reqs], logits=logits)
        for i, r in enumerate(reqs):
            check(logits[i:i + 1], expected(models, name, r)[k:][:1], dtype, (k, i))
    eng.close()


def plant_far_key(config, weights, layer, token, gain):
    """A token whose key of one attention head meets every query: the head's first channel of all
    queries is driven by the embedding's first column, and so is that token's key."""
    w = {k: v.copy() for k, v in weights.items()}
    W = config["width"]
    left = config["layers"][layer]["mixer"]["left"]
    p = f"l{layer}.mix.left."
    w["embed"][:, 0] = 3.0            # every token: the query's direction
    w["embed"][:, 1] = 0.0
    w["embed"][token, 1] = 40.0       # that token only: the key's direction
    w["pos"][:, :2] = 0.0
    per = left["heads"] // left["kv_heads"]
    for h in range(left["heads"]):
        w[p + "q"][h * left["dim"], :] = 0.0
        w[p + "q"][h * left["dim"], 0] = gain
    for g in range(left["kv_heads"]):
        w[p + "k"][g * left["dim"], :] = 0.0
        w[p + "k"][g * left["dim"], 1] = gain
    assert per >= 1 and W > 2
    return w


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("window,keep", [(37, 6), (32, 16)])
def test_a_standing_out_key_at_every_edge(hb, cuda, tmp_path, window, keep, dtype):
    """The same strong token placed first, at the last kept place, right after it, at block edges and
    far inside: its presence shows in every position that sees it, in prompts and in decoding."""
    config = model(64, 40, 2, [par(4, 2, 16, 24, 1.0, (window, keep), 1, 8, 8, [0.9], 32)])
    w = plant_far_key(config, R.random_weights(config, seed=9), 0, 7, 2.5)
    R.write_model(str(tmp_path), config, w)
    eng = load(hb, str(tmp_path), dtype)
    far = []
    for at in (0, keep - 1, keep, keep + 1, 47, 48, 63):
        toks = np.random.default_rng(at).integers(8, 40, 130)
        toks[at] = 7
        want = R.forward(config, w, toks)
        for sizes in ([130], [50, 2, 3], [70] + [1] * 60):
            seq = eng.create_kv_cache()
            check(feed(eng, seq, toks, sizes), want, dtype, (at, sizes[0]))
            seq.free()
        # the oracle itself must feel the token: without the kept places the logits move
        config2 = json.loads(json.dumps(config))
        config2["layers"][0]["mixer"]["left"]["mask"] = dict(size=window + 1, keep_first=keep)
        e = errors(R.forward(config2, w, toks), want)
        far.append(float(e[min(129, at + window)]) if at >= keep else 1.0)
    assert min(far) > 4 * LIMIT["bf16"], far
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
    assert eng.num_free_state_slots() == 3 and eng.num_free_blocks() == 25
    # drawing: the same seed gives the same tokens whatever else is in the batch
    one = serve.generate(eng, prompts[:1], 10, temperature=0.8, top_p=0.9, seed=4)
    many = serve.generate(eng, prompts, 10, max_live=3, temperature=0.8, top_p=0.9, seed=4)
    assert one[0] == many[0] and max(max(o) for o in many) < config["vocab"]
    eng.close()


def test_generate_and_replay_commands(hb, cuda, models, tmp_path):
    config, w, path = models["one"]
    p = prompt(models, "one", 21, 5)
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
    want = expected(models, "one", p)
    check(np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(2, -1), want[[0, 8]], "f32")
    check(np.fromfile(tmp_path / "2.f32", dtype="<f4").reshape(1, -1), want[[20]], "f32")
    assert not (tmp_path / "1.f32").exists()


def test_limits_and_refusals(hb, cuda, models, tmp_path):
    config, w, path = models["one"]
    eng = load(hb, path, "bf16", tokens=1200, max_seqs=2)
    a, b, c = (eng.create_kv_cache() for _ in range(3))
    eng.step([(a, [1, 2, 3], [2]), (b, [4], [0])])
    with pytest.raises(hb.HbError, match="state slot"):
        eng.step([(c, [1], [0])])
    b.free()
    eng.step([(c, [1], [0])])                      # the freed slot serves the next sequence
    with pytest.raises(hb.HbError, match="recurrent state"):
        eng.truncate(a, 1)
    eng.truncate(a, 0)                             # forgetting everything is possible
    toks = prompt(models, "one", 20, 2)
    check(feed(eng, a, toks, [20]), expected(models, "one", toks), "bf16")
    with pytest.raises(hb.HbError, match="recurrent state"):
        eng.decode_batch_tables([1], [0], [[0]])
    with pytest.raises(hb.HbError, match="recurrent state"):
        eng.kv_copy_blocks([(0, 1)])
    with pytest.raises(hb.HbError, match="positions"):
        eng.step([(a, prompt(models, "one", 500, 1), [])])
    with pytest.raises(hb.HbError, match="vocabulary"):
        eng.step([(a, [48], [])])
    with pytest.raises(hb.HbError, match="repeated"):
        eng.step([(a, [1], []), (a, [2], [])])
    with pytest.raises(hb.HbError, match="ascend"):
        eng.step([(a, [1, 2], [1, 0])])
    eng.close()
    with pytest.raises(hb.HbError, match="f16"):
        hb.Engine.load(path, bf16=False)
    for change, text in (({"architecture": "Unheard"}, "not served"), ({"streams": 99}, "streams"), ({"norm": {}}, "eps"),
                         ({"layers": [dict(config["layers"][1], type="other")]}, "unknown type"), ({"width": 72}, "shape")):
        bad = dict(json.loads(json.dumps(config)), **change)
        R.write_model(str(tmp_path), bad, w)
        with pytest.raises(hb.HbError, match=text):
            load(hb, str(tmp_path), "bf16")
    R.write_model(str(tmp_path), config, {k: v for k, v in w.items() if k != "l1.mix.a1"})
    with pytest.raises(hb.HbError, match="l1.mix.a1"):
        load(hb, str(tmp_path), "bf16")


def test_random_engine_and_profile(hb, cuda):
    config = CONFIGS["wide"][0]
    eng = hb.Engine.create_random_config(config, max_seq_len=128, max_batch=128, max_seqs=4)
    seqs = [eng.create_kv_cache() for _ in range(4)]
    eng.step([(s, np.arange(20) + i, []) for i, s in enumerate(seqs)])
    nxt, ms = eng.profile_step(seqs, np.arange(4))
    assert len(nxt) == 4 and ms["recurrence"] > 0 and ms["attention"] > 0 and ms["gemm"] > 0
    assert eng.step_bytes([20] * 4) > 0 and eng.gemm_bytes(4) > 0 and eng.last_step_launches() > 10
    eng.close()
