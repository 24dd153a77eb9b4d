"""Badolix through the engine: whole prompts, portions, token by token, mixed batches, reused blocks and
state slots, long decoding, greedy generation — against the plain NumPy form of the whole model."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

from oracle import badolix_ref as R
from tests.test_gpu_biberax import LIMIT, check, errors, feed, greedy_margin, load

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None):
    router = dict(experts=experts, top=top)
    if groups:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    return {"kind": "moe", "expert": dict(ff=ff), "router": router}


def windowed(heads, kv, dim, vdim, scale, cap, size, keep, rot, mlp, factor=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, softcap=cap, mask=dict(size=size, keep_first=keep),
             rot=dict(base=rot[0], dims=rot[1]))
    if factor:
        m["rot"]["scaling"] = dict(factor=factor)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def latent(heads, dim, rot_dim, vdim, rank, scale, base, mlp, scaling=None):
    rot = dict(base=base, dims=rot_dim)
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank, scale=scale, rot=rot)}


def mamba(heads, vdim, state, groups, taps, norm_groups, mlp):
    return {"type": "mamba2", "mlp": mlp,
            "mixer": dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=taps, norm_groups=norm_groups)}


def model(width, vocab, layers, eps=1e-5, embed=1.0, mult=1.0, logit=1.0):
    return {"architecture": "Badolix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "residual_mult": mult, "logit_scale": logit, "layers": layers}


YARN = (8.0, 96, 12.0, 1.0)

CONFIGS = {
    "narrow": model(80, 61, [windowed(4, 2, 24, 40, 0.25, 9.0, 19, 3, (1e3, 16), moe(6, 2, 40, (3, 2)), 4.0),
                             mamba(4, 16, 24, 2, 4, 4, dense(72)),
                             latent(3, 16, 8, 24, 40, 0.2, 1e3, None, YARN),
                             windowed(6, 2, 24, 40, 0.3, 4.0, 40, 0, (1e3, 16), dense(40), 4.0, kv_from=0)], 1e-5, 2.0, 0.7, 0.5),
    # sizes that are multiples of nothing
    "odd": model(75, 64, [latent(5, 9, 6, 7, 11, 0.3, 50.0, moe(9, 2, 11, (3, 1))),
                          mamba(3, 7, 5, 1, 3, 3, dense(50)),
                          windowed(3, 1, 9, 15, 0.2, 2.5, 7, 2, (100.0, 6), moe(7, 1, 20)),
                          windowed(2, 1, 9, 15, 0.4, 30.0, 33, 1, (100.0, 6), dense(19), kv_from=2)], 1e-3, 1.4, 0.6, 1.7),
    "one": model(64, 48, [mamba(1, 8, 8, 1, 1, 1, moe(1, 1, 16)),
                          latent(1, 8, 2, 8, 8, 0.5, 10.0, None),
                          windowed(1, 1, 16, 8, 0.5, 1.0, 1, 0, (10.0, 2), dense(8))]),
    "wide": model(128, 200, [mamba(8, 64, 128, 1, 2, 1, moe(12, 3, 24, (4, 2))),
                             latent(8, 64, 32, 64, 256, 0.06, 1e4, dense(264), (4.0, 64, 20.0, 2.0)),
                             mamba(6, 72, 144, 3, 6, 2, None),
                             windowed(8, 1, 128, 128, 0.09, 20.0, 70, 16, (1e4, 128), moe(16, 4, 24, (2, 2)), 2.0),
                             windowed(16, 1, 128, 128, 0.05, 50.0, 33, 5, (1e4, 128), dense(72), 2.0, kv_from=3)], 1e-6, 0.5, 0.8, 2.0),
    # plans whose last K chunk and last feature tile are ragged, a latent beyond one value slice
    "broad": model(520, 1001, [latent(6, 48, 16, 40, 320, 0.1, 2e4, dense(1100)),
                               mamba(10, 48, 40, 5, 4, 5, moe(9, 3, 296, (3, 2)))]),
    # more heads than a tile or a row's CTA takes
    "many": model(72, 56, [latent(70, 8, 8, 8, 24, 0.4, 80.0, moe(40, 6, 16, (8, 3)), (2.0, 32, 5.0, 1.0)),
                           windowed(34, 2, 8, 16, 0.4, 3.0, 40, 17, (50.0, 4), moe(10, 9, 24)),
                           mamba(40, 8, 16, 8, 5, 8, dense(32))]),
}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for i, (name, config) in enumerate(CONFIGS.items()):
        w = R.steady_routers(config, R.random_weights(config, seed=70 + i))
        path = tmp_path_factory.mktemp("badolix_" + name)
        R.write_model(str(path), config, w)
        out[name] = (config, w, str(path))
    return out


_clear = {}


def prompt(models, name, n, seed):
    """Random tokens whose experts hang on no close call: a choice that rounding turns over would be felt
    by all later tokens, through attention and states."""
    if name not in _clear:
        config, w, _ = models[name]
        margins = []
        for t in range(config["vocab"]):
            own = []
            R.forward(config, w, [t], margins_out=own)
            margins.append(min((float(m[0]) for m in own), default=np.inf))
        _clear[name] = np.flatnonzero(np.array(margins) > 0.08)
        assert len(_clear[name]) >= 12, name
    return np.random.default_rng(seed).choice(_clear[name], n)


_expected = {}


def expected(models, name, tokens):
    """(logits, least router margin of every position over the layers)"""
    key = (name, tuple(int(t) for t in tokens))
    if key not in _expected:
        margins = []
        logits = R.forward(models[name][0], models[name][1], tokens, margins_out=margins)
        _expected[key] = logits, np.min(margins, axis=0) if margins else np.full(len(tokens), np.inf)
    return _expected[key]


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
    """Unequal requests come and go: portions beside single tokens, some left out of a step, pool and
    slots just large enough, so that later requests get what earlier ones held."""
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


def plant_key(weights, places, token, gain):
    """A token whose key meets every query: column 0 of the embedding drives the queries' channel, column
    1 (set for that token alone) the key's.  places: (tensor, first row of a head) of either side."""
    w = {k: v.copy() for k, v in weights.items()}
    w["embed"][:, 0] = 3.0
    w["embed"][:, 1] = 0.0
    w["embed"][token, 1] = 40.0
    for name, row, col in places:
        w[name][row, :] = 0.0
        w[name][row, col] = gain
    return w


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("size,keep", [(37, 5), (32, 16), (48, 17), (16, 1)])
def test_a_standing_out_key_at_every_edge_of_a_window(hb, cuda, tmp_path, size, keep, dtype):
    """The same strong token among the kept ones, first after them, at block edges: it shows wherever a
    window still holds it and nowhere else, in prompts and in decoding, also for a layer that borrows the
    keys and has a window of its own."""
    attn = [windowed(4, 2, 16, 24, 1.0, 8.0, size, keep, (100.0, 8), None),
            windowed(4, 2, 16, 24, 1.0, 8.0, size + 9, keep + 1, (100.0, 8), dense(32), kv_from=0)]
    config = model(64, 40, attn)
    p = "l0.mix."
    places = [(p + "k", g * 16 + 15, 1) for g in range(2)]
    places += [(f"l{i}.mix.q", h * 16 + 15, 0) for i in range(2) for h in range(4)]
    w = plant_key(R.random_weights(config, seed=9), places, 7, 2.5)
    R.write_model(str(tmp_path), config, w)
    eng = load(hb, str(tmp_path), dtype)
    felt = []
    for at in (0, keep - 1, keep, keep + 1, 47, 48, 63):
        toks = np.random.default_rng(at).integers(8, 40, 130)
        toks[at] = 7
        want = R.forward(config, w, toks)
        for sizes in ([130], [50, 2, 3], [70] + [1] * 60):
            seq = eng.create_kv_cache()
            check(feed(eng, seq, toks, sizes), want, dtype, (at, sizes[0]))
            seq.free()
        # the plain form itself feels an edge that is one off
        for layer, change in ((0, dict(size=size + 1, keep_first=keep)), (1, dict(size=size + 9, keep_first=keep + 2))):
            other = json.loads(json.dumps(config))
            other["layers"][layer]["mixer"]["mask"] = change
            felt.append((layer, at, errors(R.forward(other, w, toks), want).max()))
    assert max(e for l, a, e in felt if l == 0 and a > keep + 1) > 4 * LIMIT["bf16"], felt
    assert max(e for l, a, e in felt if l == 1 and a == keep + 1) > 4 * LIMIT["bf16"], felt
    eng.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_a_standing_out_far_key_of_a_latent(hb, cuda, tmp_path, dtype):
    """A single strong key hundreds of positions away, met through the latent."""
    config = model(64, 40, [latent(4, 16, 8, 16, 24, 1.0, 100.0, dense(32), YARN)])
    w = R.random_weights(config, seed=10)
    w["l0.mix.uk"][:, 3] = 0.0
    places = [("l0.mix.dkv", 3, 1)] + [("l0.mix.q", h * 24 + 15, 0) for h in range(4)]
    w = plant_key(w, places, 7, 1.5)
    for h in range(4):
        w["l0.mix.uk"][h * 16 + 15, :] = 0.0
        w["l0.mix.uk"][h * 16 + 15, 3] = 1.0
    R.write_model(str(tmp_path), config, w)
    eng = load(hb, str(tmp_path), dtype)
    for at in (0, 1, 15, 16, 100):
        toks = np.random.default_rng(at).integers(8, 40, 350)
        toks[at] = 7
        want = R.forward(config, w, toks)
        for sizes in ([350], [190, 2, 3], [280] + [1] * 70):
            seq = eng.create_kv_cache()
            check(feed(eng, seq, toks, sizes), want, dtype, (at, sizes[0]))
            seq.free()
    toks[100] = 8
    assert errors(R.forward(config, w, toks), want)[280:].max() > 4 * LIMIT["bf16"]
    eng.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_a_state_remembers_and_starts_empty(hb, cuda, tmp_path, dtype):
    """Slow decays: a strong first token is still felt at the end, whatever the portions; and a sequence
    that takes over a slot feels nothing of the one before it."""
    config = model(64, 40, [mamba(4, 16, 16, 2, 4, 2, dense(32))])
    w = R.random_weights(config, seed=12)
    w["l0.mix.A_log"][:] = -3.0
    w["l0.mix.dt_bias"][:] = -3.0
    w["embed"][7] *= 8.0
    R.write_model(str(tmp_path), config, w)
    eng = load(hb, str(tmp_path), dtype, max_seqs=1)
    toks = np.random.default_rng(1).integers(8, 40, 300)
    toks[0] = 7
    plain = toks.copy()
    plain[0] = 9
    want, without = R.forward(config, w, toks), R.forward(config, w, plain)
    assert errors(without, want)[-60:].max() > 4 * LIMIT["f32"]
    for sizes in ([300], [2], [1] * 300, [128, 1, 3], [7, 65]):
        for t, e in ((toks, want), (plain, without)):
            seq = eng.create_kv_cache()
            check(feed(eng, seq, t, sizes), e, dtype, sizes[0])
            seq.free()
    eng.close()


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
def test_caller_owned_tables_copies_swaps_and_truncation(hb, cuda, tmp_path, dtype):
    """A model without recurrent state: blocks of the latent and of shared keys and values are copied,
    swapped out and in, and a sequence is wound back."""
    config = model(80, 61, [CONFIGS["narrow"]["layers"][0], CONFIGS["narrow"]["layers"][2],
                            windowed(2, 2, 24, 40, 0.3, 4.0, 40, 0, (1e3, 16), dense(40), 4.0, kv_from=0)])
    w = R.steady_routers(config, R.random_weights(config, seed=5))
    R.write_model(str(tmp_path), config, w)
    eng = load(hb, str(tmp_path), dtype, tokens=640)
    rng = np.random.default_rng(21)
    toks = rng.integers(0, 61, 70)
    other = np.concatenate([toks[:40], rng.integers(0, 61, 30)])
    want, want2 = R.forward(config, w, toks), R.forward(config, w, other)
    table = [30, 5, 17, 2, 9]
    check(eng.forward_tables(toks[:40], 0, table)[None], want, dtype, rows=slice(39, 40))
    eng.kv_copy_blocks([(17, 21)])
    table2 = [30, 5, 21, 3, 4]
    check(eng.forward_tables(toks[40:], 40, table)[None], want, dtype, rows=slice(69, 70))
    check(eng.forward_tables(other[40:], 40, table2)[None], want2, dtype, rows=slice(69, 70))
    eng.reserve_cpu_blocks(8)
    eng.kv_swap_blocks([(b, i) for i, b in enumerate(table)], to_cpu=True)
    eng.forward_tables(rng.integers(0, 61, 70), 0, table)
    back = [11, 12, 13, 14, 15]
    eng.kv_swap_blocks([(i, b) for i, b in enumerate(back)], to_cpu=False)
    logits = np.empty((1, 61), dtype=np.float32)
    eng.decode_batch_tables([toks[69]], [69], [back], logits=logits)
    check(logits, want, dtype, rows=slice(69, 70))
    seq = eng.create_kv_cache()
    feed(eng, seq, toks[:61], [61])
    eng.truncate(seq, 40)
    check(feed(eng, seq, other[40:], [7]), want2, dtype, rows=slice(40, None))
    eng.close()


def test_refusals(hb, cuda, models, tmp_path):
    config, w, path = models["narrow"]
    with pytest.raises(hb.HbError, match="f16"):
        hb.Engine.load(path, bf16=False)
    eng = load(hb, path, "bf16")
    with pytest.raises(hb.HbError, match="recurrent state"):
        eng.kv_copy_blocks([(1, 2)])
    eng.close()

    def altered(layer, key="mixer", **change):
        c = json.loads(json.dumps(config))
        c["layers"][layer][key].update(change)
        return c

    cases = [(dict(config, norm={}), "eps"), (dict(config, width=72), "shape"), (dict(config, layers=[]), "no layers"),
             (dict(config, layers=[dict(config["layers"][0], type="other")]), "unknown type"),
             (altered(0, heads=0), "sizes"), (altered(0, kv_heads=3), "sizes"), (altered(0, mask=dict(size=0)), "mask"),
             (altered(0, rot=dict(base=10.0, dims=26)), "rotation"), (altered(0, rot=dict(base=10.0, dims=5)), "rotation"),
             (altered(0, softcap=-1.0), "sizes"), (altered(0, rot=dict(base=10.0, dims=4, scaling=dict(factor=0))), "scaling"),
             (altered(1, groups=3), "sizes"), (altered(1, norm_groups=5), "sizes"), (altered(1, conv=0), "sizes"),
             (altered(1, conv=5), "conv"), (altered(2, kv_rank=0), "sizes"), (altered(2, rot=dict(base=9.0, dims=10)), "rotation"),
             (altered(3, kv_from=1), "no keys"), (altered(3, kv_from=3), "no keys"), (altered(3, kv_heads=3), "no keys"),
             (altered(3, kv_from=None), "l3.mix.k"), (altered(0, "mlp", kind="other"), "unknown kind"),
             (altered(0, "mlp", router=dict(experts=6, top=7)), "experts"),
             (altered(0, "mlp", router=dict(experts=6, top=3, groups=dict(count=3, keep=1))), "groups"),
             (altered(0, "mlp", router=dict(experts=6, top=3, groups=dict(count=4, keep=2))), "groups"),
             (altered(0, "mlp", router=dict(experts=7, top=2)), "l0.mlp.e6")]
    for bad, text in cases:
        R.write_model(str(tmp_path), bad, w)
        with pytest.raises(hb.HbError, match=text):
            load(hb, str(tmp_path), "bf16")
    for missing in ("l0.mix.v", "l1.mix.conv", "l1.mix.in", "l1.mix.D", "l2.mix.uk", "l2.mix.dkv.norm", "l1.mlp.gate.b", "l0.mlp.router",
                    "l3.mlp.down.b", "final.norm"):
        R.write_model(str(tmp_path), config, {k: v for k, v in w.items() if k != missing})
        with pytest.raises(hb.HbError, match=missing):
            load(hb, str(tmp_path), "bf16")


def test_random_engine_and_profile(hb, cuda):
    eng = hb.Engine.create_random_config(CONFIGS["wide"], max_seq_len=128, max_batch=128, max_seqs=4)
    seqs = [eng.create_kv_cache() for _ in range(4)]
    eng.step([(s, np.arange(20) + i, []) for i, s in enumerate(seqs)])
    nxt, ms = eng.profile_step(seqs, np.arange(4))
    assert len(nxt) == 4
    assert min(ms[k] for k in ("routing", "experts_gate_up", "experts_down", "attention", "gemm", "latent", "convolution", "recurrence")) > 0
    assert eng.step_bytes([20] * 4) > 0 and eng.gemm_bytes(4) > 0 and eng.last_step_launches() > 10
    eng.close()
