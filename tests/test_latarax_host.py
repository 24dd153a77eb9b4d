"""Host side, no GPU: the scheduler against a fake engine that keeps books, and the plain model's
mechanisms against second formulations of the same formulas."""
import numpy as np
import pytest

from oracle import latarax_ref as R


class FakeSeq:
    def __init__(self, eng):
        self.eng, self.len = eng, 0

    def free(self):
        self.eng.blocks += -(-self.len // 16)
        self.eng.slots += 1
        self.eng.live.remove(self)


class FakeEngine:
    """Next token = (sum of all fed tokens + their number) mod 50; blocks and slots are counted."""

    max_batch = 24

    def __init__(self, blocks, slots):
        self.blocks, self.slots, self.live, self.steps, self.sums = blocks, slots, [], [], {}

    def num_free_blocks(self):
        return self.blocks

    def num_free_state_slots(self):
        return self.slots

    def create_kv_cache(self):
        s = FakeSeq(self)
        self.live.append(s)
        self.slots -= 1
        assert self.slots >= 0
        return s

    def step(self, entries, logits=True):
        assert entries and len({id(e[0]) for e in entries}) == len(entries)
        assert sum(len(t) for _, t, _ in entries) <= self.max_batch
        out = []
        for seq, toks, want in entries:
            self.blocks -= -(-(seq.len + len(toks)) // 16) - -(-seq.len // 16)
            assert self.blocks >= 0
            seq.len += len(toks)
            self.sums[id(seq)] = self.sums.get(id(seq), 0) + sum(toks) if seq.len > len(toks) else sum(toks)
            if want:
                assert list(want) == [len(toks) - 1]
                out.append((self.sums[id(seq)] + seq.len) % 50)
        self.steps.append([len(t) for _, t, _ in entries])
        return np.asarray(out, dtype=np.uint32), None


def reference(prompt, n, stop=()):
    toks = list(prompt)
    for _ in range(n):
        toks.append((sum(toks) + len(toks)) % 50)
        if toks[-1] in stop:
            break
    return toks[len(prompt):]


def test_scheduler_batches_and_gives_back(hb):
    from vllm_hb_b200 import serve

    rng = np.random.default_rng(0)
    eng = FakeEngine(blocks=20, slots=3)
    sched = serve.Scheduler(eng, max_live=8, step_tokens=100)
    reqs = {}
    for i, n in enumerate([5, 60, 1, 33, 16, 100, 2]):
        reqs[str(i)] = (rng.integers(0, 50, n).tolist(), int(rng.integers(1, 12)))
        sched.submit(serve.Request(str(i), list(reqs[str(i)][0]), reqs[str(i)][1]))
    done = sched.run()
    for k, (p, n) in reqs.items():
        assert done[k] == reference(p, n), k
    assert eng.blocks == 20 and eng.slots == 3 and not eng.live and sched.reserved == 0
    assert any(1 in s and max(s) > 1 for s in eng.steps)  # portions ran beside single tokens
    assert sched.step_tokens == 24 and sched.max_live == 3


def test_scheduler_stops_and_refuses(hb):
    from vllm_hb_b200 import serve

    eng = FakeEngine(blocks=4, slots=2)
    sched = serve.Scheduler(eng)
    with pytest.raises(ValueError):
        sched.submit(serve.Request("a", [], 3))
    with pytest.raises(ValueError, match="blocks"):
        sched.submit(serve.Request("a", [1] * 60, 10))
    want = reference([3, 4], 30)
    sched.submit(serve.Request("a", [3, 4], 30, stop_ids=(want[4],)))
    assert sched.run()["a"] == want[:want.index(want[4]) + 1]


def test_window_mask_by_hand():
    for size, keep in ((None, 0), (1, 0), (4, 0), (4, 2), (3, 9)):
        m = R.window_mask(12, size, keep)
        for i in range(12):
            for j in range(12):
                want = j <= i and (size is None or i - j < size or j < keep)
                assert m[i, j] == want


def test_recurrence_closed_form():
    """o_t = sum_j (prod of the decays after j . k_j . q_t) v_j, written as one masked product."""
    rng = np.random.default_rng(1)
    n, H, D, V = 9, 2, 4, 5
    q, k, v = rng.standard_normal((n, H, D)), rng.standard_normal((n, H, D)), rng.standard_normal((n, H, V))
    a = rng.uniform(0.2, 1.0, (n, H, D))
    o, s = R.decayed_recurrence(q, k, v, a)
    b = np.cumsum(np.log(a), axis=0)
    w = np.einsum("thd,jhd,tjhd->htj", q, k, np.exp(np.minimum(b[:, None] - b[None], 0.0)))
    w = np.where(np.tril(np.ones((n, n), bool)), w, 0.0)
    assert np.allclose(o, np.einsum("htj,jhv->thv", w, v))
    assert np.allclose(s, np.einsum("jhd,jhv->hdv", k * np.exp(b[-1] - b), v))
    o2, s2 = R.decayed_recurrence(q[5:], k[5:], v[5:], a[5:], R.decayed_recurrence(q[:5], k[:5], v[:5], a[:5])[1])
    assert np.allclose(o2, o[5:]) and np.allclose(s2, s)


def test_attention_and_model_against_torch():
    import torch

    rng = np.random.default_rng(2)
    n, H, G, D, V = 11, 4, 2, 6, 5
    q, k, v = rng.standard_normal((n, H, D)), rng.standard_normal((n, G, D)), rng.standard_normal((n, G, V))
    mask = R.window_mask(n, 4, 2)
    t = lambda x: torch.from_numpy(x).transpose(0, 1)
    want = torch.nn.functional.scaled_dot_product_attention(
        t(q), t(k).repeat_interleave(2, 0), t(v).repeat_interleave(2, 0), attn_mask=torch.from_numpy(mask), scale=0.3)
    assert np.allclose(R.attention(q, k, v, 0.3, mask), want.transpose(0, 1).numpy())
    # one stream with an identity mix is the plain residual
    config = {"width": 8, "vocab": 7, "streams": 1, "max_positions": 16, "norm": {"eps": 1e-5},
              "layers": [{"type": "gla", "mixer": dict(heads=1, dim=4, vdim=4, tau=2.0), "mlp": {"kind": "dense", "ff": 6}}]}
    w = R.random_weights(config, seed=3, rank=2)
    for hc in ("hc1", "hc2"):
        for leaf, val in (("in", [1.0]), ("out", [1.0]), ("mix", [[1.0]])):
            w[f"l0.{hc}.{leaf}"] = np.asarray(val)
    toks = [1, 2, 3, 3]
    x = w["embed"][toks] + w["pos"][:4]
    sub = lambda p: R.sub(w, p)
    x = x + R.gla_mixer(R.rms_norm_around_zero(x, w["l0.norm1"], 1e-5), sub("l0.mix."), config["layers"][0]["mixer"], 1e-5)
    h = R.rms_norm_around_zero(x, w["l0.norm2"], 1e-5)
    x = x + R.gated_ffn(h, w["l0.mlp.gate"], w["l0.mlp.up"], w["l0.mlp.down"])
    want = R.rms_norm_around_zero(x, w["final.norm"], 1e-5) @ w["head"].T
    assert np.allclose(R.forward(config, w, toks), want)
