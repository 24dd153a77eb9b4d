"""hb_step on the Llama family: any mix of portions and tokens equals the per-sequence path, and
the scheduler generates what the oracle generates."""
import numpy as np
import pytest

from oracle import llama_ref as R

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def tiny(tmp_path_factory):
    cfg = R.LlamaTpConfig(hidden_size=256, intermediate_size=320, num_hidden_layers=2, num_attention_heads=4,
                          num_key_value_heads=2, vocab_size=500, rms_norm_eps=1e-5, rope_theta=10000.0)
    w = R.random_weights(cfg, seed=2, std=0.05, norm_ones=True)
    path = tmp_path_factory.mktemp("llama_mixed")
    R.write_model(str(path), cfg, w)
    return cfg, w, str(path)


def test_mixed_step_matches_sequences(hb, cuda, tiny):
    cfg, w, path = tiny
    eng = hb.Engine.load(path, max_seq_len=128, bf16=False, force_f32=True, max_batch=16)
    oracle = R.LlamaTpOracle(cfg, w, world_size=1, dtype="f32")
    rng = np.random.default_rng(0)
    reqs = [rng.integers(0, 500, n).tolist() for n in (40, 9, 21)]
    seqs = [eng.create_kv_cache() for _ in reqs]
    at = [0, 0, 0]
    # 20 + 1 + 5 rows exceed max_batch: the step is cut where it must be, the results are not
    for sizes in ((20, 1, 5), (1, 1, 16), (3, 0, 0), (16, 7, 0)):
        entries, where = [], []
        for i, n in enumerate(sizes):
            if n:
                entries.append((seqs[i], reqs[i][at[i]:at[i] + n], [0, n - 1] if n > 1 else [0]))
                where += [(i, at[i])] + ([(i, at[i] + n - 1)] if n > 1 else [])
                at[i] += n
        nxt, logits = eng.step(entries)
        for (i, p), row, tok in zip(where, logits, nxt):
            want = oracle.forward(reqs[i][:p + 1], 0, oracle.new_cache())
            assert np.max(np.abs(row - want)) <= 1e-3 * np.max(np.abs(want)), (i, p)
            assert tok == np.argmax(row)
    assert at == [40, 9, 21]
    eng.close()


def test_scheduler_greedy(hb, cuda, tiny):
    from vllm_hb_b200 import serve

    cfg, w, path = tiny
    eng = hb.Engine.load(path, max_seq_len=128, bf16=False, force_f32=True, max_batch=24, num_kv_blocks=12)
    oracle = R.LlamaTpOracle(cfg, w, world_size=1, dtype="f32")
    rng = np.random.default_rng(4)
    prompts = [rng.integers(0, 500, n).tolist() for n in (30, 3, 12, 50)]
    got = serve.generate(eng, prompts, 8, max_live=3, step_tokens=20)
    for g, p in zip(got, prompts):
        toks, rows = oracle.greedy_generate(p, 8)
        top = np.sort(np.asarray(rows), axis=1)[:, -2:]
        clear = (top[:, 1] - top[:, 0]) > 2e-3 * np.abs(np.asarray(rows)).max(axis=1)
        n = len(clear) if clear.all() else int(np.argmin(clear))
        assert g[:n] == list(toks)[:n]
    drawn = serve.generate(eng, prompts, 5, temperature=1.0, seed=3)
    assert [len(d) for d in drawn] == [5] * 4 and eng.num_free_blocks() == 12
    eng.close()
