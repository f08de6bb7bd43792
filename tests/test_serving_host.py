"""Host logic without a device: checkpoint files, the registry's checks, scheduling and sampling over a fake model."""
import json

import numpy as np
import pytest

from wayruntime_b200 import checkpoint, models
from wayruntime_b200.engine import Engine, Request, Sampling, sample


def test_checkpoint_round_trip_and_damaged_files(tmp_path):
    a = np.arange(12, dtype=np.float32).reshape(3, 4)
    b = checkpoint.f32_to_bf16(np.array([1.0, -2.5, 3e38, 1e-40], np.float32))
    checkpoint.save(str(tmp_path), {"x": 1}, {"a": a, "b": b})
    c = checkpoint.Checkpoint(str(tmp_path))
    assert np.array_equal(c.get("a", (3, 4)), a) and np.array_equal(c.get("b"), b)
    assert c.f32("b")[1] == -2.5 and checkpoint.read_config(str(tmp_path)) == {"x": 1}
    with pytest.raises(checkpoint.CheckpointError):
        c.get("a", (4, 3))
    with pytest.raises(checkpoint.CheckpointError):
        c.get("missing")
    path = tmp_path / "model.safetensors"
    blob = path.read_bytes()
    path.write_bytes(blob[:-4])
    with pytest.raises(checkpoint.CheckpointError):
        checkpoint.Checkpoint(str(tmp_path))
    path.write_bytes((10 ** 9).to_bytes(8, "little") + b"{}")
    with pytest.raises(checkpoint.CheckpointError):
        checkpoint.Checkpoint(str(tmp_path))


def test_bf16_rounds_to_nearest_even():
    import torch
    v = np.random.default_rng(0).standard_normal(4096).astype(np.float32) * 10 ** np.linspace(-30, 30, 4096, dtype=np.float32)
    want = torch.from_numpy(v).to(torch.bfloat16).view(torch.int16).numpy().view(np.uint16)
    assert np.array_equal(checkpoint.f32_to_bf16(v), want)


def test_layer_runs():
    assert models.layer_runs(4, None) == [0, 1, 2, 3]
    assert models.layer_runs(5, {"start": 1, "stop": 3, "times": 3}) == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert models.layer_runs(2, {"start": 0, "stop": 2, "times": 1}) == [0, 1]
    with pytest.raises(checkpoint.CheckpointError):
        models.layer_runs(2, {"start": 1, "stop": 3, "times": 2})


def test_unknown_architectures_are_refused():
    with pytest.raises(checkpoint.CheckpointError, match="unknown architecture"):
        models.architecture_of({"architecture": "Nothing"})
    assert models.architecture_of({"architectures": ["Qwen3ForCausalLM"]}) == "Qwen3ForCausalLM"


class FakeModel:
    """Next token = sum of everything the session has seen, modulo the vocabulary."""
    FWD_DECODE, FWD_PREFILL, vocab, max_rows = 0, 1, 97, 8

    def __init__(self):
        self.calls, self.live = [], 0

    def kv_create(self, max_ctx):
        model = self
        model.live += 1

        class KV:
            seen, cap = [], max_ctx

            def close(self):
                model.live -= 1
        kv = KV()
        kv.seen = []
        return kv

    def forward(self, mode, kvs, positions, tokens, out_from=0, *, logits=False, argmax=False):
        self.calls.append((mode, len(tokens)))
        rows = []
        if mode == self.FWD_PREFILL:
            assert len(kvs) == 1 and positions[0] == len(kvs[0].seen) and len(tokens) <= self.max_rows
            for t in tokens:
                kvs[0].seen.append(t)
                rows.append(sum(kvs[0].seen) % self.vocab)
        else:
            for kv, p, t in zip(kvs, positions, tokens):
                assert p == len(kv.seen) < kv.cap
                kv.seen.append(t)
                rows.append(sum(kv.seen) % self.vocab)
        rows = rows[out_from:]
        res = {"argmax": np.array(rows)} if argmax else {}
        places = range(len(rows)) if logits is True else (logits or [])
        res["logits"] = np.array([np.eye(self.vocab, dtype=np.float32)[rows[i]] for i in places]).reshape(-1, self.vocab)
        return res


def expected(prompt, n, vocab=97):
    toks = list(prompt)
    for _ in range(n):
        toks.append(sum(toks) % vocab)
    return toks[len(prompt):]


def test_scheduler_mixes_portions_and_decode_batches():
    rng = np.random.default_rng(1)
    prompts = [[int(t) for t in rng.integers(0, 97, n)] for n in (1, 3, 30, 8, 9, 17, 2, 25)]
    m = FakeModel()
    reqs = Engine(m, max_sessions=3).run([Request(p, 5 + i) for i, p in enumerate(prompts)])
    for i, (r, p) in enumerate(zip(reqs, prompts)):
        assert r.output == expected(p, 5 + i)
    assert m.live == 0
    assert max(n for mode, n in m.calls if mode == m.FWD_DECODE) > 1      # requests did share decode passes


def test_stop_ids_and_sampled_requests():
    m = FakeModel()
    want = expected([4, 5], 10)
    r = Engine(m).run([Request([4, 5], 10, stop=frozenset([want[3]]))])[0]
    assert r.output == want[:want.index(want[3]) + 1]
    r = Engine(m).run([Request([4, 5], 10, Sampling(temperature=1e-3))])[0]     # all but greedy: one-hot logits / 1e-3
    assert r.output == want


def test_sampling_filters():
    rng = np.random.default_rng(2)
    logits = np.log(np.array([0.5, 0.25, 0.15, 0.1]))
    assert sample(logits, Sampling(), rng) == 0
    draws = [sample(logits, Sampling(temperature=1.0, top_k=2), rng) for _ in range(300)]
    assert set(draws) == {0, 1}
    draws = [sample(logits, Sampling(temperature=1.0, top_p=0.8), rng) for _ in range(500)]
    assert set(draws) == {0, 1, 2}
    draws = np.bincount([sample(logits, Sampling(temperature=1.0), rng) for _ in range(4000)], minlength=4) / 4000
    assert np.abs(draws - [0.5, 0.25, 0.15, 0.1]).max() < 0.04


def test_advance_returns_wanted_places_in_order():
    m = FakeModel()
    e = Engine(m)
    s = e.session(64)
    toks = list(range(1, 21))
    rows = e.advance([s], [toks], [[19, 0, 9]])[0]                        # three passes of at most eight rows
    assert [int(np.argmax(r)) for r in rows] == [sum(toks[:k + 1]) % 97 for k in (19, 0, 9)]
    assert e.advance([s], [[3]], [[]])[0].shape == (0, 97)


def test_plain_forward_has_no_lookahead():
    """The restatement the GPU tests trust: a prefix's logits do not change with what follows."""
    import _plain_tumadra as plain
    from _tumadra_models import attn, config, mamba, tokens, weights, with_mlp
    cfg = config([with_mlp(mamba(), 20), with_mlp(attn(), 0)], loop=(0, 2, 2))
    w = weights(cfg, 1)
    t = tokens(cfg, 30, 2)
    full = plain.forward(cfg, w, t)
    assert np.abs(plain.forward(cfg, w, t[:12]) - full[:12]).max() < 1e-10
    assert json.dumps(cfg)
