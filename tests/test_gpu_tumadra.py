"""GPU: the mixed layer stack running Tumadra against the plain numpy restatement (_plain_tumadra.py).

float32 models are held to 32-bit rounding, bfloat16 models to what 16-bit matrix products cost.  Mechanisms are
isolated by models that hold nothing else; the schedules (whole prompts, portions, token by token, batches,
sessions reused) are compared with each other and with the plain forward pass.
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import _plain_tumadra as plain
from _tumadra_models import Weights, attn, config, mamba, tokens, weights, with_mlp

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# difference of logits or residual rows over the row's root mean square
TOL = {"float32": 3e-5, "bfloat16": 4e-2}
DTYPES = ("float32", "bfloat16")


@pytest.fixture(scope="module")
def ctx():
    import wayruntime_b200 as wr
    c = wr.Context(0, attn_max_seq=8192)
    yield c
    c.close()


def build(ctx, cfg, w, dtype, max_rows=512):
    from wayruntime_b200 import models
    return models.build(ctx, cfg, Weights(w), dtype, max_rows)


def rel(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    rms = np.sqrt((want * want).mean(axis=-1, keepdims=True))
    return float((np.sqrt(((got - want) ** 2).mean(axis=-1, keepdims=True)) / rms).max())


def run_cuts(model, toks, cuts, max_ctx=1024, kv=None):
    """Logits of every position with the prompt cut into portions; a portion of one token is a decode step."""
    own = kv is None
    kv = kv or model.kv_create(max_ctx)
    pos, out = 0, []
    for n in cuts:
        mode = model.FWD_DECODE if n == 1 else model.FWD_PREFILL
        out.append(model.forward(mode, [kv], [pos], toks[pos:pos + n], logits=True)["logits"])
        pos += n
    assert pos == len(toks)
    if own:
        kv.close()
    return np.concatenate(out)


def cuts_of(n, size):
    return [size] * (n // size) + ([n % size] if n % size else [])


# ---------------------------------------------------------------- mechanisms alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer,width,groups", [
    (attn(), 48, 3), (attn(heads=3, kv_heads=3, dim=10, vdim=7, every=1), 45, 5), (attn(heads=6, kv_heads=1, dim=64, vdim=128), 64, 1),
    (attn(heads=2, kv_heads=1, dim=80, vdim=72), 40, 2), (attn(heads=2, kv_heads=2, dim=96, vdim=192, diff=0.8), 56, 7),
    (attn(heads=4, kv_heads=2, dim=36, vdim=150, coef=0.0), 51, 3), (attn(heads=2, kv_heads=1, dim=8, vdim=300), 32, 32),
    (mamba(), 48, 3), (mamba(inner=37, state=1, dt_rank=1, conv=1), 33, 1), (mamba(inner=130, state=20, dt_rank=11, conv=5), 60, 4),
    (mamba(inner=24, state=140, dt_rank=3, conv=2), 26, 13), (mamba(inner=9, state=64, dt_rank=17, conv=4), 21, 3),
], ids=lambda v: "-".join(str(x) for x in v["mixer"].values() if not isinstance(x, dict)) if isinstance(v, dict) else str(v))
def test_one_mixer(ctx, dtype, layer, width, groups):
    """One mixer without a feed-forward: residual rows after it, prompt wide (77 rows), short (9), token by token."""
    cfg = config([with_mlp(layer, 0)], width=width, groups=groups)
    w = weights(cfg, 5)
    toks = tokens(cfg, 77, 6)
    want = []
    plain.forward(cfg, w, toks, want)
    m = build(ctx, cfg, w, dtype)
    for cuts in ([77], cuts_of(77, 9), [70] + [1] * 7, [1] * 77):
        kv, pos = m.kv_create(128), 0
        for n in cuts:
            tap = np.zeros((1, n, width), np.float32)
            m.set_hidden_tap(tap)
            m.forward(m.FWD_PREFILL if n > 1 else m.FWD_DECODE, [kv], [pos], toks[pos:pos + n], out_from=n)
            assert rel(tap[0], want[0][pos:pos + n]) <= TOL[dtype], (len(cuts), pos)
            pos += n
        m.set_hidden_tap(None)
        kv.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_and_positions(ctx, dtype):
    """A mixer whose output projection is zero leaves the embedding and the position vector, far positions included."""
    cfg = config([with_mlp(mamba(inner=8, state=2, dt_rank=1, conv=1), 0)], width=50, groups=2)
    w = weights(cfg, 1)
    w["l0.mix.o"][:] = 0
    toks = tokens(cfg, 3000, 2)
    want = []
    plain.forward(cfg, w, toks, want)
    m = build(ctx, cfg, w, dtype, max_rows=3000)
    kv = m.kv_create(3000)
    got = m.forward(m.FWD_PREFILL, [kv], [0], toks, hidden=True)["hidden"]
    assert np.abs(got - want[0]).max() <= 2e-6
    kv.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,act", [(56, (0.7, -0.4, 0.3, 0.2)), (1, (1.0, 0.5, 0.25, -1.0)), (333, (0.0, 0.0, 1.0, 0.0)),
                                    (100, (0.0, 1.0, 0.0, 0.5))])
def test_feed_forward(ctx, dtype, ff, act):
    cfg = config([with_mlp(mamba(inner=8, state=2, dt_rank=1, conv=1), ff)], width=52, groups=4)
    w = weights(cfg, 3)
    w["l0.mix.o"][:] = 0
    w["l0.mlp.act"] = np.float32(np.round(np.array(act) * 64) / 64)
    toks = tokens(cfg, 40, 4)
    want = []
    plain.forward(cfg, w, toks, want)
    m = build(ctx, cfg, w, dtype)
    for n in (40, 10, 1):
        kv = m.kv_create(64)
        got = m.forward(m.FWD_PREFILL if n > 1 else m.FWD_DECODE, [kv], [0], toks[:n], hidden=True)["hidden"]
        assert rel(got, want[0][:n]) <= TOL[dtype] / 4
        kv.close()
    m.close()


# ----------------------------------------------------------------- whole models

MODELS = {
    "mixed": config([with_mlp(mamba(), 56), with_mlp(attn(), 72), with_mlp(attn(heads=2, kv_heads=2, dim=12, vdim=20), 0)],
                    loop=(0, 2, 3)),
    "attention-first": config([with_mlp(attn(heads=6, kv_heads=2, dim=20, vdim=28), 31), with_mlp(mamba(conv=4), 0),
                               with_mlp(mamba(inner=50, state=12), 40)], width=70, groups=7, loop=(1, 3, 2)),
    "no-loop": config([with_mlp(attn(heads=2, kv_heads=1, dim=100, vdim=90), 24), with_mlp(mamba(), 24)], width=36, groups=1,
                      vocab=67),
    "loop-of-one": config([with_mlp(mamba(), 24), with_mlp(attn(), 24)], loop=(1, 2, 1)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MODELS)
def test_whole_portions_and_token_by_token(ctx, name, dtype):
    cfg = MODELS[name]
    w = weights(cfg, 11)
    toks = tokens(cfg, 200, 12)
    want = plain.forward(cfg, w, toks)
    m = build(ctx, cfg, w, dtype)
    for cuts in ([200], cuts_of(200, 2), cuts_of(200, 17), cuts_of(200, 64), [3, 61, 2, 63, 1, 65, 5], [130] + [1] * 70):
        got = run_cuts(m, toks, cuts)
        assert rel(got, want) <= TOL[dtype], cuts[:4]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_over_page_borders(ctx, dtype):
    cfg = MODELS["mixed"]
    w = weights(cfg, 21)
    toks = tokens(cfg, 400, 22)
    want = plain.forward(cfg, w, toks)
    m = build(ctx, cfg, w, dtype)
    got = run_cuts(m, toks, [1] * 400)                               # from the first token on
    assert rel(got, want) <= TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [(16, 24), (80, 72)])
def test_one_key_among_hundreds(ctx, dtype, dims):
    """One query-key pair stands far out of the scores: a key that is lost, doubled or shifted by one shows.  The key
    sits at the first token, around page borders and right before the query; it is asked for from a prompt's rows
    and from decoding."""
    kd, vd = dims
    cfg = config([with_mlp(attn(heads=2, kv_heads=1, dim=kd, vdim=vd, scale=1.0, coef=0.1, every=50), 0)], width=48, groups=1)
    w = weights(cfg, 31)
    a, b = 7, 8                                                      # the asking token and the asked-for one
    d = cfg["width"]
    w["embed"] *= 0.25
    w["embed"][a] = 0
    w["embed"][b] = 0
    w["embed"][a, 0], w["embed"][b, 1] = 32.0, 32.0                  # far above the position vector
    for n in ("q", "k"):
        w[f"l0.mix.{n}"] *= 0.0625
        w[f"l0.mix.{n}.b"] *= 0.0625
    w["l0.mix.q"][:, 0] = 1.0
    w["l0.mix.k"][:, 1] = np.where(np.arange(2 * kd) < kd, 1.0, 0.25)      # map 1 much sharper than map 2
    w["l0.mix.o"] *= 32.0                                           # beside a residual row of 32
    w["l0.shift"][:] = 0.0
    w["l0.norm1"][:] = 1.0
    n = 330
    m = build(ctx, cfg, w, dtype)
    base = [t if t not in (a, b) else 20 for t in tokens(cfg, n, 33)]
    for key in (0, 1, 62, 63, 64, 65, 127, 128, 191, 192, 255, 256, 257, n - 2):
        toks = list(base)
        toks[key], toks[-1] = b, a
        want = plain.forward(cfg, w, toks)
        without = plain.forward(cfg, w, toks[:key] + [20] + toks[key + 1:])
        assert rel(without[-1:], want[-1:]) > 10 * TOL["bfloat16"], "the planted key must matter"
        for cuts in ([n], [n - 1, 1], [100, n - 102, 2]):
            got = run_cuts(m, toks, cuts)
            assert rel(got[-1:], want[-1:]) <= TOL[dtype], (key, cuts)
            assert rel(got, want) <= 4 * TOL[dtype], (key, cuts)      # (rows whose two maps nearly cancel)
    m.close()


# ------------------------------------------------------- sessions, batches, state

def test_batch_of_unequal_sessions_equals_each_alone(ctx):
    """Bit for bit: decode rows do not depend on what else is in the step."""
    for dtype in DTYPES:
        for name in ("mixed", "no-loop"):
            cfg = MODELS[name]
            w = weights(cfg, 41)
            m = build(ctx, cfg, w, dtype)
            lens = [1, 3, 64, 65, 130, 18, 250, 7, 33, 100, 63, 2, 129, 5, 90, 40]
            seqs = [tokens(cfg, n + 4, 50 + i) for i, n in enumerate(lens)]
            alone = []
            for n, t in zip(lens, seqs):
                alone.append(run_cuts(m, t, ([n] if n > 1 else [1]) + [1] * 4, max_ctx=300)[-4:])
            kvs = [m.kv_create(300 + 64 * (i % 3)) for i in range(len(lens))]
            for kv, n, t in zip(kvs, lens, seqs):
                m.forward(m.FWD_PREFILL if n > 1 else m.FWD_DECODE, [kv], [0], t[:n], out_from=n)
            for k in range(4):
                got = m.forward(m.FWD_DECODE, kvs, [n + k for n in lens], [t[n + k] for n, t in zip(lens, seqs)],
                                logits=True)["logits"]
                for i in range(len(lens)):
                    assert np.array_equal(got[i], alone[i][k]), (dtype, name, i, k)
            for kv in kvs:
                kv.close()
            m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_used_again(ctx, dtype):
    """A session on pages and state slots that another one filled, and a session that starts over, know nothing of it."""
    cfg = MODELS["attention-first"]
    w = weights(cfg, 61)
    m = build(ctx, cfg, w, dtype)
    t1, t2 = tokens(cfg, 180, 62), tokens(cfg, 75, 63)
    fresh = run_cuts(m, t2, [40, 20] + [1] * 15, max_ctx=256)
    others = [m.kv_create(256) for _ in range(3)]
    for kv in others:
        run_cuts(m, t1, [100, 60] + [1] * 20, kv=kv)
    for kv in (others[1], others[0]):
        kv.close()
    assert np.array_equal(run_cuts(m, t2, [40, 20] + [1] * 15, max_ctx=256), fresh)          # their pages, new owner
    assert np.array_equal(run_cuts(m, t2, [40, 20] + [1] * 15, kv=others[2]), fresh)         # the same session from 0 again
    others[2].close()
    assert rel(fresh, plain.forward(cfg, w, t2)) <= TOL[dtype]
    m.close()


def test_a_step_can_be_taken_again_and_a_wrong_position_is_refused(ctx):
    import wayruntime_b200 as wr
    cfg = MODELS["mixed"]
    w = weights(cfg, 71)
    m = build(ctx, cfg, w, "float32")
    toks = tokens(cfg, 60, 72)
    want = run_cuts(m, toks, [30, 10, 20])
    kv = m.kv_create(64)
    m.forward(m.FWD_PREFILL, [kv], [0], toks[:30], out_from=30)
    m.forward(m.FWD_PREFILL, [kv], [30], toks[::-1][:25], out_from=25)                       # tokens nobody keeps
    got = m.forward(m.FWD_PREFILL, [kv], [30], toks[30:40], logits=True)["logits"]           # the step again, other tokens
    assert np.array_equal(got, want[30:40])
    for bad in (20, 41, 55):
        with pytest.raises(wr.WrCudaError) as e:
            m.forward(m.FWD_DECODE, [kv], [bad], [1])
        assert e.value.status == -7                                                          # WR_ERR_STATE
    with pytest.raises(wr.WrCudaError) as e:
        m.forward(m.FWD_PREFILL, [kv], [40], toks[:25])
    assert e.value.status == -6                                                              # WR_ERR_CTX_FULL
    with pytest.raises(wr.WrCudaError) as e:
        m.forward(m.FWD_PREFILL, [kv], [40], [cfg["vocab"]] * 2)
    assert e.value.status == -4
    got = m.forward(m.FWD_PREFILL, [kv], [40], toks[40:], logits=True)["logits"]             # refusals consumed nothing
    assert np.array_equal(got, want[40:])
    kv.close()
    m.close()


def test_more_wanted_rows_than_one_pass_finishes(ctx):
    cfg = MODELS["loop-of-one"]
    w = weights(cfg, 81)
    toks = tokens(cfg, 300, 82)
    want = plain.forward(cfg, w, toks)
    for dtype in DTYPES:
        m = build(ctx, cfg, w, dtype)
        kv = m.kv_create(300)
        places = [0, 1, 5, 130, 128, 299, 77] + list(range(140, 290))
        got = m.forward(m.FWD_PREFILL, [kv], [0], toks, logits=places)["logits"]
        assert rel(got, want[places]) <= TOL[dtype]
        kv.close()
        m.close()


# ------------------------------------------------ serving loop, command line, trace

def greedy_plain(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(plain.forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler(ctx):
    from wayruntime_b200.engine import Engine, Request
    cfg = MODELS["mixed"]
    w = weights(cfg, 91)
    m = build(ctx, cfg, w, "float32", max_rows=64)
    prompts = [tokens(cfg, n, 92 + i) for i, n in enumerate((1, 2, 70, 33, 150))]
    want = [greedy_plain(cfg, w, p, 12) for p in prompts]
    for max_sessions, portion in ((16, None), (2, 7)):
        reqs = Engine(m, max_sessions=max_sessions, portion=portion).run([Request(p, 12) for p in prompts])
        assert [r.output for r in reqs] == want
    m.close()


def test_dense_models_come_through_the_same_registry_and_loop(ctx, tmp_path):
    """A Qwen3-class folder: registry, serving loop, and the layer stack called directly give the same ids."""
    from wayruntime_b200 import checkpoint, models
    from wayruntime_b200.engine import Engine, Request
    hid, ffn, nq, nkv, hd, vocab = 64, 96, 4, 2, 128, 101
    rng = np.random.default_rng(5)
    t = {"model.embed_tokens.weight": (vocab, hid), "model.norm.weight": (hid,)}
    for i in range(2):
        p = f"model.layers.{i}."
        t.update({p + "input_layernorm.weight": (hid,), p + "post_attention_layernorm.weight": (hid,),
                  p + "self_attn.q_proj.weight": (nq * hd, hid), p + "self_attn.k_proj.weight": (nkv * hd, hid),
                  p + "self_attn.v_proj.weight": (nkv * hd, hid), p + "self_attn.o_proj.weight": (hid, nq * hd),
                  p + "self_attn.q_norm.weight": (hd,), p + "self_attn.k_norm.weight": (hd,),
                  p + "mlp.gate_proj.weight": (ffn, hid), p + "mlp.up_proj.weight": (ffn, hid), p + "mlp.down_proj.weight": (hid, ffn)})
    w = {k: (1 + 0.1 * rng.standard_normal(s) if len(s) == 1 else rng.standard_normal(s) / np.sqrt(s[1])).astype(np.float32)
         for k, s in t.items()}
    cfg = {"architectures": ["Qwen3ForCausalLM"], "hidden_size": hid, "intermediate_size": ffn, "num_attention_heads": nq,
           "num_key_value_heads": nkv, "head_dim": hd, "num_hidden_layers": 2, "vocab_size": vocab, "tie_word_embeddings": True,
           "rope_theta": 10000.0, "rms_norm_eps": 1e-6}
    checkpoint.save(str(tmp_path), cfg, w)
    with pytest.raises(models.UnsupportedDtype):
        models.load(ctx, str(tmp_path), "bfloat16")
    m = models.load(ctx, str(tmp_path), "float32", max_rows=32)
    prompt = [3, 77, 15, 9, 60]
    kv, ids = ctx.kv_create(2, nkv, hd, 64), []
    nxt = int(m.forward(m.FWD_PREFILL, [kv], [0], prompt, out_from=4, argmax=True)["argmax"][0])
    for k in range(6):
        ids.append(nxt)
        nxt = int(m.forward(m.FWD_DECODE, [kv], [5 + k], [nxt], argmax=True)["argmax"][0])
    kv.close()
    got = Engine(m).run([Request(prompt, 6), Request(prompt[:2], 6)])
    assert got[0].output == ids
    m.close()


def test_command_line_and_trace_replay(tmp_path):
    """Both programs on a saved folder, in processes of their own."""
    from wayruntime_b200 import checkpoint
    cfg = MODELS["mixed"]
    w = weights(cfg, 101)
    folder = str(tmp_path / "model")
    checkpoint.save(folder, cfg, {k: checkpoint.f32_to_bf16(v) for k, v in w.items()})
    prompt = tokens(cfg, 20, 102)
    out = subprocess.run([sys.executable, "-m", "wayruntime_b200.cli", "generate", "--model", folder, "--dtype", "float32",
                          "--prompt", ",".join(map(str, prompt)), "--prompt", "5", "--max-new", "6"],
                         cwd=ROOT, stdout=subprocess.PIPE, text=True, timeout=300, check=True).stdout
    lines = [json.loads(x) for x in out.splitlines()]
    assert lines[0]["output"] == greedy_plain(cfg, w, prompt, 6) and lines[1]["output"] == greedy_plain(cfg, w, [5], 6)

    a, b = tokens(cfg, 90, 103), tokens(cfg, 41, 104)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [49, 0, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[50:51], "want": []}, {"id": "b", "tokens": b[:2], "want": [1]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[2:], "want": [3, 38]}, {"id": "a", "tokens": a[51:52], "want": [0]}],
              "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[52:], "want": [37]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "c", "tokens": b[:1], "want": [0]}], "end": ["c"]}]
    want_a, want_b = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    want = {0: want_a[[49, 0, 7]], 2: np.concatenate([want_b[[5, 40]], want_a[[51]]]), 3: want_a[[89]], 4: want_b[[0]], 1: want_b[[1]]}
    for dtype in DTYPES:
        dst = tmp_path / dtype
        dst.mkdir()
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(dst),
                            "--max-tokens", "160"], input="\n".join(json.dumps(s) for s in steps) + "\n", cwd=ROOT,
                           stdout=subprocess.PIPE, text=True, timeout=300, check=True)
        assert p.stdout.split("\n")[:5] == [f"done {i}" for i in range(5)]
        for i, rows in want.items():
            got = np.fromfile(dst / f"{i}.f32", "<f4").reshape(rows.shape)
            assert rel(got, rows) <= TOL[dtype], i
