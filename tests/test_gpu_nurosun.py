"""GPU: the mixed layer stack running Nurosun against the plain numpy restatement (_plain_nurosun.py).

float32 models are held to 32-bit rounding, bfloat16 models to what 16-bit matrix products cost.  The schedules (whole
prompts, portions, token by token, batches, sessions used again) are compared with the plain forward pass and, where the
arithmetic is the same, bit for bit with each other.
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import _plain_nurosun as plain
from _nurosun_models import Weights, config, dense, latent, moe, tokens, weights

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


def residuals(model, cfg, toks, cuts, layers):
    """Residual rows after every layer, [layers, tokens, width]."""
    kv, pos, out = model.kv_create(len(toks) + 8), 0, []
    for n in cuts:
        tap = np.zeros((layers, n, cfg["width"]), np.float32)
        model.set_hidden_tap(tap)
        model.forward(model.FWD_PREFILL if n > 1 else model.FWD_DECODE, [kv], [pos], toks[pos:pos + n], out_from=n)
        out.append(tap)
        pos += n
    model.set_hidden_tap(None)
    kv.close()
    return np.concatenate(out, axis=1)


def cuts_of(n, size):
    return [size] * (n // size) + ([n % size] if n % size else [])


def silence(w, i, *names):
    for n in names:
        w[f"l{i}.{n}"][:] = 0


# ---------------------------------------------------------------- mechanisms alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer,width", [
    (latent(), 48), (latent(heads=1, dim=1, rot=2, vdim=1, q_rank=1, kv_rank=1, scale=1.0), 33),
    (latent(heads=5, dim=33, rot=6, vdim=17, q_rank=70, kv_rank=65, base=500.0), 52),
    (latent(heads=2, dim=64, rot=64, vdim=64, q_rank=64, kv_rank=64), 64),
    (latent(heads=4, dim=128, rot=64, vdim=128, q_rank=96, kv_rank=256, scale=0.07), 72),
    (latent(heads=16, dim=16, rot=16, vdim=32, q_rank=48, kv_rank=320, scale=0.15), 40),
    (latent(heads=2, dim=150, rot=34, vdim=200, q_rank=30, kv_rank=130, scale=0.08), 56),
    (latent(heads=20, dim=8, rot=80, vdim=8, q_rank=100, kv_rank=512, scale=0.1), 44),
], ids=lambda v: "-".join(str(x) for x in v["mixer"].values() if not isinstance(x, dict)) if isinstance(v, dict) else str(v))
def test_attention_alone(ctx, dtype, layer, width):
    """One layer without a feed-forward: residual rows after it, prompt wide (150 rows), short (9), token by token."""
    cfg = config([layer], width=width)
    w = weights(cfg, 5)
    toks = tokens(cfg, 150, 6)
    want = []
    plain.forward(cfg, w, toks, want)
    m = build(ctx, cfg, w, dtype)
    for cuts in ([150], cuts_of(150, 9), [20, 123] + [1] * 7, [1] * 150):
        assert rel(residuals(m, cfg, toks, cuts, 1)[0], want[0]) <= TOL[dtype], len(cuts)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", [dense(56), dense(1), dense(333), moe(), moe(1, 1, 8, 4.0), moe(5, 5, 13, 0.3), moe(40, 3, 72, 1.0),
                                 moe(130, 1, 9, 100.0)],
                         ids=lambda v: json.dumps(v).replace(" ", "").replace('"', ""))
def test_feed_forward_alone(ctx, dtype, mlp):
    cfg = config([latent(mlp=mlp)], width=52)
    w = weights(cfg, 3)
    silence(w, 0, "mix.o")
    toks = tokens(cfg, 300, 4)
    want = []
    plain.forward(cfg, w, toks, want)
    m = build(ctx, cfg, w, dtype)
    for n in (300, 40, 16, 10, 1):
        got = residuals(m, cfg, toks[:n], [n], 1)[0]
        assert rel(got, want[0][:n]) <= TOL[dtype] / 2, n
    m.close()


def test_limits_of_the_experts_cut(ctx):
    """Weights so large that most gate and up values lie beyond the limits, on both sides."""
    for dtype in DTYPES:
        cfg = config([latent(mlp=moe(3, 2, 16, 0.75))], width=48)
        w = weights(cfg, 13)
        silence(w, 0, "mix.o")
        for e in range(3):
            w[f"l0.mlp.e{e}.gate"] *= 4
            w[f"l0.mlp.e{e}.up"] *= 4
        toks = tokens(cfg, 60, 14)
        want = []
        plain.forward(cfg, w, toks, want)
        m = build(ctx, cfg, w, dtype)
        for cuts in ([60], cuts_of(60, 6), [1] * 60):
            assert rel(residuals(m, cfg, toks, cuts, 1)[0], want[0]) <= TOL[dtype], cuts[:3]
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_equal_logits_choose_the_lower_expert(ctx, dtype):
    cfg = config([latent(mlp=moe(9, 3, 16, 1.0))], width=48)
    w = weights(cfg, 15)
    silence(w, 0, "mix.o", "mlp.router", "mlp.router.b")
    w["l0.mlp.router.b"][[2, 5, 6, 8]] = 1.0
    toks = tokens(cfg, 30, 16)
    want = []
    plain.forward(cfg, w, toks, want)
    m = build(ctx, cfg, w, dtype)
    for cuts in ([30], [1] * 30):
        assert rel(residuals(m, cfg, toks, cuts, 1)[0], want[0]) <= TOL[dtype] / 2
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,scale,mult,eps", [(48, 1.0, 1.0, 1e-5), (51, 6.5, 0.25, 1e-5), (256, 16.0, 1.5, 1e-2), (640, 0.5, 0.5, 1.0)])
def test_embedding_norm_and_residual_factors(ctx, dtype, width, scale, mult, eps):
    """Constants at and away from 1; rows with a mean away from zero, which the layer norm has to take off."""
    cfg = config([latent(mlp=dense(40)), latent(source=0, mlp=moe())], width=width, scale=scale, mult=mult, eps=eps)
    w = weights(cfg, 17)
    w["embed"] += 0.75
    w["embed"] = np.float32(np.round(w["embed"] * 32) / 32)
    toks = tokens(cfg, 40, 18)
    want = []
    logits = plain.forward(cfg, w, toks, want)
    m = build(ctx, cfg, w, dtype)
    for cuts in ([40], [20, 4] + [1] * 16):
        got = residuals(m, cfg, toks, cuts, 2)
        assert rel(got[0], want[0]) <= TOL[dtype] and rel(got[1], want[1]) <= TOL[dtype]
        assert rel(run_cuts(m, toks, cuts), logits) <= TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", [dense(56), moe(6, 2, 24)], ids=["dense", "experts"])
def test_sublayers_one_after_the_other(ctx, dtype, mlp):
    """The same mechanisms in a stack of another make: root-mean-square norms, the feed-forward with a norm of its own
    behind the attention's residual, layers run twice (a borrowing run reads the latest rows)."""
    from wayruntime_b200 import binding as B
    from wayruntime_b200.models import DTYPES as TYPES
    cfg = config([latent(mlp=mlp), latent(heads=2, source=0, mlp=mlp)], width=48)
    w, runs, eps = weights(cfg, 51), [0, 1, 0, 1], cfg["norm"]["eps"]
    w.update({f"l{i}.norm2": w[f"l{1 - i}.norm1"] for i in (0, 1)})
    toks = tokens(cfg, 70, 52)

    x, want, rows = w["embed"][toks].astype(np.float64) * 1.5, [], None
    d = {k: v.astype(np.float64) for k, v in w.items()}
    for i in runs:
        pre, mx = f"l{i}.", cfg["layers"][i]["mixer"]
        h = plain.rms_norm(x, d[pre + "norm1"], eps)
        rows = plain.latent_rows(h, d, pre + "mix.", mx, eps) if i == 0 else rows
        x = x + 0.8 * plain.latent_attention(h, d, pre + "mix.", mx, eps, rows)
        x = x + 0.8 * plain.feed_forward(plain.rms_norm(x, d[pre + "norm2"], eps), d, pre + "mlp.", mlp)
        want.append(x)

    layers = []
    for lay in cfg["layers"]:
        mx = lay["mixer"]
        s = dict(mixer=B.MIXER_LATENT, n_q_heads=mx["heads"], k_dim=mx["dim"], v_dim=mx["vdim"], rot_dim=mx["rot_dim"], q_rank=mx["q_rank"],
                 kv_rank=mx["kv_rank"], rope_base=mx["rot"]["base"], attn_scale=mx["scale"], latent_eps=eps, kv_from=int("kv_from" in mx))
        if mlp["kind"] == "dense":
            s.update(ffn=B.FFN_SWIGLU, ffn_dim=mlp["ff"])
        else:
            s.update(ffn=B.FFN_MOE, ffn_dim=mlp["expert"]["ff"], n_experts=6, top_k=2, moe_alpha=1.702, moe_limit=mlp["expert"]["limit"])
        layers.append(s)
    names = {"w_dq": "mix.dq", "dq_norm": "mix.dq.norm", "w_uq": "mix.uq", "w_dkv": "mix.dkv", "dkv_norm": "mix.dkv.norm",
             "w_uk": "mix.uk", "w_uv": "mix.uv", "wo": "mix.o", "w_gate_up": "mlp.gate", "w_up": "mlp.up", "w_down": "mlp.down",
             "router": "mlp.router", "router_b": "mlp.router.b", "norm1": "norm1", "norm2": "norm2"}

    def tensor(i, field):
        if i is None:
            return w[field.replace("_", ".")]
        if field == "experts":
            return [w[f"l{i}.mlp.e{e}.{n}"] for e in range(6) for n in ("gate", "up", "down")]
        return w.get(f"l{i}.{names[field]}") if field in names else None

    m = B.MixedModel(ctx, layers, runs, tensor, compute=TYPES[dtype], width=48, vocab=cfg["vocab"], norm_groups=1, norm_eps=eps,
                     embed_scale=1.5, residual_mult=0.8, max_rows=128)
    for cuts in ([70], cuts_of(70, 8), [40] + [1] * 30):
        got = residuals(m, cfg, toks, cuts, len(runs))
        for k in range(len(runs)):
            assert rel(got[k], want[k]) <= TOL[dtype], (k, cuts[:3])
    m.close()


# ----------------------------------------------------------------- whole models

MODELS = {
    "mixed": config([latent(mlp=dense(56)), latent(heads=4, dim=12, vdim=9, source=0, scale=0.3, mlp=moe()), latent(kv_rank=72, rot=16),
                     latent(heads=1, dim=40, vdim=40, q_rank=25, kv_rank=72, rot=16, source=2, mlp=dense(31)),
                     latent(heads=2, source=0, mlp=moe(7, 3, 17))]),
    "experts-first": config([latent(heads=2, mlp=moe(20, 4, 30)), latent(mlp=moe(3, 1, 10)), latent(source=1, mlp=dense(20))], width=70,
                            vocab=67, mult=0.5),
    "wide-heads": config([latent(heads=2, dim=128, rot=64, vdim=128, q_rank=64, kv_rank=192, scale=0.07, mlp=dense(80)),
                          latent(heads=3, dim=64, rot=64, vdim=64, q_rank=40, kv_rank=192, scale=0.1, source=0, mlp=moe(4, 2, 64))],
                         width=128, mult=1.0, scale=1.0),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MODELS)
def test_whole_portions_and_token_by_token(ctx, name, dtype):
    cfg = MODELS[name]
    w = weights(cfg, 11)
    toks = tokens(cfg, 300, 12)
    want = plain.forward(cfg, w, toks)
    m = build(ctx, cfg, w, dtype)
    for cuts in ([300], cuts_of(300, 2), cuts_of(300, 17), cuts_of(300, 64), [3, 61, 2, 63, 1, 65, 5, 100], [130, 100] + [1] * 70):
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


def planted(dims, w, a, b):
    """Token a asks for token b: one score stands far out of the others.  The query and the latent get one number each
    that only these two tokens have."""
    heads, dim, rot = dims[:3]
    w["embed"][:, 3:5] = 0
    w["embed"][[a, b]] = 0
    w["embed"][a, 3], w["embed"][b, 4] = 8.0, 8.0
    w["l0.norm1"][:] = 1
    for n in ("mix.dq", "mix.dkv"):
        w["l0." + n][:, 3:5] = 0
        w["l0." + n][0] = 0
    w["l0.mix.dq"][0, 3], w["l0.mix.dkv"][0, 4] = 8.0, 8.0
    uq, uk = w["l0.mix.uq"].reshape(heads, dim + rot, -1), w["l0.mix.uk"].reshape(heads, dim, -1)
    uq *= 0.25
    uk *= 0.25
    uq[:, 0], uk[:, 0] = 0, 0
    uq[:, 0, 0], uk[:, 0, 0] = 2.0, 2.0
    w["l0.mix.o"][:] *= 4.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [(2, 20, 8, 24, 40), (4, 128, 64, 128, 256), (3, 150, 20, 140, 70)])
def test_one_key_among_hundreds(ctx, dtype, dims):
    """A key that is lost, doubled or shifted by one shows: it sits at the first token, around page and tile borders and
    right before the query, and is asked for from a prompt's rows, from portions and from decoding."""
    heads, dim, rot, vdim, rank = dims
    cfg = config([latent(heads=heads, dim=dim, rot=rot, vdim=vdim, q_rank=24, kv_rank=rank, scale=0.5)], width=48, scale=1.0)
    w = weights(cfg, 31)
    a, b, n = 7, 8, 330
    planted(dims, w, a, b)
    m = build(ctx, cfg, w, dtype)
    base = [t if t not in (a, b) else 20 for t in tokens(cfg, n, 33)]
    for key in (0, 1, 62, 63, 64, 65, 127, 128, 129, 191, 192, 255, 256, 257, n - 3, n - 2):
        toks = list(base)
        toks[key], toks[-1] = b, a
        want = plain.forward(cfg, w, toks)
        without = plain.forward(cfg, w, toks[:key] + [20] + toks[key + 1:])
        assert rel(without[-1:], want[-1:]) > 10 * TOL["bfloat16"], "the planted key must matter"
        for cuts in ([n], [n - 1, 1], [100, n - 102, 2], [n - 17, 17]):
            got = run_cuts(m, toks, cuts)
            assert rel(got[-1:], want[-1:]) <= TOL[dtype], (key, cuts)
            assert rel(got, want) <= 2 * TOL[dtype], (key, cuts)
    m.close()


@pytest.mark.parametrize("dims", [(2, 20, 8, 24, 40), (18, 16, 64, 32, 256)])
def test_one_key_among_thousands(ctx, dims):
    """Long sessions, where a decoding row's keys come in chunks of several tiles: a far-out score in the first or second
    tile of a chunk, at a chunk's first and last key, or in the last chunk."""
    heads, dim, rot, vdim, rank = dims
    cfg = config([latent(heads=heads, dim=dim, rot=rot, vdim=vdim, q_rank=24, kv_rank=rank, scale=0.5)], width=48, scale=1.0)
    w = weights(cfg, 41)
    a, b, n = 7, 8, 2700
    planted(dims, w, a, b)
    base = [t if t not in (a, b) else 20 for t in tokens(cfg, n, 43)]
    models_ = {d: build(ctx, cfg, w, d, max_rows=1024) for d in DTYPES}
    for key in (0, 127, 128, 255, 256, 1500, 2303, 2304, 2500, 2559, 2560, n - 2):
        toks = list(base)
        toks[key], toks[-1] = b, a
        want = plain.forward(cfg, w, toks, last_only=True)
        without = plain.forward(cfg, w, toks[:key] + [20] + toks[key + 1:], last_only=True)
        assert rel(without, want) > 10 * TOL["bfloat16"], "the planted key must matter"
        for dtype, m in models_.items():
            for cuts in ([1000, 1000, 699, 1], [1024, 1024, 652 - 9, 9]):
                kv, pos = m.kv_create(n), 0
                for c in cuts:
                    mode = m.FWD_DECODE if c == 1 else m.FWD_PREFILL
                    got = m.forward(mode, [kv], [pos], toks[pos:pos + c], out_from=c - 1, logits=True)["logits"]
                    pos += c
                kv.close()
                assert pos == n and rel(got, want) <= TOL[dtype], (key, dtype, cuts)
    for m in models_.values():
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_far_out(ctx, dtype):
    """Only the rotated part decides, on positions up to 1500: a frequency or a position that is off turns the scores."""
    cfg = config([latent(heads=2, dim=8, rot=20, vdim=16, q_rank=24, kv_rank=24, base=300.0, scale=0.5)], width=48)
    w = weights(cfg, 35)
    uq = w["l0.mix.uq"].reshape(2, 28, -1)
    uq[:, :8] = 0
    toks = tokens(cfg, 1500, 36)
    want = []
    plain.forward(cfg, w, toks, want)
    m = build(ctx, cfg, w, dtype, max_rows=2048)
    for cuts in ([1500], [1400, 60] + [1] * 40, [700, 790, 10]):
        got = residuals(m, cfg, toks, cuts, 1)[0]
        assert rel(got, want[0]) <= TOL[dtype]
    m.close()


# ------------------------------------------------------- sessions, batches, pages

@pytest.mark.parametrize("name", MODELS)
def test_batch_of_unequal_sessions_equals_each_alone(ctx, name):
    """Bit for bit: decode rows do not depend on what else is in the step."""
    for dtype in DTYPES:
        cfg = MODELS[name]
        w = weights(cfg, 41)
        m = build(ctx, cfg, w, dtype)
        lens = [1, 3, 64, 65, 130, 18, 250, 7, 33, 100, 63, 2, 129, 5, 500, 40]
        seqs = [tokens(cfg, n + 4, 50 + i) for i, n in enumerate(lens)]
        alone = []
        for n, t in zip(lens, seqs):
            alone.append(run_cuts(m, t, ([n] if n > 1 else [1]) + [1] * 4, max_ctx=600)[-4:])
        kvs = [m.kv_create(600 + 64 * (i % 3)) for i in range(len(lens))]
        for kv, n, t in zip(kvs, lens, seqs):
            m.forward(m.FWD_PREFILL if n > 1 else m.FWD_DECODE, [kv], [0], t[:n], out_from=n)
        for k in range(4):
            got = m.forward(m.FWD_DECODE, kvs, [n + k for n in lens], [t[n + k] for n, t in zip(lens, seqs)],
                            logits=True)["logits"]
            for i in range(len(lens)):
                assert np.array_equal(got[i], alone[i][k]), (dtype, i, k)
        for kv in kvs:
            kv.close()
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_used_again(ctx, dtype):
    """A session on pages that others filled (in another order), and one that starts over or steps back, know nothing of it."""
    cfg = MODELS["mixed"]
    w = weights(cfg, 61)
    m = build(ctx, cfg, w, dtype)
    t1, t2 = tokens(cfg, 180, 62), tokens(cfg, 175, 63)
    cuts = [40, 100, 20] + [1] * 15
    fresh = run_cuts(m, t2, cuts, max_ctx=256)
    others = [m.kv_create(256) for _ in range(3)]
    for kv in others:
        run_cuts(m, t1, [100, 60] + [1] * 20, kv=kv)
    for kv in (others[1], others[0]):
        kv.close()
    assert np.array_equal(run_cuts(m, t2, cuts, max_ctx=256), fresh)
    assert np.array_equal(run_cuts(m, t2, cuts, kv=others[2]), fresh)
    others[2].close()
    kv = m.kv_create(256)
    m.forward(m.FWD_PREFILL, [kv], [0], t2[:40], out_from=40)
    m.forward(m.FWD_PREFILL, [kv], [40], t1[:120], out_from=120)          # tokens nobody keeps
    got = m.forward(m.FWD_PREFILL, [kv], [40], t2[40:140], logits=True)["logits"]
    assert np.array_equal(got, fresh[40:140])
    kv.close()
    assert rel(fresh, plain.forward(cfg, w, t2)) <= TOL[dtype]
    m.close()


def test_bad_models_are_refused(ctx):
    from wayruntime_b200.checkpoint import CheckpointError
    ok = config([latent(), latent(source=0)])
    w = weights(ok, 1)
    for layers in ([latent(), latent(), latent(source=2)], [latent(), latent(source=0), latent(source=1)],
                   [latent(), latent(kv_rank=32, source=0)], [latent(), latent(base=5.0, source=0)],
                   [dict(latent(), type="other"), latent()], [latent(mlp={"kind": "other"})]):
        with pytest.raises(CheckpointError):
            build(ctx, config(layers), w, "float32")
    build(ctx, ok, w, "float32").close()


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
    prompts = [tokens(cfg, n, 92 + i) for i, n in enumerate((1, 2, 70, 33, 150))]
    m = build(ctx, cfg, w, "float32", max_rows=64)
    want = [greedy_plain(cfg, w, p, 12) for p in prompts]
    for max_sessions, portion in ((16, None), (2, 7)):
        reqs = Engine(m, max_sessions=max_sessions, portion=portion).run([Request(p, 12) for p in prompts])
        assert [r.output for r in reqs] == want
    m.close()


def test_command_line_and_trace_replay(tmp_path):
    """Both programs on a saved folder, in processes of their own."""
    from wayruntime_b200 import checkpoint
    cfg = MODELS["experts-first"]
    w = weights(cfg, 101)
    folder = str(tmp_path / "model")
    checkpoint.save(folder, cfg, {k: checkpoint.f32_to_bf16(v) for k, v in w.items()})
    prompt = tokens(cfg, 20, 102)
    out = subprocess.run([sys.executable, "-m", "wayruntime_b200.cli", "generate", "--model", folder, "--dtype", "float32",
                          "--prompt", ",".join(map(str, prompt)), "--prompt", "5", "--max-new", "6"],
                         cwd=ROOT, stdout=subprocess.PIPE, text=True, timeout=300, check=True).stdout
    lines = [json.loads(x) for x in out.splitlines()]
    assert lines[0]["output"] == greedy_plain(cfg, w, prompt, 6) and lines[1]["output"] == greedy_plain(cfg, w, [5], 6)
    a = tokens(cfg, 90, 103)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [49, 0, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[50:51], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[51:], "want": [0, 38]}], "end": ["a"]}]
    full = plain.forward(cfg, w, a)
    for dtype in DTYPES:
        dst = tmp_path / dtype
        dst.mkdir()
        subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(dst),
                        "--max-tokens", "160"], input="\n".join(json.dumps(s) for s in steps) + "\n", cwd=ROOT,
                       stdout=subprocess.PIPE, text=True, timeout=300, check=True)
        for i, rows in ((0, full[[49, 0, 7]]), (2, full[[51, 89]])):
            got = np.fromfile(dst / f"{i}.f32", "<f4").reshape(rows.shape)
            assert rel(got, rows) <= TOL[dtype], i
        assert not (dst / "1.f32").exists()
