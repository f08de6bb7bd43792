"""Small Tumadra configurations with random weights for the tests (weights are exact in bfloat16)."""
import numpy as np

from wayruntime_b200.checkpoint import bf16_to_f32, f32_to_bf16


def attn(heads=4, kv_heads=2, dim=16, vdim=24, coef=0.4, every=7, scale=0.3, diff=0.35):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "diff": diff, "q_temp": {"coef": coef, "every": every}}}


def mamba(inner=40, state=8, dt_rank=6, conv=3):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}


def with_mlp(layer, ff=56):
    return dict(layer, mlp={"kind": "dense", "ff": ff} if ff else None)


def config(layers, width=48, vocab=131, groups=3, eps=1e-5, loop=None):
    c = {"architecture": "Tumadra", "layers": layers, "width": width, "vocab": vocab, "norm": {"groups": groups, "eps": eps}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def weights(cfg, seed):
    """float32 arrays under the checkpoint's names; every value survives a round trip through bfloat16."""
    rng = np.random.default_rng(seed)
    d, w = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        w[name] = rng.standard_normal((n, k)) * (gain / np.sqrt(k))

    def near_one(name, n):
        w[name] = 1.0 + 0.2 * rng.standard_normal(n)

    w["embed"] = rng.standard_normal((cfg["vocab"], d))
    mat("head", cfg["vocab"], d)
    near_one("final.norm", d)
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        near_one(p + "norm1", d)
        w[p + "shift"] = rng.uniform(0.05, 0.9, d)
        if lay["type"] == "attention":
            H, G, kd, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", H * 2 * kd), ("k", G * 2 * kd), ("v", G * vd)):
                mat(p + "mix." + n, rows, d)
                w[p + f"mix.{n}.b"] = 0.3 * rng.standard_normal(rows)
            mat(p + "mix.g", H * vd, d)
            mat(p + "mix.o", d, H * vd)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[p + "mix." + n] = 0.4 * rng.standard_normal(kd) / np.sqrt(kd)
        else:
            e, n, r, k = m["inner"], m["state"], m["dt_rank"], m["conv"]
            mat(p + "mix.in", 2 * e, d)
            w[p + "mix.conv"] = rng.standard_normal((e, k)) / np.sqrt(k)
            w[p + "mix.conv.b"] = 0.2 * rng.standard_normal(e)
            mat(p + "mix.x", r + 2 * n, e, 1.5)
            mat(p + "mix.dt", e, r)
            w[p + "mix.dt.b"] = rng.uniform(-4.0, 0.0, e)
            w[p + "mix.A_log"] = rng.uniform(-2.0, 2.0, (e, n))
            w[p + "mix.D"] = rng.standard_normal(e)
            mat(p + "mix.o", d, e)
        if lay.get("mlp"):
            near_one(p + "norm2", d)
            mat(p + "mlp.up", lay["mlp"]["ff"], d)
            mat(p + "mlp.down", d, lay["mlp"]["ff"])
            w[p + "mlp.act"] = rng.standard_normal(4) * 0.6
    return {k: bf16_to_f32(f32_to_bf16(v.astype(np.float32))) for k, v in w.items()}


def tokens(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


class Weights:
    """Stands for a Checkpoint: BF16 bits under get(), as a file would give them."""

    def __init__(self, w):
        self._w = w

    def __contains__(self, name):
        return name in self._w

    def get(self, name, shape=None):
        a = f32_to_bf16(self._w[name])
        assert shape is None or a.shape == tuple(shape), (name, a.shape, shape)
        return a
