"""Small Nurosun configurations with random weights for the tests (weights are exact in bfloat16)."""
import numpy as np

from _tumadra_models import Weights, tokens  # noqa: F401
from wayruntime_b200.checkpoint import bf16_to_f32, f32_to_bf16


def latent(heads=3, dim=20, rot=8, vdim=24, q_rank=18, kv_rank=40, base=10000.0, scale=0.2, source=None, mlp=None):
    mx = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
          "rot": {"base": base, "dims": rot}}
    if source is not None:
        mx["kv_from"] = source
    return {"type": "latent_attention", "mixer": mx, "mlp": mlp}


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(layers, width=48, vocab=131, eps=1e-5, scale=3.0, mult=0.7):
    return {"architecture": "Nurosun", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "residual_mult": mult}


SIGNS = 3


def clear_router(rng, experts, top, signs):
    """Router weights and biases under which, of several draws, the last chosen and the first left out expert lie furthest
    apart in the worst sign pattern."""
    patterns = np.array(np.meshgrid(*[[-1.0, 1.0]] * signs)).reshape(signs, -1)
    best = (-1.0, None, None)
    for _ in range(1500):
        r, b = rng.standard_normal((experts, signs)), 0.5 * rng.standard_normal(experts)
        if top == experts:
            return r, b
        z = np.sort(r @ patterns + b[:, None], axis=0)[::-1]
        gap = (z[top - 1] - z[top]).min()
        if gap > best[0]:
            best = (gap, r, b)
    return best[1:]


def weights(cfg, seed):
    """float32 arrays under the checkpoint's names; every value survives a round trip through bfloat16."""
    rng = np.random.default_rng(seed)
    d, w = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        w[name] = rng.standard_normal((n, k)) * (gain / np.sqrt(k))

    def near_one(name, n):
        w[name] = 1.0 + 0.2 * rng.standard_normal(n)

    w["embed"] = rng.standard_normal((cfg["vocab"], d)) / 3
    # routers look at the first columns alone, which hold a sign pattern per token that no layer changes: choices do not
    # hang on rounding
    signs = min(SIGNS, d)
    w["embed"][:, :signs] = rng.choice([-1.0, 1.0], (cfg["vocab"], signs))
    mat("head", cfg["vocab"], d)
    near_one("final.norm", d)
    for i, lay in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", lay["mixer"], lay["mlp"]
        near_one(p + "norm1", d)
        H, rank = m["heads"], m["kv_rank"]
        mat(p + "mix.dq", m["q_rank"], d)
        near_one(p + "mix.dq.norm", m["q_rank"])
        mat(p + "mix.uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.5)
        if "kv_from" not in m:
            mat(p + "mix.dkv", rank + m["rot_dim"], d)
            near_one(p + "mix.dkv.norm", rank)
        mat(p + "mix.uk", H * m["dim"], rank)
        mat(p + "mix.uv", H * m["vdim"], rank)
        mat(p + "mix.o", d, H * m["vdim"])
        if mlp and mlp["kind"] == "dense":
            for n, rows, k in (("gate", mlp["ff"], d), ("up", mlp["ff"], d), ("down", d, mlp["ff"])):
                mat(p + "mlp." + n, rows, k)
        elif mlp:
            ff, E = mlp["expert"]["ff"], mlp["router"]["experts"]
            for e in range(E):
                for n, rows, k in (("gate", ff, d), ("up", ff, d), ("down", d, ff)):
                    mat(f"{p}mlp.e{e}.{n}", rows, k, 1.5)
            w[p + "mlp.router"], w[p + "mlp.router.b"] = np.zeros((E, d)), np.zeros(E)
            w[p + "mlp.router"][:, :signs], w[p + "mlp.router.b"][:] = clear_router(rng, E, mlp["router"]["top"], signs)
    for name in w:
        if name.endswith(("mix.o", ".down")):
            w[name][:signs] = 0
        if name.endswith("norm1"):
            w[name][:signs] = 1
    return {k: bf16_to_f32(f32_to_bf16(v.astype(np.float32))) for k, v in w.items()}
