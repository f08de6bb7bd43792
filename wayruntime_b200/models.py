"""Model registry: which architecture a config.json names, and how it becomes a device model.

An architecture is a function (ctx, config, weights, dtype, max_rows) -> DeviceModel, registered under the name
its config carries ("architecture", or the first entry of "architectures").  `weights` answers get(name, shape)
and f32(name, shape) as checkpoint.Checkpoint does.
"""
from __future__ import annotations

import numpy as np

from . import binding as B
from .checkpoint import Checkpoint, CheckpointError, read_config

_REGISTRY: dict = {}
DTYPES = {"float32": B.F32, "bfloat16": B.BF16}


class UnsupportedDtype(ValueError):
    """The architecture does not run in this number format."""


def register(*names):
    def add(fn):
        for n in names:
            _REGISTRY[n] = fn
        return fn
    return add


def architectures():
    return sorted(_REGISTRY)


def architecture_of(config: dict) -> str:
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in _REGISTRY:
        raise CheckpointError(f"unknown architecture {name!r}; known: {', '.join(architectures())}")
    return name


def load(ctx, folder: str, dtype: str = "bfloat16", max_rows: int = 2048):
    """The device model of a folder with config.json and safetensors weights."""
    config = read_config(folder)
    return build(ctx, config, Checkpoint(folder), dtype, max_rows)


def build(ctx, config: dict, weights, dtype: str = "bfloat16", max_rows: int = 2048):
    return _REGISTRY[architecture_of(config)](ctx, config, weights, dtype, max_rows)


# ---- Llama / Qwen3-class models on the F32 layer stack (wr_cuda_model_create)

@register("LlamaForCausalLM", "Qwen3ForCausalLM")
def dense_f32(ctx, c, w, dtype, max_rows):
    if dtype != "float32":
        raise UnsupportedDtype("the dense layer stack keeps its weights in float32")
    if c.get("rope_scaling") or c.get("attention_bias") or c.get("use_sliding_window"):
        raise CheckpointError("rope scaling, attention biases and sliding windows are not part of the dense stack")
    hid, nq, vocab, ffn = c["hidden_size"], c["num_attention_heads"], c["vocab_size"], c["intermediate_size"]
    nkv, n = c.get("num_key_value_heads", nq), c["num_hidden_layers"]
    hd = c.get("head_dim") or hid // nq
    t = {"embed": w.f32("model.embed_tokens.weight", (vocab, hid)), "final_norm": w.f32("model.norm.weight", (hid,))}
    t["lm_head"] = t["embed"] if c.get("tie_word_embeddings") else w.f32("lm_head.weight", (vocab, hid))
    for i in range(n):
        p = f"model.layers.{i}."
        for ours, theirs, shape in (("attn_norm", "input_layernorm", (hid,)), ("wq", "self_attn.q_proj", (nq * hd, hid)),
                                    ("wk", "self_attn.k_proj", (nkv * hd, hid)), ("wv", "self_attn.v_proj", (nkv * hd, hid)),
                                    ("wo", "self_attn.o_proj", (hid, nq * hd)), ("ffn_norm", "post_attention_layernorm", (hid,)),
                                    ("w_gate", "mlp.gate_proj", (ffn, hid)), ("w_up", "mlp.up_proj", (ffn, hid)),
                                    ("w_down", "mlp.down_proj", (hid, ffn)), ("q_norm", "self_attn.q_norm", (hd,)),
                                    ("k_norm", "self_attn.k_norm", (hd,))):
            name = f"{p}{theirs}.weight"
            if ours in ("q_norm", "k_norm") and name not in w:
                continue
            t[f"l{i}.{ours}"] = w.f32(name, shape)
    return B.DeviceModel(ctx, t, n_layers=n, hidden=hid, n_q_heads=nq, n_kv_heads=nkv, head_dim=hd, vocab=vocab, ffn=ffn,
                         rms_eps=c.get("rms_norm_eps", 1e-6), rope_theta=c.get("rope_theta", 10000.0), max_rows=max_rows)


# ---- Tumadra on the mixed layer stack (wr_cuda_model_create_mixed)

SINUSOIDAL_BASE = 10000.0


def _integer(v, what):
    if int(v) != v:
        raise CheckpointError(f"{what} must be a whole number, got {v}")
    return int(v)


def layer_runs(n_layers: int, loop) -> list[int]:
    """Layer indices in the order they are applied: loop = {start, stop, times} repeats layers start .. stop-1."""
    if not loop:
        return list(range(n_layers))
    a, b, k = loop["start"], loop["stop"], loop["times"]
    if not 0 <= a <= b <= n_layers or k < 0:
        raise CheckpointError(f"loop {loop} does not fit {n_layers} layers")
    return list(range(a)) + list(range(a, b)) * k + list(range(b, n_layers))


# tensor fields of a mixed layer -> (name after 'l<i>.', shape from the scalars s and the width)
_COMMON = {"norm1": ("norm1", lambda s, d: (d,)), "shift": ("shift", lambda s, d: (d,))}
_ATTENTION = {
    "wq": ("mix.q", lambda s, d: (s["n_q_heads"] * 2 * s["k_dim"], d)), "bq": ("mix.q.b", lambda s, d: (s["n_q_heads"] * 2 * s["k_dim"],)),
    "wk": ("mix.k", lambda s, d: (s["n_kv_heads"] * 2 * s["k_dim"], d)), "bk": ("mix.k.b", lambda s, d: (s["n_kv_heads"] * 2 * s["k_dim"],)),
    "wv": ("mix.v", lambda s, d: (s["n_kv_heads"] * s["v_dim"], d)), "bv": ("mix.v.b", lambda s, d: (s["n_kv_heads"] * s["v_dim"],)),
    "w_gate": ("mix.g", lambda s, d: (s["n_q_heads"] * s["v_dim"], d)), "wo": ("mix.o", lambda s, d: (d, s["n_q_heads"] * s["v_dim"])),
    "lq1": ("mix.lq1", lambda s, d: (s["k_dim"],)), "lk1": ("mix.lk1", lambda s, d: (s["k_dim"],)),
    "lq2": ("mix.lq2", lambda s, d: (s["k_dim"],)), "lk2": ("mix.lk2", lambda s, d: (s["k_dim"],)),
}
_MAMBA1 = {
    "w_in": ("mix.in", lambda s, d: (2 * s["inner"], d)), "conv": ("mix.conv", lambda s, d: (s["inner"], s["taps"])),
    "conv_b": ("mix.conv.b", lambda s, d: (s["inner"],)), "w_x": ("mix.x", lambda s, d: (s["dt_rank"] + 2 * s["state"], s["inner"])),
    "w_dt": ("mix.dt", lambda s, d: (s["inner"], s["dt_rank"])), "dt_b": ("mix.dt.b", lambda s, d: (s["inner"],)),
    "a_log": ("mix.A_log", lambda s, d: (s["inner"], s["state"])), "d": ("mix.D", lambda s, d: (s["inner"],)),
    "w_out": ("mix.o", lambda s, d: (d, s["inner"])),
}
_POLYNORM = {
    "norm2": ("norm2", lambda s, d: (d,)), "w_up": ("mlp.up", lambda s, d: (s["ffn_dim"], d)),
    "w_down": ("mlp.down", lambda s, d: (d, s["ffn_dim"])), "act": ("mlp.act", lambda s, d: (4,)),
}


@register("Tumadra")
def tumadra(ctx, c, w, dtype, max_rows):
    """Grouped-RMS pre-norm decoder with token shift; per layer differential attention or a selective scan, and a
    PolyNorm feed-forward or none; absolute sinusoidal positions; a span of layers may be looped."""
    width, vocab = c["width"], c["vocab"]
    eps = float(c["norm"]["eps"])
    layers, fields = [], []
    for i, lay in enumerate(c["layers"]):
        mx, f = lay["mixer"], dict(_COMMON)
        if lay["type"] == "attention":
            temp = mx.get("q_temp")
            s = dict(mixer=B.MIXER_ATTENTION, n_q_heads=mx["heads"], n_kv_heads=mx["kv_heads"], n_maps=2, k_dim=mx["dim"],
                     v_dim=mx["vdim"], attn_scale=mx["scale"], diff_init=mx["diff"], diff_eps=eps,
                     q_temp_every=_integer(temp["every"], "q_temp.every") if temp else 0,
                     q_temp_coef=temp["coef"] if temp else 0.0)
            f.update(_ATTENTION)
        elif lay["type"] == "mamba1":
            s = dict(mixer=B.MIXER_MAMBA1, inner=mx["inner"], state=mx["state"], dt_rank=mx["dt_rank"], taps=mx["conv"])
            f.update(_MAMBA1)
        else:
            raise CheckpointError(f"layer {i} has an unknown mixer {lay['type']!r}")
        mlp = lay.get("mlp")
        if mlp:
            if mlp["kind"] != "dense":
                raise CheckpointError(f"layer {i} has an unknown feed-forward {mlp['kind']!r}")
            s.update(ffn=B.FFN_POLYNORM, ffn_dim=mlp["ff"], ffn_eps=eps)
            f.update(_POLYNORM)
        layers.append(s)
        fields.append(f)
    top = {"embed": ("embed", (vocab, width)), "head": ("head", (vocab, width)), "final_norm": ("final.norm", (width,))}

    def tensor(i, field):
        if i is None:
            return w.get(*top[field])
        if field not in fields[i]:
            return None
        name, shape = fields[i][field]
        return w.get(f"l{i}.{name}", shape(layers[i], width))

    return B.MixedModel(ctx, layers, layer_runs(len(layers), c.get("loop")), tensor, compute=DTYPES[dtype], width=width,
                        vocab=vocab, norm_groups=c["norm"]["groups"], norm_eps=eps, position=B.POS_SINUSOIDAL,
                        position_base=SINUSOIDAL_BASE, max_rows=max_rows)


# ---- Nurosun on the mixed layer stack

EXPERT_ALPHA = 1.702
_LATENT = {
    "w_dq": ("mix.dq", lambda s, d: (s["q_rank"], d)), "dq_norm": ("mix.dq.norm", lambda s, d: (s["q_rank"],)),
    "w_uq": ("mix.uq", lambda s, d: (s["n_q_heads"] * (s["k_dim"] + s["rot_dim"]), s["q_rank"])),
    "w_uk": ("mix.uk", lambda s, d: (s["n_q_heads"] * s["k_dim"], s["kv_rank"])),
    "w_uv": ("mix.uv", lambda s, d: (s["n_q_heads"] * s["v_dim"], s["kv_rank"])),
    "wo": ("mix.o", lambda s, d: (d, s["n_q_heads"] * s["v_dim"])),
}
_LATENT_ROWS = {
    "w_dkv": ("mix.dkv", lambda s, d: (s["kv_rank"] + s["rot_dim"], d)), "dkv_norm": ("mix.dkv.norm", lambda s, d: (s["kv_rank"],)),
}
_SWIGLU = {
    "w_gate_up": ("mlp.gate", lambda s, d: (s["ffn_dim"], d)), "w_up": ("mlp.up", lambda s, d: (s["ffn_dim"], d)),
    "w_down": ("mlp.down", lambda s, d: (d, s["ffn_dim"])),
}
_MOE = {
    "router": ("mlp.router", lambda s, d: (s["n_experts"], d)), "router_b": ("mlp.router.b", lambda s, d: (s["n_experts"],)),
}


@register("Nurosun")
def nurosun(ctx, c, w, dtype, max_rows):
    """Layer-norm decoder with parallel sublayers: latent attention with rotary positions, whose rows a later layer
    may borrow, beside a SwiGLU feed-forward, a mixture of limited experts, or nothing."""
    width, vocab = c["width"], c["vocab"]
    eps = float(c["norm"]["eps"])
    layers, fields = [], []
    for i, lay in enumerate(c["layers"]):
        mx, f = lay["mixer"], {"norm1": ("norm1", lambda s, d: (d,)), **_LATENT}
        if lay["type"] != "latent_attention":
            raise CheckpointError(f"layer {i} has an unknown mixer {lay['type']!r}")
        if mx["rot"]["dims"] != mx["rot_dim"]:
            raise CheckpointError(f"layer {i} rotates {mx['rot']['dims']} of {mx['rot_dim']} dimensions")
        s = dict(mixer=B.MIXER_LATENT, parallel=1, n_q_heads=mx["heads"], k_dim=mx["dim"], v_dim=mx["vdim"], rot_dim=mx["rot_dim"],
                 q_rank=mx["q_rank"], kv_rank=mx["kv_rank"], rope_base=mx["rot"]["base"], attn_scale=mx["scale"], latent_eps=eps)
        source = mx.get("kv_from")
        if source is None:
            f.update(_LATENT_ROWS)
        else:
            if not 0 <= source < i or c["layers"][source]["mixer"].get("kv_from") is not None:
                raise CheckpointError(f"layer {i} takes its rows from layer {source}, which has none of its own before it")
            theirs = c["layers"][source]["mixer"]
            if any(theirs[k] != mx[k] for k in ("kv_rank", "rot_dim", "rot")):
                raise CheckpointError(f"the rows of layers {i} and {source} differ")
            s["kv_from"] = source + 1
        mlp = lay.get("mlp")
        if mlp and mlp["kind"] == "dense":
            s.update(ffn=B.FFN_SWIGLU, ffn_dim=mlp["ff"])
            f.update(_SWIGLU)
        elif mlp and mlp["kind"] == "moe":
            s.update(ffn=B.FFN_MOE, ffn_dim=mlp["expert"]["ff"], n_experts=mlp["router"]["experts"], top_k=mlp["router"]["top"],
                     moe_alpha=EXPERT_ALPHA, moe_limit=mlp["expert"]["limit"])
            f.update(_MOE)
        elif mlp:
            raise CheckpointError(f"layer {i} has an unknown feed-forward {mlp['kind']!r}")
        layers.append(s)
        fields.append(f)
    top = {"embed": ("embed", (vocab, width)), "head": ("head", (vocab, width)), "final_norm": ("final.norm", (width,))}

    def tensor(i, field):
        if i is None:
            return w.get(*top[field])
        if field == "experts":
            ff = layers[i]["ffn_dim"]
            return [w.get(f"l{i}.mlp.e{e}.{n}", shape) for e in range(layers[i]["n_experts"])
                    for n, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))]
        if field not in fields[i]:
            return None
        name, shape = fields[i][field]
        return w.get(f"l{i}.{name}", shape(layers[i], width))

    return B.MixedModel(ctx, layers, list(range(len(layers))), tensor, compute=DTYPES[dtype], width=width, vocab=vocab,
                        norm_groups=1, norm_eps=eps, norm=B.NORM_LAYER, embed_scale=c["embedding"]["scale"],
                        residual_mult=c["residual_mult"], max_rows=max_rows)
