"""Plain float64 numpy restatement of the Nurosun design, one function per mechanism.

Slow on purpose: whole sequences, no cache, no batching, keys and values written out per head.  It shares no code
with the product; the GPU tests compare against it.  A model is (config dict, weights dict of float arrays under
the checkpoint's tensor names).
"""
import numpy as np


def layer_norm(x, w, eps):
    centred = x - x.mean(axis=-1, keepdims=True)
    return centred / np.sqrt((centred ** 2).mean(axis=-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x ** 2).mean(axis=-1, keepdims=True) + eps) * w


def rotate_half(x, pos, base):
    """x [t, ..., dims]: component i and i + dims/2 turn by pos * base^(-2i/dims)."""
    half = x.shape[-1] // 2
    angle = np.asarray(pos, np.float64)[:, None] * base ** (-2.0 * np.arange(half) / x.shape[-1])
    angle = angle.reshape((len(pos),) + (1,) * (x.ndim - 2) + (half,))
    u, v = x[..., :half], x[..., half:]
    return np.concatenate([u * np.cos(angle) - v * np.sin(angle), v * np.cos(angle) + u * np.sin(angle)], axis=-1)


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def causal(scores, first=0):
    t, s = scores.shape[-2:]
    return np.where(np.arange(s)[None, :] <= first + np.arange(t)[:, None], scores, -np.inf)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def latent_rows(h, w, pre, cfg, eps):
    """What a layer's cache holds for every position: the latent, and the key part all heads share (rotated)."""
    both = h @ w[pre + "dkv"].T
    rank = cfg["kv_rank"]
    c = rms_norm(both[:, :rank], w[pre + "dkv.norm"], eps)
    return c, rotate_half(both[:, rank:], np.arange(h.shape[0]), cfg["rot"]["base"])


def queries(h, w, pre, cfg, eps):
    cq = rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps)
    q = (cq @ w[pre + "uq"].T).reshape(h.shape[0], cfg["heads"], cfg["dim"] + cfg["rot_dim"])
    return q[..., :cfg["dim"]], rotate_half(q[..., cfg["dim"]:], np.arange(h.shape[0]), cfg["rot"]["base"])


def latent_attention(h, w, pre, cfg, eps, latent, first=0):
    """Rows from `first` on."""
    t, H, c, kr = h.shape[0], cfg["heads"], *latent
    qn, qr = (q[first:] for q in queries(h, w, pre, cfg, eps))
    k = (c @ w[pre + "uk"].T).reshape(t, H, cfg["dim"])
    v = (c @ w[pre + "uv"].T).reshape(t, H, cfg["vdim"])
    out = np.zeros((t - first, H, cfg["vdim"]))
    for head in range(H):
        scores = (qn[:, head] @ k[:, head].T + qr[:, head] @ kr.T) * cfg["scale"]
        out[:, head] = softmax(causal(scores, first)) @ v[:, head]
    return out.reshape(t - first, -1) @ w[pre + "o"].T


def swiglu(h, gate, up, down):
    g = h @ gate.T
    return (g * sigmoid(g) * (h @ up.T)) @ down.T


def limited_expert(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, w, bias, top):
    """Chosen experts of every row (largest logit first) and their weights."""
    z = h @ w.T + bias
    chosen = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    return chosen, softmax(np.take_along_axis(z, chosen, axis=-1))


def mixture(h, w, pre, cfg):
    chosen, weight = route(h, w[pre + "router"], w[pre + "router.b"], cfg["router"]["top"])
    y = np.zeros_like(h)
    for e in range(cfg["router"]["experts"]):
        rows, slot = np.nonzero(chosen == e)
        if len(rows):
            out = limited_expert(h[rows], *(w[f"{pre}e{e}.{n}"] for n in ("gate", "up", "down")), cfg["expert"]["limit"])
            y[rows] += weight[rows, slot][:, None] * out
    return y


def feed_forward(h, w, pre, cfg):
    if not cfg:
        return 0.0
    if cfg["kind"] == "dense":
        return swiglu(h, w[pre + "gate"], w[pre + "up"], w[pre + "down"])
    return mixture(h, w, pre, cfg)


def forward(cfg, weights, tokens, layers_out=None, last_only=False):
    """Logits [n, vocab] of a whole sequence; layers_out, a list, gets the residual after every layer.  last_only: the
    last layer works on the last row alone (logits [1, vocab])."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    latents = {}
    for i, lay in enumerate(cfg["layers"]):
        pre, mx = f"l{i}.", lay["mixer"]
        h = layer_norm(x, w[pre + "norm1"], eps)
        if mx.get("kv_from") is None:
            latents[i] = latent_rows(h, w, pre + "mix.", mx, eps)
        rows = latents[i if mx.get("kv_from") is None else mx["kv_from"]]
        first = len(tokens) - 1 if last_only and i + 1 == len(cfg["layers"]) else 0
        mixed = latent_attention(h, w, pre + "mix.", mx, eps, rows, first)
        x, h = x[first:], h[first:]
        x = x + cfg["residual_mult"] * (mixed + feed_forward(h, w, pre + "mlp.", lay.get("mlp")))
        if layers_out is not None:
            layers_out.append(x.copy())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T
