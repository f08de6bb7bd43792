"""Plain float64 numpy restatement of the Tumadra design, one function per mechanism.

Slow on purpose: whole sequences, no cache, no batching, one token after another where the
design is recurrent.  It shares no code with the product; the GPU tests compare against it.
A model is (config dict, weights dict of float arrays under the checkpoint's tensor names).
"""
import numpy as np


def group_rms_norm(x, w, groups, eps):
    """Each of `groups` equal parts of the last axis over its own root mean square, times w."""
    parts = x.reshape(*x.shape[:-1], groups, -1)
    parts = parts / np.sqrt(np.mean(parts * parts, axis=-1, keepdims=True) + eps)
    return parts.reshape(x.shape) * w


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sinusoidal_positions(n, width, first=0):
    p = np.arange(first, first + n, dtype=np.float64)[:, None]
    e = np.arange(width)
    angle = p * 10000.0 ** (-(2.0 * (e // 2)) / width)
    return np.where(e % 2 == 0, np.sin(angle), np.cos(angle))


def token_shift(h, mix):
    """h[t] + (h[t-1] - h[t]) * mix with h[-1] = 0."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mix


def query_temperature(pos, coef, every):
    return 1.0 + coef * np.log(np.floor((pos + 1.0) / every) + 1.0)


def softmax_causal(scores):
    t, s = scores.shape[-2:]
    seen = np.arange(s)[None, :] <= np.arange(t)[:, None]
    scores = np.where(seen, scores, -np.inf)
    e = np.exp(scores - scores.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def diff_lambda(lq1, lk1, lq2, lk2, diff):
    return np.exp(np.sum(lq1 * lk1)) - np.exp(np.sum(lq2 * lk2)) + diff


def diff_combine(a1, a2, lam, diff, eps):
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention(h, w, pre, cfg, eps):
    H, G, dim, vdim = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    t = h.shape[0]
    q = (h @ w[pre + "q"].T + w[pre + "q.b"]).reshape(t, H, 2, dim)
    k = (h @ w[pre + "k"].T + w[pre + "k.b"]).reshape(t, G, 2, dim)
    v = (h @ w[pre + "v"].T + w[pre + "v.b"]).reshape(t, G, vdim)
    temp = query_temperature(np.arange(t), cfg["q_temp"]["coef"], cfg["q_temp"]["every"])
    q = q * temp[:, None, None, None]
    lam = diff_lambda(*(w[pre + n] for n in ("lq1", "lk1", "lq2", "lk2")), cfg["diff"])
    out = np.zeros((t, H, vdim))
    for head in range(H):
        g = head // (H // G)
        a = [softmax_causal(q[:, head, m] @ k[:, g, m].T * cfg["scale"]) @ v[:, g] for m in (0, 1)]
        out[:, head] = diff_combine(a[0], a[1], lam, cfg["diff"], eps)
    y = out.reshape(t, H * vdim) * sigmoid(h @ w[pre + "g"].T)
    return y @ w[pre + "o"].T


def causal_conv(x, w, b):
    """Per channel; the last tap multiplies the current token."""
    taps = w.shape[1]
    xp = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return sum(xp[j:j + x.shape[0]] * w[:, j] for j in range(taps)) + b


def selective_scan(x, dt, A, B, C, D):
    s = np.zeros(A.shape)
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        s = np.exp(dt[t][:, None] * A) * s + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = s @ C[t] + D * x[t]
    return y


def mamba1(h, w, pre, cfg):
    inner, state, rank = cfg["inner"], cfg["state"], cfg["dt_rank"]
    xz = h @ w[pre + "in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w[pre + "conv"], w[pre + "conv.b"]))
    dbc = x @ w[pre + "x"].T
    dt, B, C = dbc[:, :rank], dbc[:, rank:rank + state], dbc[:, rank + state:]
    dt = softplus(dt @ w[pre + "dt"].T + w[pre + "dt.b"])
    y = selective_scan(x, dt, -np.exp(w[pre + "A_log"]), B, C, w[pre + "D"])
    return (y * silu(z)) @ w[pre + "o"].T


def polynorm(z, abce, eps):
    a, b, c, e = abce
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def feed_forward(h, w, pre, eps):
    return polynorm(h @ w[pre + "up"].T, w[pre + "act"], eps) @ w[pre + "down"].T


def layer_runs(cfg):
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b, k = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * k + list(range(b, n))


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [n, vocab] of a whole sequence; layers_out, a list, gets the residual after every layer run."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][np.asarray(tokens)] + sinusoidal_positions(len(tokens), cfg["width"])
    for i in layer_runs(cfg):
        lay, pre = cfg["layers"][i], f"l{i}."
        h = token_shift(group_rms_norm(x, w[pre + "norm1"], groups, eps), w[pre + "shift"])
        if lay["type"] == "attention":
            x = x + attention(h, w, pre + "mix.", lay["mixer"], eps)
        else:
            x = x + mamba1(h, w, pre + "mix.", lay["mixer"])
        if lay.get("mlp"):
            x = x + feed_forward(group_rms_norm(x, w[pre + "norm2"], groups, eps), w, pre + "mlp.", eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return group_rms_norm(x, w["final.norm"], groups, eps) @ w["head"].T
