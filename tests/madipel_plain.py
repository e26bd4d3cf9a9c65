"""A plain, slow statement of the Madipel design, one function per mechanism: what the GPU tests compare the framework with.

Whole sequences, no cache, no batching, float64 by default; nothing is shared with the package or its kernels.  Weights are a dict of
numpy arrays by tensor name (`l<i>.mix.q`, ...), the configuration is the dict of a config.json.
"""
import numpy as np


def rms_norm(x, gain, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * gain


def layer_norm(x, gain, bias, eps):
    c = x - np.mean(x, axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * gain + bias


def sinusoid(positions, width, dtype=np.float64):
    """Pairs of (sine, cosine) of position * frequency, the frequencies falling geometrically from 1 towards 1 / 10000."""
    e = np.arange(width)
    ang = np.asarray(positions, dtype)[:, None] * np.power(10000.0, -(2.0 * (e // 2)) / width).astype(dtype)
    return np.where(e % 2 == 0, np.sin(ang), np.cos(ang))


def xielu(z, p, q):
    sp, sq = np.log1p(np.exp(p)), np.log1p(np.exp(q))
    neg = np.minimum(z, 0)
    return np.where(z > 0, sp * z * z, (0.5 + sq) * (np.expm1(neg) - neg)) + z / 2


def window_mask(n, size):
    """visible[i, j]: position i sees j when 0 <= i - j < size (size None: every earlier position)."""
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (d >= 0) & (d < (n if size is None else size))


def distance_bias(n, r1, r2):
    """[heads, i, j]: r1_h * ln(1 + r2_h * (i - j)) for j <= i."""
    d = np.maximum(np.arange(n)[:, None] - np.arange(n)[None, :], 0)
    return r1[:, None, None] * np.log1p(r2[:, None, None] * d)


def softmax(s):
    e = np.exp(s - np.max(s, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def mix_values(v, v_first, lam):
    return (1 - lam) * v + lam * v_first


def attention(q, k, v, heads, kv_heads, scale, temp, r1, r2, size):
    """q [n, heads * dim], k [n, kv_heads * dim], v [n, kv_heads * vdim] -> [n, heads * vdim]."""
    n = q.shape[0]
    q = q.reshape(n, heads, -1).transpose(1, 0, 2)
    share = heads // kv_heads
    k = np.repeat(k.reshape(n, kv_heads, -1).transpose(1, 0, 2), share, axis=0)
    v = np.repeat(v.reshape(n, kv_heads, -1).transpose(1, 0, 2), share, axis=0)
    s = (q @ k.transpose(0, 2, 1)) * scale * temp[:, None, None] - distance_bias(n, r1, r2)
    s = np.where(window_mask(n, size)[None], s, -np.inf)
    return (softmax(s) @ v).transpose(1, 0, 2).reshape(n, -1)


def forward(cfg, weights, tokens, dtype=np.float64, layers_out=None, rows=None):
    """Logits [len(rows or tokens), vocab]; layers_out (a list) receives the residual stream after every layer; with `rows` the
    vocabulary product runs for those positions only."""
    W = {k: np.asarray(a, dtype) for k, a in weights.items()}
    eps, width = cfg["norm"]["eps"], cfg["width"]
    x = W["embed"][np.asarray(tokens)] + sinusoid(np.arange(len(tokens)), width, dtype)
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        L, mx, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = layer_norm(x, W[L + "norm1"], W[L + "norm1.b"], eps)
        q = rms_norm(h @ W[L + "mix.q"].T, W[L + "mix.q.norm"], eps)
        k = rms_norm(h @ W[L + "mix.k"].T, W[L + "mix.k.norm"], eps)
        v = h @ W[L + "mix.v"].T
        if mx.get("v_mix"):
            if v_first is None:
                v_first = v
            else:
                v = mix_values(v, v_first, W[L + "mix.vmix"])
        mask = mx.get("mask")
        y = attention(q, k, v, mx["heads"], mx["kv_heads"], mx["scale"], W[L + "mix.temp"], W[L + "mix.r1"], W[L + "mix.r2"],
                      mask["size"] if mask else None) @ W[L + "mix.o"].T
        if mlp:
            p, q2 = W[L + "mlp.act"]
            y = y + xielu(h @ W[L + "mlp.up"].T, p, q2) @ W[L + "mlp.down"].T
        x = x + cfg["residual_mult"] * y
        if layers_out is not None:
            layers_out.append(x)
    out = layer_norm(x if rows is None else x[np.asarray(rows)], W["final.norm"], W["final.norm.b"], eps)
    return (out @ W["head"].T) * cfg["logit_scale"]
