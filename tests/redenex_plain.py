"""A plain, slow statement of the Redenex design, one function per mechanism: what the tests compare the framework with.

Whole sequences, no cache, no batching, float64 by default; nothing is shared with the package or its kernels.  Weights are a dict of
numpy arrays by tensor name (`l<i>.mix.q`, ...), the configuration is the dict of a config.json.
"""
import numpy as np


def root_mean_square(x, eps):
    return np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def centred_rms_norm(x, w, eps):
    """RMS norm whose stored weight is the gain's distance from one."""
    return x / root_mean_square(x, eps) * (1.0 + w)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def short_conv(u, w):
    """u [n, channels], w [channels, taps]: a weighted sum of each channel's last `taps` values, zeros before the first."""
    n, taps = u.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1]), u.dtype), u])
    return sum(padded[j:j + n] * w[:, j] for j in range(taps))


def block_diagonal(u, w, b):
    """u [n, blocks * size], w [blocks, size, size] (out, in), b [blocks, size]."""
    blocks, size, _ = w.shape
    return np.concatenate([u[:, k * size:(k + 1) * size] @ w[k].T + b[k] for k in range(blocks)], axis=1)


def gated_recurrence(u, r, i, lam):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with ln a_t = -8 r_t softplus(lam), S before the first token zero."""
    log_a = -8.0 * r * softplus(lam)
    a, g = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a))
    out, s = np.empty_like(u), np.zeros_like(u[0])
    for t in range(len(u)):
        s = a[t] * s + g[t] * i[t] * u[t]
        out[t] = s
    return out


def recurrent_block(h, W, p):
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = short_conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"]) + W[p + "conv.b"]
    r = sigmoid(block_diagonal(u, W[p + "ra"], W[p + "ra.b"]))
    i = sigmoid(block_diagonal(u, W[p + "ri"], W[p + "ri.b"]))
    return (gated_recurrence(u, r, i, W[p + "lam"]) * y) @ W[p + "o"].T


def rotate(x, positions, dims, base):
    """x [n, heads, dim]: the first `dims` of each head turn, element k together with element k + dims / 2."""
    half = dims // 2
    f = np.power(float(base), -2.0 * np.arange(half) / dims)
    ang = (np.asarray(positions, np.float64)[:, None] * f)[:, None, :].astype(x.dtype)
    c, s, a, b = np.cos(ang), np.sin(ang), x[..., :half], x[..., half:dims]
    return np.concatenate([a * c - b * s, b * c + a * s, x[..., dims:]], axis=-1)


def chunk_mask(n, size):
    """visible[i, j]: j is not later than i and in the same chunk of `size` positions (None: no chunks)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i // size == j // size) if size else True)


def softmax(s):
    e = np.exp(s - np.max(s, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def difference_weight(lq1, lk1, lq2, lk2, diff):
    return np.exp(np.sum(lq1 * lk1)) - np.exp(np.sum(lq2 * lk2)) + diff


def differential_attention(q, k, v, heads, kv_heads, scale, lam, diff, size, eps):
    """q [n, heads, 2, dim], k [n, kv_heads, 2, dim], v [n, kv_heads, vdim] -> [n, heads * vdim]."""
    n, out = q.shape[0], []
    seen = chunk_mask(n, size)
    for h in range(heads):
        g = h // (heads // kv_heads)
        a = [softmax(np.where(seen, q[:, h, m] @ k[:, g, m].T * scale, -np.inf)) @ v[:, g] for m in (0, 1)]
        o = a[0] - lam * a[1]
        out.append(o / root_mean_square(o, eps) * (1.0 - diff))
    return np.concatenate(out, axis=1)


def attention_block(h, W, p, mx, eps):
    n, H, G, dim, vdim = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (short_conv(h @ W[p + c].T + W[p + c + ".b"], W[p + c + ".conv"]) for c in "qkv")
    q, k = q.reshape(n, H * 2, dim), k.reshape(n, G * 2, dim)
    q = q / root_mean_square(q, eps) * W[p + "q.norm"]
    k = k / root_mean_square(k, eps) * W[p + "k.norm"]
    q = rotate(q, np.arange(n), mx["rot"]["dims"], mx["rot"]["base"])
    k = rotate(k, np.arange(n), mx["rot"]["dims"], mx["rot"]["base"])
    lam = difference_weight(W[p + "lq1"], W[p + "lk1"], W[p + "lq2"], W[p + "lk2"], mx["diff"])
    mask = mx.get("mask")
    o = differential_attention(q.reshape(n, H, 2, dim), k.reshape(n, G, 2, dim), v.reshape(n, G, vdim), H, G, mx["scale"], lam, mx["diff"],
                               mask["size"] if mask else None, eps)
    return o @ W[p + "o"].T


def clamped_gate(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, W, p, limit):
    return clamped_gate(h @ W[p + "gate"].T, h @ W[p + "up"].T, limit) @ W[p + "down"].T


def stream_input(xs, w_in):
    """xs [streams, n, width]."""
    return np.einsum("s,snd->nd", w_in, xs)


def stream_update(xs, mix, out, y):
    """mix [from, to]."""
    return np.einsum("st,snd->tnd", mix, xs) + out[:, None, None] * y[None]


def layer_order(n_layers, loop):
    if not loop:
        return list(range(n_layers))
    inner = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inner * loop["times"] + list(range(loop["stop"], n_layers))


def forward(cfg, weights, tokens, dtype=np.float64, layers_out=None, rows=None):
    """Logits [len(rows or tokens), vocab]; layers_out (a list) receives the sum of the streams after every layer run; with `rows` the
    vocabulary product runs for those positions only."""
    W = {k: np.asarray(a, dtype) for k, a in weights.items()}
    eps = cfg["norm"]["eps"]
    xs = np.repeat((W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"])[None], cfg["streams"], axis=0)
    for i in layer_order(len(cfg["layers"]), cfg.get("loop")):
        layer, L = cfg["layers"][i], f"l{i}."
        h = centred_rms_norm(stream_input(xs, W[L + "hc1.in"]), W[L + "norm1"], eps)
        if layer["type"] == "rglru":
            y = recurrent_block(h, W, L + "mix.")
        else:
            y = attention_block(h, W, L + "mix.", layer["mixer"], eps)
        xs = stream_update(xs, W[L + "hc1.mix"], W[L + "hc1.out"], y)
        if layer.get("mlp"):
            h = centred_rms_norm(stream_input(xs, W[L + "hc2.in"]), W[L + "norm2"], eps)
            xs = stream_update(xs, W[L + "hc2.mix"], W[L + "hc2.out"], feed_forward(h, W, L + "mlp.", layer["mlp"]["limit"]))
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    x = xs.sum(0)
    return centred_rms_norm(x if rows is None else x[np.asarray(rows)], W["final.norm"], eps) @ W["head"].T
