"""Small Madipel models for the tests: configurations, random weights, checkpoint folders, and a driver over the runtime."""
import json
import os

import numpy as np


def layer(heads, kv, dim, vdim, window, ff, mix=True, scale=None):
    mx = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "v_mix": mix}
    if window:
        mx["mask"] = {"size": window}
    return {"type": "attention", "mixer": mx, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=88, vocab=203, mult=0.63, logit_scale=0.37, eps=1e-5):
    return {"architecture": "Madipel", "layers": layers, "width": width, "vocab": vocab, "residual_mult": mult, "logit_scale": logit_scale,
            "norm": {"eps": eps}}


# every layer another shape: odd head sizes, 1 / 3 / 10 query heads per K/V head, windows of several lengths and none, no feed-forward,
# no value mixing in the first layer, sizes that fill no tile or chunk
MIXED = config([layer(6, 2, 40, 24, 50, 100, mix=False), layer(4, 4, 24, 12, 7, None), layer(10, 1, 64, 48, 130, 72, scale=0.2),
                layer(2, 2, 33, 24, None, 33)])
# sizes on the tensor-core attention path only: wide heads, windows around a tile of keys
WIDE = config([layer(12, 4, 80, 112, 64, 200), layer(4, 4, 128, 112, 65, 96), layer(16, 1, 48, 448, 100, 64, mix=False), layer(8, 4, 176, 112, 63, None)],
              width=272, vocab=331, mult=1.0, logit_scale=1.0)


def bf16(a):
    """Rounded to bfloat16 (round to nearest even), as float32 values."""
    u = np.asarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def weights(cfg, seed, sharp=1.0):
    """Random weights of sensible size, exact in bf16.  ``sharp`` scales the query gains: large values make single keys stand out."""
    rng = np.random.default_rng(seed)
    D = cfg["width"]

    def lin(n, k, g=1.0):
        return rng.standard_normal((n, k)) * g / np.sqrt(k)

    W = {"embed": rng.standard_normal((cfg["vocab"], D)), "final.norm": 1 + 0.2 * rng.standard_normal(D), "final.norm.b": 0.2 * rng.standard_normal(D),
         "head": lin(cfg["vocab"], D, 2.0)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        W.update({p + "norm1": 1 + 0.2 * rng.standard_normal(D), p + "norm1.b": 0.2 * rng.standard_normal(D), p + "mix.q": lin(H * dk, D),
                  p + "mix.k": lin(G * dk, D), p + "mix.v": lin(G * dv, D), p + "mix.o": lin(D, H * dv), p + "mix.temp": rng.uniform(0.5, 1.5, H),
                  p + "mix.q.norm": sharp * (1 + 0.3 * rng.standard_normal(H * dk)), p + "mix.k.norm": 1 + 0.3 * rng.standard_normal(G * dk),
                  p + "mix.r1": rng.uniform(0.05, 1.0, H), p + "mix.r2": rng.uniform(0.05, 0.6, H)})
        if m["v_mix"]:
            W[p + "mix.vmix"] = np.array(rng.uniform(0.2, 0.8))
        if l["mlp"]:
            F = l["mlp"]["ff"]
            W.update({p + "mlp.up": lin(F, D, 1.5), p + "mlp.down": lin(D, F, 0.5), p + "mlp.act": np.array([0.6, -0.4]) + 0.2 * rng.standard_normal(2)})
    return {k: bf16(v).reshape(np.shape(v)) for k, v in W.items()}


def save(pkg, folder, cfg, W):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    bits = {k: ("bf16", (np.ascontiguousarray(v, np.float32).view(np.uint32) >> 16).astype(np.uint16).reshape(np.shape(v))) for k, v in W.items()}
    pkg.safetensors_write(os.path.join(folder, "model.safetensors"), bits)
    return str(folder)


def tokens(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def run(rt, toks, cuts, slot=0, start=0):
    """Logits of every token, taken in portions of the given sizes (the last size repeats)."""
    rt.seq_select(slot)
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        rt.want_logits(range(n))
        rt.set_data(toks[at:at + n])
        rt.execute({"s": n, "p": start + at})
        out.append(rt.get_wanted())
        at, i = at + n, i + 1
    return np.concatenate(out)


def errors(got, want):
    """Per position: root mean square of the difference (mean taken off) over that of the expected logits as a whole."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt(np.mean((want - want.mean(-1, keepdims=True)) ** 2))


TOL = {"float32": 2e-5, "bfloat16": 4e-2}
