"""Small Redenex models for the tests: configurations and random weights (checkpoint folders and the driver are madipel_cases')."""
import numpy as np

from madipel_cases import bf16, errors, run, save, tokens  # noqa: F401


def rec(width, blocks, ff=None, conv=4, limit=1.0):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp(ff, limit)}


def att(heads, kv, dim, vdim, size, ff=None, conv=4, diff=0.3, rot=None, base=10000.0, scale=None, limit=1.0):
    mx = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "diff": diff, "scale": dim ** -0.5 if scale is None else scale,
          "rot": {"dims": dim if rot is None else rot, "base": base}}
    if size:
        mx["mask"] = {"size": size}
    return {"type": "attention", "mixer": mx, "mlp": mlp(ff, limit)}


def mlp(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit} if ff else None


def config(layers, width=88, vocab=203, streams=3, loop=None, scale=0.7, eps=1e-5):
    cfg = {"architecture": "Redenex", "layers": layers, "width": width, "vocab": vocab, "streams": streams, "embedding": {"scale": scale}, "norm": {"eps": eps}}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# every layer another shape: blocks of sizes that fill no group of 8, 3 / 1 / 10 query heads per K/V head, chunks of several lengths and
# none, taps 1 .. 5, part of a head rotated, no feed-forward; three passes over the middle
MIXED = config([rec(84, 7, 100, conv=3), att(6, 2, 40, 24, 50, 70, rot=24, limit=0.8), rec(40, 1, None, conv=2), att(4, 4, 24, 12, 7, None, conv=1, diff=0.6),
                att(10, 1, 64, 48, 130, 72, scale=0.2, conv=5, base=500.0), att(2, 2, 34, 20, None, 33, rot=2)], loop=(1, 3, 3))
# sizes on the tensor-core paths: wide heads, chunks around a tile of keys, gates of whole and broken chunks of K
WIDE = config([att(12, 4, 80, 112, 64, 200), rec(288, 3, 96), att(4, 4, 128, 112, 65, 96, rot=64), rec(512, 2, 40), att(16, 1, 48, 208, 100, 64), att(8, 4, 112, 80, 63)],
              width=272, vocab=331, streams=2, loop=(2, 4, 2), scale=1.0)


def weights(cfg, seed, sharp=1.0):
    """Random weights of sensible size, exact in bf16.  ``sharp`` scales the query gains: large values make single keys stand out."""
    rng = np.random.default_rng(seed)
    D, S, normal = cfg["width"], cfg["streams"], rng.standard_normal

    def lin(n, k, g=1.0):
        return normal((n, k)) * g / np.sqrt(k)

    def taps(channels, n):
        w = 0.4 * normal((channels, n))
        w[:, -1] += 1.0
        return w

    W = {"embed": normal((cfg["vocab"], D)), "final.norm": 0.2 * normal(D), "head": lin(cfg["vocab"], D, 2.0)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        x = p + "mix."
        for q in (1, 2) if l["mlp"] else (1,):
            W.update({p + f"norm{q}": 0.2 * normal(D), p + f"hc{q}.in": 1.0 / S + 0.3 * normal(S), p + f"hc{q}.out": 1.0 + 0.3 * normal(S),
                      p + f"hc{q}.mix": np.eye(S) * 0.8 + 0.2 * normal((S, S)) / np.sqrt(S)})
        if l["type"] == "rglru":
            w, b = m["width"], m["blocks"]
            n = w // b
            W.update({x + "y": lin(w, D), x + "y.b": 0.3 * normal(w), x + "x": lin(w, D), x + "x.b": 0.3 * normal(w), x + "conv": taps(w, m["conv"]),
                      x + "conv.b": 0.2 * normal(w), x + "ra": normal((b, n, n)) / np.sqrt(n), x + "ra.b": 0.5 * normal((b, n)),
                      x + "ri": normal((b, n, n)) / np.sqrt(n), x + "ri.b": 0.5 * normal((b, n)), x + "lam": rng.uniform(-8.0, 0.5, w), x + "o": lin(D, w)})
        else:
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for c, n in (("q", H * 2 * dk), ("k", G * 2 * dk), ("v", G * dv)):
                W.update({x + c: lin(n, D), x + c + ".b": 0.3 * normal(n), x + c + ".conv": taps(n, m["conv"])})
            W.update({x + "q.norm": sharp * (1 + 0.3 * normal(dk)), x + "k.norm": 1 + 0.3 * normal(dk), x + "o": lin(D, H * dv)})
            W.update({x + c: 0.5 * normal(dk) / np.sqrt(dk) for c in ("lq1", "lk1", "lq2", "lk2")})
        if l["mlp"]:
            F = l["mlp"]["ff"]
            W.update({p + "mlp.gate": lin(F, D, 1.5), p + "mlp.up": lin(F, D, 1.5), p + "mlp.down": lin(D, F)})
    return {k: bf16(v).reshape(np.shape(v)) for k, v in W.items()}


TOL = {"float32": 2e-5, "bfloat16": 4e-2}
