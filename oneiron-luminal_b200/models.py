"""Model registry: a config.json's ``architecture`` names the function that turns it into what the runtime loads.

A ``ModelSpec`` is a ``ModelDesc`` plus, for models whose layers differ, one ``LayerDesc`` per layer; sizes and constants all come from
the configuration.  ``B200Runtime.load_pretrained(folder)`` goes through here; the fixed shapes of ``runtime.CONFIGS`` (benchmarks,
tests) need no configuration file.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Union

from .runtime import DTYPE, LayerDesc, ModelDesc, _desc, layer_order


@dataclass
class ModelSpec:
    architecture: str
    desc: ModelDesc
    layers: Optional[List[LayerDesc]]

    def tensor_names(self) -> List[str]:
        """Labels of the tensors a checkpoint of this model must hold (models with per-layer descriptors)."""
        d = self.desc
        if d.block_kind == 2:
            return self._sequential_names()
        top = ["embed", "final.norm", "head"] + (["final.norm.b"] if d.norm_kind == 1 else [])
        out = list(top)
        for i, g in enumerate(self.layers or []):
            names = ["norm1", "mix.q", "mix.k", "mix.v", "mix.o"]
            if d.norm_kind == 1:
                names.append("norm1.b")
            if d.qk_norm:
                names += ["mix.q.norm", "mix.k.norm"]
            if g.v_mix:
                names.append("mix.vmix")
            if d.dist_bias:
                names += ["mix.temp", "mix.r1", "mix.r2"]
            if g.ffn:
                names += ["mlp.up", "mlp.down", "mlp.act"]
            out += [f"l{i}.{n}" for n in names]
        return out

    def _sequential_names(self) -> List[str]:
        out = ["embed", "final.norm", "head"]
        for i, g in enumerate(self.layers or []):
            if g.mixer == 1:
                names = ["mix." + n for n in ("y", "y.b", "x", "x.b", "ra", "ra.b", "ri", "ri.b", "lam", "o")]
                names += ["mix.conv", "mix.conv.b"] if g.conv_taps else []
            else:
                names = ["mix." + n for n in ("q", "k", "v", "o")]
                names += [f"mix.{c}.b" for c in "qkv"] if g.qkv_bias else []
                names += [f"mix.{c}.conv" for c in "qkv"] if g.conv_taps else []
                names += ["mix.q.norm", "mix.k.norm"] if g.head_norm else []
                names += ["mix.lq1", "mix.lk1", "mix.lq2", "mix.lk2"] if g.maps == 2 else []
            names += ["norm1"] + (["norm2", "mlp.gate", "mlp.up", "mlp.down"] if g.ffn else [])
            if self.desc.streams:
                names += [f"hc{q}.{n}" for q in ((1, 2) if g.ffn else (1,)) for n in ("in", "out", "mix")]
            out += [f"l{i}.{n}" for n in names]
        return out

    def weight_elems_per_token(self) -> int:
        """Elements of the linear weights one decode step streams."""
        d, n = self.desc, self.desc.vocab * self.desc.hidden
        if d.block_kind == 2:
            for i in layer_order(d, len(self.layers)):
                g = self.layers[i]
                n += 3 * d.hidden * g.ffn
                if g.mixer == 1:
                    n += 3 * d.hidden * g.rec_width + 2 * g.rec_width * (g.rec_width // g.rec_blocks)
                else:
                    m = max(1, g.maps)
                    n += d.hidden * (m * g.qk_dim * (g.n_q_heads + g.n_kv_heads) + g.n_kv_heads * g.v_dim + g.n_q_heads * g.v_dim)
            return n
        for g in self.layers or []:
            n += d.hidden * (g.n_q_heads * g.qk_dim + g.n_kv_heads * (g.qk_dim + g.v_dim) + g.n_q_heads * g.v_dim + 2 * g.ffn)
        return n


REGISTRY: Dict[str, Callable[..., ModelSpec]] = {}


def register(name: str):
    def deco(fn):
        REGISTRY[name] = fn
        return fn
    return deco


def from_config(config: Union[str, dict], dtype: str = "bfloat16", max_seq: int = 4096, max_batch: int = 1, max_new_tokens: int = 4096,
                kv_page_rows: int = 0, kv_pool_pages: int = 0) -> ModelSpec:
    """``config``: a parsed config.json, its path, or the folder that holds it.  ``dtype``: "bfloat16" (bf16 weights, matrix operands and
    cache) or "float32" (32-bit throughout).  The rest sizes the cache, as in ``lum_model_desc``."""
    if not isinstance(config, dict):
        path = os.path.join(config, "config.json") if os.path.isdir(config) else config
        with open(path) as f:
            config = json.load(f)
    arch = config.get("architecture")
    if arch not in REGISTRY:
        raise ValueError(f"no model is registered for architecture {arch!r} (known: {', '.join(sorted(REGISTRY))})")
    if dtype not in ("bfloat16", "float32"):
        raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
    spec = REGISTRY[arch](config, DTYPE["bf16" if dtype == "bfloat16" else "f32"])
    for k, v in dict(max_seq=max_seq, max_batch=max_batch, max_new_tokens=max_new_tokens, kv_page_rows=kv_page_rows, kv_pool_pages=kv_pool_pages).items():
        setattr(spec.desc, k, v)
    return spec


def _int(d: dict, key: str, where: str) -> int:
    v = d.get(key)
    if not isinstance(v, int) or isinstance(v, bool) or v <= 0:
        raise ValueError(f"{where}: {key} must be a positive integer, not {v!r}")
    return v


@register("Madipel")
def madipel(cfg: dict, dtype: int) -> ModelSpec:
    """Parallel attention + feed-forward blocks: layer norm with bias, projection-wide q / k norms, no rotation (sinusoidal vector at
    the embedding, learned temperature and logarithmic distance bias on the scores), sliding windows, value mixing, xIELU."""
    layers: List[LayerDesc] = []
    for i, layer in enumerate(cfg["layers"]):
        where = f"layers[{i}]"
        if layer.get("type") != "attention":
            raise ValueError(f"{where}: type {layer.get('type')!r} (this design has attention layers)")
        mx, mlp = layer["mixer"], layer.get("mlp")
        if mlp is not None and mlp.get("kind") != "dense":
            raise ValueError(f"{where}: feed-forward kind {mlp.get('kind')!r} (this design has dense ones)")
        heads, kv_heads = _int(mx, "heads", where), _int(mx, "kv_heads", where)
        if heads % kv_heads:
            raise ValueError(f"{where}: {heads} query heads are not a multiple of {kv_heads} K/V heads")
        layers.append(LayerDesc(n_q_heads=heads, n_kv_heads=kv_heads, qk_dim=_int(mx, "dim", where), v_dim=_int(mx, "vdim", where),
                                window=_int(mx["mask"], "size", where + ".mask") if mx.get("mask") else 0,
                                v_mix=1 if mx.get("v_mix") else 0, ffn=_int(mlp, "ff", where) if mlp else 0, scale=float(mx["scale"])))
    if not layers:
        raise ValueError("a model needs at least one layer")
    g = layers[0]
    desc = _desc(n_layers=len(layers), hidden=_int(cfg, "width", "config"), vocab=_int(cfg, "vocab", "config"), n_q_heads=g.n_q_heads,
                 n_kv_heads=g.n_kv_heads, head_dim=g.qk_dim, ffn=g.ffn, rms_eps=float(cfg["norm"]["eps"]), rope_theta=10000.0, qk_norm=2,
                 weight_dtype=dtype, embed_dtype=dtype, kv_dtype=dtype, block_kind=1, norm_kind=1, pos_kind=1, dist_bias=1,
                 residual_mult=float(cfg["residual_mult"]), logit_scale=float(cfg["logit_scale"]))
    return ModelSpec("Madipel", desc, layers)


@register("Redenex")
def redenex(cfg: dict, dtype: int) -> ModelSpec:
    """Sequential sublayers over several residual streams: gated linear recurrences and differential attention in chunks (short
    convolutions, per-head q / k norms, rotation of part of a head), clamped gated feed-forwards, and a loop over some of the layers."""
    layers: List[LayerDesc] = []
    width = _int(cfg, "width", "config")
    for i, layer in enumerate(cfg["layers"]):
        where = f"layers[{i}]"
        mx, mlp = layer["mixer"], layer.get("mlp")
        g = LayerDesc(conv_taps=_int(mx, "conv", where) if mx.get("conv") else 0)
        if layer.get("type") == "rglru":
            g.mixer, g.rec_width, g.rec_blocks = 1, _int(mx, "width", where), _int(mx, "blocks", where)
            if g.rec_width % g.rec_blocks:
                raise ValueError(f"{where}: width {g.rec_width} does not divide into {g.rec_blocks} blocks")
        elif layer.get("type") == "attention":
            g.n_q_heads, g.n_kv_heads = _int(mx, "heads", where), _int(mx, "kv_heads", where)
            if g.n_q_heads % g.n_kv_heads:
                raise ValueError(f"{where}: {g.n_q_heads} query heads are not a multiple of {g.n_kv_heads} K/V heads")
            g.qk_dim, g.v_dim, g.scale = _int(mx, "dim", where), _int(mx, "vdim", where), float(mx["scale"])
            g.maps, g.diff, g.head_norm, g.qkv_bias = 2, float(mx["diff"]), 1, 1
            g.chunk = _int(mx["mask"], "size", where + ".mask") if mx.get("mask") else 0
            if mx.get("rot"):
                g.rot_dims, g.rot_base = _int(mx["rot"], "dims", where + ".rot"), float(mx["rot"]["base"])
                if g.rot_dims % 2 or g.rot_dims > g.qk_dim:
                    raise ValueError(f"{where}: {g.rot_dims} rotated dimensions of {g.qk_dim}")
        else:
            raise ValueError(f"{where}: type {layer.get('type')!r} (this design has attention and rglru layers)")
        if mlp is not None:
            if mlp.get("kind") != "dense":
                raise ValueError(f"{where}: feed-forward kind {mlp.get('kind')!r} (this design has dense ones)")
            g.ffn, g.ffn_kind, g.ffn_limit = _int(mlp, "ff", where), 1, float(mlp["limit"])
        layers.append(g)
    if not layers:
        raise ValueError("a model needs at least one layer")
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    if not (0 <= loop["start"] <= loop["stop"] <= len(layers)) or loop["times"] < 1:
        raise ValueError(f"loop {loop!r} over {len(layers)} layers")
    desc = _desc(n_layers=len(layers), hidden=width, vocab=_int(cfg, "vocab", "config"), rms_eps=float(cfg["norm"]["eps"]), rope_theta=10000.0,
                 weight_dtype=dtype, embed_dtype=dtype, kv_dtype=dtype, block_kind=2, norm_kind=2, residual_mult=1.0, logit_scale=1.0,
                 streams=_int(cfg, "streams", "config"), embed_scale=float(cfg["embedding"]["scale"]),
                 loop_start=loop["start"], loop_stop=loop["stop"], loop_times=loop["times"])
    return ModelSpec("Redenex", desc, layers)
