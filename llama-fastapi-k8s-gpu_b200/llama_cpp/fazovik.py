"""Fazovik: a decoder of parallel blocks over latent attention, served by the layer-list graph of the native engine.

A model folder holds `config.json` and `model.safetensors`. Every layer is
    x <- x + (mixer(norm1(x)) + ff(norm2(x)))            (`mlp` may be null)
with layer norms that carry a weight and a bias, both of the same x. The embedding adds a row of the table `bigram`, hashed
from the previous and the current token (`embedding.bigram`); the output map is the embedding table. Token mixers:
  "latent_attention":   queries through a normed latent of their own, keys and values as per-head linear maps of one cached,
                        normed latent per token plus one rotated key part shared by all heads (pairs 2i, 2i+1; frequencies
                        blended for long contexts when `rot.scaling` is given); one sigmoid output gate per head
  "latent_attention_2": the same without rotated part and gate; with `kv_from` a layer reads the latent that an earlier layer
                        caches instead of making its own (it has no `dkv`)
Feed-forward: "dense" (a gated unit with the tanh form of GELU) or "moe" (sigmoid scores, the `top` largest, not
renormalised; a gated SiLU expert whose INPUT is multiplied by its score).

This module turns the config into the C ABI's `b2_layer_desc` list (every size and constant comes from the file) and
checks the tensor set; the arithmetic is in csrc/layered.cu, latent_attn.cu, mixers.cu, moe.cu and dense.cu.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

from . import _cabi
from .goponex import LayeredDims, _need
from .models import Family, register


def _rotation(d: _cabi.B2LayerDesc, m: dict, where: str):
    rot = _need(m, "rot", where)
    d.rot_dims = int(rot.get("dims", d.la_rot_dim))
    d.rope_base = float(_need(rot, "base", where + ".rot"))
    d.rope_factor = 0.0
    sc = rot.get("scaling")
    if sc:
        d.rope_factor, d.rope_orig_ctx = float(sc["factor"]), int(sc["original"])
        d.rope_fast, d.rope_slow = float(sc["fast"]), float(sc["slow"])


def layer_desc(i: int, layer: dict) -> _cabi.B2LayerDesc:
    where = f"layers[{i}]"
    kind = _need(layer, "type", where)
    mix = _need(layer, "mixer", where)
    d = _cabi.B2LayerDesc()
    d.mixer = _cabi.B2_MIX_LATENT_ATTN
    if kind not in ("latent_attention", "latent_attention_2"):
        raise ValueError(f"config.json: {where}: unknown layer type {kind!r}")
    d.n_head, d.head_dim = int(_need(mix, "heads", where)), int(_need(mix, "dim", where))
    d.la_vdim, d.la_rank = int(_need(mix, "vdim", where)), int(_need(mix, "kv_rank", where))
    d.la_q_rank = int(_need(mix, "q_rank", where))
    d.attn_scale = float(_need(mix, "scale", where))
    d.attn_flags = _cabi.B2_ATTN_NO_SINK
    if kind == "latent_attention":
        d.la_rot_dim = int(_need(mix, "rot_dim", where))
        d.attn_flags |= _cabi.B2_ATTN_HEAD_GATE | _cabi.B2_ATTN_ROT_PAIRS
        _rotation(d, mix, where + ".mixer")
        if mix.get("kv_from") is not None:
            raise ValueError(f"config.json: {where}: kv_from belongs to latent_attention_2")
    else:
        d.attn_flags |= _cabi.B2_ATTN_NO_GATE
        if mix.get("kv_from") is not None:
            j = int(mix["kv_from"])
            if not 0 <= j < i:
                raise ValueError(f"config.json: {where}: kv_from {j} is no earlier layer")
            d.kv_from = j + 1
    mlp = layer.get("mlp")
    if mlp:
        fk = _need(mlp, "kind", where + ".mlp")
        if fk == "dense":
            d.ff_kind, d.n_ff, d.ff_act = _cabi.B2_FF_GLU, int(_need(mlp, "ff", where + ".mlp")), _cabi.B2_ACT_GELU_TANH
        elif fk == "moe":
            r, ex = _need(mlp, "router", where + ".mlp"), _need(mlp, "expert", where + ".mlp")
            d.ff_kind, d.n_ff = _cabi.B2_FF_MOE, int(_need(ex, "ff", where + ".mlp.expert"))
            d.moe_experts, d.moe_identity, d.moe_top = int(_need(r, "experts", where)), 0, int(_need(r, "top", where))
            d.moe_groups = d.moe_keep = 1
            d.moe_scale = 1.0
            d.moe_route, d.moe_scale_input, d.moe_expert = _cabi.B2_ROUTE_SIGMOID, 1, _cabi.B2_EXPERT_SILU
        else:
            raise ValueError(f"config.json: {where}: unknown feed-forward kind {fk!r}")
    return d


def _bigram(cfg: dict) -> Optional[dict]:
    return (cfg.get("embedding") or {}).get("bigram")


def read_dims(cfg: dict) -> LayeredDims:
    layers = _need(cfg, "layers", "the config")
    descs = [layer_desc(i, L) for i, L in enumerate(layers)]
    for i, d in enumerate(descs):
        if d.kv_from:
            j = descs[d.kv_from - 1]
            if j.kv_from or j.la_rank != d.la_rank:
                raise ValueError(f"config.json: layers[{i}]: kv_from names a layer without a latent of its own, or of another size")
    bg = _bigram(cfg)
    hashed = (0, 0, 0)
    if bg:
        n = int(_need(bg, "buckets", "embedding.bigram"))
        if n <= 0:
            raise ValueError("config.json: embedding.bigram: buckets must be positive")
        hashed = (n, int(_need(bg, "mul_prev", "embedding.bigram")) % n, int(_need(bg, "mul_cur", "embedding.bigram")) % n)
    return LayeredDims(n_layer=len(descs), n_embd=int(_need(cfg, "width", "the config")), n_vocab=int(_need(cfg, "vocab", "the config")),
                       norm_eps=float(_need(_need(cfg, "norm", "the config"), "eps", "norm")), residual_scale=1.0, layers=descs,
                       block_style=_cabi.B2_BLOCK_PARALLEL_LN, tie_head=True, bigram=hashed)


def tensor_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    """Every tensor the design needs, with its shape ([out, in] for linear maps)."""
    W, V = int(cfg["width"]), int(cfg["vocab"])
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, W), "final.norm": (W,), "final.norm.b": (W,)}
    bg = _bigram(cfg)
    if bg:
        out["bigram"] = (int(bg["buckets"]) + 1, W)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        rotated = L["type"] == "latent_attention"
        H, d, dv, rank, qr = int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["kv_rank"]), int(m["q_rank"])
        dr = int(m["rot_dim"]) if rotated else 0
        out.update({p + "norm1": (W,), p + "norm1.b": (W,), p + "mix.dq": (qr, W), p + "mix.dq.norm": (qr,), p + "mix.uq": (H * (d + dr), qr),
                    p + "mix.uk": (H * d, rank), p + "mix.uv": (H * dv, rank), p + "mix.o": (W, H * dv)})
        if m.get("kv_from") is None:
            out.update({p + "mix.dkv": (rank + dr, W), p + "mix.dkv.norm": (rank,)})
        if rotated:
            out[p + "mix.g"] = (H, W)
        mlp = L.get("mlp")
        if mlp:
            out.update({p + "norm2": (W,), p + "norm2.b": (W,)})
            units = [p + "mlp."]
            F = int((mlp["expert"] if mlp["kind"] == "moe" else mlp)["ff"])
            if mlp["kind"] == "moe":
                E = int(mlp["router"]["experts"])
                out[p + "mlp.router"] = (E, W)
                units = [f"{p}mlp.e{e}." for e in range(E)]
            for u in units:
                out.update({u + "gate": (F, W), u + "up": (F, W), u + "down": (W, F)})
    return out


def synthetic(width: int, heads: int, ff: int, vocab: int, pattern: str = "rpls", experts: int = 16, top: int = 4, rank: int = 512,
              q_rank: int = 0, seed: int = 0):
    """A random-weight model of realistic layer sizes, in memory (timing and smoke runs). `pattern` lists the layers: "r"
    rotated latent attention, "p" the plain one, "s" the plain one over the latent of the latest "p" before it; a "d" after a
    letter makes that layer's feed-forward dense (width 4 * `ff`), the others have a mixture of `experts` experts of width
    `ff`. Returns (config dict, {name: tensor})."""
    import numpy as np
    from .safetensors_file import STensor
    q_rank = q_rank or max(64, 3 * width // 8)
    rot = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": rank, "q_rank": q_rank, "scale": 192 ** -0.5,
           "rot": {"base": 1e4, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    plain = {"heads": heads, "dim": 128, "vdim": 128, "kv_rank": rank, "q_rank": q_rank, "scale": 128 ** -0.5}
    layers, last_plain = [], None
    for n, ch in enumerate(pattern.replace("d", "")):
        if ch == "s" and last_plain is None:
            raise ValueError("pattern: an 's' needs a 'p' before it")
        mix = rot if ch == "r" else dict(plain, kv_from=last_plain) if ch == "s" else plain
        last_plain = n if ch == "p" else last_plain
        layers.append({"type": "latent_attention" if ch == "r" else "latent_attention_2", "mixer": mix,
                       "mlp": {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}})
    n = -1
    for ch in pattern:
        if ch != "d":
            n += 1
        else:
            layers[n]["mlp"] = {"kind": "dense", "ff": 4 * ff}
    cfg = {"architecture": "Fazovik", "embedding": {"bigram": {"buckets": 4093, "mul_cur": 31, "mul_prev": 1009}}, "layers": layers,
           "norm": {"eps": 1e-5}, "vocab": vocab, "width": width}
    rng = np.random.default_rng(seed)
    tensors = {}
    for name, shape in tensor_shapes(cfg).items():
        size = int(np.prod(shape))
        leaf = name.rsplit(".", 1)[-1]
        if len(shape) == 2:
            a = rng.standard_normal(size, dtype=np.float32) / np.sqrt(shape[1])
        elif leaf == "b":
            a = rng.standard_normal(size, dtype=np.float32) * 0.05
        else:
            a = np.ones(size, dtype=np.float32)
        bits = (np.ascontiguousarray(a, dtype=np.float32).view(np.uint32) >> 16).astype(np.uint16)       # truncation is fine for random weights
        tensors[name] = STensor(name, "BF16", tuple(shape), bits.reshape(shape))
    return cfg, tensors


def open_synthetic(cfg, tensors, **kw):
    from .engine import LayeredEngine
    return LayeredEngine(read_dims(cfg), tensors, **kw)


def _open(src, **kw):
    from .engine import LayeredEngine
    have = src.weights.tensors
    dims = read_dims(src.config)
    want = tensor_shapes(src.config)
    for name, shape in want.items():
        if name not in have:
            raise ValueError(f"{src.path}: tensor {name} is missing")
        if tuple(have[name].shape) != tuple(shape):
            raise ValueError(f"{src.path}: tensor {name} has shape {tuple(have[name].shape)}, the config asks for {tuple(shape)}")
    return LayeredEngine(dims, {n: have[n] for n in want}, **kw)


FAZOVIK = register(Family(name="Fazovik", source="folder", open_engine=_open))
