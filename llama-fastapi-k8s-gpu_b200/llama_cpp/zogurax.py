"""Zogurax: a decoder of parallel blocks behind one norm, with a looped run of layers and experts chosen by token id, served by
the layer-list graph of the native engine.

A model folder holds `config.json` and `model.safetensors`. The embedding output is the embedding row plus a sinusoid of the
position. Every layer is
    x <- x + (mixer(n) + ff(n)),  n = LayerNorm(x) * norm1            (`mlp` may be null)
`loop` passes layers start .. stop-1 `times` times with the same weights; ahead of pass t the stream becomes
`loop.in` [x; x0] + `loop.step`[t], x0 being the embedding output. Every pass keeps a cache and state of its own, which is why
the engine gets one layer entry per RUN with `weights_of` naming the layer whose tensors it uses and `loop_pass` marking the
entries a pass starts with. Token mixers, both causal softmax attention with grouped query heads, capped scores, queries
scaled by a slowly growing function of the position (`q_temp`) and a value size of its own:
  "attention":   a short causal convolution on every channel of q, k and v, q and k RMS-normed over the whole projection, one
                 sigmoid gate per head
  "attention_2": biases on q, k, v and the output map, one added to the softmax denominator
Feed-forward "moe": squared-ReLU experts; `mlp.table` [vocab, top] (int32) gives each token id its experts, all with weight
1 / top; the shared expert runs for every token, times a sigmoid gate.

This module turns the config into the C ABI's `b2_layer_desc` list (every size and constant comes from the file) and
checks the tensor set; the arithmetic is in csrc/layered.cu, sink_attn.cu, mixers.cu, moe.cu and dense.cu.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

from . import _cabi
from .goponex import LayeredDims, _need
from .models import Family, register
from .nafelix import layer_runs


def pass_starts(cfg: dict) -> List[Tuple[int, Optional[int]]]:
    """(layer index, number of the pass that starts ahead of it or None) for every run of a layer, in order."""
    runs, loop = layer_runs(cfg), cfg.get("loop")
    if not loop:
        return [(i, None) for i in runs]
    a, b = int(loop["start"]), int(loop["stop"])
    if a == b:
        raise ValueError(f"config.json: loop {loop!r} holds no layers")
    return [(i, (r - a) // (b - a) if a <= r < a + (b - a) * int(loop["times"]) and i == a else None) for r, i in enumerate(runs)]


def layer_desc(i: int, layer: dict, weights_of: int = 0, loop_pass: Optional[int] = None) -> _cabi.B2LayerDesc:
    where = f"layers[{i}]"
    kind = _need(layer, "type", where)
    m = _need(layer, "mixer", where)
    d = _cabi.B2LayerDesc()
    d.mixer = _cabi.B2_MIX_SINK_ATTN
    d.weights_of = weights_of
    d.loop_pass = 0 if loop_pass is None else loop_pass + 1
    if kind == "attention":
        d.attn_flags = _cabi.B2_ATTN_CONV | _cabi.B2_ATTN_FULL_NORM | _cabi.B2_ATTN_HEAD_GATE | _cabi.B2_ATTN_NO_SINK
        d.conv_taps = int(_need(m, "conv", where + ".mixer"))
    elif kind == "attention_2":
        d.attn_flags = _cabi.B2_ATTN_BIAS | _cabi.B2_ATTN_OUT_BIAS | _cabi.B2_ATTN_UNIT_SINK | _cabi.B2_ATTN_NO_GATE
    else:
        raise ValueError(f"config.json: {where}: unknown layer type {kind!r}")
    d.n_head, d.head_dim = int(_need(m, "heads", where)), int(_need(m, "dim", where))
    d.n_head_kv = int(m.get("kv_heads", d.n_head))
    d.attn_vdim = int(m.get("vdim", d.head_dim))
    d.attn_scale = float(_need(m, "scale", where))
    d.softcap = float(_need(m, "softcap", where))
    if not d.softcap > 0.0:
        raise ValueError(f"config.json: {where}: softcap must be positive")
    qt = _need(m, "q_temp", where)
    d.qtemp_coef, d.qtemp_every = float(_need(qt, "coef", where + ".q_temp")), float(_need(qt, "every", where + ".q_temp"))
    if not d.qtemp_every > 0.0:
        raise ValueError(f"config.json: {where}: q_temp.every must be positive")
    mlp = layer.get("mlp")
    if mlp:
        if mlp.get("kind", "moe") != "moe":
            raise ValueError(f"config.json: {where}: unknown feed-forward kind {mlp.get('kind')!r}")
        r, ex = _need(mlp, "router", where + ".mlp"), _need(mlp, "expert", where + ".mlp")
        d.ff_kind, d.n_ff = _cabi.B2_FF_MOE, int(_need(ex, "ff", where + ".mlp.expert"))
        d.moe_experts, d.moe_identity, d.moe_top = int(_need(r, "experts", where)), 0, int(_need(r, "top", where))
        d.moe_groups = d.moe_keep = 1
        d.moe_scale = 1.0
        d.moe_route, d.moe_expert = _cabi.B2_ROUTE_TABLE, _cabi.B2_EXPERT_RELU2
        if mlp.get("shared"):
            d.moe_shared_ff, d.moe_shared_gate = int(_need(mlp["shared"], "ff", where + ".mlp.shared")), 1
    return d


def read_dims(cfg: dict) -> LayeredDims:
    layers = _need(cfg, "layers", "the config")
    descs = [layer_desc(i, layers[i], weights_of=i + 1, loop_pass=t) for i, t in pass_starts(cfg)]
    return LayeredDims(n_layer=len(descs), n_embd=int(_need(cfg, "width", "the config")), n_vocab=int(_need(cfg, "vocab", "the config")),
                       norm_eps=float(_need(_need(cfg, "norm", "the config"), "eps", "norm")), residual_scale=1.0, layers=descs,
                       block_style=_cabi.B2_BLOCK_PARALLEL_ONE_LN, embed_sinusoid=True,
                       loop_times=int(cfg["loop"]["times"]) if cfg.get("loop") else 0)


def tensor_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    """Every tensor the design needs, with its shape ([out, in] for linear maps); `mlp.table` holds integers."""
    W, V = int(cfg["width"]), int(cfg["vocab"])
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    if cfg.get("loop"):
        out.update({"loop.in": (W, 2 * W), "loop.step": (int(cfg["loop"]["times"]), W)})
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        a = p + "mix."
        H, d = int(m["heads"]), int(m["dim"])
        G, dv = int(m.get("kv_heads", H)), int(m.get("vdim", d))
        rows = {"q": H * d, "k": G * d, "v": G * dv}
        out[p + "norm1"] = (W,)
        out.update({a + n: (r, W) for n, r in rows.items()})
        out[a + "o"] = (W, H * dv)
        if L["type"] == "attention":
            out.update({f"{a}{n}.conv": (r, int(m["conv"])) for n, r in rows.items()})
            out.update({a + "q.norm": (H * d,), a + "k.norm": (G * d,), a + "g": (H, W)})
        else:
            out.update({f"{a}{n}.b": (r,) for n, r in rows.items()})
            out[a + "o.b"] = (W,)
        mlp = L.get("mlp")
        if mlp:
            E, F = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
            out[p + "mlp.table"] = (V, int(mlp["router"]["top"]))
            for e in range(E):
                out.update({f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
            if mlp.get("shared"):
                S = int(mlp["shared"]["ff"])
                out.update({p + "mlp.shared.up": (S, W), p + "mlp.shared.down": (W, S), p + "mlp.shared.sg": (1, W)})
    return out


def synthetic(width: int, heads: int, ff: int, vocab: int, pattern: str = "ba", experts: int = 16, top: int = 4, loop=None, seed: int = 0):
    """A random-weight model of realistic layer sizes, in memory (timing and smoke runs). `pattern` lists the layers: "a"
    attention, "b" attention_2; experts and the shared expert have width `ff`; `loop` = (start, stop, times). Returns
    (config dict, {name: tensor})."""
    import numpy as np
    from .safetensors_file import STensor
    kv = max(1, heads // 4)
    common = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    a = dict(common, conv=4, softcap=30.0, q_temp={"coef": 0.1, "every": 1024})
    b = dict(common, softcap=50.0, q_temp={"coef": 0.2, "every": 512})
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": ff}}
    layers = [{"type": "attention" if ch == "a" else "attention_2", "mixer": a if ch == "a" else b, "mlp": mlp} for ch in pattern]
    cfg = {"architecture": "Zogurax", "layers": layers, "norm": {"eps": 1e-5}, "vocab": vocab, "width": width}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    rng = np.random.default_rng(seed)
    tensors = {}
    for name, shape in tensor_shapes(cfg).items():
        size = int(np.prod(shape))
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "table":
            first = rng.integers(0, experts, size=shape[0])
            t = (first[:, None] + np.arange(top) * max(1, experts // top)) % experts        # distinct while top <= experts
            tensors[name] = STensor(name, "I32", tuple(shape), t.astype(np.int32))
            continue
        if leaf == "conv":
            v = rng.standard_normal(size, dtype=np.float32) * 0.5
        elif len(shape) == 2:
            v = rng.standard_normal(size, dtype=np.float32) / np.sqrt(shape[1])
        elif leaf == "b":
            v = rng.standard_normal(size, dtype=np.float32) * 0.05
        else:
            v = np.ones(size, dtype=np.float32)
        bits = (np.ascontiguousarray(v, dtype=np.float32).view(np.uint32) >> 16).astype(np.uint16)       # truncation is fine for random weights
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
        if name.endswith(".table") and have[name].dtype != "I32":
            raise ValueError(f"{src.path}: tensor {name} has dtype {have[name].dtype}, expected I32")
    return LayeredEngine(dims, {n: have[n] for n in want}, **kw)


ZOGURAX = register(Family(name="Zogurax", source="folder", open_engine=_open))
