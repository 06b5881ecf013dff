"""Small random Zogurax models for the tests: a config, bf16-rounded random weights, the folder the product loads."""
import numpy as np

from goponex_util import bf16_round, rel_err, write_model  # noqa: F401  (shared helpers)


def moe(experts=6, top=2, ff=24, shared=20):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _mixer(heads, kv_heads, dim, vdim, scale, softcap, coef, every):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": softcap, "q_temp": {"coef": coef, "every": every},
            "scale": float(scale if scale is not None else 1.5 * dim ** -0.5)}


def conved(mlp=None, heads=4, kv_heads=2, dim=20, vdim=12, conv=3, scale=None, softcap=4.0, coef=0.6, every=9):
    return {"type": "attention", "mixer": dict(_mixer(heads, kv_heads, dim, vdim, scale, softcap, coef, every), conv=conv), "mlp": mlp}


def biased(mlp=None, heads=6, kv_heads=3, dim=18, vdim=14, scale=None, softcap=6.0, coef=0.4, every=7):
    return {"type": "attention_2", "mixer": _mixer(heads, kv_heads, dim, vdim, scale, softcap, coef, every), "mlp": mlp}


def config(layers, width=72, vocab=131, eps=1e-5, loop=None):
    cfg = {"architecture": "Zogurax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def random_weights(cfg, seed=0):
    """Weights at a scale that keeps every mechanism alive (scores into their caps, gates unsaturated, biases and the vectors of
    the passes as large as what they are added to), rounded to bf16 so the file and the oracle hold the same numbers."""
    from llama_cpp.zogurax import tensor_shapes
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "table":
            i = int(name[1:].split(".")[0])
            E = int(cfg["layers"][i]["mlp"]["router"]["experts"])
            w[name] = np.stack([rng.permutation(E)[:shape[1]] for _ in range(shape[0])]).astype(np.int32)
            continue
        if name == "embed":
            a = rng.standard_normal(shape)
        elif leaf == "conv":
            a = rng.standard_normal(shape) * 0.7
        elif leaf == "step":
            a = rng.standard_normal(shape) * 0.5
        elif leaf in ("q", "k"):
            a = rng.standard_normal(shape) * 1.3 / np.sqrt(shape[1])
        elif leaf == "o":
            a = rng.standard_normal(shape) * 2.0 / np.sqrt(shape[1])
        elif leaf == "sg":
            a = rng.standard_normal(shape) * 1.5 / np.sqrt(shape[1])
        elif len(shape) == 2:
            a = rng.standard_normal(shape) / np.sqrt(shape[1])
        elif leaf == "b":
            a = rng.standard_normal(shape) * 0.5
        else:                                           # norm weights
            a = 1.0 + 0.3 * rng.standard_normal(shape)
        w[name] = bf16_round(a)
    return w
