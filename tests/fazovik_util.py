"""Small random Fazovik models for the tests: a config, bf16-rounded random weights, the folder the product loads."""
import numpy as np

from goponex_util import bf16_round, rel_err, write_model  # noqa: F401  (shared helpers)


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def scaling(factor=3.0, original=40, fast=6.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def rotated(mlp=None, heads=3, dim=20, rot_dim=12, vdim=14, rank=28, q_rank=22, base=3000.0, scale=None, yarn=scaling()):
    rot = {"base": base, "dims": rot_dim}
    if yarn:
        rot["scaling"] = yarn
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "rot": rot,
                      "scale": float(scale if scale is not None else (dim + rot_dim) ** -0.5)}}


def plain(mlp=None, heads=4, dim=18, vdim=10, rank=26, q_rank=30, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": float(scale if scale is not None else dim ** -0.5)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention_2", "mixer": m, "mlp": mlp}


def bigram(buckets=53, mul_prev=17, mul_cur=5):
    return {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}


def config(layers, width=72, vocab=131, eps=1e-5, hashed=bigram()):
    return {"architecture": "Fazovik", "embedding": {"bigram": hashed} if hashed else {}, "layers": layers, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


def random_weights(cfg, seed=0):
    """Weights at a scale that keeps every mechanism alive (gates and scores unsaturated, norm biases and the bigram row as
    large as what they are added to), rounded to bf16 so the file and the oracle hold the same numbers."""
    from llama_cpp.fazovik import tensor_shapes
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "router":
            a = rng.standard_normal(shape) * 2.0 / np.sqrt(shape[1])
        elif name in ("embed", "bigram"):
            a = rng.standard_normal(shape)
        elif leaf in ("gate", "up") and ".mlp." in name:
            a = rng.standard_normal(shape) * 1.5 / np.sqrt(shape[1])
        elif leaf in ("uq", "uk", "dkv"):               # scores spread enough that single keys and their positions matter
            a = rng.standard_normal(shape) * (1.4 if leaf != "dkv" else 2.0) / np.sqrt(shape[1])
        elif leaf == "o":
            a = rng.standard_normal(shape) * 2.0 / np.sqrt(shape[1])
        elif len(shape) == 2:
            a = rng.standard_normal(shape) / np.sqrt(shape[1])
        elif leaf == "b":
            a = rng.standard_normal(shape) * 0.5
        else:                                           # norm weights
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        w[name] = bf16_round(a)
    return w
