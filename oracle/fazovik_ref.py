"""Plain float64 restatement of the Fazovik decoder (test oracle only; the product path never imports it).

Fazovik is a pre-norm decoder with parallel blocks: x <- x + mixer(norm1(x)) + ff(norm2(x)), both norms (mean and variance,
weight and bias) of the same x. Two token mixers, both attention over one cached low-rank latent per token: one with an
interleaved rotation on a separate query / key part and a sigmoid gate per head, one without positions that may read the
latent of an earlier layer instead of making its own. Feed-forward: a gated GELU unit or a mixture of gated SiLU experts
whose sigmoid score scales the expert's INPUT. The embedding adds a row hashed from the token pair (previous, current).

One function per mechanism, whole sequences at a time, no cache and no batching: every token's output is computed from the
full prefix the slow way. `w` maps tensor names to float arrays, `cfg` is the parsed config.json dictionary.

Notation: h [T, W] is a sublayer's input, positions count from 0, linear maps are stored [out, in].
"""
from __future__ import annotations

import math

import numpy as np

F = np.float64


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, weight, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * weight


def layer_norm(x, weight, bias, eps):
    mean = x.mean(-1, keepdims=True)
    var = ((x - mean) ** 2).mean(-1, keepdims=True)
    return (x - mean) / np.sqrt(var + eps) * weight + bias


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Table row of every token: a hash of (previous, current); the extra last row for the first token."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return np.array(rows[:len(tokens)], dtype=np.int64)


def embed(w, tokens, bigram):
    x = w["embed"][np.asarray(tokens, dtype=np.int64)]
    if bigram:
        x = x + w["bigram"][bigram_rows(list(tokens), int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"]))]
    return x


def rotation_frequencies(rot):
    """Frequencies of the pairs and the factor on cos and sin. With scaling: pairs that turn slowly over the original context
    are slowed down by `factor`, fast ones stay, a linear ramp over the pair index between the two."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor = float(sc["factor"])

    def index_of(turns):
        return dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(index_of(float(sc["slow"]))), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, positions, rot):
    """x [T, ..., d]: entries 2i and 2i+1 of the first rot.dims are one pair; the rest pass through."""
    f, mag = rotation_frequencies(rot)
    n = int(rot["dims"])
    ang = np.asarray(positions, dtype=F)[:, None] * f[None, :]
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (n // 2,)
    c, s = (np.cos(ang) * mag).reshape(shape), (np.sin(ang) * mag).reshape(shape)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.copy()
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


def causal_softmax(scores):
    T = scores.shape[0]
    s = np.where(np.tril(np.ones((T, T), dtype=bool)), scores, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


def latent_queries(h, w, pre, width, heads, eps):
    cq = rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps)
    return (cq @ w[pre + "uq"].T).reshape(h.shape[0], heads, width)


def rotated_latent_attention(h, w, pre, m, eps, latents, layer):
    T = h.shape[0]
    H, d, dr, dv, rank = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    pos = np.arange(T)
    q = latent_queries(h, w, pre, d + dr, H, eps)
    qr = rotate_pairs(q[..., d:], pos, m["rot"])
    down = h @ w[pre + "dkv"].T
    c = rms_norm(down[:, :rank], w[pre + "dkv.norm"], eps)
    latents[layer] = c
    kr = rotate_pairs(down[:, rank:], pos, m["rot"])
    k = (c @ w[pre + "uk"].T).reshape(T, H, d)
    v = (c @ w[pre + "uv"].T).reshape(T, H, dv)
    gate = sigmoid(h @ w[pre + "g"].T)
    out = np.zeros((T, H, dv), dtype=F)
    for a in range(H):
        p = causal_softmax((q[:, a, :d] @ k[:, a].T + qr[:, a] @ kr.T) * float(m["scale"]))
        out[:, a] = (p @ v[:, a]) * gate[:, a:a + 1]
    return out.reshape(T, H * dv) @ w[pre + "o"].T


def plain_latent_attention(h, w, pre, m, eps, latents, layer):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = latent_queries(h, w, pre, d, H, eps)
    if m.get("kv_from") is None:
        latents[layer] = rms_norm(h @ w[pre + "dkv"].T, w[pre + "dkv.norm"], eps)
        c = latents[layer]
    else:
        c = latents[int(m["kv_from"])]
    k = (c @ w[pre + "uk"].T).reshape(T, H, d)
    v = (c @ w[pre + "uv"].T).reshape(T, H, dv)
    out = np.zeros((T, H, dv), dtype=F)
    for a in range(H):
        out[:, a] = causal_softmax((q[:, a] @ k[:, a].T) * float(m["scale"])) @ v[:, a]
    return out.reshape(T, H * dv) @ w[pre + "o"].T


MIXERS = {"latent_attention": rotated_latent_attention, "latent_attention_2": plain_latent_attention}


def gated_unit(h, w, pre, act):
    return (act(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(h, w, pre, r):
    """Chosen experts [T, top] and their scores (sigmoid, not renormalised)."""
    s = sigmoid(h @ w[pre + "router"].T)
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :int(r["top"])]
    return chosen, np.take_along_axis(s, chosen, axis=-1)


def mixture(h, w, pre, mlp):
    chosen, score = route(h, w, pre, mlp["router"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], score[t]):
            out[t] += gated_unit((s * h[t])[None], w, f"{pre}e{e}.", silu)[0]
    return out


def feed_forward(h, w, pre, mlp):
    return mixture(h, w, pre, mlp) if mlp["kind"] == "moe" else gated_unit(h, w, pre, gelu_tanh)


def forward(cfg, weights, tokens, return_layers=False):
    """logits [T, vocab] (and the residual stream after every layer [L, T, W])."""
    w = {k: np.asarray(v, dtype=F) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = embed(w, tokens, (cfg.get("embedding") or {}).get("bigram"))
    trace, latents = [], {}
    for li, L in enumerate(cfg["layers"]):
        p = f"l{li}."
        y = MIXERS[L["type"]](layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps), w, p + "mix.", L["mixer"], eps, latents, li)
        if L.get("mlp"):
            y = y + feed_forward(layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps), w, p + "mlp.", L["mlp"])
        x = x + y
        trace.append(x.copy())
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
    return (logits, np.stack(trace)) if return_layers else logits
