"""Plain float64 restatement of the Zogurax decoder (test oracle only; the product path never imports it).

Zogurax is a pre-norm decoder whose two sublayers run side by side behind ONE bias-free layer norm:
x <- x + (mixer(n) + ff(n)), n = norm1(x). The embedding adds a sinusoid of the position; nothing else but the temperature of the
queries knows a position. A run of layers is passed several times: ahead of every pass the stream is mixed with the embedding
output by one linear map and a learned vector of the pass is added. Two token mixers, both softmax attention over capped scores:
one with short convolutions on q, k, v, RMS norms over whole projections and a sigmoid gate per head, one with biases and a one
added to the softmax denominator. Feed-forward: experts (squared ReLU, no biases) chosen by a table of token ids, all with the
same weight, beside a shared expert with a sigmoid gate per token.

One function per mechanism, whole sequences at a time, no cache and no batching: every token's output is computed from the
full prefix the slow way. `w` maps tensor names to arrays, `cfg` is the parsed config.json dictionary.

Notation: h [T, W] is a sublayer's input, positions count from 0, linear maps are stored [out, in].
"""
from __future__ import annotations

import math

import numpy as np

F = np.float64


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def relu2(z):
    return np.maximum(z, 0.0) ** 2


def rms_norm(x, weight, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * weight


def layer_norm(x, weight, eps):
    mean = x.mean(-1, keepdims=True)
    return (x - mean) / np.sqrt(((x - mean) ** 2).mean(-1, keepdims=True) + eps) * weight


def position_sinusoid(positions, width):
    """[T, width]: entry 2i = sin(p * 10000^(-2i/width)), entry 2i + 1 = cos of the same."""
    out = np.zeros((len(positions), width), dtype=F)
    for c in range(width):
        angle = np.asarray(positions, dtype=F) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = np.sin(angle) if c % 2 == 0 else np.cos(angle)
    return out


def embed(w, tokens):
    return w["embed"][np.asarray(tokens, dtype=np.int64)] + position_sinusoid(np.arange(len(tokens)), w["embed"].shape[1])


def causal_conv(u, taps):
    """u [T, C], taps [C, n]: y_t = sum_j taps[:, j] u_(t - n + 1 + j), zeros before the start."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, u.shape[1]), dtype=F), u])
    return sum(taps[:, j] * padded[j:j + u.shape[0]] for j in range(n))


def query_temperature(positions, q_temp):
    p = np.asarray(positions, dtype=F)
    return 1.0 + float(q_temp["coef"]) * np.log(np.floor((p + 1.0) / float(q_temp["every"])) + 1.0)


def cap(s, softcap):
    return softcap * np.tanh(s / softcap)


def causal_weights(scores, extra):
    """exp(s) / (extra + sum exp(s)) over the keys up to the query; extra = 0 is the ordinary softmax, 1 adds one to the sum."""
    T = scores.shape[0]
    s = np.where(np.tril(np.ones((T, T), dtype=bool)), scores, -np.inf)
    m = np.maximum(s.max(-1, keepdims=True), 0.0) if extra else s.max(-1, keepdims=True)
    p = np.exp(s - m)
    return p / (extra * np.exp(-m) + p.sum(-1, keepdims=True))


def attend(q, k, v, m, extra):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head a reads key/value head a // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    q = q * query_temperature(np.arange(T), m["q_temp"])[:, None, None]
    out = np.zeros((T, H, v.shape[2]), dtype=F)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = causal_weights(cap(q[:, a] @ k[:, g].T * float(m["scale"]), float(m["softcap"])), extra) @ v[:, g]
    return out


def sizes(m):
    return int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])


def convolved_attention(h, w, pre, m, eps):
    T = h.shape[0]
    H, G, d, dv = sizes(m)
    q, k, v = (causal_conv(h @ w[pre + n].T, w[pre + n + ".conv"]) for n in "qkv")
    q, k = rms_norm(q, w[pre + "q.norm"], eps), rms_norm(k, w[pre + "k.norm"], eps)
    o = attend(q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, dv), m, extra=0.0)
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[pre + "o"].T


def biased_attention(h, w, pre, m, eps):
    T = h.shape[0]
    H, G, d, dv = sizes(m)
    q, k, v = (h @ w[pre + n].T + w[pre + n + ".b"] for n in "qkv")
    o = attend(q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, dv), m, extra=1.0)
    return o.reshape(T, H * dv) @ w[pre + "o"].T + w[pre + "o.b"]


MIXERS = {"attention": convolved_attention, "attention_2": biased_attention}


def expert(h, w, pre):
    return relu2(h @ w[pre + "up"].T) @ w[pre + "down"].T


def table_mixture(h, w, pre, mlp, tokens):
    """Experts by token id, equal weights; the shared expert for every token, times its sigmoid gate."""
    table, top = w[pre + "table"], int(mlp["router"]["top"])
    out = np.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in table[int(tok)]:
            out[t] += expert(h[t:t + 1], w, f"{pre}e{int(e)}.")[0] / top
    if mlp.get("shared"):
        out += sigmoid(h @ w[pre + "shared.sg"].T) * expert(h, w, pre + "shared.")
    return out


def runs(cfg):
    """(layer index, pass that starts ahead of it or None) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    out = [(i, None) for i in range(a)]
    for t in range(int(loop["times"])):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def start_pass(x, x0, w, t):
    return np.concatenate([x, x0], axis=-1) @ w["loop.in"].T + w["loop.step"][t]


def forward(cfg, weights, tokens, return_layers=False):
    """logits [T, vocab] (and the residual stream after every layer run [runs, T, W])."""
    w = {k: np.asarray(v) if np.issubdtype(np.asarray(v).dtype, np.integer) else np.asarray(v, dtype=F) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x0 = x = embed(w, tokens)
    trace = []
    for li, begins in runs(cfg):
        L, p = cfg["layers"][li], f"l{li}."
        if begins is not None:
            x = start_pass(x, x0, w, begins)
        h = layer_norm(x, w[p + "norm1"], eps)
        y = MIXERS[L["type"]](h, w, p + "mix.", L["mixer"], eps)
        if L.get("mlp"):
            y = y + table_mixture(h, w, p + "mlp.", L["mlp"], tokens)
        x = x + y
        trace.append(x.copy())
    logits = layer_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, np.stack(trace)) if return_layers else logits
