"""Host-side pieces of the Zogurax family (no GPU): config -> layer descriptors (one per run of a layer), the tensor set, the
registry, refusals, and sanity properties of the float64 oracle's mechanisms."""
import math

import numpy as np
import pytest

import zogurax_util as zu
from oracle import zogurax_ref as ref


def f64(w):
    return {k: v if np.issubdtype(np.asarray(v).dtype, np.integer) else np.asarray(v, dtype=np.float64) for k, v in w.items()}


def test_config_to_descriptors():
    from llama_cpp import _cabi, zogurax
    cfg = zu.config([zu.biased(mlp=zu.moe(experts=7, top=3, ff=16, shared=11), heads=6, kv_heads=2, dim=10, vdim=14, scale=0.3, softcap=9.0, coef=0.25, every=33),
                     zu.conved(mlp=zu.moe(shared=None), heads=5, kv_heads=1, dim=8, vdim=6, conv=4, scale=0.7, softcap=2.5, coef=0.5, every=12),
                     zu.conved(mlp=None)], loop=(1, 3, 2))
    d = zogurax.read_dims(cfg)
    assert d.block_style == _cabi.B2_BLOCK_PARALLEL_ONE_LN and d.embed_sinusoid and d.loop_times == 2 and not d.tie_head
    assert d.n_layer == 5 and [x.weights_of for x in d.layers] == [1, 2, 3, 2, 3] and [x.loop_pass for x in d.layers] == [0, 1, 0, 2, 0]
    a, b, c = d.layers[:3]
    assert all(x.mixer == _cabi.B2_MIX_SINK_ATTN for x in d.layers)
    assert (a.n_head, a.n_head_kv, a.head_dim, a.attn_vdim, a.attn_scale, a.softcap, a.qtemp_coef, a.qtemp_every) == (6, 2, 10, 14, 0.3, 9.0, 0.25, 33.0)
    assert a.attn_flags == _cabi.B2_ATTN_BIAS | _cabi.B2_ATTN_OUT_BIAS | _cabi.B2_ATTN_UNIT_SINK | _cabi.B2_ATTN_NO_GATE and a.conv_taps == 0
    assert (a.ff_kind, a.n_ff, a.moe_experts, a.moe_top, a.moe_route, a.moe_expert, a.moe_shared_ff, a.moe_shared_gate) == (
        _cabi.B2_FF_MOE, 16, 7, 3, _cabi.B2_ROUTE_TABLE, _cabi.B2_EXPERT_RELU2, 11, 1)
    assert (b.n_head, b.n_head_kv, b.head_dim, b.attn_vdim, b.conv_taps, b.softcap, b.qtemp_every) == (5, 1, 8, 6, 4, 2.5, 12.0)
    assert b.attn_flags == _cabi.B2_ATTN_CONV | _cabi.B2_ATTN_FULL_NORM | _cabi.B2_ATTN_HEAD_GATE | _cabi.B2_ATTN_NO_SINK
    assert (b.moe_shared_ff, b.moe_shared_gate, c.n_ff) == (0, 0, 0)
    s = zogurax.tensor_shapes(cfg)
    assert s["loop.in"] == (72, 144) and s["loop.step"] == (2, 72) and s["head"] == (131, 72) and "final.norm.b" not in s
    assert s["l0.mix.q"] == (60, 72) and s["l0.mix.k.b"] == (20,) and s["l0.mix.v"] == (28, 72) and s["l0.mix.o"] == (72, 84) and s["l0.mix.o.b"] == (72,)
    assert "l0.mix.g" not in s and "l0.mix.q.norm" not in s and "l0.norm2" not in s
    assert s["l0.mlp.table"] == (131, 3) and s["l0.mlp.e6.down"] == (72, 16) and s["l0.mlp.shared.up"] == (11, 72) and s["l0.mlp.shared.sg"] == (1, 72)
    assert s["l1.mix.q.conv"] == (40, 4) and s["l1.mix.v.conv"] == (6, 4) and s["l1.mix.k.norm"] == (8,) and s["l1.mix.g"] == (5, 72) and "l1.mix.q.b" not in s
    assert "l1.mlp.shared.up" not in s and not any(k.startswith("l2.mlp") for k in s)
    plain = zu.config([zu.biased()])
    assert zogurax.read_dims(plain).loop_times == 0 and "loop.in" not in zogurax.tensor_shapes(plain)


def test_passes():
    from llama_cpp import zogurax
    cfg = zu.config([zu.biased()] * 4, loop=(1, 3, 3))
    assert zogurax.pass_starts(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)] == ref.runs(cfg)
    cfg = zu.config([zu.biased()] * 2, loop=(0, 1, 2))
    assert zogurax.pass_starts(cfg) == [(0, 0), (0, 1), (1, None)] == ref.runs(cfg)
    with pytest.raises(ValueError):
        zogurax.pass_starts(zu.config([zu.biased()] * 2, loop=(1, 1, 2)))


def test_registry_and_folder(tmp_path):
    from llama_cpp import models, zogurax
    cfg = zu.config([zu.conved(mlp=zu.moe())], loop=(0, 1, 1))
    path = zu.write_model(str(tmp_path / "m"), cfg, zu.random_weights(cfg))
    src = models.open_model(path)
    assert src.family.name == "Zogurax" and "Zogurax" in models.architectures() and src.weights.tensors["l0.mlp.table"].dtype == "I32"
    no_cap = zu.biased()
    del no_cap["mixer"]["softcap"]
    bad = [dict(zu.biased(), type="nope"), no_cap, zu.biased(softcap=0.0), zu.biased(every=0), zu.biased(mlp={"kind": "dense", "ff": 4})]
    for layer in bad:
        with pytest.raises(ValueError):
            zogurax.read_dims(zu.config([layer]))
    with pytest.raises(ValueError):
        zogurax.read_dims(zu.config([zu.biased()], loop=(0, 2, 1)))


def test_sinusoid_by_hand():
    s = ref.position_sinusoid([0, 3], 5)
    assert np.allclose(s[0], [0, 1, 0, 1, 0])
    f = [1.0, 10000.0 ** (-2 / 5), 10000.0 ** (-4 / 5)]
    assert np.allclose(s[1], [math.sin(3 * f[0]), math.cos(3 * f[0]), math.sin(3 * f[1]), math.cos(3 * f[1]), math.sin(3 * f[2])])


def test_query_temperature_steps():
    t = ref.query_temperature(np.arange(12), {"coef": 0.5, "every": 4})
    assert np.allclose(t[:3], 1.0) and np.allclose(t[3:7], 1 + 0.5 * math.log(2)) and np.allclose(t[7:11], 1 + 0.5 * math.log(3)) and t[11] > t[10]


def test_causal_conv():
    u, taps = np.arange(1.0, 6.0)[:, None], np.array([[0.5, 2.0, 3.0]])
    assert np.allclose(ref.causal_conv(u, taps)[:, 0], [3.0, 2 + 6, 0.5 + 4 + 9, 1 + 6 + 12, 1.5 + 8 + 15])


def test_one_in_the_denominator():
    s = np.array([[-3.0, 9.0], [1.0, 2.0]])
    p = ref.causal_weights(s, 1.0)
    e = np.exp(1.0)
    assert np.allclose(p[0], [np.exp(-3) / (1 + np.exp(-3)), 0]) and np.allclose(p[1], np.array([e, e * e]) / (1 + e + e * e))
    assert np.allclose(ref.causal_weights(s, 0.0).sum(-1), 1.0)
    assert abs(ref.cap(np.array(1e9), 7.0) - 7.0) < 1e-9 and abs(ref.cap(np.array(1e-3), 7.0) - 1e-3) < 1e-9


def test_experts_by_token_id():
    mlp = zu.moe(experts=5, top=2, ff=8, shared=6)
    cfg = zu.config([zu.biased(mlp=mlp)])
    w = f64(zu.random_weights(cfg, seed=4))
    h = np.random.default_rng(5).standard_normal((3, 72))
    y = ref.table_mixture(h, w, "l0.mlp.", mlp, [9, 4, 9])
    a, b = w["l0.mlp.table"][4]
    want = (ref.expert(h[1:2], w, f"l0.mlp.e{a}.") + ref.expert(h[1:2], w, f"l0.mlp.e{b}."))[0] / 2
    gate = ref.sigmoid(w["l0.mlp.shared.sg"][0] @ h[1])
    want = want + gate * (w["l0.mlp.shared.down"] @ np.maximum(w["l0.mlp.shared.up"] @ h[1], 0) ** 2)
    assert np.allclose(y[1], want)
    assert len(set(w["l0.mlp.table"][7])) == 2


def test_a_pass_mixes_in_the_embedding_output():
    cfg = zu.config([zu.biased()], loop=(0, 1, 2))
    w = zu.random_weights(cfg, seed=6)
    toks = [3, 8, 1]
    _, layers = ref.forward(cfg, w, toks, return_layers=True)
    wd = f64(w)
    x0 = ref.embed(wd, toks)
    x = layers[0]
    start = x @ wd["loop.in"][:, :72].T + x0 @ wd["loop.in"][:, 72:].T + wd["loop.step"][1]
    y = ref.biased_attention(ref.layer_norm(start, wd["l0.norm1"], 1e-5), wd, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5)
    assert layers.shape[0] == 2 and np.allclose(layers[1], start + y)


def test_oracle_is_causal_and_parallel():
    cfg = zu.config([zu.conved(mlp=zu.moe()), zu.biased(mlp=zu.moe())], loop=(0, 1, 2))
    w = zu.random_weights(cfg, seed=4)
    toks = [int(t) for t in np.random.default_rng(5).integers(0, cfg["vocab"], size=30)]
    full = ref.forward(cfg, w, toks)
    assert np.allclose(ref.forward(cfg, w, toks[:17]), full[:17], atol=1e-10)


def test_synthetic_models():
    from llama_cpp import zogurax
    cfg, tensors = zogurax.synthetic(64, 4, 16, 50, pattern="abb", experts=8, top=3, loop=(1, 3, 2))
    assert [L["type"] for L in cfg["layers"]] == ["attention", "attention_2", "attention_2"] and cfg["loop"]["times"] == 2
    assert {n: tuple(t.shape) for n, t in tensors.items()} == zogurax.tensor_shapes(cfg)
    t = tensors["l0.mlp.table"]
    assert t.dtype == "I32" and all(len(set(r)) == 3 for r in np.asarray(t.data)) and np.asarray(t.data).max() < 8
