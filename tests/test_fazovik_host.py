"""Host-side pieces of the Fazovik family (no GPU): config -> layer descriptors, the tensor set, the registry, and sanity
properties of the float64 oracle's mechanisms."""
import copy
import math

import numpy as np
import pytest

import fazovik_util as fu
from oracle import fazovik_ref as ref


def f64(w):
    return {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}


def test_config_to_descriptors():
    from llama_cpp import _cabi, fazovik
    cfg = fu.config([fu.rotated(mlp=fu.dense(44), heads=5, dim=10, rot_dim=6, vdim=14, rank=21, q_rank=33, base=777.0, scale=0.3,
                                yarn=fu.scaling(5.0, 96, 8.0, 2.0)),
                     fu.plain(mlp=fu.moe(experts=7, top=3, ff=16), heads=2, dim=9, vdim=11, rank=19, q_rank=13, scale=0.7),
                     fu.plain(rank=19, kv_from=1), fu.rotated(yarn=None)], hashed=fu.bigram(10, 37, 12))
    d = fazovik.read_dims(cfg)
    assert d.block_style == _cabi.B2_BLOCK_PARALLEL_LN and d.tie_head and d.bigram == (10, 7, 2)
    a, b, c, e = d.layers
    assert all(x.mixer == _cabi.B2_MIX_LATENT_ATTN for x in d.layers)
    assert (a.n_head, a.head_dim, a.la_rot_dim, a.la_vdim, a.la_rank, a.la_q_rank, a.rot_dims, a.rope_base, a.attn_scale) == (5, 10, 6, 14, 21, 33, 6, 777.0, 0.3)
    assert (a.rope_factor, a.rope_orig_ctx, a.rope_fast, a.rope_slow, a.kv_from) == (5.0, 96, 8.0, 2.0, 0)
    assert a.attn_flags == _cabi.B2_ATTN_NO_SINK | _cabi.B2_ATTN_HEAD_GATE | _cabi.B2_ATTN_ROT_PAIRS
    assert (a.ff_kind, a.n_ff, a.ff_act) == (_cabi.B2_FF_GLU, 44, _cabi.B2_ACT_GELU_TANH)
    assert (b.n_head, b.head_dim, b.la_rot_dim, b.rot_dims, b.la_vdim, b.la_rank, b.la_q_rank, b.attn_scale) == (2, 9, 0, 0, 11, 19, 13, 0.7)
    assert b.attn_flags == _cabi.B2_ATTN_NO_SINK | _cabi.B2_ATTN_NO_GATE
    assert (b.ff_kind, b.n_ff, b.moe_experts, b.moe_top, b.moe_route, b.moe_scale_input, b.moe_expert) == (
        _cabi.B2_FF_MOE, 16, 7, 3, _cabi.B2_ROUTE_SIGMOID, 1, _cabi.B2_EXPERT_SILU)
    assert (c.kv_from, c.n_ff) == (2, 0) and e.rope_factor == 0.0
    s = fazovik.tensor_shapes(cfg)
    assert s["bigram"] == (11, 72) and "head" not in s and s["final.norm.b"] == (72,)
    assert s["l0.mix.dkv"] == (27, 72) and s["l0.mix.g"] == (5, 72) and s["l0.mix.uq"] == (80, 33) and s["l0.mix.o"] == (72, 70)
    assert s["l1.mix.dkv"] == (19, 72) and s["l1.mix.uv"] == (22, 19) and "l1.mix.g" not in s and s["l1.mlp.router"] == (7, 72)
    assert "l2.mix.dkv" not in s and "l2.mix.dkv.norm" not in s and s["l2.mix.uk"] == (72, 19) and "l2.norm2" not in s
    bare = fu.config([fu.plain()], hashed=None)
    assert fazovik.read_dims(bare).bigram == (0, 0, 0) and "bigram" not in fazovik.tensor_shapes(bare)


def test_registry_and_folder(tmp_path):
    from llama_cpp import fazovik, models
    cfg = fu.config([fu.rotated(mlp=fu.moe())])
    path = fu.write_model(str(tmp_path / "m"), cfg, fu.random_weights(cfg))
    assert models.open_model(path).family.name == "Fazovik" and "Fazovik" in models.architectures()
    bad = [fu.config([dict(fu.plain(), type="nope")]), fu.config([fu.plain(kv_from=0)]), fu.config([fu.plain(), fu.plain(kv_from=0, rank=30)]),
           fu.config([fu.plain(), fu.plain(kv_from=0), fu.plain(kv_from=1)]), fu.config([fu.plain(mlp={"kind": "other", "ff": 4})]),
           fu.config([fu.plain()], hashed=fu.bigram(0))]
    for b in bad:
        with pytest.raises(ValueError):
            fazovik.read_dims(b)


def test_bigram_rows():
    assert list(ref.bigram_rows([4, 9, 2], 10, 3, 5)) == [10, (12 + 45) % 10, (27 + 10) % 10]
    w = f64(fu.random_weights(fu.config([fu.plain()])))
    x = ref.embed(w, [7, 7], fu.bigram())
    assert np.allclose(x[0] - w["embed"][7], w["bigram"][53]) and np.allclose(x[1] - w["embed"][7], w["bigram"][(7 * 22) % 53])


def test_rotation_depends_on_distance_only_and_scales():
    rot = {"base": 500.0, "dims": 8, "scaling": fu.scaling(4.0, 64, 4.0, 1.0)}
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 10)), rng.standard_normal((1, 10))
    at = lambda v, p: ref.rotate_pairs(v, [p], rot)[0]
    near, far = at(q, 9)[:8] @ at(k, 4)[:8], at(q, 105)[:8] @ at(k, 100)[:8]
    assert abs(near - far) < 1e-10
    mag = 0.1 * math.log(4.0) + 1.0
    assert np.allclose(at(q, 0)[:8], q[0, :8] * mag) and np.array_equal(at(q, 77)[8:], q[0, 8:])
    f, _ = ref.rotation_frequencies(rot)
    plain, one = ref.rotation_frequencies({"base": 500.0, "dims": 8})
    assert one == 1.0 and f[0] == plain[0] and abs(f[3] - plain[3] / 4.0) < 1e-15 and (f <= plain).all()
    assert np.allclose(at(np.eye(1, 10), 1)[:2], [math.cos(1.0) * mag, math.sin(1.0) * mag])      # pair (0, 1), frequency 1


def test_shared_latent():
    """A layer with kv_from uses the other layer's latent through its own maps: with equal maps and inputs it returns the same."""
    cfg = fu.config([fu.plain(), fu.plain(kv_from=0)])
    w = f64(fu.random_weights(cfg, seed=2))
    h = np.random.default_rng(3).standard_normal((9, 72))
    lat = {}
    a = ref.plain_latent_attention(h, w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5, lat, 0)
    for leaf in ("dq", "dq.norm", "uq", "uk", "uv", "o"):
        w["l1.mix." + leaf] = w["l0.mix." + leaf]
    assert np.allclose(ref.plain_latent_attention(h, w, "l1.mix.", cfg["layers"][1]["mixer"], 1e-5, lat, 1), a)
    assert sorted(lat) == [0]


def test_scores_scale_the_experts_input():
    mlp = fu.moe(experts=4, top=1, ff=8)
    cfg = fu.config([fu.plain(mlp=mlp)])
    w = f64(fu.random_weights(cfg, seed=4))
    h = np.random.default_rng(5).standard_normal((6, 72))
    chosen, score = ref.route(h, w, "l0.mlp.", mlp["router"])
    y = ref.mixture(h, w, "l0.mlp.", mlp)
    e, s = chosen[2, 0], score[2, 0]
    p = f"l0.mlp.e{e}."
    assert np.allclose(y[2], w[p + "down"] @ (ref.silu(s * (w[p + "gate"] @ h[2])) * (s * (w[p + "up"] @ h[2]))))
    assert not np.allclose(y[2], s * ref.gated_unit(h[2:3], w, p, ref.silu)[0], rtol=0.05)
    assert (np.diff(np.sort(ref.sigmoid(h @ w["l0.mlp.router"].T), -1)) >= 0).all() and (score < 1).all() and (score > 0).all()


def test_gelu_and_layer_norm_by_hand():
    z = np.array([-2.0, 0.0, 0.5])
    want = [0.5 * v * (1 + math.tanh(math.sqrt(2 / math.pi) * (v + 0.044715 * v ** 3))) for v in z]
    assert np.allclose(ref.gelu_tanh(z), want)
    y = ref.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 5.0]), np.array([0.1, 0.2]), 0.0)
    assert np.allclose(y, [[-2.0 + 0.1, 5.0 + 0.2]])


def test_oracle_is_causal_and_parallel():
    cfg = fu.config([fu.rotated(mlp=fu.moe()), fu.plain(mlp=fu.dense()), fu.plain(kv_from=1, heads=2)])
    w = fu.random_weights(cfg, seed=4)
    toks = [int(t) for t in np.random.default_rng(5).integers(0, cfg["vocab"], size=30)]
    full = ref.forward(cfg, w, toks)
    assert np.allclose(ref.forward(cfg, w, toks[:17]), full[:17], atol=1e-10)
    # without mixers a layer is x + ff(norm2(x)) of the SAME x: two branches of one layer are not two sublayers
    one = copy.deepcopy(cfg)
    one["layers"] = one["layers"][:1]
    x = ref.embed(f64(w), toks, fu.bigram())
    wd = f64(w)
    a = ref.rotated_latent_attention(ref.layer_norm(x, wd["l0.norm1"], wd["l0.norm1.b"], 1e-5), wd, "l0.mix.", one["layers"][0]["mixer"], 1e-5, {}, 0)
    b = ref.mixture(ref.layer_norm(x, wd["l0.norm2"], wd["l0.norm2.b"], 1e-5), wd, "l0.mlp.", one["layers"][0]["mlp"])
    assert np.allclose(ref.forward(one, w, toks, return_layers=True)[1][0], x + a + b)


def test_synthetic_patterns():
    from llama_cpp import fazovik
    cfg, tensors = fazovik.synthetic(64, 2, 16, 50, pattern="rdpsr", experts=3, top=2, rank=32, q_rank=24)
    kinds = [(L["type"], L["mlp"]["kind"], L["mixer"].get("kv_from")) for L in cfg["layers"]]
    assert kinds == [("latent_attention", "dense", None), ("latent_attention_2", "moe", None), ("latent_attention_2", "moe", 1),
                     ("latent_attention", "moe", None)]
    assert {n: tuple(t.shape) for n, t in tensors.items()} == fazovik.tensor_shapes(cfg)
