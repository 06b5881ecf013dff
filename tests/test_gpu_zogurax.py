"""Zogurax through the native engine against the float64 oracle (oracle/zogurax_ref.py), on small random models the tests
make themselves: each kind of layer alone, every mechanism shown to matter, prompt against token-by-token decoding, portions down
to two tokens, unequal batches against each request alone, slots, convolution states and pages used again, marked keys far away
and at page and portion borders, the first tokens, long decoding over many steps of the query temperature, degenerate and odd
sizes, and greedy generation through `Llama` and the scheduler."""
import copy
import threading

import numpy as np
import pytest

import zogurax_util as zu
from oracle import zogurax_ref as ref

pytestmark = pytest.mark.gpu

TOL = {"float32": 3e-5, "bfloat16": 5e-2}


def open_engine(path, dtype="float32", n_ctx=512, max_seqs=4, kv_tokens=None, max_step_tokens=None, flags=0):
    from llama_cpp import models
    return models.open_engine(models.open_model(path), n_ctx=n_ctx, max_seqs=max_seqs, dtype=dtype, kv_tokens=kv_tokens,
                              max_step_tokens=max_step_tokens, flags=flags)


def run_cut(eng, seqs, key, tokens, cuts):
    """All logits of `tokens`, fed in portions of the given sizes (cycled)."""
    rows, pos, k = [], 0, 0
    seqs.open(key)
    while pos < len(tokens):
        n = min(cuts[k % len(cuts)], len(tokens) - pos)
        k += 1
        slot = seqs.extend(key, n)
        lg, _ = eng.step([(slot, tokens[pos:pos + n])], want=[list(range(n))])
        rows.append(lg)
        pos += n
    seqs.close(key)
    return np.concatenate(rows)


def row_errors(got, want):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt(((want - want.mean(-1, keepdims=True)) ** 2).mean())


def close(got, want, dtype):
    """Every row within the tolerance (the experts of a token do not depend on rounding, so bfloat16 has no row to excuse), the
    typical bfloat16 row well inside."""
    rows = row_errors(got, want)
    return rows.max() < TOL[dtype] and (dtype == "float32" or np.median(rows) < TOL[dtype] / 3)


def tokens_for(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], size=n)]


@pytest.fixture(scope="module")
def model(native_lib, tmp_path_factory):
    """All mechanisms in one model: both mixers inside and outside a loop that starts after the first layer, with and without a
    feed-forward block and a shared expert."""
    cfg = zu.config([zu.biased(mlp=zu.moe()), zu.conved(mlp=zu.moe(experts=9, top=3, ff=16, shared=24), heads=4, kv_heads=1, dim=16, vdim=24, conv=4),
                     zu.biased(mlp=None, heads=2, kv_heads=2, dim=24, vdim=8, every=5), zu.conved(mlp=zu.moe(experts=4, top=1, shared=None))],
                    loop=(1, 3, 2))
    w = zu.random_weights(cfg, seed=3)
    path = zu.write_model(str(tmp_path_factory.mktemp("zogurax_model")), cfg, w)
    return cfg, w, path


LAYERS = {
    "conved": lambda: ([zu.conved()], None),
    "conved_moe": lambda: ([zu.conved(mlp=zu.moe(experts=10, top=4, ff=20, shared=33), heads=6, kv_heads=3, dim=16, vdim=32, conv=4)], None),
    "conved_two_taps": lambda: ([zu.conved(mlp=zu.moe(shared=None), heads=2, kv_heads=1, dim=40, vdim=24, conv=2)], None),
    "conved_one_tap": lambda: ([zu.conved(heads=3, kv_heads=3, dim=12, vdim=20, conv=1)], None),
    "conved_seven_taps": lambda: ([zu.conved(mlp=zu.moe(), heads=2, kv_heads=2, dim=32, vdim=16, conv=7)], None),
    "biased": lambda: ([zu.biased()], None),
    "biased_moe": lambda: ([zu.biased(mlp=zu.moe(experts=5, top=5, ff=32, shared=40), heads=8, kv_heads=2, dim=64, vdim=32)], None),
    "biased_one_choice": lambda: ([zu.biased(mlp=zu.moe(experts=5, top=1, ff=17, shared=None), heads=3, kv_heads=1, dim=9, vdim=7)], None),
    "one_pass": lambda: ([zu.biased(mlp=zu.moe())], (0, 1, 1)),
    "passes": lambda: ([zu.conved(mlp=zu.moe())], (0, 1, 3)),
    "passes_in_the_middle": lambda: ([zu.biased(), zu.conved(), zu.biased(mlp=zu.moe()), zu.conved()], (1, 3, 2)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", sorted(LAYERS))
def test_each_kind_of_layer_alone(native_lib, tmp_path, layer, dtype):
    from llama_cpp.kv_pages import SequenceSlots
    layers, loop = LAYERS[layer]()
    cfg = zu.config(layers, loop=loop)
    w = zu.random_weights(cfg, seed=11)
    eng = open_engine(zu.write_model(str(tmp_path / "m"), cfg, w), dtype)
    toks = tokens_for(cfg, 90, 1)
    want_logits, want_layers = ref.forward(cfg, w, toks, return_layers=True)
    seqs = SequenceSlots(eng)
    eng.trace_layers(True)
    seqs.open("a")
    slot = seqs.extend("a", len(toks))
    got, _ = eng.step([(slot, toks)], want=[list(range(len(toks)))])
    layers = eng.layer_outputs(len(toks))
    seqs.close("a")
    eng.trace_layers(False)
    single = run_cut(eng, seqs, "s", toks, [1])
    eng.close()
    assert layers.shape == want_layers.shape
    for have, want in zip(layers, want_layers):
        assert close(have, want, dtype)
    assert close(got, want_logits, dtype)
    assert close(single, want_logits, dtype)


def test_mechanisms_are_not_trivial(model):
    """Leaving out or changing any one mechanism of the test model moves the logits by far more than the tolerances."""
    cfg, w, _ = model
    toks = tokens_for(cfg, 120, 2)
    want = ref.forward(cfg, w, toks)

    def moved(c=cfg, weights=w):
        return float(np.median(row_errors(ref.forward(c, weights, toks), want)[10:]))

    def changed(f, *ends):
        return {k: (f(v) if k.endswith(ends) else v) for k, v in w.items()}

    assert moved(weights=changed(np.zeros_like, ".q.b", ".k.b", ".v.b")) > 0.1
    assert moved(weights=changed(np.zeros_like, ".o.b")) > 0.1
    assert moved(weights=changed(np.zeros_like, "mix.g")) > 0.05
    assert moved(weights=changed(np.zeros_like, "shared.sg")) > 0.02
    assert moved(weights=changed(np.ones_like, "q.norm", "k.norm")) > 0.02
    assert moved(weights=changed(np.zeros_like, "loop.step")) > 0.1
    assert moved(weights=changed(lambda v: v[::-1], "loop.step")) > 0.1
    assert moved(weights=changed(lambda v: np.concatenate([v[:, :72], 0 * v[:, 72:]], 1), "loop.in")) > 0.1
    assert moved(weights=changed(lambda v: np.concatenate([v[:, 72:], v[:, :72]], 1), "loop.in")) > 0.1
    assert moved(weights=changed(lambda v: np.roll(v, 1, axis=0), "mlp.table")) > 0.1
    for leaf in ("q.conv", "k.conv", "v.conv"):
        assert moved(weights=changed(lambda v: np.concatenate([0 * v[:, :-1], v[:, -1:]], 1), leaf)) > 0.02

    def other(**kw):
        c = copy.deepcopy(cfg)
        for L in c["layers"]:
            for k, v in kw.items():
                L["mixer"][k] = v
        return c

    assert moved(other(softcap=1e6)) > 0.02
    assert moved(other(q_temp={"coef": 0.0, "every": 9})) > 0.02
    assert moved(other(q_temp={"coef": 0.5, "every": 11})) > 0.01


def test_one_in_the_denominator_matters(native_lib, tmp_path):
    """The first tokens of a biased layer: with one visible key its weight is far from one."""
    cfg = zu.config([zu.biased()])
    w = zu.random_weights(cfg, seed=12)
    toks = tokens_for(cfg, 5, 3)
    wd = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    h = ref.layer_norm(ref.embed(wd, toks), wd["l0.norm1"], 1e-5)
    k = (h @ wd["l0.mix.k"].T + wd["l0.mix.k.b"]).reshape(5, 3, 18)
    q = (h @ wd["l0.mix.q"].T + wd["l0.mix.q.b"]).reshape(5, 6, 18)
    s = ref.cap(q[0, 0] @ k[0, 0] * cfg["layers"][0]["mixer"]["scale"], 6.0)
    assert abs(1 - np.exp(s) / (1 + np.exp(s))) > 0.02
    eng = open_engine(zu.write_model(str(tmp_path / "m"), cfg, w), "float32")
    from llama_cpp.kv_pages import SequenceSlots
    assert close(run_cut(eng, SequenceSlots(eng), "a", toks, [1]), ref.forward(cfg, w, toks), "float32")
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_against_token_by_token(model, dtype):
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    eng = open_engine(path, dtype)
    seqs = SequenceSlots(eng)
    toks = tokens_for(cfg, 150, 2)
    want = ref.forward(cfg, w, toks)
    whole = run_cut(eng, seqs, "w", toks, [len(toks)])
    single = run_cut(eng, seqs, "s", toks, [1])
    eng.close()
    assert close(whole, want, dtype)
    assert close(single, want, dtype)
    assert close(single, whole, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cuts", [[2], [3, 2, 5, 1], [17, 64, 2, 9], [63, 1, 1, 70]])
def test_portions(model, cuts, dtype):
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    eng = open_engine(path, dtype)
    toks = tokens_for(cfg, 140, 4)
    got = run_cut(eng, SequenceSlots(eng), "p", toks, cuts)
    eng.close()
    assert close(got, ref.forward(cfg, w, toks), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone(model, dtype):
    """Three requests of different lengths advance together, portions of some beside single tokens of others."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    eng = open_engine(path, dtype)
    seqs = SequenceSlots(eng)
    reqs = {"a": tokens_for(cfg, 131, 5), "b": tokens_for(cfg, 40, 6), "c": tokens_for(cfg, 77, 7)}
    alone = {k: run_cut(eng, seqs, k + "_alone", t, [len(t)]) for k, t in reqs.items()}
    plan = {"a": [50, 1, 1, 30, 2, 1], "b": [1, 1, 9, 1], "c": [2, 40, 1, 1, 20]}
    at, turn, got = {k: 0 for k in reqs}, {k: 0 for k in reqs}, {k: [] for k in reqs}
    for k in reqs:
        seqs.open(k)
    while any(at[k] < len(reqs[k]) for k in reqs):
        entries, want, who = [], [], []
        for k, t in reqs.items():
            if at[k] >= len(t):
                continue
            n = min(plan[k][turn[k] % len(plan[k])], len(t) - at[k])
            turn[k] += 1
            entries.append((seqs.extend(k, n), t[at[k]:at[k] + n]))
            want.append(list(range(n)))
            who.append((k, n))
            at[k] += n
        lg, _ = eng.step(entries, want=want)
        r = 0
        for k, n in who:
            got[k].append(lg[r:r + n])
            r += n
    eng.close()
    for k, t in reqs.items():
        mixed = np.concatenate(got[k])
        assert row_errors(mixed, alone[k]).max() < 2e-5 if dtype == "float32" else close(mixed, alone[k], dtype)
        assert close(mixed, ref.forward(cfg, w, t), dtype)


def test_slots_and_pages_used_again(model):
    """One slot, a pool of three pages: every sequence runs in the pages and over the convolution states the previous one left."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    eng = open_engine(path, "float32", n_ctx=192, max_seqs=1, kv_tokens=192)
    seqs = SequenceSlots(eng)
    for i, n in enumerate([150, 70, 192, 3, 1]):
        toks = tokens_for(cfg, n, 20 + i)
        got = run_cut(eng, seqs, f"s{i}", toks, [1, 40, 2, 23] if i % 2 else [40, 1, 23])
        assert seqs.free_slots == 1 and eng.pages.free_pages == 3
        assert close(got, ref.forward(cfg, w, toks), "float32"), i
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_convolution_state_across_cuts_and_idle_steps(native_lib, tmp_path, dtype):
    """The last inputs of a convolution span portions, single tokens, steps in which other requests run in between, and portions
    shorter than the convolution; nine requests in a step take the prompt path, fewer the one for few tokens."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = zu.config([zu.conved(mlp=zu.moe(), conv=5), zu.conved(conv=4, dim=16, vdim=16)], loop=(0, 2, 2))
    w = zu.random_weights(cfg, seed=9)
    eng = open_engine(zu.write_model(str(tmp_path / "m"), cfg, w), dtype, max_seqs=10)
    seqs = SequenceSlots(eng)
    reqs = {k: tokens_for(cfg, 40, i) for i, k in enumerate("abcdefghi")}
    got, at = {k: [] for k in reqs}, {k: 0 for k in reqs}
    for k in reqs:
        seqs.open(k)
    plan = [{"a": 2}, {"b": 1}, {"b": 1, "a": 1}, {"c": 3}, {"a": 1, "c": 1}, {k: 1 for k in reqs}, {k: 2 for k in reqs}, {"b": 30}, {"a": 3, "b": 1, "d": 4},
            {k: 1 for k in "bcdefghi"}]
    while True:
        step = plan.pop(0) if plan else {k: 9 for k in reqs}
        step = {k: min(n, 40 - at[k]) for k, n in step.items() if at[k] < 40}
        if not step:
            break
        lg, _ = eng.step([(seqs.extend(k, n), reqs[k][at[k]:at[k] + n]) for k, n in step.items()], want=[list(range(n)) for n in step.values()])
        r = 0
        for k, n in step.items():
            got[k].append(lg[r:r + n])
            r += n
            at[k] += n
    eng.close()
    for k, t in reqs.items():
        assert close(np.concatenate(got[k]), ref.forward(cfg, w, t), dtype), k


PROBE, MARK = 5, 7


def _peaky_model(tmp_path, kind):
    """Attention in which the token PROBE looks for the token MARK: queries are a map of the first half of the stream, keys the
    same map of the second half, and the two embedding rows hold one vector in those halves, so MARK's key is parallel to
    PROBE's query wherever it stands. The rows are large against the position's sinusoid. The marked key holds most of the weight."""
    d, H, G, W = 32, 4, 2, 64
    size = dict(heads=H, kv_heads=G, dim=d, vdim=24, softcap=20.0, coef=0.02, every=64)
    layer = zu.conved(scale=0.42, conv=4, **size) if kind == "conved" else zu.biased(scale=0.42, **size)
    cfg = zu.config([layer], width=W)
    w = zu.random_weights(cfg, seed=5)
    rng = np.random.default_rng(6)
    w["embed"] = zu.bf16_round(6.0 * w["embed"])
    A = rng.standard_normal((d, W // 2)) / np.sqrt(W // 2)
    vec = 6.0 * rng.standard_normal(W // 2)
    w["embed"][PROBE, :W // 2] = w["embed"][MARK, W // 2:] = zu.bf16_round(vec - vec.mean())
    p = "l0."
    w[p + "norm1"] = np.ones(W, dtype=np.float32)
    w[p + "mix.q"] = zu.bf16_round(np.tile(np.concatenate([A, 0 * A], 1), (H, 1)))
    w[p + "mix.k"] = zu.bf16_round(np.tile(np.concatenate([0 * A, A], 1), (G, 1)))
    for n in "qk":
        if kind == "conved":
            w[p + f"mix.{n}.norm"] = np.ones_like(w[p + f"mix.{n}.norm"])
            taps = np.zeros_like(w[p + f"mix.{n}.conv"])
            taps[:, -1], taps[:, 0] = 1.0, 0.03125
            w[p + f"mix.{n}.conv"] = taps
        else:
            w[p + f"mix.{n}.b"] = zu.bf16_round(0.02 * w[p + f"mix.{n}.b"])
    w[p + "mix.o"] = zu.bf16_round(30.0 * w[p + "mix.o"])            # the mixer's output stands out in the stream
    return cfg, w, zu.write_model(str(tmp_path / "peaky"), cfg, w)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("kind", ["conved", "biased"])
def test_far_keys_and_page_borders(native_lib, tmp_path, kind, decode, dtype):
    """The marked token is the sequence's first, at a page border (a page's last / first place), a portion's last / first, at the
    border of a key range of the few-token kernel, or the one just before the probing position; a key that is lost or counted twice
    changes the probe's logits by far more than the tolerance."""
    from llama_cpp.kv_pages import SequenceSlots
    n = 450
    cfg, w, path = _peaky_model(tmp_path, kind)
    eng = open_engine(path, dtype)
    tol = TOL["float32"] if dtype == "float32" else 0.03
    seqs = SequenceSlots(eng)
    base = [int(t) for t in np.random.default_rng(9).integers(8, cfg["vocab"], size=n)]
    probe = n - 1
    without = list(base)
    without[probe] = PROBE
    lost = ref.forward(cfg, w, without)[probe]
    for at in (0, 1, 63, 64, 127, 128, 199, 200, 255, 256, 319, 320, 383, 384, 447, 448, probe - 1):
        toks = list(without)
        toks[at] = MARK
        true = ref.forward(cfg, w, toks)[probe]
        assert row_errors(lost[None], true[None])[0] > 0.3, "the test model does not show the marked key"
        key = f"k{at}"
        seqs.open(key)
        if decode:
            eng.step([(seqs.extend(key, 200), toks[:200])])
            eng.step([(seqs.extend(key, probe - 4 - 200), toks[200:probe - 4])])
            for t in range(probe - 4, probe):
                eng.step([(seqs.extend(key, 1), [toks[t]])])
            got, _ = eng.step([(seqs.extend(key, 1), [toks[probe]])], want=[[0]])
        else:
            eng.step([(seqs.extend(key, 200), toks[:200])])
            got, _ = eng.step([(seqs.extend(key, n - 200), toks[200:])], want=[[probe - 200]])
        seqs.close(key)
        err = row_errors(got, true[None])[0]
        assert err < tol, (at, err)
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_few_token_ranges(native_lib, tmp_path, dtype):
    """The few-token kernel cuts the visible keys into eight ranges when the context is long: decoding at lengths around every
    count of keys per range, from a context that starts with fewer keys than ranges, for the three lane layouts."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = zu.config([zu.conved(heads=2, kv_heads=1, dim=16, vdim=64), zu.biased(heads=4, kv_heads=2, dim=128, vdim=40),
                     zu.conved(heads=2, kv_heads=2, dim=72, vdim=200, conv=4), zu.biased(heads=1, kv_heads=1, dim=256, vdim=8)])
    w = zu.random_weights(cfg, seed=15)
    eng = open_engine(zu.write_model(str(tmp_path / "m"), cfg, w), dtype, n_ctx=640)
    seqs = SequenceSlots(eng)
    toks = tokens_for(cfg, 600, 16)
    want = ref.forward(cfg, w, toks)
    got = run_cut(eng, seqs, "s", toks, [1] * 40 + [86, 1, 1, 1, 1] + [123, 2, 1, 1, 1, 3] * 10)
    eng.close()
    assert close(got, want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kv_heads", [1, 4, 19])
def test_prompt_tiles(native_lib, tmp_path, kv_heads, dtype):
    """Sizes the tensor-core kernels take (key and value sizes up to and above 64, up to 38 heads, enough (token, expert) pairs for
    128-row expert tiles); a 300-token prompt at once and in portions that straddle the tiles, and decoded tokens."""
    from llama_cpp.kv_pages import SequenceSlots
    mlp = zu.moe(experts=6, top=4, ff=16, shared=24)
    cfg = zu.config([zu.conved(mlp=mlp, heads=2 * kv_heads, kv_heads=kv_heads, dim=16, vdim=48, conv=3),
                     zu.biased(mlp=mlp, heads=kv_heads, kv_heads=kv_heads, dim=80, vdim=16),
                     zu.biased(mlp=None, heads=kv_heads, kv_heads=kv_heads, dim=64, vdim=112),
                     zu.conved(mlp=zu.moe(experts=3, top=2, ff=8, shared=None), heads=2 * kv_heads, kv_heads=kv_heads, dim=128, vdim=128, conv=4)],
                    width=64, loop=(1, 3, 2))
    w = zu.random_weights(cfg, seed=13)
    eng = open_engine(zu.write_model(str(tmp_path / "m"), cfg, w), dtype)
    toks = tokens_for(cfg, 300, 14)
    want = ref.forward(cfg, w, toks)
    seqs = SequenceSlots(eng)
    whole = run_cut(eng, seqs, "w", toks, [300])
    parts = run_cut(eng, seqs, "p", toks, [100, 7, 64, 100] + [1] * 29)
    eng.close()
    assert close(whole, want, dtype)
    assert close(parts, want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_of_another_size(model, dtype):
    """Pages that do not hold whole 64-key blocks, so that a block of the prompt kernel spans several pages."""
    from llama_cpp import models
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    for block in (16, 48):
        eng = models.open_engine(models.open_model(path), n_ctx=384, max_seqs=2, dtype=dtype, kv_block_tokens=block)
        toks = tokens_for(cfg, 200, 17)
        got = run_cut(eng, SequenceSlots(eng), "a", toks, [150, 1, 2, 30])
        eng.close()
        assert close(got, ref.forward(cfg, w, toks), dtype), block


def test_steps_larger_than_the_engine_takes_at_once(model):
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    eng = open_engine(path, "float32", max_step_tokens=16)
    seqs = SequenceSlots(eng)
    reqs = {"a": tokens_for(cfg, 50, 70), "b": tokens_for(cfg, 3, 71), "c": tokens_for(cfg, 37, 72)}
    for k in reqs:
        seqs.open(k)
    entries = [(seqs.extend(k, len(t)), t) for k, t in reqs.items()]
    want = [[0, 17, 49], [2], list(range(37))]
    got, _ = eng.step(entries, want=want)
    eng.close()
    expect = np.concatenate([ref.forward(cfg, w, t)[wi] for t, wi in zip(reqs.values(), want)])
    assert got.shape == expect.shape and close(got, expect, "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replayed_steps_equal_direct_launches(model, dtype):
    """Repeating small steps are replayed as CUDA graphs; the logits are bit-identical to launching the kernels directly."""
    from llama_cpp import _cabi
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    toks = {"a": tokens_for(cfg, 40, 80), "b": tokens_for(cfg, 30, 81)}
    outs = []
    for flags in (0, _cabi.B2_FLAG_NO_GRAPH):
        eng = open_engine(path, dtype, n_ctx=256, max_seqs=2, flags=flags)
        seqs = SequenceSlots(eng)
        rows = []
        for k, t in toks.items():
            seqs.open(k)
            eng.step([(seqs.extend(k, 5), t[:5])])
        for i in range(5, 30):
            lg, _ = eng.step([(seqs.extend(k, 1), [t[i]]) for k, t in toks.items()], want=[[0], [0]])
            rows.append(lg)
        eng.close()
        outs.append(np.concatenate(rows))
    assert np.array_equal(outs[0], outs[1])
    full = {k: ref.forward(cfg, w, t) for k, t in toks.items()}
    want = np.concatenate([np.stack([f[i] for f in full.values()]) for i in range(5, 30)])
    assert close(outs[0], want, dtype)


def test_first_tokens(model):
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    eng = open_engine(path, "float32")
    seqs = SequenceSlots(eng)
    for n in (1, 2, 3, 5):
        toks = tokens_for(cfg, n, 30 + n)
        want = ref.forward(cfg, w, toks)
        assert close(run_cut(eng, seqs, f"w{n}", toks, [n]), want, "float32")
        assert close(run_cut(eng, seqs, f"s{n}", toks, [1]), want, "float32")
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(model, dtype):
    """A short prompt and 300 single-token steps: over many steps of the query temperature and over page borders."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    eng = open_engine(path, dtype)
    toks = tokens_for(cfg, 310, 40)
    got = run_cut(eng, SequenceSlots(eng), "d", toks, [10] + [1] * 300)
    eng.close()
    assert close(got, ref.forward(cfg, w, toks), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_positions(native_lib, tmp_path, dtype):
    """Positions in the thousands: the sinusoid's fast entries have turned many times, the temperature grows slowly."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = zu.config([zu.biased(heads=1, kv_heads=1, dim=8, vdim=8, every=500), zu.conved(heads=1, kv_heads=1, dim=8, vdim=8, every=700)], width=24, vocab=40)
    w = zu.random_weights(cfg, seed=19)
    eng = open_engine(zu.write_model(str(tmp_path / "m"), cfg, w), dtype, n_ctx=2600)
    toks = tokens_for(cfg, 2500, 18)
    got = run_cut(eng, SequenceSlots(eng), "a", toks, [1000, 900, 590, 1])
    eng.close()
    assert close(got, ref.forward(cfg, w, toks), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_are_one_odd_or_large(native_lib, tmp_path, dtype):
    """One head, expert, choice, tap, pass; keys and values of one entry or 256; all experts chosen; odd sizes that no vector path
    takes; expert and shared widths of one; sixteen taps; heads whose queries are normed together and do not fill a warp."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = zu.config([
        zu.conved(mlp=zu.moe(experts=1, top=1, ff=8, shared=1), heads=1, kv_heads=1, dim=8, vdim=1, conv=1, coef=0.0, every=1),
        zu.biased(mlp=zu.moe(experts=5, top=5, ff=1, shared=9), heads=1, kv_heads=1, dim=1, vdim=1, scale=1.0, softcap=0.5),
        zu.conved(mlp=zu.moe(experts=3, top=2, ff=7, shared=11), heads=6, kv_heads=3, dim=7, vdim=5, conv=16, every=1),
        zu.biased(mlp=None, heads=5, kv_heads=5, dim=13, vdim=19, softcap=80.0, every=1000),
        zu.conved(mlp=zu.moe(experts=33, top=5, ff=11, shared=None), heads=33, kv_heads=11, dim=3, vdim=2, conv=2),
        zu.biased(mlp=zu.moe(experts=2, top=1, ff=130, shared=130), heads=2, kv_heads=1, dim=256, vdim=256),
    ], width=40, vocab=50, eps=1e-3, loop=(2, 5, 1))
    w = zu.random_weights(cfg, seed=8)
    eng = open_engine(zu.write_model(str(tmp_path / "m"), cfg, w), dtype)
    toks = tokens_for(cfg, 100, 3)
    got = run_cut(eng, SequenceSlots(eng), "x", toks, [5, 1, 2, 30])
    eng.close()
    assert close(got, ref.forward(cfg, w, toks), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [45, 50])
def test_widths_no_vector_path_takes(native_lib, tmp_path, width, dtype):
    """A model width that is odd (the last sine of the position has no cosine), or even but no multiple of four: every product over
    the width takes its scalar path."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = zu.config([zu.conved(mlp=zu.moe(ff=10)), zu.biased(mlp=zu.moe(ff=7, shared=13))], width=width, vocab=77, loop=(0, 2, 2))
    w = zu.random_weights(cfg, seed=21)
    eng = open_engine(zu.write_model(str(tmp_path / "m"), cfg, w), dtype)
    toks = tokens_for(cfg, 150, 22)
    got = run_cut(eng, SequenceSlots(eng), "x", toks, [70, 1, 3, 20, 1])
    eng.close()
    assert close(got, ref.forward(cfg, w, toks), dtype)


def random_config(seed):
    """A random model: layer count and order, loop, every size and constant drawn anew (sizes of the scale small real models have)."""
    rng = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(rng.integers(0, len(xs)))]

    def ff():
        if rng.random() < 0.2:
            return None
        experts = pick(2, 5, 8, 12, 24)
        return zu.moe(experts=experts, top=int(rng.integers(1, min(experts, 4) + 1)), ff=pick(8, 24, 56, 72), shared=pick(None, 16, 40, 96, 100))

    layers = []
    for _ in range(int(rng.integers(2, 6))):
        G = pick(1, 2, 3, 4)
        size = dict(heads=G * pick(1, 2, 3, 4), kv_heads=G, dim=pick(16, 24, 32, 48, 64, 96), vdim=pick(16, 24, 32, 48, 64, 100),
                    softcap=pick(2.0, 10.0, 30.0, 50.0), coef=pick(0.1, 0.5, 1.0), every=pick(16, 50, 64, 128))
        layers.append(zu.conved(mlp=ff(), conv=pick(2, 3, 4, 5), **size) if rng.random() < 0.5 else zu.biased(mlp=ff(), **size))
    start = int(rng.integers(0, len(layers)))
    loop = (start, int(rng.integers(start + 1, len(layers) + 1)), pick(1, 2, 3))
    return zu.config(layers, width=pick(64, 96, 128, 200, 320), vocab=pick(97, 256, 500), eps=pick(1e-5, 1e-6), loop=None if rng.random() < 0.15 else loop)


@pytest.mark.parametrize("seed", range(10))
def test_random_configurations(native_lib, tmp_path, seed):
    """Ten models nobody chose: each runs a 330-token prompt at once and in uneven portions with decoded tokens at the end,
    in both modes, from a pool that forces page reuse."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = random_config(100 + seed)
    w = zu.random_weights(cfg, seed=seed)
    path = zu.write_model(str(tmp_path / "m"), cfg, w)
    toks = tokens_for(cfg, 330, seed)
    want = ref.forward(cfg, w, toks)
    for dtype in ("float32", "bfloat16"):
        eng = open_engine(path, dtype, n_ctx=384, max_seqs=2, kv_tokens=384 + 128)
        seqs = SequenceSlots(eng)
        whole = run_cut(eng, seqs, "w", toks, [330])
        parts = run_cut(eng, seqs, "p", toks, [61, 3, 128, 2, 70, 37] + [1] * 29)
        eng.close()
        assert close(whole, want, dtype), (seed, dtype, "whole")
        assert close(parts, want, dtype), (seed, dtype, "parts")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(model, tmp_path, dtype):
    """`bin/trace_run` as a user starts it: six requests, at most four live, portions of some beside single tokens of others, a
    request that sits out steps, a pool of --max-tokens sized for the live ones only, so pages and slots are used again; every
    written row against the oracle."""
    import json
    import os
    import subprocess
    import sys
    cfg, w, path = model
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    reqs = {f"r{i}": tokens_for(cfg, n, 90 + i) for i, n in enumerate([130, 7, 64, 201, 33, 90])}
    plans = {"r0": [64, 2, 1, 1, 40, 1], "r1": [1, 1], "r2": [3, 61], "r3": [100, 1, 1, 64, 2], "r4": [33], "r5": [2, 1, 50, 1]}
    order, live, at, turn, steps, wanted = list(reqs), [], {k: 0 for k in reqs}, {k: 0 for k in reqs}, [], []
    most = 0
    while order or live:
        while order and len(live) < 4:
            live.append(order.pop(0))
        entries, end = [], []
        for k in list(live):
            if k == "r3" and len(steps) % 3 == 1:          # sits this step out
                continue
            n = min(plans[k][turn[k] % len(plans[k])], len(reqs[k]) - at[k])
            turn[k] += 1
            want = sorted({0, n - 1})
            entries.append({"id": k, "tokens": reqs[k][at[k]:at[k] + n], "want": want})
            wanted.append((len(steps), k, [at[k] + x for x in want]))
            at[k] += n
        most = max(most, sum((at[k] + 63) // 64 * 64 for k in live))
        for k in list(live):
            if at[k] == len(reqs[k]):
                end.append(k)
                live.remove(k)
        steps.append({"step": len(steps), "entries": entries, "end": end})
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out),
                        "--max-tokens", str(most)], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [ln for ln in p.stdout.split("\n") if ln.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    refs = {k: ref.forward(cfg, w, t) for k, t in reqs.items()}
    got, expect = [], []
    for i in range(len(steps)):
        rows = [(k, pos) for st, k, ps in wanted if st == i for pos in ps]
        got.append(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"]))
        expect.append(np.stack([refs[k][pos] for k, pos in rows]))
    assert close(np.concatenate(got), np.concatenate(expect), dtype)


def test_greedy_generation_through_llama_and_the_scheduler(model):
    """`Llama(model_path=<folder>)`: three callers at once, prompts of different lengths, greedy. Every generated token is
    the oracle's argmax for the sequence so far wherever the oracle's top-two margin is clear."""
    from llama_cpp import Llama
    cfg, w, path = model
    llm = Llama(model_path=path, n_gpu_layers=-1, n_ctx=256, n_seq_max=3, verbose=False, dtype="float32")
    prompts = [tokens_for(cfg, n, 50 + n) for n in (9, 70, 33)]
    outs = [None] * len(prompts)

    def call(i):
        outs[i] = llm.create_completion(prompts[i], max_tokens=12, temperature=0.0, repeat_penalty=1.0)

    threads = [threading.Thread(target=call, args=(i,)) for i in range(len(prompts))]
    for t in threads:
        t.start()
    for t in threads:
        t.join()
    stats = llm._scheduler.stats
    llm.close()
    assert stats["max_batch"] >= 2
    for p, o in zip(prompts, outs):
        assert o["usage"]["completion_tokens"] == 12
        gen = [int(x[1:-1]) for x in o["choices"][0]["text"].replace("><", "> <").split()]
        logits = ref.forward(cfg, w, p + gen)
        for i, g in enumerate(gen):
            row = logits[len(p) + i - 1]
            top = np.sort(row)[-2:]
            if top[1] - top[0] > 1e-3:
                assert int(np.argmax(row)) == g


def test_direct_eval_and_scores(model):
    from llama_cpp import Llama
    cfg, w, path = model
    llm = Llama(model_path=path, n_gpu_layers=-1, n_ctx=128, verbose=False, dtype="float32")
    toks = tokens_for(cfg, 40, 60)
    llm.eval(toks[:30])
    for t in toks[30:]:
        llm.eval([t])
    got = llm.scores[0]
    llm.close()
    assert close(got[None], ref.forward(cfg, w, toks)[-1:], "float32")


def test_a_large_batch_of_single_tokens(model):
    """Sixteen sequences decoding together: more tokens than the few-token kernels take, each a segment of its own."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    for dtype in ("float32", "bfloat16"):
        eng = open_engine(path, dtype, n_ctx=128, max_seqs=16)
        seqs = SequenceSlots(eng)
        reqs = {i: tokens_for(cfg, 20 + 3 * i, 200 + i) for i in range(16)}
        for i, t in reqs.items():
            seqs.open(i)
            eng.step([(seqs.extend(i, len(t) - 12), t[:-12])])
        rows = []
        for n in range(12):
            lg, _ = eng.step([(seqs.extend(i, 1), [t[len(t) - 12 + n]]) for i, t in reqs.items()], want=[[0]] * 16)
            rows.append(lg)
        eng.close()
        want = [ref.forward(cfg, w, t)[-12:] for t in reqs.values()]
        assert close(np.stack(rows, 1).reshape(-1, cfg["vocab"]), np.concatenate(want), dtype)


def test_engine_refuses_what_it_cannot_run(native_lib, tmp_path):
    """Descriptors whose parts do not go together, and tables that name no expert."""
    from llama_cpp import _cabi, models, zogurax
    from llama_cpp._cabi import B2Error
    from llama_cpp.engine import LayeredEngine
    cfg = zu.config([zu.conved(mlp=zu.moe()), zu.biased()], loop=(0, 1, 2))

    def refused(f):
        dims = zogurax.read_dims(cfg)
        f(dims)
        with pytest.raises(B2Error):
            LayeredEngine(dims, {}, n_ctx=64)

    def put(i, **kw):
        return lambda dims: [setattr(dims.layers[i], k, v) for k, v in kw.items()]

    refused(put(0, rot_dims=4))
    refused(put(0, attn_flags=_cabi.B2_ATTN_CONV | _cabi.B2_ATTN_UNIT_QK))
    refused(put(0, attn_flags=_cabi.B2_ATTN_TALK))
    refused(put(0, conv_taps=0))
    refused(put(0, qtemp_every=0.0))
    refused(put(0, loop_pass=3))
    refused(put(0, moe_shared_gate=0))
    refused(put(0, moe_top=7))
    refused(put(0, n_head_kv=3))
    refused(lambda dims: setattr(dims, "block_style", _cabi.B2_BLOCK_PRENORM_RMS))
    w = zu.random_weights(cfg, seed=1)
    w["l0.mlp.table"] = w["l0.mlp.table"].copy()
    w["l0.mlp.table"][9, 1] = 6
    with pytest.raises(B2Error):
        open_engine(zu.write_model(str(tmp_path / "bad"), cfg, w))
    assert models.architectures()
