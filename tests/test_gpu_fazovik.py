"""Fazovik through the native engine against the float64 oracle (oracle/fazovik_ref.py), on small random models the tests
make themselves: each mixer and feed-forward kind alone, prompt against token-by-token decoding, portions down to two tokens,
unequal batches against each request alone, slots and pages used again, marked keys far away and at page borders, the token
pair of the bigram embedding across cuts, the first tokens, long decoding, degenerate and odd sizes, and greedy generation
through `Llama` and the scheduler."""
import copy
import threading

import numpy as np
import pytest

import fazovik_util as fu
from oracle import fazovik_ref as ref

pytestmark = pytest.mark.gpu

TOL = {"float32": 3e-5, "bfloat16": 6e-2}


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
    """float32: every row within the tolerance. bfloat16: the rounded activations can tip a near-tie of the router the other
    way than the oracle's, which moves that row (and, slightly, later ones) by a whole expert; so the typical row must be
    well inside the tolerance and at most one row in ten may leave it."""
    rows = row_errors(got, want)
    if dtype == "float32":
        return rows.max() < TOL[dtype]
    return np.median(rows) < TOL[dtype] / 3 and (rows > TOL[dtype]).mean() <= 0.1


def tokens_for(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], size=n)]


@pytest.fixture(scope="module")
def model(native_lib, tmp_path_factory):
    """All mechanisms in one model: both mixers, a latent read by two later layers (one of them right after a rotated layer),
    both feed-forward kinds and a layer without one."""
    cfg = fu.config([fu.rotated(mlp=fu.moe()), fu.plain(mlp=fu.dense(), rank=32, q_rank=24), fu.plain(mlp=fu.moe(experts=9, top=3, ff=16), rank=32, kv_from=1, heads=5, dim=12, vdim=20, q_rank=18),
                     fu.rotated(mlp=None, heads=2, dim=16, rot_dim=16, vdim=16, rank=48, q_rank=40, base=900.0, yarn=fu.scaling(2.0, 100, 5.0, 1.5)),
                     fu.plain(mlp=fu.moe(experts=4, top=1), rank=32, kv_from=1, heads=2)])
    w = fu.random_weights(cfg, seed=3)
    path = fu.write_model(str(tmp_path_factory.mktemp("fazovik_model")), cfg, w)
    return cfg, w, path


LAYERS = {
    "rotated": lambda: [fu.rotated()],
    "rotated_plain_frequencies_dense": lambda: [fu.rotated(mlp=fu.dense(72), heads=2, dim=32, rot_dim=8, vdim=40, rank=64, q_rank=32, yarn=None)],
    "rotated_moe": lambda: [fu.rotated(mlp=fu.moe(experts=10, top=4, ff=20), heads=4, dim=24, rot_dim=24, vdim=8, rank=40, q_rank=50)],
    "plain": lambda: [fu.plain()],
    "plain_dense": lambda: [fu.plain(mlp=fu.dense(), heads=2, dim=64, vdim=48, rank=80, q_rank=16)],
    "plain_moe_one": lambda: [fu.plain(mlp=fu.moe(experts=5, top=1, ff=32))],
    "shared": lambda: [fu.plain(), fu.plain(kv_from=0, heads=3, dim=22, vdim=16, q_rank=12)],
    "shared_of_rotated": lambda: [fu.rotated(rank=30, rot_dim=6), fu.plain(rank=30, kv_from=0)],
    "shared_of_rotated_aligned": lambda: [fu.rotated(rank=32, rot_dim=16), fu.plain(rank=32, kv_from=0, heads=2, dim=16, vdim=16)],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", sorted(LAYERS))
def test_each_kind_of_layer_alone(native_lib, tmp_path, layer, dtype):
    from llama_cpp.kv_pages import SequenceSlots
    cfg = fu.config(LAYERS[layer]())
    w = fu.random_weights(cfg, seed=11)
    eng = open_engine(fu.write_model(str(tmp_path / "m"), cfg, w), dtype)
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
    for have, want in zip(layers, want_layers):
        assert close(have, want, dtype)
    assert close(got, want_logits, dtype)
    assert close(single, want_logits, dtype)


def test_mechanisms_are_not_trivial(model):
    """Leaving out any one mechanism of the test model moves the logits by far more than the tolerances."""
    cfg, w, _ = model
    toks = tokens_for(cfg, 120, 2)
    want = ref.forward(cfg, w, toks)

    def moved(c=cfg, weights=w):
        return float(np.median(row_errors(ref.forward(c, weights, toks), want)[10:]))

    zero = lambda *names: {k: (np.zeros_like(v) if any(k.endswith(n) for n in names) else v) for k, v in w.items()}
    assert moved(weights=zero("bigram")) > 0.1
    assert moved(weights=zero(".b")) > 0.1
    assert moved(weights=zero("mix.g")) > 0.05
    ones = {k: (np.ones_like(v) if k.endswith((".dq.norm", ".dkv.norm")) else v) for k, v in w.items()}
    assert moved(weights=ones) > 0.05
    c = copy.deepcopy(cfg)
    for L in c["layers"]:
        if "rot" in L["mixer"]:
            L["mixer"]["rot"].pop("scaling")
    assert moved(c) > 0.05
    rolled = dict(w)                                        # the latent that three layers read
    rolled["l1.mix.dkv"] = np.roll(w["l1.mix.dkv"], 1, axis=0)
    assert moved(weights=rolled) > 0.05


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
    """One slot, a pool of three pages: every sequence runs in the pages the previous one left, and its first token has no
    predecessor although the slot's last sequence ended with one."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    eng = open_engine(path, "float32", n_ctx=192, max_seqs=1, kv_tokens=192)
    seqs = SequenceSlots(eng)
    for i, n in enumerate([150, 70, 192, 3, 1]):
        toks = tokens_for(cfg, n, 20 + i)
        got = run_cut(eng, seqs, f"s{i}", toks, [40, 1, 23])
        assert seqs.free_slots == 1 and eng.pages.free_pages == 3
        assert close(got, ref.forward(cfg, w, toks), "float32"), i
    eng.close()


def test_bigram_pair_across_cuts_and_idle_steps(native_lib, tmp_path):
    """The pair (previous, current) spans portions, single tokens, and steps in which another request runs in between; the
    hash multiplies beyond 32 bits before it is reduced."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = fu.config([fu.plain(mlp=None, heads=1, dim=8, vdim=8, rank=8, q_rank=8)], vocab=3000, width=32, hashed=fu.bigram(99991, 2 ** 33 + 17, 2 ** 31 + 99))
    w = fu.random_weights(cfg, seed=9)
    w["embed"] = fu.bf16_round(w["embed"] * 0.3)
    eng = open_engine(fu.write_model(str(tmp_path / "m"), cfg, w), "float32")
    seqs = SequenceSlots(eng)
    a, b = tokens_for(cfg, 40, 1), tokens_for(cfg, 40, 2)
    want = {"a": ref.forward(cfg, w, a), "b": ref.forward(cfg, w, b)}
    wrong = dict(w)
    wrong["bigram"] = np.roll(w["bigram"], 1, axis=0)
    assert row_errors(ref.forward(cfg, wrong, a), want["a"]).min() > 0.1
    got = {"a": [], "b": []}
    for k in got:
        seqs.open(k)
    at = {"a": 0, "b": 0}
    for step in [{"a": 3}, {"b": 1}, {"b": 2}, {"a": 1}, {"a": 1, "b": 5}, {"b": 1, "a": 20}, {"a": 15}, {"b": 31}]:
        entries, who = [], []
        for k, n in step.items():
            toks = (a if k == "a" else b)[at[k]:at[k] + n]
            entries.append((seqs.extend(k, n), toks))
            who.append((k, n))
            at[k] += n
        lg, _ = eng.step(entries, want=[list(range(n)) for _, n in who])
        r = 0
        for k, n in who:
            got[k].append(lg[r:r + n])
            r += n
    eng.close()
    for k in got:
        assert close(np.concatenate(got[k]), want[k], "float32")


PROBE, MARK = 5, 7


def _peaky_model(tmp_path, kind):
    """Attention in which the token PROBE looks for the token MARK: queries are a map of the first half of the stream, keys the
    same map of the second half, and the two embedding rows hold one vector in those halves, so MARK's key is parallel to
    PROBE's query wherever it stands (both per-head maps are the identity; a small rotated part is all that tells positions
    apart). Its score is about six standard deviations above the random keys', some nine tenths of the weight."""
    d, H, W = 32, 2, 64
    size = dict(heads=H, dim=d, vdim=24, rank=d, q_rank=d, scale=0.3)
    layers = {"rotated": [fu.rotated(rot_dim=16, **size)], "plain": [fu.plain(**size)], "shared": [fu.plain(**size), fu.plain(kv_from=0, **size)]}[kind]
    cfg = fu.config(layers, width=W, hashed=None)
    w = fu.random_weights(cfg, seed=5)
    rng = np.random.default_rng(6)
    A = rng.standard_normal((d, W // 2)) / np.sqrt(W // 2)
    vec = rng.standard_normal(W // 2)
    w["embed"][PROBE, :W // 2] = w["embed"][MARK, W // 2:] = fu.bf16_round(vec - vec.mean())
    for i, L in enumerate(layers):
        p = f"l{i}."
        w[p + "norm1"], w[p + "norm1.b"] = np.ones(W), np.zeros(W)
        dr = L["mixer"].get("rot_dim", 0)
        w[p + "mix.dq"] = fu.bf16_round(np.concatenate([A, 0 * A], 1))
        w[p + "mix.dq.norm"] = np.ones(d)
        if p + "mix.dkv" in w:
            w[p + "mix.dkv"][:d] = fu.bf16_round(np.concatenate([0 * A, A], 1))
            w[p + "mix.dkv.norm"] = np.ones(d)
        uq = np.zeros((H, d + dr, d))
        uq[:, :d] = np.eye(d)
        uq[:, d:] = 0.03 * rng.standard_normal((H, dr, d))
        w[p + "mix.uq"] = fu.bf16_round(uq.reshape(H * (d + dr), d))
        w[p + "mix.uk"] = np.tile(np.eye(d), (H, 1))
        w[p + "mix.o"] = fu.bf16_round(2.0 * w[p + "mix.o"])            # the mixer's output stands out in the stream
    if kind == "shared":                    # the second layer's queries are to find the first layer's keys: nothing comes in between
        w["l0.mix.o"] = np.zeros_like(w["l0.mix.o"])
    return cfg, w, fu.write_model(str(tmp_path / "peaky"), cfg, w)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("kind", ["rotated", "plain", "shared"])
def test_far_keys_and_page_borders(native_lib, tmp_path, kind, decode, dtype):
    """The marked token is the sequence's first, at a page border (a page's last / first place), a portion's last / first, or
    the one just before the probing position; a key that is lost or counted twice changes the probe's logits by far more
    than the tolerance. 450 keys are enough for several key ranges per decoded token and eight key blocks per prompt tile."""
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
    for at in (0, 1, 63, 64, 199, 200, 255, 256, 383, 384, 447, 448, probe - 1):
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
@pytest.mark.parametrize("heads", [1, 4, 16, 19])
def test_prompt_tiles(native_lib, tmp_path, heads, dtype):
    """Sizes the tensor-core kernels take: latents up to and above 128 and 256, up to 19 heads, enough (token, expert) pairs
    for 128-row expert tiles; a 300-token prompt at once and in portions that straddle the tiles, and decoded tokens."""
    from llama_cpp.kv_pages import SequenceSlots
    mlp = fu.moe(experts=6, top=4, ff=16)
    cfg = fu.config([fu.rotated(mlp=mlp, heads=heads, dim=16, rot_dim=16, vdim=32, rank=144, q_rank=32),
                     fu.plain(mlp=fu.dense(80), heads=heads, dim=32, vdim=16, rank=272, q_rank=48),
                     fu.plain(mlp=mlp, heads=2 * heads, dim=16, vdim=16, rank=272, q_rank=16, kv_from=1),
                     fu.rotated(mlp=None, heads=heads, dim=16, rot_dim=32, vdim=16, rank=64, q_rank=64)], width=64)
    w = fu.random_weights(cfg, seed=13)
    eng = open_engine(fu.write_model(str(tmp_path / "m"), cfg, w), dtype)
    toks = tokens_for(cfg, 300, 14)
    want = ref.forward(cfg, w, toks)
    seqs = SequenceSlots(eng)
    whole = run_cut(eng, seqs, "w", toks, [300])
    parts = run_cut(eng, seqs, "p", toks, [100, 7, 64, 100] + [1] * 29)
    eng.close()
    assert close(whole, want, dtype)
    assert close(parts, want, dtype)


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
    """A short prompt and 300 single-token steps: past the original context of the frequency scaling and over page borders."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg, w, path = model
    eng = open_engine(path, dtype)
    toks = tokens_for(cfg, 310, 40)
    got = run_cut(eng, SequenceSlots(eng), "d", toks, [10] + [1] * 300)
    eng.close()
    assert close(got, ref.forward(cfg, w, toks), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_are_one_odd_or_large(native_lib, tmp_path, dtype):
    """One head, expert, choice, bucket; latents, keys and values of one entry; all experts chosen; odd sizes that no vector
    path takes; latents above 320 entries and with an odd row length shared by another layer; hidden sizes that differ."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = fu.config([
        fu.rotated(mlp=fu.moe(experts=1, top=1, ff=8), heads=1, dim=8, rot_dim=2, vdim=1, rank=8, q_rank=4, base=10.0, yarn=fu.scaling(1.5, 8, 1.0, 0.5)),
        fu.plain(mlp=fu.dense(1), heads=1, dim=1, vdim=1, rank=4, q_rank=1, scale=1.0),
        fu.plain(mlp=fu.moe(experts=5, top=5, ff=9), heads=3, dim=7, vdim=5, rank=4, q_rank=3, kv_from=1),
        fu.rotated(mlp=None, heads=5, dim=13, rot_dim=10, vdim=7, rank=171, q_rank=37, yarn=fu.scaling(30.0, 500, 2.0, 1.9)),
        fu.plain(mlp=fu.moe(experts=33, top=5, ff=11), heads=2, dim=20, vdim=9, rank=171, q_rank=45, kv_from=3),
        fu.plain(mlp=fu.dense(130), heads=2, dim=24, vdim=24, rank=530, q_rank=20),
        fu.rotated(mlp=fu.dense(33), heads=33, dim=3, rot_dim=4, vdim=3, rank=9, q_rank=5),
    ], width=40, vocab=50, eps=1e-3, hashed=fu.bigram(1, 5, 3))
    w = fu.random_weights(cfg, seed=8)
    eng = open_engine(fu.write_model(str(tmp_path / "m"), cfg, w), dtype)
    toks = tokens_for(cfg, 100, 3)
    got = run_cut(eng, SequenceSlots(eng), "x", toks, [5, 1, 2, 30])
    eng.close()
    assert close(got, ref.forward(cfg, w, toks), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [45, 50])
def test_widths_no_vector_path_takes(native_lib, tmp_path, width, dtype):
    """A model width that is odd, or even but no multiple of four: every product over the width takes its scalar path; no
    bigram table, as a model may come without one."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = fu.config([fu.rotated(mlp=fu.moe(ff=10)), fu.plain(mlp=fu.dense(30)), fu.plain(mlp=fu.moe(ff=7), kv_from=1)], width=width, vocab=77, hashed=None)
    w = fu.random_weights(cfg, seed=21)
    eng = open_engine(fu.write_model(str(tmp_path / "m"), cfg, w), dtype)
    toks = tokens_for(cfg, 150, 22)
    got = run_cut(eng, SequenceSlots(eng), "x", toks, [70, 1, 3, 20, 1])
    eng.close()
    assert close(got, ref.forward(cfg, w, toks), dtype)


def random_config(seed):
    """A random model: layer count and order, every size and constant drawn anew (sizes of the scale small real models have)."""
    rng = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(rng.integers(0, len(xs)))]

    def ff():
        kind = pick("none", "dense", "dense", "moe", "moe", "moe")
        if kind == "none":
            return None
        if kind == "dense":
            return fu.dense(pick(40, 64, 160, 300))
        experts = pick(2, 5, 8, 12, 24)
        return fu.moe(experts=experts, top=int(rng.integers(1, min(experts, 4) + 1)), ff=pick(8, 24, 56, 72))

    layers, owners = [], []
    for i in range(int(rng.integers(3, 7))):
        if rng.random() < 0.5:
            layers.append(fu.rotated(mlp=ff(), heads=pick(1, 2, 4, 5, 8, 12), dim=pick(16, 32, 48, 64), rot_dim=pick(4, 8, 16, 32), vdim=pick(16, 32, 48, 72),
                                     rank=pick(32, 48, 64, 112, 160), q_rank=pick(24, 64, 96, 130), base=pick(500.0, 1e4, 1e6),
                                     yarn=None if rng.random() < 0.3 else fu.scaling(pick(2.0, 8.0, 40.0), pick(32, 128, 1000), pick(32.0, 8.0), pick(1.0, 2.0))))
        else:
            share = bool(owners) and rng.random() < 0.5
            j = pick(*owners) if share else None
            layers.append(fu.plain(mlp=ff(), heads=pick(1, 2, 3, 6, 8), dim=pick(16, 24, 64, 96), vdim=pick(16, 40, 64, 100),
                                   rank=layers[j]["mixer"]["kv_rank"] if share else pick(32, 64, 96, 144, 288), q_rank=pick(24, 64, 100), kv_from=j))
            if not share:
                owners.append(i)
    buckets = pick(17, 211, 1500)
    return fu.config(layers, width=pick(64, 96, 128, 200, 320), vocab=pick(97, 256, 500), eps=pick(1e-5, 1e-6),
                     hashed=fu.bigram(buckets, int(rng.integers(1, 3000)), int(rng.integers(1, 3000))))


@pytest.mark.parametrize("seed", range(10))
def test_random_configurations(native_lib, tmp_path, seed):
    """Ten models nobody chose: each runs a 330-token prompt at once and in uneven portions with decoded tokens at the end,
    in both modes, from a pool that forces page reuse."""
    from llama_cpp.kv_pages import SequenceSlots
    cfg = random_config(100 + seed)
    w = fu.random_weights(cfg, seed=seed)
    path = fu.write_model(str(tmp_path / "m"), cfg, w)
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


def test_engine_refuses_what_it_cannot_share(native_lib):
    """Descriptors that name rows of a later layer, of another size, or of a layer without rows of its own."""
    from llama_cpp import fazovik
    from llama_cpp._cabi import B2Error
    from llama_cpp.engine import LayeredEngine
    cfg = fu.config([fu.plain(), fu.plain(kv_from=0), fu.plain(kv_from=0)])
    for i, j in ((1, 3), (2, 2), (1, 2)):
        dims = fazovik.read_dims(cfg)
        dims.layers[i].kv_from = j
        with pytest.raises(B2Error):
            LayeredEngine(dims, {}, n_ctx=64)
    dims = fazovik.read_dims(cfg)
    dims.layers[1].la_rank = 20
    with pytest.raises(B2Error):
        LayeredEngine(dims, {}, n_ctx=64)
