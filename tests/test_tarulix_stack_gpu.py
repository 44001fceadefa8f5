"""The Tarulix design on the GPU against the plain restatement: each mechanism alone, edges of windows, blocks, biases and pages, far keys, sinks, routing,
states, prompts, portions, decoding, mixed batches, slots and pages used again, generation, programs."""
import json
import os
import subprocess

import numpy as np
import pytest

import stack_util as U
from oracle import layer_stack as LS

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ("float32", "bfloat16")
BF16_MODEL = 0.1         # worst row of a whole random model in bfloat16; single mechanisms are held to far less below
PORTIONS = ([200], [65, 1, 2, 64, 1, 31, 36], [1] * 6 + [130] + [2, 3, 4, 16, 15, 24], [17, 63, 120])


def tol(dtype):
    return U.F32_TOL if dtype == "float32" else BF16_MODEL


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return tmp_path_factory.mktemp("tarulix")


@pytest.fixture(scope="module")
def opened(root):
    from forge_llm_b200 import runtime
    models = {}

    def get(name, dtype, seed=0):
        key = (name, dtype, seed)
        if key not in models:
            folder, orc = U.make(root, "tarulix_" + name, seed)
            models[key] = (runtime.Model.open(folder, dtype), orc)
        return models[key]

    yield get
    for m, _ in models.values():
        m.close()


def open_custom(root, cfg, tensors, dtype, name):
    from forge_llm_b200 import runtime
    folder = str(root / (name + "-" + dtype))
    LS.write_model(folder, cfg, tensors)
    return runtime.Model.open(folder, dtype), LS.LayerStack(cfg, tensors)


def all_logits(model, toks, cache, seq=0):
    return model.step([(seq, toks, list(range(len(toks))))], cache)[0]


def traced(m, toks, portions, kv):
    """Residual stream after every layer run over the whole prompt, fed in portions."""
    m.trace(True)
    out, at = [], 0
    for n in portions:
        m.step([(0, toks[at:at + n], [])], kv)
        out.append(m.read_trace(n))
        at += n
    m.trace(False)
    assert at == len(toks)
    return np.concatenate(out, axis=1)


def embedded(orc, toks):
    return orc.t["embed"][toks]


# ------------------------------------------------------------------------------------------------ each mechanism alone
DISTANCE = {
    "small": LS.distance_mixer(),
    "wide": LS.distance_mixer(4, 2, 128, 96, 70, 33),
    "odd": LS.distance_mixer(5, 5, 9, 13, 64, 200, 0.5),
    "past": LS.distance_mixer(7, 1, 40, 264, 500, 90),
    "all": LS.distance_mixer(6, 2, 128, 160, None, 150),
    "long": LS.distance_mixer(4, 2, 24, 40, 180, 9000),
    "blocks": LS.distance_mixer(40, 2, 64, 64, 90, 64),      # more heads on a key head than one tile holds
    "one": LS.distance_mixer(2, 1, 8, 8, 1, 3),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,buckets", [(n, 16) for n in DISTANCE] + [("small", 2), ("long", 33), ("all", 7)])
def test_attention_with_distances_alone(root, dtype, name, buckets):
    """Two layers, the second one's values blended with the first one's."""
    mx = DISTANCE[name]
    cfg = LS.make_tarulix(104, 90, [("attention", mx, None), ("attention", mx, None)], eps=1e-3)
    t = LS.random_tarulix(cfg, 5, buckets=buckets)
    m, orc = open_custom(root, cfg, t, dtype, f"distance-{name}-{buckets}")
    toks = U.tokens(cfg, 200, 6)
    want, e = orc.residuals(toks), embedded(orc, toks)
    for portions in PORTIONS:
        kv = m.new_cache(max_seq=256)
        got = traced(m, toks, portions, kv)
        assert U.err(got[0] - e, want[0] - e) < (2e-5 if dtype == "float32" else 8e-2), portions
        assert U.err(got[1] - e, want[1] - e) < (2e-5 if dtype == "float32" else 8e-2), portions
        for run, x in ((0, e), (1, want[0])):
            p = f"l{run}.mix."
            k = LS.unit_rms((x @ orc.t[p + "k"].T + orc.t[p + "k.b"]).reshape(200, mx["kv_heads"], -1), 1e-3).reshape(200, -1)
            v = x @ orc.t[p + "v"].T + orc.t[p + "v.b"]
            if run:
                first = e @ orc.t["l0.mix.v"].T + orc.t["l0.mix.v.b"]
                v = (1 - orc.t[p + "vmix"]) * v + orc.t[p + "vmix"] * first
            for which, y in ((0, k), (1, v)):
                assert np.abs(kv.read(run, which) - y).max() < (1e-5 if dtype == "float32" else 4e-2) * np.abs(y).max(), (portions, run, which)
        kv.close()
    m.close()


POOLED = {
    "small": LS.scan_pair(),
    "divides": LS.scan_pair(6, 3, 64, 64, 50, 16, 32),
    "uneven": LS.scan_pair(4, 2, 24, 24, 37, 24, 8),
    "long_blocks": LS.scan_pair(4, 4, 16, 16, 30, 70, 4),
    "single": LS.scan_pair(2, 1, 16, 24, 5, 1, 16),
    "wide": LS.scan_pair(8, 2, 128, 128, 66, 8, 128),
    "many_groups": LS.scan_pair(8, 8, 32, 72, 40, 10, 16),          # values of sixteen column blocks
    "many_heads": LS.scan_pair(40, 2, 24, 40, 40, 8, 0),            # more heads on a key head than one tile holds, more than sixteen to mix
    "past": LS.scan_pair(6, 2, 24, 40, None, 0, 24),
    "beyond": LS.scan_pair(3, 1, 72, 300, 40, 12, 8),
    "odd": LS.scan_pair(3, 3, 9, 7, 33, 5, 2),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(POOLED))
def test_pooled_attention_with_mixed_heads_alone(root, dtype, name):
    mx = POOLED[name]
    cfg = LS.make_tarulix(104, 90, [("parallel", mx, None)], eps=1e-3)
    t = LS.random_tensors(cfg, 15)
    t["l0.mix.right.o"] = t["l0.mix.right.o"] * 0
    m, orc = open_custom(root, cfg, t, dtype, f"pooled-{name}")
    toks = U.tokens(cfg, 200, 16)
    e = embedded(orc, toks)
    want = orc.residuals(toks)[0] - e
    for portions in PORTIONS:
        kv = m.new_cache(max_seq=256)
        assert U.err(traced(m, toks, portions, kv)[0] - e, want) < (2e-5 if dtype == "float32" else 8e-2), portions
        kv.close()
    m.close()


SCAN = {"small": (72, 16, 12, 4), "one": (8, 1, 1, 1), "odd": (37, 5, 3, 5), "wide": (320, 64, 96, 4), "beyond": (40, 250, 70, 16), "whole": (64, 32, 64, 2), "lanes": (33, 128, 8, 3), "eight": (48, 8, 20, 4), "ranks": (24, 16, 200, 4), "far_ranks": (16, 4, 300, 2)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SCAN))
@pytest.mark.parametrize("steps", ("mixed", "strong", "none"))
def test_selective_scan_alone(root, dtype, name, steps):
    inner, state, rank, conv = SCAN[name]
    mx = LS.scan_pair(1, 1, 8, 8, 4, 2, 0, inner=inner, state=state, rank=rank, conv=conv)
    cfg = LS.make_tarulix(104, 90, [("parallel", mx, None)], eps=1e-3)
    t = LS.random_tensors(cfg, 3)
    t["l0.mix.left.o"] = t["l0.mix.left.o"] * 0
    t["l0.mix.left.o.b"] = t["l0.mix.left.o.b"] * 0
    if steps != "mixed":      # a token takes the state over, or hardly touches it
        t["l0.mix.right.dt.b"] = t["l0.mix.right.dt.b"] * 0 + (6.0 if steps == "strong" else -7.0)
    m, orc = open_custom(root, cfg, t, dtype, f"scan-{name}-{steps}")
    toks = U.tokens(cfg, 200, 4)
    e = embedded(orc, toks)
    want = orc.residuals(toks)[0] - e
    w = lambda n: orc.t["l0.mix.right." + n]
    x, dt, B, C, _ = LS.selective_inputs(e, w, mx["right"])
    _, S = LS.selective_scan(x, dt, -np.exp(w("A_log")), B, C, w("D"))
    lim = 2e-5 if dtype == "float32" else 6e-2
    for portions in PORTIONS:
        kv = m.new_cache(max_seq=256)
        assert U.err(traced(m, toks, portions, kv)[0] - e, want) < lim, portions
        s = kv.read_state(0).reshape(S.shape)
        assert np.linalg.norm(s - S) < (1e-5 if dtype == "float32" else 2e-2) * np.linalg.norm(S), portions
        kv.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("scales", ((1.0, 1.0), (0.3, 2.0), (-1.5, 0.25)))
def test_both_sides_of_a_pair(root, dtype, scales):
    cfg = LS.make_tarulix(104, 90, [("parallel", LS.scan_pair(scales=scales), None)])
    m, orc = open_custom(root, cfg, LS.random_tensors(cfg, 9), dtype, f"sides{scales}")
    toks = U.tokens(cfg, 100, 5)
    e = embedded(orc, toks)
    kv = m.new_cache(max_seq=128)
    assert U.err(traced(m, toks, [40, 1, 2, 1, 56], kv)[0] - e, orc.residuals(toks)[0] - e) < (1e-5 if dtype == "float32" else 5e-2)
    kv.close(); m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", (-50.0, 4.0, 12.0, 60.0))
def test_sinks_of_any_size(root, dtype, sink):
    """From none at all to one that takes everything (then the bias of the output is what is left)."""
    cfg = LS.make_tarulix(64, 64, [("attention", LS.distance_mixer(4, 2, 16, 16, 30, 12, 1.0), None)])
    t = LS.random_tensors(cfg, 8)
    t["l0.mix.sink"] = np.array([sink, sink / 2, -sink, 0.0], np.float32)
    m, orc = open_custom(root, cfg, t, dtype, f"sink{sink}")
    toks = U.tokens(cfg, 90, 9)
    want = orc.residuals(toks)[0] - embedded(orc, toks)
    for portions in ([90], [1] * 20 + [70], [31, 59]):
        kv = m.new_cache(max_seq=128)
        assert U.err(traced(m, toks, portions, kv)[0] - embedded(orc, toks), want) < (2e-5 if dtype == "float32" else 6e-2)
        kv.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("buckets,longest", ((16, 128), (32, 256), (6, 24), (12, 6 * 3 ** 3)))
def test_where_a_bucket_of_distances_begins(root, dtype, buckets, longest):
    """One bucket stands out of the biases at a time, in one head each; edges that are whole numbers."""
    cfg = LS.make_tarulix(64, 64, [("attention", LS.distance_mixer(8, 2, 16, 16, None, longest, 0.1), None)])
    t = LS.random_tarulix(cfg, 8, buckets=buckets)
    rel = np.zeros((buckets, 8), np.float32)
    rel[buckets // 2 + np.arange(8) % (buckets - buckets // 2), np.arange(8)] = 6.0
    t["l0.mix.rel"] = rel
    m, orc = open_custom(root, cfg, t, dtype, f"buckets{buckets}")
    toks = U.tokens(cfg, 300, 9)
    want = orc.residuals(toks)[0] - embedded(orc, toks)
    for portions in ([300], [20] * 6 + [1] * 60 + [120]):
        kv = m.new_cache(max_seq=320)
        assert U.err(traced(m, toks, portions, kv)[0] - embedded(orc, toks), want) < (2e-5 if dtype == "float32" else 6e-2)
        kv.close()
    m.close()


# experts, top, size, identity choices, shared size
EXPERTS = [(5, 2, 24, 2, 40), (1, 1, 40, 0, 8), (4, 6, 64, 2, 130), (8, 1, 130, 7, 24), (70, 6, 20, 10, 64), (300, 3, 8, 100, 16), (2, 3, 16, 30, 100)]


@pytest.mark.parametrize("experts", EXPERTS)
@pytest.mark.parametrize("clear", (True, False))
def test_experts_alone(root, experts, clear):
    """The mixer writes nothing.  Batches from one token to several hundred: experts that many, few and no tokens use, tokens that only pass themselves on.
    A router that reads the whole stream (float32) and one whose choices rounding cannot change."""
    cfg = LS.make_tarulix(104, 90, [("attention", LS.distance_mixer(1, 1, 8, 8), experts)], eps=1e-3)
    t = LS.random_tarulix(cfg, 11, clear=clear)
    t["l0.mix.o"] = t["l0.mix.o"] * 0
    t["l0.mix.o.b"] = t["l0.mix.o.b"] * 0
    if clear:
        t["embed"][40:, :LS.MARKERS] = t["embed"][40, :LS.MARKERS]      # most tokens agree
    toks = U.tokens(cfg, 300, 12)
    for dtype in DTYPES if clear else DTYPES[:1]:
        m, orc = open_custom(root, cfg, t, dtype, f"moe{experts[0]}-{experts[3]}-{clear}")
        e = embedded(orc, toks)
        want = orc.residuals(toks)[0] - e
        if not clear and experts[1] < experts[0] + experts[3]:
            z = e @ orc.t["l0.mlp.router"].T
            s = np.exp(z - z.max(1, keepdims=True))
            s = np.sort(s / s.sum(1, keepdims=True) + orc.t["l0.mlp.correction"], axis=1)
            assert (s[:, -experts[1]] - s[:, -experts[1] - 1]).min() > 2e-6
        for portions in ([300], [1, 2, 16, 17, 32, 33, 64, 65, 70], [1] * 30 + [128, 142]):
            kv = m.new_cache(max_seq=320)
            assert U.err(traced(m, toks, portions, kv)[0] - e, want) < (1e-5 if dtype == "float32" else 3e-2), portions
            kv.close()
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("only", (0, 1))
def test_nobody_uses_an_expert(root, dtype, only):
    """Corrections that send every token to the identity choices alone, or to one expert."""
    cfg = LS.make_tarulix(72, 60, [("attention", LS.distance_mixer(1, 1, 8, 8), (5, 1, 24, 3, 32))])
    t = LS.random_tensors(cfg, 2)
    t["l0.mlp.correction"] = np.array([0, 0, 9.0 * only, 0, 0, 0, 9.0 * (1 - only), 0], np.float32)
    m, orc = open_custom(root, cfg, t, dtype, f"only{only}")
    toks = U.tokens(cfg, 80, 3)
    want = orc.residuals(toks)[0] - embedded(orc, toks)
    for portions in ([80], [1, 7, 32, 40]):
        kv = m.new_cache(max_seq=128)
        assert U.err(traced(m, toks, portions, kv)[0] - embedded(orc, toks), want) < (1e-5 if dtype == "float32" else 5e-2)
        kv.close()
    m.close()


# ------------------------------------------------------------------------------------------------ edges of windows, blocks and pages
def _beacon(window, pool=None):
    """The query of token 0 meets one key, token 1's, whose score stands out (as one of a block's, too) and whose value alone reaches the output."""
    if pool is None:
        kind, p, mx = "attention", "l0.mix.", LS.distance_mixer(4, 2, 16, 16, window, 50, 1.0)
    else:
        kind, p, mx = "parallel", "l0.mix.left.", LS.scan_pair(4, 2, 16, 16, window, pool, 0, softcap=400.0, scale=float(pool), inner=8, state=2, rank=2)
    cfg = LS.make_tarulix(64, 64, [(kind, mx, None)])
    t = LS.random_tarulix(cfg, 11)
    rng = np.random.default_rng(12)
    emb = 0.3 * rng.standard_normal((64, 64)).astype(np.float32)
    emb[:, :8] = 0
    emb[0, 0], emb[1, 1] = 8.0, 8.0
    emb[2:, 2] = 4.0
    q, k, v = (np.zeros_like(t[p + n]) for n in "qkv")
    q[::16, 0], q[1::16, 2] = 5.0, 5.0              # token 0 asks along one axis, the others along another
    k[::16, 1], k[1::16, 0], k[2::16, 2] = 5.0, 5.0, 5.0
    v[:] = LS.bf16_round(0.1 * rng.standard_normal(v.shape))
    v[:, 1] = 3.0 * np.sign(rng.standard_normal(len(v)))
    t.update({"embed": LS.bf16_round(emb), p + "q": q, p + "k": k, p + "v": LS.bf16_round(v)})
    for n in "qkv":
        t[f"{p}{n}.b"] = 0 * t[f"{p}{n}.b"]
    if pool is None:
        t[p + "rel"] = LS.bf16_round(0.3 * t[p + "rel"])
    else:
        t["l0.mix.right.o"] = t["l0.mix.right.o"] * 0
    return cfg, t


def _meet(m, orc, cases, dtype, rng, max_seq):
    kv = m.new_cache(max_seq=max_seq, batch=3)
    lim = U.F32_TOL if dtype == "float32" else 5e-2
    for i, j, seen in cases:
        toks = [int(x) for x in rng.integers(2, 64, i + 1)]
        toks[j], toks[i] = 1, 0
        lost = list(toks)
        lost[j] = 5
        want, without = orc.logits(toks)[-1:], orc.logits(lost)[-1:]
        assert (U.err(without, want) > 0.2) == seen, (i, j, U.err(without, want))
        got = m.step([(0, toks, [i])], kv)[0]                                        # in a prompt's portion
        m.step([(1, toks[:-1], [])], kv)
        one = m.forward(toks[-1], kv, seq=1)[None]                                   # decoded
        cut = max(1, j)
        m.step([(2, toks[:cut], [])], kv)
        two = m.step([(2, toks[cut:], [i - cut])], kv)[0]                            # a portion that starts at the key
        for g in (got, one, two):
            assert U.err(g, want) < lim, (i, j)
        for s in range(3):
            kv.free_seq(s)
    kv.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", (48, 64, 100, 129, 1))
def test_keys_just_inside_and_outside_a_window(root, dtype, window):
    cfg, t = _beacon(window)
    m, orc = open_custom(root, cfg, t, dtype, f"beacon-{window}")
    cases = []                                    # (query position, key position, seen)
    for i in (window, window + 1, 2 * window, 3 * window + 5, 127, 128, 129, 255, 256):
        for j in (i - window - 1, i - window, i - window + 1, i - 1, 0):
            if 0 <= j < i:
                cases.append((i, j, i - j < window))
    cases += [(i, j, i - j < window) for i, j in ((1, 0), (65, 64), (64, 63), (192, 128), (300, 64), (300, 63))]
    _meet(m, orc, sorted(set(cases)), dtype, np.random.default_rng(13), 512)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,pool", ((48, 16), (30, 5), (20, 48), (65, 8), (10, 64)))
def test_tokens_that_left_the_window_and_blocks_just_seen(root, dtype, window, pool):
    cfg, t = _beacon(window, pool)
    m, orc = open_custom(root, cfg, t, dtype, f"blocks-{window}-{pool}")
    seen = lambda i, j: i - j < window or j // pool * pool + pool - 1 <= i - window
    cases = set()
    for b in (0, 1, 64 // pool, 128 // pool):
        last = b * pool + pool - 1
        for j in (b * pool, last):
            for i in (last + window - 1, last + window, last + window + 1, last + window + 90):     # not yet, just, seen; far behind
                cases.add((i, j))
    for i in (window, 127, 128, 191, 192, 256):
        for j in (i - window, i - window + 1, 0, 63, 64):
            if 0 <= j < i:
                cases.add((i, j))
    _meet(m, orc, [(i, j, seen(i, j)) for i, j in sorted(cases)], dtype, np.random.default_rng(13), 512)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,pool", ((None, None), (700, 16)))
def test_far_keys(root, dtype, window, pool):
    """Over more keys than one group of warps takes: several ranges of keys per row, several tiles of blocks."""
    cfg, t = _beacon(window, pool)
    m, orc = open_custom(root, cfg, t, dtype, f"far{window}")
    seen = lambda i, j: window is None or i - j < window or j // pool * pool + pool - 1 <= i - window
    cases = [(i, j) for i, j in ((1, 0), (64, 0), (64, 63), (129, 64), (700, 0), (700, 1), (700, 63), (700, 64), (700, 511), (700, 512), (1290, 0), (1290, 640), (1290, 1289), (2300, 3), (2300, 1500), (2300, 1599), (2300, 1600))]
    _meet(m, orc, [(i, j, seen(i, j)) for i, j in cases], dtype, np.random.default_rng(14), 2368)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_what_was_written_first_is_read_last(root, dtype):
    """A scan whose states hardly decay: the first token still shows hundreds of tokens later, in prompts and decoded."""
    cfg = LS.make_tarulix(64, 64, [("parallel", LS.scan_pair(1, 1, 8, 8, 4, 2, 0, inner=64, state=16, rank=4), None)])
    t = LS.random_tensors(cfg, 14)
    t["l0.mix.left.o"] *= 0
    t["l0.mix.right.A_log"] = t["l0.mix.right.A_log"] * 0 - 7.0
    m, orc = open_custom(root, cfg, t, dtype, "far-state")
    toks = [int(x) for x in np.random.default_rng(16).integers(2, 64, 420)]
    want = orc.logits(toks)
    assert U.err(orc.logits([1] + toks[1:])[-1:], want[-1:]) > 10 * U.F32_TOL
    lim = U.F32_TOL if dtype == "float32" else 6e-2
    kv = m.new_cache(max_seq=448, batch=2)
    assert U.err(all_logits(m, toks, kv, 0), want) < lim
    m.step([(1, toks[:20], [])], kv)
    assert U.err([m.forward(x, kv, seq=1) for x in toks[20:]], want[20:]) < lim
    kv.close(); m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ("all", "ones", "odd"))
def test_the_first_tokens(opened, dtype, name):
    """Sequences of one to twelve tokens, in every cut into two portions, in slots that other sequences have used."""
    m, orc = opened(name, dtype)
    cfg = U.TARULIX[name]
    kv = m.new_cache(max_seq=128, batch=2)
    m.step([(0, U.tokens(cfg, 90, 1), []), (1, U.tokens(cfg, 20, 2), [])], kv)
    toks = U.tokens(cfg, 12, 17)
    want = orc.logits(toks)
    for n in range(1, 13):
        kv.free_seq(0)
        assert U.err(all_logits(m, toks[:n], kv), want[:n]) < tol(dtype), n
    for cut in range(1, 12):
        kv.free_seq(1)
        got = list(all_logits(m, toks[:cut], kv, 1)) + list(all_logits(m, toks[cut:], kv, 1))
        assert U.err(got, want) < tol(dtype), cut
    kv.close()


# ------------------------------------------------------------------------------------------------ prompts, decoding, portions, batches
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(U.TARULIX))
def test_prompt_decode_and_portions(opened, dtype, name):
    m, orc = opened(name, dtype)
    toks = U.tokens(U.TARULIX[name], 170)
    want = orc.logits(toks)
    kv = m.new_cache(max_seq=192, batch=3)
    assert U.err(all_logits(m, toks, kv, 0), want) < tol(dtype)
    got = [m.forward(t, kv, seq=1) for t in toks[:3]]
    got += list(all_logits(m, toks[3:140], kv, 1))
    got += [m.forward(t, kv, seq=1) for t in toks[140:]]
    assert U.err(got, want) < tol(dtype)
    at, got = 0, []
    for n in (2, 37, 2, 3, 31, 32, 16, 15, 30, 2):
        got += list(all_logits(m, toks[at:at + n], kv, 2))
        at += n
    assert at == 170 and U.err(got, want) < tol(dtype)
    kv.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_in_one_step(root, dtype):
    """More rows than the passes in front of the attention take one by one, an uneven number of them."""
    cfg = LS.make_tarulix(104, 90, [("parallel", LS.scan_pair(6, 2, 40, 24, 150, 16), None), ("attention", LS.distance_mixer(6, 2, 40, 24, 200, 100), (5, 2, 24, 1, 40))])
    m, orc = open_custom(root, cfg, LS.random_tensors(cfg, 6), dtype, "long")
    toks = U.tokens(cfg, 1031, 8)
    kv = m.new_cache(max_seq=1088)
    assert U.err(all_logits(m, toks, kv), orc.logits(toks)) < tol(dtype)
    kv.close(); m.close()


def test_a_router_that_reads_the_whole_stream(root):
    """A whole model in 32 bits whose choices depend on everything."""
    cfg = U.TARULIX["all"]
    m, orc = open_custom(root, cfg, LS.random_tarulix(cfg, 5, clear=False), "float32", "general")
    toks = U.tokens(cfg, 150, 3)
    want = orc.logits(toks)
    kv = m.new_cache(max_seq=192, batch=2)
    assert U.err(all_logits(m, toks, kv), want) < U.F32_TOL
    got = list(all_logits(m, toks[:50], kv, 1)) + [m.forward(t, kv, seq=1) for t in toks[50:]]
    assert U.err(got, want) < U.F32_TOL
    kv.close(); m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ("all", "odd"))
def test_mixed_batches_equal_each_request_alone(opened, dtype, name):
    from forge_llm_b200.engine import Engine
    m, orc = opened(name, dtype)
    cfg = U.TARULIX[name]
    lens = {"a": 170, "b": 9, "c": 64, "d": 129, "e": 1, "f": 200, "g": 65, "h": 130}
    toks = {k: U.tokens(cfg, n, seed=i) for i, (k, n) in enumerate(lens.items())}
    want = {k: orc.logits(v) for k, v in toks.items()}
    eng = Engine(m, pool_tokens=640, slots=4)       # far less than all requests together: pages and slots are used again
    rng = np.random.default_rng(21)
    pages = {k: -(-n // 64) * 64 for k, n in lens.items()}
    fed, waiting, live, seen, reserved, used = {k: 0 for k in lens}, list(lens), [], {k: [] for k in lens}, 0, []
    while waiting or live:
        while waiting and len(live) < 4 and reserved + pages[waiting[0]] <= 640:
            k = waiting.pop(0)
            live.append(k)
            reserved += pages[k]
        entries = []
        for k in live:
            if len(live) > 1 and rng.random() < 0.2:
                continue                             # left out of this step
            n = int(min(lens[k] - fed[k], rng.choice([1, 1, 2, 3, 15, 16, 32, 33, 64, 100])))
            entries.append((k, toks[k][fed[k]:fed[k] + n], list(range(n))))
        if not entries:
            continue
        for (k, t, _), rows in zip(entries, eng.step(entries)):
            seen[k] += list(rows)
            fed[k] += len(t)
        for k in [k for k in live if fed[k] == lens[k]]:
            used.append(eng._slot[k])
            eng.release(k)
            live.remove(k)
            reserved -= pages[k]
    assert len(used) == 8 and len(set(used)) <= 4 and eng.cache.free_tokens() == 640
    for k in lens:
        assert U.err(seen[k], want[k]) < tol(dtype), k
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_do_not_matter(opened, dtype):
    """The same steps on a fresh cache and on one whose pages and slots were used by others, in another order: the same bits."""
    m, _ = opened("all", dtype)
    cfg = U.TARULIX["all"]
    a, b = U.tokens(cfg, 180, 30), U.tokens(cfg, 100, 31)

    def play(kv, sa, sb):
        out = [m.step([(sa, a[:100], [99]), (sb, b[:5], [4])], kv)]
        out.append(m.step([(sa, a[100:120], [0, 19]), (sb, b[5:70], [3])], kv))
        for i in range(30):
            out.append(m.step([(sa, [a[120 + i]], [0]), (sb, [b[70 + i]], [0])], kv))
        return np.concatenate([r for o in out for r in o])

    kv1 = m.new_cache(max_seq=256, batch=4, pool_tokens=512)
    x = play(kv1, 0, 1)
    kv2 = m.new_cache(max_seq=256, batch=4, pool_tokens=512)
    for s, n in ((0, 70), (1, 200), (3, 65)):
        m.step([(s, U.tokens(cfg, n, 40 + s), [])], kv2)
    kv2.free_seq(1)
    kv2.free_seq(0)
    m.step([(2, U.tokens(cfg, 30, 44), [])], kv2)
    kv2.free_seq(3)
    assert np.array_equal(x, play(kv2, 3, 0))
    kv1.close(); kv2.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ("all", "ones"))
def test_long_decoding(opened, dtype, name):
    """From the third token to the three-hundredth one by one (graph replays), over many window, block and page borders."""
    m, orc = opened(name, dtype)
    toks = U.tokens(U.TARULIX[name], 300, 50)
    want = orc.logits(toks)
    kv = m.new_cache(max_seq=320)
    m.forward_prefill(toks[:2], kv)
    assert U.err([m.forward(t, kv) for t in toks[2:]], want[2:]) < tol(dtype)
    kv.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch", (2, 5, 19, 40))
def test_batched_decode_equals_each_alone(opened, dtype, batch):
    m, orc = opened("all", dtype)
    cfg = U.TARULIX["all"]
    seqs = [U.tokens(cfg, 20 + 5 * (i % 20), 60 + i) for i in range(batch)]
    kv = m.new_cache(max_seq=192, batch=batch)
    for b in range(batch):
        m.forward_prefill(seqs[b][:-3], kv, seq=b)
    for k in (3, 2, 1):
        lg = m.forward_batch([s[len(s) - k] for s in seqs], kv)
    assert U.err(lg, np.stack([orc.logits(s)[-1] for s in seqs])) < tol(dtype)
    kv.close()


def test_more_wanted_places_than_tokens(opened):
    """A place may be asked for twice."""
    m, orc = opened("all", "bfloat16")
    toks = U.tokens(U.TARULIX["all"], 20, 5)
    kv = m.new_cache(max_seq=64)
    want = [i % 20 for i in range(45)]
    assert U.err(m.step([(0, toks, want)], kv)[0], orc.logits(toks)[want]) < BF16_MODEL
    kv.close()


# ------------------------------------------------------------------------------------------------ generation
def test_greedy_generation_everywhere(opened):
    """The session's greedy loop, the batched loop and the scheduler give the restatement's tokens (float32)."""
    from forge_llm_b200.engine import Engine, Sampling, Scheduler
    m, orc = opened("all", "float32")
    cfg = U.TARULIX["all"]
    prompts = [U.tokens(cfg, n, 70 + n) for n in (1, 3, 40, 64, 75)]
    want = [orc.generate_greedy(p, 10) for p in prompts]
    kv = m.new_cache(max_seq=128, batch=5)
    for p, w in zip(prompts, want):
        kv.reset()
        assert list(m.generate_greedy(p, 10, kv)) == w
    kv.reset()
    for b, p in enumerate(prompts):
        m.forward_prefill(p, kv, seq=b)
    out = m.decode_greedy_batch([w[0] for w in want], 9, kv)
    for b in range(5):
        assert list(out[:, b]) == want[b][:9]
    kv.close()
    eng = Engine(m, pool_tokens=256, slots=3)
    s = Scheduler(eng, step_tokens=48)
    for i, p in enumerate(prompts):
        s.submit(i, p, 10, Sampling())
    got = s.run()
    assert [got[i] for i in range(5)] == want
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_cache_persistence(opened, dtype):
    """Blocks and states travel with a sequence: what follows is the same to the bit, also when blocks come into sight later."""
    from forge_llm_b200._lib import ForgeError
    m, _ = opened("all", dtype)
    other, _ = opened("ones", dtype)
    cfg = U.TARULIX["all"]
    kv = m.new_cache(max_seq=192, batch=3)
    m.step([(2, U.tokens(cfg, 50, 91), [])], kv)
    m.forward_prefill(U.tokens(cfg, 100, 90), kv, seq=0)
    blob = kv.save(0)
    kv.load(blob, 2)
    assert kv.len(2) == 100
    for x in range(5, 45):
        a, b = m.step([(0, [x], [0]), (2, [x], [0])], kv)
        assert np.array_equal(a, b)
    with pytest.raises(ForgeError):
        kv.load(blob[:-1], 1)
    okv = other.new_cache(max_seq=192)
    with pytest.raises(ForgeError):
        okv.load(blob)
    kv.close(); okv.close()


def test_scoring_and_scratch_growth(opened):
    """Per-token scoring, and a captured decode step beside prompts that grow the step's buffers."""
    m, orc = opened("ones", "float32")
    cfg = U.TARULIX["ones"]
    toks = U.tokens(cfg, 60, 81)
    lg = orc.logits(toks)
    kv = m.new_cache(max_seq=64)
    m.forward_prefill(toks[:10], kv)
    got = [m.forward(t, kv) for t in toks[10:20]]
    kv2 = m.new_cache(max_seq=2048, batch=3)
    m.step([(0, U.tokens(cfg, 700, 92), []), (1, U.tokens(cfg, 30, 93), []), (2, U.tokens(cfg, 300, 94), [])], kv2)
    got += [m.forward(t, kv) for t in toks[20:]]
    assert U.err(got, lg[10:]) < U.F32_TOL
    kv2.close()
    lse = np.log(np.exp(lg - lg.max(-1, keepdims=True)).sum(-1)) + lg.max(-1)
    mean, _, count = m.score_corpus(toks, kv)
    assert count == 59 and abs(mean - np.mean([lse[i] - lg[i, toks[i + 1]] for i in range(59)])) < 1e-4
    kv.close()


# ------------------------------------------------------------------------------------------------ programs
def test_programs(root, tmp_path, capsys):
    from forge_llm_b200.__main__ import main
    folder, orc = U.make(root, "tarulix_all")
    cfg = U.TARULIX["all"]
    a, b = U.tokens(cfg, 90, 95), U.tokens(cfg, 40, 96)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:50], "want": [0, 49]}, {"id": "y", "tokens": b, "want": [39]}], "end": ["y"]},
             {"step": 1, "entries": [{"id": "x", "tokens": a[50:88], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "z", "tokens": b[:2], "want": [1]}, {"id": "x", "tokens": a[88:89], "want": [0]}], "end": ["z"]},
             {"step": 3, "entries": [{"id": "x", "tokens": a[89:], "want": [0]}], "end": ["x"]}]
    la, lb = orc.logits(a), orc.logits(b)
    want = {0: [la[0], la[49], lb[39]], 2: [lb[1], la[88]], 3: [la[89]]}
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "192"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        for s, rows in want.items():
            got = np.fromfile(out / f"{s}.f32", "<f4").reshape(len(rows), cfg["vocab"])
            assert U.err(got, rows) < tol(dtype)
    prompts = [U.tokens(cfg, n, 97 + n) for n in (5, 50)]
    args = ["generate", "--model", folder, "--dtype", "float32", "--max-new", "6", "--repeat-penalty", "1.0"]
    for p in prompts:
        args += ["--prompt", ",".join(map(str, p))]
    assert main(args) == 0
    lines = capsys.readouterr().out.strip().splitlines()
    assert [[int(x) for x in l.split()] for l in lines] == [orc.generate_greedy(p, 6) for p in prompts]
