"""The Mokatar design on the GPU against the plain restatement: each mechanism alone, edges of windows, kept tokens and pages, far keys,
sinks, routing, states, prompts, portions, decoding, mixed batches, slots and pages used again, generation, programs."""
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
    return tmp_path_factory.mktemp("experts")


@pytest.fixture(scope="module")
def opened(root):
    from forge_llm_b200 import runtime
    models = {}

    def get(name, dtype, seed=0):
        key = (name, dtype, seed)
        if key not in models:
            folder, orc = U.make(root, "mokatar_" + name, seed)
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
    """What layer 0 finds."""
    e = orc.cfg["embedding"]
    return orc.t["embed"][toks] * e["scale"] + orc.t["bigram"][LS.bigram_rows(toks, e["bigram"])]


# ------------------------------------------------------------------------------------------------ each mechanism alone
LINEAR = {"small": (3, 24, 40, 8.0), "one": (1, 8, 8, 1.0), "odd": (2, 11, 9, 5.0), "wide": (2, 128, 136, 16.0), "beyond": (1, 136, 40, 2.0)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(LINEAR))
@pytest.mark.parametrize("decay", ("mixed", "strong", "none"))
def test_gated_linear_attention_alone(root, dtype, name, decay):
    sizes = LS.linear_mixer(*LINEAR[name])
    cfg = LS.make_mokatar(104, 90, [("gla", sizes, None)], eps=1e-3)
    t = LS.random_tensors(cfg, 3)
    if decay != "mixed":      # almost nothing of a channel survives a token, or everything does
        t["l0.mix.a2.b"] = t["l0.mix.a2.b"] * 0 + (-60.0 if decay == "strong" else 40.0)
    if decay == "strong":     # then a token reads little but itself: q k must not vanish in front of the norm
        t["l0.mix.q"] = t["l0.mix.k"]
    m, orc = open_custom(root, cfg, t, dtype, f"{name}-{decay}")
    toks = U.tokens(cfg, 200, 4)
    e = embedded(orc, toks)
    want = orc.residuals(toks)[0] - e
    _, state = LS.linear_attention_states(orc.norm(e, "l0.norm1"), lambda n: orc.t["l0.mix." + n], sizes)
    lim = 1e-5 if dtype == "float32" else 4e-2
    for portions in PORTIONS:
        kv = m.new_cache(max_seq=256)
        got = traced(m, toks, portions, kv)[0] - e
        assert U.err(got, want) < lim, portions
        s = kv.read_state(0).reshape(state.shape)
        assert np.linalg.norm(s - state) < (1e-5 if dtype == "float32" else 2e-2) * np.linalg.norm(state), portions
        kv.close()
    m.close()


ATTENTION = {
    "head": ("attention", LS.head_normed_mixer()),
    "head_wide": ("attention", LS.head_normed_mixer(4, 2, 128, 96, 70, 7, LS.rotation_of(128, 5e5, factor=16.0, fast=32.0, original=64, slow=1.0))),
    "head_odd": ("attention", LS.head_normed_mixer(5, 5, 9, 13, 64, 64, LS.rotation_of(8, 30.0), 0.5)),
    "head_past": ("attention", LS.head_normed_mixer(7, 1, 40, 264, 500, 3)),
    "row": ("attention_2", LS.row_normed_mixer()),
    "row_wide": ("attention_2", LS.row_normed_mixer(6, 2, 128, 160, LS.rotation_of(96, 1e6, factor=5.0))),
    "row_odd": ("attention_2", LS.row_normed_mixer(3, 1, 7, 11, LS.rotation_of(2, 9.0), 0.7)),
    "row_blocks": ("attention_2", LS.row_normed_mixer(40, 2, 64, 64, LS.rotation_of(64, 200.0, factor=1.5))),     # more heads on a key head than one tile holds
    "row_many": ("attention_2", LS.row_normed_mixer(21, 7, 16, 24, LS.rotation_of(16, 200.0, factor=1.5))),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(ATTENTION))
def test_attention_alone(root, dtype, name):
    kind, mx = ATTENTION[name]
    cfg = LS.make_mokatar(104, 90, [(kind, mx, None)], eps=1e-3)
    t = LS.random_tensors(cfg, 5)
    t["l0.mix.q.norm"] = LS.bf16_round(t["l0.mix.q.norm"] * 2)       # single keys that decide
    m, orc = open_custom(root, cfg, t, dtype, name)
    toks = U.tokens(cfg, 200, 6)
    e = embedded(orc, toks)
    want = orc.residuals(toks)[0] - e
    h, w, G = orc.norm(e, "l0.norm1"), lambda n: orc.t["l0.mix." + n], mx["kv_heads"]
    k, v = h @ w("k").T, h @ w("v").T
    if kind == "attention":
        f, c = LS.rotation(mx["rot"], "yarn")
        k = LS.rotate(LS.rms_norm(k.reshape(200, G, -1), w("k.norm"), 1e-3), np.arange(200), f, c, True).reshape(200, -1)
    else:
        f, c = LS.rotation(mx["rot"], "linear")
        k = LS.rotate(LS.rms_norm(k + w("k.b"), w("k.norm"), 1e-3).reshape(200, G, -1), np.arange(200), f, c, False).reshape(200, -1)
        v = v + w("v.b")
    for portions in PORTIONS:
        kv = m.new_cache(max_seq=256)
        got = traced(m, toks, portions, kv)[0] - e
        assert U.err(got, want) < (2e-5 if dtype == "float32" else 8e-2), portions
        for which, x in ((0, k), (1, v)):
            assert np.abs(kv.read(0, which) - x).max() < (1e-5 if dtype == "float32" else 3e-2) * np.abs(x).max(), portions
        kv.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", (-50.0, 4.0, 12.0, 60.0))
def test_sinks_of_any_size(root, dtype, sink):
    """From none at all to one that takes everything, beside scores that stand out themselves."""
    cfg = LS.make_mokatar(64, 64, [("attention", LS.head_normed_mixer(4, 2, 16, 16, 30, 2), None)])
    t = LS.random_tensors(cfg, 8)
    t["l0.mix.q.norm"] = LS.bf16_round(t["l0.mix.q.norm"] * 2)
    t["l0.mix.sink"] = np.array([sink, sink / 2, -sink, 0.0], np.float32)
    m, orc = open_custom(root, cfg, t, dtype, f"sink{sink}")
    toks = U.tokens(cfg, 90, 9)
    want = orc.residuals(toks)[0] - embedded(orc, toks)
    for portions in ([90], [1] * 20 + [70], [31, 59]):
        kv = m.new_cache(max_seq=128)
        assert U.err(traced(m, toks, portions, kv)[0] - embedded(orc, toks), want) < (2e-5 if dtype == "float32" else 6e-2)
        kv.close()
    m.close()


EXPERTS = [(5, 2, 24), (1, 1, 40), (4, 4, 64), (8, 1, 130), (70, 6, 20), (300, 3, 8)]


@pytest.mark.parametrize("experts", EXPERTS)
@pytest.mark.parametrize("clear", (True, False))
def test_experts_alone(root, experts, clear):
    """The mixer writes nothing.  Batches from one token to several hundred: experts that many, few and no tokens use.  A router that reads
    the whole stream (float32) and one whose choices rounding cannot change."""
    cfg = LS.make_mokatar(104, 90, [("gla", LS.linear_mixer(1, 8, 8), experts)], eps=1e-3)
    t = LS.random_mokatar(cfg, 11, clear=clear)
    t["l0.mix.o"] = t["l0.mix.o"] * 0
    if clear:
        t["embed"][40:, :LS.MARKERS] = t["embed"][40, :LS.MARKERS]      # most tokens agree
    toks = U.tokens(cfg, 300, 12)
    for dtype in DTYPES if clear else DTYPES[:1]:
        m, orc = open_custom(root, cfg, t, dtype, f"moe{experts[0]}-{clear}")
        e = embedded(orc, toks)
        want = orc.residuals(toks)[0] - e
        if not clear:
            z = np.sort(orc.norm(e, "l0.norm2") @ orc.t["l0.mlp.router"].T + orc.t["l0.mlp.router.b"], axis=1)
            assert experts[0] == experts[1] or (z[:, -experts[1]] - z[:, -experts[1] - 1]).min() > 2e-5
        for portions in ([300], [1, 2, 16, 17, 32, 33, 64, 65, 70], [1] * 30 + [128, 142]):
            kv = m.new_cache(max_seq=320)
            assert U.err(traced(m, toks, portions, kv)[0] - e, want) < (1e-5 if dtype == "float32" else 3e-2), portions
            kv.close()
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("loop", ((0, 3, 3), (1, 2, 4), (2, 3, 1), None))
def test_embedding_loop_and_norms_alone(root, dtype, loop):
    """The mixers write nothing: embeddings, dense feed-forwards, passes of the loop, the last norm and the scaled head."""
    mx = LS.linear_mixer(1, 8, 8)
    cfg = LS.make_mokatar(104, 90, [("gla", mx, 88), ("gla", mx, None), ("gla", mx, 56)], loop, scale=7.5, logit_scale=1.7)
    t = LS.random_tensors(cfg, 7)
    for i in range(3):
        t[f"l{i}.mix.o"] *= 0
    m, orc = open_custom(root, cfg, t, dtype, f"ff{loop}")
    toks = U.tokens(cfg, 70)
    want = orc.residuals(toks)
    for portions in ([70], [1] * 10 + [2, 3, 20, 35]):
        kv = m.new_cache(max_seq=128)
        got = traced(m, toks, portions, kv)
        assert got.shape == want.shape
        for g, w in zip(got, want):
            assert U.err(g, w) < (3e-6 if dtype == "float32" else 3e-2)
        kv.close()
    kv = m.new_cache(max_seq=128)
    got = all_logits(m, toks, kv)
    lim = 1e-5 if dtype == "float32" else 3e-2
    assert U.err(got, orc.logits(toks)) < lim and np.abs(got - orc.logits(toks)).max() < 2 * lim * np.abs(got).max()
    kv.close(); m.close()


# ------------------------------------------------------------------------------------------------ edges of windows, kept tokens and pages
def _beacon(kind, window=None, keep=0):
    """The query of token 0 meets one key, token 1's, whose score stands out and whose value alone reaches the output."""
    none = LS.rotation_of(0, 10.0)
    mx = LS.head_normed_mixer(4, 2, 16, 16, window, keep, none, 1.0) if kind == "attention" else LS.row_normed_mixer(4, 2, 16, 16, none, 1.0)
    cfg = LS.make_mokatar(64, 64, [(kind, mx, None)], scale=1.0)
    t = LS.random_tensors(cfg, 11)
    rng = np.random.default_rng(12)
    emb = 0.3 * rng.standard_normal((64, 64)).astype(np.float32)
    emb[:, :8] = 0
    emb[0, 0], emb[1, 1] = 8.0, 8.0
    emb[2:, 2] = 4.0
    q, k, v = (np.zeros_like(t["l0.mix." + n]) for n in "qkv")
    q[::16, 0], q[1::16, 2] = 5.0, 5.0              # token 0 asks along one axis, the others along another
    k[::16, 1], k[1::16, 0], k[2::16, 2] = 5.0, 5.0, 5.0
    v[:] = LS.bf16_round(0.1 * rng.standard_normal(v.shape))
    v[:, 1] = 3.0 * np.sign(rng.standard_normal(len(v)))
    t.update({"embed": LS.bf16_round(emb), "bigram": 0 * t["bigram"], "l0.norm1": np.zeros(64, np.float32), "l0.mix.q": q, "l0.mix.k": k, "l0.mix.v": LS.bf16_round(v),
              "l0.mix.q.norm": np.full_like(t["l0.mix.q.norm"], 1.0), "l0.mix.k.norm": np.full_like(t["l0.mix.k.norm"], 1.0)})
    for n in "qkv":
        if kind == "attention_2":
            t[f"l0.mix.{n}.b"] = 0 * t[f"l0.mix.{n}.b"]
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
        assert (U.err(without, want) > 0.2) == seen, (i, j)
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
@pytest.mark.parametrize("window,keep", ((48, 0), (64, 4), (100, 70), (129, 1), (20, 66)))
def test_keys_just_inside_and_outside_a_window(root, dtype, window, keep):
    cfg, t = _beacon("attention", window, keep)
    m, orc = open_custom(root, cfg, t, dtype, f"beacon-{window}-{keep}")
    cases = []                                    # (query position, key position, seen)
    for i in (window, window + 1, 2 * window, 3 * window + 5, 127, 128, 129, 255, 256):
        for j in (i - window - 1, i - window, i - window + 1, i - 1, keep - 1, keep, 0):
            if 0 <= j < i:
                cases.append((i, j, i - j < window or j < keep))
    cases += [(i, j, i - j < window or j < keep) for i, j in ((1, 0), (65, 64), (64, 63), (192, 128), (300, 64), (300, 63))]
    _meet(m, orc, sorted(set(cases)), dtype, np.random.default_rng(13), 512)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_of_the_whole_past(root, dtype):
    """Also over more keys than one group of warps takes: the clusters of the row attention."""
    cfg, t = _beacon("attention_2")
    m, orc = open_custom(root, cfg, t, dtype, "beacon-far")
    _meet(m, orc, [(i, j, True) for i, j in ((1, 0), (64, 0), (64, 63), (129, 64), (700, 0), (700, 1), (700, 63), (700, 64), (700, 511), (700, 512), (1290, 0), (1290, 640), (1290, 1289))], dtype,
          np.random.default_rng(14), 1344)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_what_was_written_first_is_read_last(root, dtype):
    """Gated linear attention whose channels hardly decay: the first token still shows hundreds of tokens later, in prompts and decoded."""
    cfg = LS.make_mokatar(64, 64, [("gla", LS.linear_mixer(2, 64, 16, 16.0), None)])
    t = LS.random_tensors(cfg, 14)
    t["l0.mix.a2.b"] = t["l0.mix.a2.b"] * 0 + 12.0
    m, orc = open_custom(root, cfg, t, dtype, "far")
    toks = [int(x) for x in np.random.default_rng(16).integers(2, 64, 420)]
    toks[0], toks[-1] = 0, 0
    want = orc.logits(toks)
    assert U.err(orc.logits([1] + toks[1:])[-1:], want[-1:]) > 10 * U.F32_TOL
    lim = U.F32_TOL if dtype == "float32" else 4e-2
    kv = m.new_cache(max_seq=448, batch=2)
    assert U.err(all_logits(m, toks, kv, 0), want) < lim
    m.step([(1, toks[:20], [])], kv)
    assert U.err([m.forward(x, kv, seq=1) for x in toks[20:]], want[20:]) < lim
    kv.close(); m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ("all", "odd"))
def test_the_first_tokens(opened, dtype, name):
    """Sequences of one to twelve tokens, in every cut into two portions, in slots that other sequences have used."""
    m, orc = opened(name, dtype)
    cfg = U.MOKATAR[name]
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
@pytest.mark.parametrize("name", list(U.MOKATAR))
def test_prompt_decode_and_portions(opened, dtype, name):
    m, orc = opened(name, dtype)
    toks = U.tokens(U.MOKATAR[name], 170)
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
    cfg = LS.make_mokatar(104, 90, [("attention", LS.head_normed_mixer(), 40), ("attention_2", LS.row_normed_mixer(6, 2, 40, 24, LS.rotation_of(24, 500.0)), (5, 2, 24))])
    m, orc = open_custom(root, cfg, LS.random_tensors(cfg, 6), dtype, "long")
    toks = U.tokens(cfg, 1031, 8)
    kv = m.new_cache(max_seq=1088)
    assert U.err(all_logits(m, toks, kv), orc.logits(toks)) < tol(dtype)
    kv.close(); m.close()


def test_a_router_that_reads_the_whole_stream(root):
    """A whole model in 32 bits whose choices depend on everything."""
    cfg = U.MOKATAR["all"]
    m, orc = open_custom(root, cfg, LS.random_mokatar(cfg, 5, clear=False), "float32", "general")
    toks = U.tokens(cfg, 150, 3)
    want = orc.logits(toks)
    kv = m.new_cache(max_seq=192, batch=2)
    assert U.err(all_logits(m, toks, kv), want) < U.F32_TOL
    got = list(all_logits(m, toks[:50], kv, 1)) + [m.forward(t, kv, seq=1) for t in toks[50:]]
    assert U.err(got, want) < U.F32_TOL
    kv.close(); m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_equal_each_request_alone(opened, dtype):
    from forge_llm_b200.engine import Engine
    m, orc = opened("all", dtype)
    cfg = U.MOKATAR["all"]
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
    cfg = U.MOKATAR["all"]
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
@pytest.mark.parametrize("name", ("all", "loop_all"))
def test_long_decoding(opened, dtype, name):
    """From the third token to the three-hundredth one by one (graph replays), over many window, chunk and page borders."""
    m, orc = opened(name, dtype)
    toks = U.tokens(U.MOKATAR[name], 300, 50)
    want = orc.logits(toks)
    kv = m.new_cache(max_seq=320)
    m.forward_prefill(toks[:2], kv)
    assert U.err([m.forward(t, kv) for t in toks[2:]], want[2:]) < tol(dtype)
    kv.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch", (2, 19, 40))
def test_batched_decode_equals_each_alone(opened, dtype, batch):
    m, orc = opened("all", dtype)
    cfg = U.MOKATAR["all"]
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
    toks = U.tokens(U.MOKATAR["all"], 20, 5)
    kv = m.new_cache(max_seq=64)
    want = [i % 20 for i in range(45)]
    assert U.err(m.step([(0, toks, want)], kv)[0], orc.logits(toks)[want]) < BF16_MODEL
    kv.close()


# ------------------------------------------------------------------------------------------------ generation
def test_greedy_generation_everywhere(opened):
    """The session's greedy loop, the batched loop and the scheduler give the restatement's tokens (float32)."""
    from forge_llm_b200.engine import Engine, Sampling, Scheduler
    m, orc = opened("all", "float32")
    cfg = U.MOKATAR["all"]
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
    from forge_llm_b200._lib import ForgeError
    m, _ = opened("all", dtype)
    other, _ = opened("loop_all", dtype)
    cfg = U.MOKATAR["all"]
    kv = m.new_cache(max_seq=192, batch=3)
    m.step([(2, U.tokens(cfg, 50, 91), [])], kv)
    m.forward_prefill(U.tokens(cfg, 100, 90), kv, seq=0)
    blob = kv.save(0)
    kv.load(blob, 2)
    assert kv.len(2) == 100
    for x in (5, 6, 7, 8):
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
    m, orc = opened("loop_all", "float32")
    cfg = U.MOKATAR["loop_all"]
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
    folder, orc = U.make(root, "mokatar_all")
    cfg = U.MOKATAR["all"]
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
