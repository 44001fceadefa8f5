"""The Robazen design on the GPU against the plain restatement: each mechanism alone, states, chunk borders, prompts, portions,
decoding, mixed batches, slots and pages used again, long runs, generation through the session calls, scheduler and programs."""
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
BF16_MODEL = 0.16        # worst row of a whole random model in bfloat16; single mechanisms are held to far less below


def tol(dtype):
    return U.F32_TOL if dtype == "float32" else BF16_MODEL


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return tmp_path_factory.mktemp("recurrent")


@pytest.fixture(scope="module")
def opened(root):
    from forge_llm_b200 import runtime
    models = {}

    def get(name, dtype, seed=0):
        key = (name, dtype, seed)
        if key not in models:
            folder, orc = U.make(root, "robazen_" + name, seed)
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


PORTIONS = ([200], [65, 1, 2, 64, 1, 31, 36], [1] * 6 + [130] + [2, 3, 4, 16, 15, 24], [17, 63, 120])


# ------------------------------------------------------------------------------------------------ each mechanism alone
MIXERS = {
    "delta": ("delta", dict(heads=4, kv_heads=2, dim=24, vdim=40, conv=4)),
    "delta_long_taps": ("delta", dict(heads=3, kv_heads=3, dim=32, vdim=16, conv=9)),
    "delta_odd": ("delta", dict(heads=2, kv_heads=1, dim=11, vdim=9, conv=3)),
    "delta_128": ("delta", dict(heads=2, kv_heads=2, dim=128, vdim=96, conv=4)),
    "channel": ("channel_delta", dict(heads=4, kv_heads=2, dim=24, vdim=40, conv=4)),
    "channel_128": ("channel_delta", dict(heads=2, kv_heads=1, dim=128, vdim=136, conv=2)),
    "channel_odd": ("channel_delta", dict(heads=3, kv_heads=3, dim=6, vdim=10, conv=1)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MIXERS))
@pytest.mark.parametrize("decay", ("mixed", "strong", "none"))
def test_delta_rules_alone(root, dtype, name, decay):
    kind, sizes = MIXERS[name]
    cfg = LS.make_robazen(104, 90, [(kind, sizes, None)], eps=1e-3)
    t = LS.random_tensors(cfg, 3)
    if decay != "mixed":      # logarithms of -30 and more per token, or none at all
        t["l0.mix.A_log"] = t["l0.mix.A_log"] * 0 + (3.5 if decay == "strong" else -30.0)
    m, orc = open_custom(root, cfg, t, dtype, f"{name}-{decay}")
    toks = U.tokens(cfg, 200, 4)
    e = orc.t["embed"][toks]
    want = orc.residuals(toks)[0] - e
    h = orc.norm(e, "l0.norm1")
    _, state = getattr(LS, {"delta": "gated_delta_states", "channel_delta": "channel_delta_states"}[kind])(h, lambda n: orc.t["l0.mix." + n], sizes)
    lim = 1e-5 if dtype == "float32" else 4e-2
    states = []
    for portions in PORTIONS:
        kv = m.new_cache(max_seq=256)
        got = traced(m, toks, portions, kv)[0] - e
        assert U.err(got, want) < lim, portions
        s = kv.read_state(0).reshape(state.shape)
        assert np.linalg.norm(s - state) < (1e-5 if dtype == "float32" else 2e-2) * np.linalg.norm(state), portions
        states.append(s)
        kv.close()
    for s in states[1:]:      # however the prompt was cut: the same state, up to what another order of sums moves
        assert np.linalg.norm(s - states[0]) < (1e-5 if dtype == "float32" else 6e-3) * np.linalg.norm(states[0])
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("side", ("left", "right", "both"))
@pytest.mark.parametrize("sizes", (dict(), dict(heads=5, kv_heads=1, dim=72, vdim=16, chunk=100, heads_r=2, dim_r=64), dict(heads=3, kv_heads=3, dim=9, vdim=130, chunk=64, heads_r=1, dim_r=128)))
def test_attention_and_time_mixing_alone(root, dtype, side, sizes):
    mx = LS.pair_mixer(**sizes)
    cfg = LS.make_robazen(104, 90, [("parallel", mx, None)], eps=1e-3)
    t = LS.random_tensors(cfg, 5)
    if side == "left":
        t["l0.mix.right.out"] *= 0
    if side == "right":
        t["l0.mix.left.out"] *= 0
    t["l0.mix.left.q"] = LS.bf16_round(t["l0.mix.left.q"] * 4)       # scores that reach the cap, single keys that decide
    m, orc = open_custom(root, cfg, t, dtype, f"pair-{side}-{mx['left']['mask']['size']}")
    toks = U.tokens(cfg, 200, 6)
    e = orc.t["embed"][toks]
    want = orc.residuals(toks)[0] - e
    h = orc.norm(e, "l0.norm1")
    s = (h @ orc.t["l0.mix.left.q"].T)[:, :mx["left"]["dim"]] @ (h @ orc.t["l0.mix.left.k"].T)[:, :mx["left"]["dim"]].T * mx["left"]["scale"]
    assert np.abs(s).max() > 0.5 * mx["left"]["softcap"]
    _, state = LS.time_mix_states(h, lambda n: orc.t["l0.mix.right." + n], mx["right"])
    for portions in PORTIONS:
        kv = m.new_cache(max_seq=256)
        got = traced(m, toks, portions, kv)[0] - e
        assert U.err(got, want) < (2e-5 if dtype == "float32" else 8e-2), portions
        s = kv.read_state(0).reshape(state.shape)
        assert np.linalg.norm(s - state) < (1e-5 if dtype == "float32" else 1e-2) * np.linalg.norm(state), portions
        k = (h @ orc.t["l0.mix.left.k"].T)
        assert np.abs(kv.read(0, 0) - k).max() < (1e-5 if dtype == "float32" else 3e-2) * np.abs(k).max()
        kv.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_and_loop_alone(root, dtype):
    """The mixers write nothing: a stream of feed-forwards, of passes through the loop, and of norms."""
    mx = LS.delta_mixer(2, 1, 8, 8, 2)
    cfg = LS.make_robazen(104, 90, [("delta", mx, 88), ("delta", mx, None), ("delta", mx, 56)], (0, 2, 3))
    t = LS.random_tensors(cfg, 7)
    for i in range(3):
        t[f"l{i}.mix.o"] *= 0
    m, orc = open_custom(root, cfg, t, dtype, "ff")
    kv = m.new_cache(max_seq=128)
    toks = U.tokens(cfg, 60)
    got, want = traced(m, toks, [60], kv), orc.residuals(toks)
    assert got.shape == want.shape == (7, 60, 104)
    assert np.array_equal(want[1], want[0]) and U.err(want[2], want[0]) > 0.1     # a pass changes the stream, an empty layer does not
    for g, w in zip(got, want):
        assert U.err(g, w) < (3e-6 if dtype == "float32" else 3e-2)
    kv.close(); m.close()


# ------------------------------------------------------------------------------------------------ edges of chunks and pages
def _beacon(chunk):
    """The query of token 0 meets one key, token 1's, whose score stands out and whose value alone reaches the output."""
    mx = LS.pair_mixer(heads=4, kv_heads=2, dim=16, vdim=16, chunk=chunk, softcap=40.0, scale=1.0, heads_r=1, dim_r=8)
    cfg = LS.make_robazen(64, 64, [("parallel", mx, None)])
    t = LS.random_tensors(cfg, 11)
    rng = np.random.default_rng(12)
    emb = 0.3 * rng.standard_normal((64, 64)).astype(np.float32)
    emb[:, :4] = 0
    emb[0, 0], emb[1, 1] = 4.0, 4.0
    t["embed"] = LS.bf16_round(emb)
    t["l0.norm1"], t["l0.norm1.b"], t["l0.norm1.alpha"] = np.ones(64, np.float32), np.zeros(64, np.float32), np.asarray(0.5, np.float32)
    q, k = np.zeros_like(t["l0.mix.left.q"]), LS.bf16_round(0.1 * t["l0.mix.left.k"])
    q[::16, 0] = 5.0
    k[::16] = 0
    k[::16, 1] = 5.0
    v = LS.bf16_round(0.3 * t["l0.mix.left.v"])
    v[:, 1] = 3.0 * np.sign(rng.standard_normal(len(v)))
    t.update({"l0.mix.left.q": q, "l0.mix.left.k": k, "l0.mix.left.v": v, "l0.mix.right.out": 0 * t["l0.mix.right.out"], "l0.mix.left.g": 0 * t["l0.mix.left.g"]})
    return cfg, t


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", (48, 64, 100, 129))
def test_keys_just_inside_and_outside_a_chunk(root, dtype, chunk):
    cfg, t = _beacon(chunk)
    m, orc = open_custom(root, cfg, t, dtype, f"beacon-{chunk}")
    rng = np.random.default_rng(13)
    cases = []                                    # (query position, key position, seen)
    for c in (1, 2, 3):
        b = c * chunk
        cases += [(b, b - 1, False), (b, b, None), (b + 1, b, True), (b + 1, b - 1, False), (b - 1, b - chunk, True), (b + chunk - 1, b, True), (b + chunk - 1, b - 1, False)]
    cases += [(1, 0, True), (chunk - 1, 0, True), (chunk, 0, False)] + [(p, p - 1, p % chunk != 0) for p in (64, 65, 128, 129, 192)]
    kv = m.new_cache(max_seq=576, batch=3)
    for i, j, seen in cases:
        if seen is None:
            continue
        toks = [int(x) for x in rng.integers(2, 64, i + 1)]
        toks[j], toks[i] = 1, 0
        lost = list(toks)
        lost[j] = 5
        want, without = orc.logits(toks)[-1:], orc.logits(lost)[-1:]
        assert (U.err(without, want) > 0.5) == seen, (i, j)
        lim = U.F32_TOL if dtype == "float32" else 5e-2
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
    kv.close(); m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_what_was_written_first_is_read_last(root, dtype):
    """Delta rules without decay: the first token's value comes back hundreds of tokens later, in prompts and decoded."""
    cfg = LS.make_robazen(64, 64, [("delta", LS.delta_mixer(2, 2, 64, 16, 1), None), ("channel_delta", LS.delta_mixer(2, 1, 64, 16, 1), None)])
    t = LS.random_tensors(cfg, 14)
    emb = LS.bf16_round(np.random.default_rng(15).standard_normal((64, 64)))
    for i in range(2):
        t[f"l{i}.mix.A_log"] = t[f"l{i}.mix.A_log"] * 0 - 40.0
        t[f"l{i}.mix.b"] = t[f"l{i}.mix.b"] * 0 - LS.bf16_round(np.full_like(t[f"l{i}.mix.b"], 0.02))
    t["embed"] = emb
    m, orc = open_custom(root, cfg, t, dtype, "far")
    toks = [int(x) for x in np.random.default_rng(16).integers(2, 64, 420)]
    toks[0], toks[-1] = 0, 0
    lost = list(toks)
    lost[0] = 1
    want = orc.logits(toks)
    lim = U.F32_TOL if dtype == "float32" else 4e-2
    assert U.err(orc.logits(lost)[-1:], want[-1:]) > 10 * U.F32_TOL
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
    cfg = U.ROBAZEN[name]
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
@pytest.mark.parametrize("name", list(U.ROBAZEN))
def test_prompt_decode_and_portions(opened, dtype, name):
    m, orc = opened(name, dtype)
    toks = U.tokens(U.ROBAZEN[name], 170)
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
def test_mixed_batches_equal_each_request_alone(opened, dtype):
    from forge_llm_b200.engine import Engine
    m, orc = opened("all", dtype)
    cfg = U.ROBAZEN["all"]
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
    cfg = U.ROBAZEN["all"]
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
    """From the third token to the three-hundredth one by one (graph replays), over many chunk and page borders."""
    m, orc = opened(name, dtype)
    toks = U.tokens(U.ROBAZEN[name], 300, 50)
    want = orc.logits(toks)
    kv = m.new_cache(max_seq=320)
    m.forward_prefill(toks[:2], kv)
    assert U.err([m.forward(t, kv) for t in toks[2:]], want[2:]) < tol(dtype)
    kv.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_decode_equals_each_alone(opened, dtype):
    m, orc = opened("all", dtype)
    cfg = U.ROBAZEN["all"]
    B = 19
    seqs = [U.tokens(cfg, 20 + 7 * i, 60 + i) for i in range(B)]
    kv = m.new_cache(max_seq=192, batch=B)
    for b in range(B):
        m.forward_prefill(seqs[b][:-3], kv, seq=b)
    for k in (3, 2, 1):
        lg = m.forward_batch([s[len(s) - k] for s in seqs], kv)
    assert U.err(lg, np.stack([orc.logits(s)[-1] for s in seqs])) < tol(dtype)
    kv.close()


def test_many_keys_in_one_row(root):
    """Rows over more keys than one group of warps takes: the clusters of the row attention."""
    cfg = LS.make_robazen(64, 64, [("parallel", LS.pair_mixer(heads=4, kv_heads=2, dim=16, vdim=24, chunk=5000, heads_r=1, dim_r=8), None)])
    t = LS.random_tensors(cfg, 18)
    toks = U.tokens(cfg, 1300, 19)
    for dtype in DTYPES:
        m, orc = open_custom(root, cfg, t, dtype, "keys")
        want = orc.logits(toks[:1290] + toks[1290:])[1285:]
        kv = m.new_cache(max_seq=1344)
        m.step([(0, toks[:1285], [])], kv)
        got = [m.forward(x, kv) for x in toks[1285:]]
        assert U.err(got, want) < (U.F32_TOL if dtype == "float32" else 4e-2)
        kv.close(); m.close()


# ------------------------------------------------------------------------------------------------ generation
def test_greedy_generation_everywhere(opened):
    """The session's greedy loop, the batched loop and the scheduler give the restatement's tokens (float32)."""
    from forge_llm_b200.engine import Engine, Sampling, Scheduler
    m, orc = opened("all", "float32")
    cfg = U.ROBAZEN["all"]
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
    cfg = U.ROBAZEN["all"]
    toks = U.tokens(cfg, 100, 90)
    kv = m.new_cache(max_seq=192, batch=3)
    m.step([(2, U.tokens(cfg, 50, 91), [])], kv)
    m.forward_prefill(toks, kv, seq=0)
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
    cfg = U.ROBAZEN["loop_all"]
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
    folder, orc = U.make(root, "robazen_all")
    cfg = U.ROBAZEN["all"]
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
