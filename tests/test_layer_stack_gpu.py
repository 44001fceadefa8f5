"""Layer-list models on the GPU against the plain restatement: each mechanism alone, whole prompts, decoding, portions, mixed
batches, pages used again, long contexts, generation through the session calls, the scheduler and the command line."""
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


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return tmp_path_factory.mktemp("stack")


@pytest.fixture(scope="module")
def opened(root):
    """Open models, one per (configuration, type, gain)."""
    from forge_llm_b200 import runtime
    models = {}

    def get(name, dtype, gain=1.0, seed=0):
        key = (name, dtype, gain, seed)
        if key not in models:
            folder, orc = U.make(root, name, seed, gain)
            models[key] = (runtime.Model.open(folder, dtype), orc)
        return models[key]

    yield get
    for m, _ in models.values():
        m.close()


def open_custom(root, cfg, tensors, dtype, name):
    from forge_llm_b200 import runtime
    folder = str(root / name)
    LS.write_model(folder, cfg, tensors)
    return runtime.Model.open(folder, dtype), LS.LayerStack(cfg, tensors)


def last_logits(model, toks, cache, seq=0):
    return model.step([(seq, toks, [len(toks) - 1])], cache)[0][0]


def all_logits(model, toks, cache, seq=0):
    return model.step([(seq, toks, list(range(len(toks))))], cache)[0]


# ------------------------------------------------------------------------------------------------ each mechanism alone
def _one_layer(mlp=True, **mix):
    m = LS.mixer(**{**dict(heads=4, dim=24, rot_dim=16, vdim=20, kv_rank=48, base=900.0), **mix})
    return LS.make_config(104, 104, [(m, 88 if mlp else None, 0.8, None)], eps=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_dynamic_tanh_alone(root, dtype):
    """Mixer and feed-forward write nothing and the head is the identity: the logits are the final norm of the embedding."""
    cfg = _one_layer()
    t = LS.random_tensors(cfg, 5)
    t["l0.mix.o"] *= 0
    t["l0.mlp.down"] *= 0
    t["head"] = np.eye(104, dtype=np.float32)
    m, orc = open_custom(root, cfg, t, dtype, "dyt-" + dtype)
    kv = m.new_cache(max_seq=128)
    toks = U.tokens(cfg, 60)
    got = all_logits(m, toks, kv)
    want = LS.dynamic_tanh(orc.t["embed"][toks], orc.t["final.norm.alpha"], orc.t["final.norm"], orc.t["final.norm.b"])
    assert np.abs(got - want).max() < (2e-6 if dtype == "float32" else 1.2e-2)
    kv.close(); m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_alone(root, dtype):
    cfg = _one_layer()
    t = LS.random_tensors(cfg, 6)
    t["l0.mix.o"] *= 0
    m, orc = open_custom(root, cfg, t, dtype, "ff-" + dtype)
    kv = m.new_cache(max_seq=128)
    toks = U.tokens(cfg, 50)
    m.trace(True)
    m.forward_prefill(toks, kv)
    x = m.read_trace(50)[0]
    m.trace(False)
    e = orc.t["embed"][toks]
    h = orc.norm(e, "l0.norm1")
    gate = h @ orc.t["l0.mlp.gate"].T
    assert (gate > 0.8).mean() > 0.05 and (np.abs(h @ orc.t["l0.mlp.up"].T) > 0.8).mean() > 0.1   # every clamp is met
    want = LS.dense_ff(h, lambda n: orc.t["l0.mlp." + n], cfg["layers"][0]["mlp"])
    assert U.err(x - e, want) < (1e-5 if dtype == "float32" else 1.5e-2)
    kv.close(); m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", (20, 90))
def test_latents_and_rotated_keys(root, dtype, n):
    """What the cache holds: the normed latents and the rotated key parts (appended by single rows and by prompt portions)."""
    cfg = _one_layer(mlp=False)
    t = LS.random_tensors(cfg, 7)
    m, orc = open_custom(root, cfg, t, dtype, f"cache-{dtype}-{n}")
    kv = m.new_cache(max_seq=128)
    toks = U.tokens(cfg, n)
    m.forward_prefill(toks, kv)
    h = orc.norm(orc.t["embed"][toks], "l0.norm1")
    down = h @ orc.t["l0.mix.dkv"].T
    c = LS.rms_norm(down[:, :48], orc.t["l0.mix.dkv.norm"], 1e-2)
    r = LS.rotate_half(down[:, 48:], np.arange(n), 900.0, 16)
    lim = 1e-6 if dtype == "float32" else 1.5e-2
    assert np.abs(kv.read(0, 0) - c).max() < lim * max(1, np.abs(c).max())
    assert np.abs(kv.read(0, 1) - r).max() < lim * max(1, np.abs(r).max())
    kv.close(); m.close()


def _mixer_residual(m, toks, portions, kv):
    """Trace of layer 0 over the whole prompt, fed in portions."""
    m.trace(True)
    out, at = [], 0
    for n in portions:
        m.step([(0, toks[at:at + n], [])], kv)
        out.append(m.read_trace(n)[0])
        at += n
    m.trace(False)
    assert at == len(toks)
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("what", ("all", "rotated_only", "unrotated_only", "gate", "scale"))
def test_latent_attention_alone(root, dtype, what):
    cfg = _one_layer(mlp=False, scale=0.9 if what == "scale" else None)
    t = LS.random_tensors(cfg, 8)
    if what == "rotated_only":        # only the shared rotated part makes the scores
        t["l0.mix.uk"] *= 0
        t = U.sharp(t, cfg, 3.0)
    if what == "unrotated_only":
        t["l0.mix.dkv"][48:] = 0
    if what == "gate":
        t["l0.mix.g"] = LS.bf16_round(t["l0.mix.g"] * 3)
    m, orc = open_custom(root, cfg, t, dtype, f"mla-{dtype}-{what}")
    toks = U.tokens(cfg, 140, seed=9)
    e = orc.t["embed"][toks]
    want = orc.residuals(toks)[0] - e
    for portions in ([140], [33, 1, 2, 60, 1, 31, 12], [1] * 5 + [135]):
        kv = m.new_cache(max_seq=192)
        got = _mixer_residual(m, toks, portions, kv) - e
        kv.close()
        assert U.err(got, want) < (1e-5 if dtype == "float32" else 2.5e-2), portions
    m.close()


# ------------------------------------------------------------------------------------------------ one far key
def _beacon(root, dtype, name, key_pos, n, heads=2):
    """A model in which the query of the last token meets one key whose score stands out: tokens 0 and 1 are the query and the
    key, the latents of token 1 are large along one direction, and only it carries a value that reaches the output."""
    cfg = LS.make_config(64, 64, [(LS.mixer(heads=heads, dim=16, rot_dim=8, vdim=16, kv_rank=32, base=1e4, scale=1.0), None, 1.0, None)], eps=1e-5)
    t = LS.random_tensors(cfg, 11)
    rng = np.random.default_rng(12)
    emb = 0.3 * rng.standard_normal((64, 64)).astype(np.float32)
    emb[:, :4] = 0
    emb[0, 0], emb[1, 1] = 4.0, 4.0      # the query's and the key's marks
    t["embed"] = LS.bf16_round(emb)
    t["l0.norm1"] = np.ones(64, np.float32)
    t["l0.norm1.b"] = np.zeros(64, np.float32)
    t["l0.norm1.alpha"] = np.asarray(0.5, np.float32)
    q = np.zeros_like(t["l0.mix.q"])
    dkv = LS.bf16_round(0.2 * t["l0.mix.dkv"])
    dkv[:, 0] = 0
    dkv[0, :] = 0
    dkv[0, 1] = 4.0                       # latent 0 is the key's mark
    uk = np.zeros_like(t["l0.mix.uk"])
    for h in range(heads):
        q[h * 24, 0] = 4.0
        uk[h * 16, 0] = 1.5
    t.update({"l0.mix.q": q, "l0.mix.dkv": dkv, "l0.mix.uk": uk, "l0.mix.dkv.norm": np.ones(32, np.float32)})
    toks = [int(x) for x in np.random.default_rng(13).integers(2, 64, n)]
    toks[key_pos], toks[-1] = 1, 0
    return cfg, t, toks


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,key_pos", [(2, 0), (65, 0), (65, 63), (66, 64), (129, 0), (193, 127), (193, 128), (400, 0), (400, 63), (400, 64), (400, 398)])
def test_one_key_stands_out(root, dtype, n, key_pos):
    cfg, t, toks = _beacon(root, dtype, "b", key_pos, n)
    m, orc = open_custom(root, cfg, t, dtype, f"beacon-{dtype}-{n}-{key_pos}")
    want = orc.logits(toks)
    lost = list(toks)
    lost[key_pos] = 5                     # the same sequence without the key answers differently
    assert U.err(orc.logits(lost)[-1:], want[-1:]) > 10 * U.BF16_TOL
    kv = m.new_cache(max_seq=448, batch=2)
    assert U.err(last_logits(m, toks, kv)[None], want[-1:]) < U.tol(dtype)            # in a prompt's portion
    if n > 2:
        m.step([(1, toks[:-1], [])], kv)
    else:
        m.step([(1, toks[:1], [])], kv)
    assert U.err(m.forward(toks[-1], kv, seq=1)[None], want[-1:]) < U.tol(dtype)      # decoded
    kv.close(); m.close()


# ------------------------------------------------------------------------------------------------ prompts, decoding, portions
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", U.BOLENEX_NAMES)
def test_prompt_decode_and_portions(opened, dtype, name):
    m, orc = opened(name, dtype)
    toks = U.tokens(U.CONFIGS[name], 150)
    want = orc.logits(toks)
    kv = m.new_cache(max_seq=192, batch=3)
    whole = all_logits(m, toks, kv, 0)
    assert U.err(whole, want) < U.tol(dtype)
    # the first tokens, one by one from nothing, then a portion, then single tokens again
    got = [m.forward(t, kv, seq=1) for t in toks[:3]]
    got += list(all_logits(m, toks[3:120], kv, 1))
    got += [m.forward(t, kv, seq=1) for t in toks[120:]]
    assert U.err(got, want) < U.tol(dtype)
    at, got = 0, []
    for n in (2, 37, 2, 3, 31, 32, 2, 41):
        got += list(all_logits(m, toks[at:at + n], kv, 2))
        at += n
    assert at == 150 and U.err(got, want) < U.tol(dtype)
    kv.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sharp_attention(opened, dtype):
    """Single keys decide (the restatement's own tests show that a lost one would be seen)."""
    m, orc = opened("mixed", dtype, 5.0, 3)
    toks = U.tokens(U.CONFIGS["mixed"], 150)
    want = orc.logits(toks)
    kv = m.new_cache(max_seq=192, batch=2)
    lim = 1e-4 if dtype == "float32" else 0.12
    assert U.err(all_logits(m, toks, kv, 0), want) < lim
    m.step([(1, toks[:-30], [])], kv)
    assert U.err([m.forward(t, kv, seq=1) for t in toks[-30:]], want[-30:]) < lim
    kv.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_equal_each_request_alone(opened, dtype):
    from forge_llm_b200.engine import Engine
    m, orc = opened("mixed", dtype)
    cfg = U.CONFIGS["mixed"]
    lens = {"a": 170, "b": 9, "c": 64, "d": 129, "e": 1, "f": 200, "g": 65, "h": 130}
    toks = {k: U.tokens(cfg, n, seed=i) for i, (k, n) in enumerate(lens.items())}
    want = {k: orc.logits(v) for k, v in toks.items()}
    eng = Engine(m, pool_tokens=640, slots=4)       # far less than all requests together: pages and slots are used again
    rng = np.random.default_rng(21)
    fed, waiting, live, seen = {k: 0 for k in lens}, list(lens), [], {k: [] for k in lens}
    reserved = 0
    pages = {k: -(-n // 64) * 64 for k, n in lens.items()}
    slots_used = []
    while waiting or live:
        while waiting and len(live) < 4 and reserved + pages[waiting[0]] <= 640:
            k = waiting.pop(0)
            live.append(k)
            reserved += pages[k]
        entries = []
        for k in live:
            if len(live) > 1 and rng.random() < 0.2:
                continue                             # left out of this step
            n = int(min(lens[k] - fed[k], rng.choice([1, 1, 2, 3, 17, 31, 32, 33, 64, 100])))
            entries.append((k, toks[k][fed[k]:fed[k] + n], list(range(n))))
        if not entries:
            continue
        for (k, t, _), rows in zip(entries, eng.step(entries)):
            seen[k] += list(rows)
            fed[k] += len(t)
            assert eng.length(k) == fed[k]
        for k in [k for k in live if fed[k] == lens[k]]:
            slots_used.append(eng._slot[k])
            eng.release(k)
            live.remove(k)
            reserved -= pages[k]
    assert len(slots_used) == 8 and len(set(slots_used)) <= 4
    assert eng.cache.free_tokens() == 640
    for k in lens:
        assert U.err(seen[k], want[k]) < U.tol(dtype), k
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_do_not_matter(opened, dtype):
    """The same steps on a fresh cache and on one whose pages were used by others, in another order: the same bits."""
    m, orc = opened("mixed", dtype)
    cfg = U.CONFIGS["mixed"]
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
    y = play(kv2, 3, 0)
    assert np.array_equal(x, y)
    kv1.close(); kv2.close()


def test_pool_limits_and_errors(opened):
    from forge_llm_b200._lib import ForgeError
    m, _ = opened("mixed", "bfloat16")
    cfg = U.CONFIGS["mixed"]
    kv = m.new_cache(max_seq=192, batch=3, pool_tokens=256)
    assert kv.free_tokens() == 256
    m.step([(0, U.tokens(cfg, 129), [])], kv)
    assert kv.free_tokens() == 64 and kv.len(0) == 129
    bad = [([(1, U.tokens(cfg, 65), [])], 3), ([(0, U.tokens(cfg, 64), [])], 3), ([(1, [203], [])], 1), ([(1, [1], [1])], 1),
           ([(1, [1], []), (1, [2], [])], 1), ([(3, [1], [])], 1), ([(1, [], [])], 1)]
    for entries, code in bad:
        with pytest.raises(ForgeError) as e:
            m.step(entries, kv)
        assert e.value.code == code, entries
        assert kv.len(0) == 129 and kv.len(1) == 0
    m.step([(0, U.tokens(cfg, 63), []), (1, U.tokens(cfg, 64), [])], kv)
    assert kv.free_tokens() == 0
    kv.free_seq(0)
    assert kv.free_tokens() == 192 and kv.len(0) == 0
    kv.close()


# ------------------------------------------------------------------------------------------------ long runs and generation
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(opened, dtype):
    """From the third token to the three-hundredth one by one (graph replays), over several page borders."""
    m, orc = opened("no_mlp", dtype)
    toks = U.tokens(U.CONFIGS["no_mlp"], 300, 50)
    want = orc.logits(toks)
    kv = m.new_cache(max_seq=320)
    m.forward_prefill(toks[:2], kv)
    got = [m.forward(t, kv) for t in toks[2:]]
    assert U.err(got, want[2:]) < U.tol(dtype)
    kv.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_decode_equals_each_alone(opened, dtype):
    m, orc = opened("mixed", dtype)
    cfg = U.CONFIGS["mixed"]
    B = 19                                # more rows than one activation tile of the smallest product
    seqs = [U.tokens(cfg, 20 + 7 * i, 60 + i) for i in range(B)]
    kv = m.new_cache(max_seq=192, batch=B)
    for b in range(B):
        m.forward_prefill(seqs[b][:-3], kv, seq=b)
    for k in (3, 2, 1):
        lg = m.forward_batch([s[len(s) - k] for s in seqs], kv)
    want = np.stack([orc.logits(s)[-1] for s in seqs])
    assert U.err(lg, want) < U.tol(dtype)
    kv.close()


def test_greedy_generation_everywhere(opened):
    """The session's greedy loop, the sampling loop, the batched loop and the scheduler give the restatement's tokens (float32)."""
    from forge_llm_b200.engine import Engine, Sampling, Scheduler
    m, orc = opened("mixed", "float32")
    cfg = U.CONFIGS["mixed"]
    prompts = [U.tokens(cfg, n, 70 + n) for n in (3, 40, 64, 75)]
    want = [orc.generate_greedy(p, 12) for p in prompts]
    kv = m.new_cache(max_seq=128, batch=4)
    for p, w in zip(prompts, want):
        kv.reset()
        assert list(m.generate_greedy(p, 12, kv)) == w
    kv.reset()
    for b, p in enumerate(prompts):
        m.forward_prefill(p, kv, seq=b)
    out = m.decode_greedy_batch([w[0] for w in want], 11, kv)
    for b in range(4):
        # a row of the history is the token each sequence was fed
        assert list(out[:, b]) == want[b][:11]
    kv.close()
    eng = Engine(m, pool_tokens=256, slots=3)
    s = Scheduler(eng, step_tokens=48)
    for i, p in enumerate(prompts):
        s.submit(i, p, 12, Sampling())
    got = s.run()
    assert [got[i] for i in range(4)] == want
    eng.close()


def test_sampling_and_scoring_take_the_model(opened):
    import ctypes as C
    from forge_llm_b200._lib import ForgeSampling, check, lib
    m, orc = opened("mixed", "float32")
    cfg = U.CONFIGS["mixed"]
    prompt = np.array(U.tokens(cfg, 30, 80), np.uint32)
    kv = m.new_cache(max_seq=96)
    out, n = np.empty(10, np.uint32), C.c_int32()
    sp = ForgeSampling(0.0, 0, 0.9, 1.0, 1)
    check(lib.forge_generate(m._h, kv._h, prompt.ctypes.data, prompt.size, 10, C.byref(sp), None, 0, out.ctypes.data, C.byref(n)))
    assert n.value == 10 and list(out) == orc.generate_greedy(prompt, 10)
    toks = U.tokens(cfg, 40, 81)
    lg = orc.logits(toks)
    lse = np.log(np.exp(lg - lg.max(-1, keepdims=True)).sum(-1)) + lg.max(-1)
    want = np.mean([lse[i] - lg[i, toks[i + 1]] for i in range(39)])
    mean, _, count = m.score_corpus(toks, kv)
    assert count == 39 and abs(mean - want) < 1e-4
    kv.close()


def test_cache_persistence(opened):
    from forge_llm_b200._lib import ForgeError
    m, _ = opened("mixed", "bfloat16")
    other, _ = opened("no_mlp", "bfloat16")
    cfg = U.CONFIGS["mixed"]
    toks = U.tokens(cfg, 100, 90)
    kv = m.new_cache(max_seq=192, batch=2)
    m.forward_prefill(toks, kv, seq=0)
    blob = kv.save(0)
    kv.load(blob, 1)
    assert kv.len(1) == 100
    assert np.array_equal(m.forward(5, kv, seq=0), m.forward(5, kv, seq=1))
    okv = other.new_cache(max_seq=192)
    with pytest.raises(ForgeError):
        okv.load(blob)
    kv.close(); okv.close()


def test_scratch_growth_between_caches_and_steps(opened):
    """A captured decode step survives the growth of the step buffers by a later prompt and by a longer cache's tables."""
    m, orc = opened("one_head", "float32")
    cfg = U.CONFIGS["one_head"]
    toks = U.tokens(cfg, 60, 91)
    kv = m.new_cache(max_seq=64)
    m.forward_prefill(toks[:10], kv)
    got = [m.forward(t, kv) for t in toks[10:20]]
    kv2 = m.new_cache(max_seq=2048, batch=3)
    m.step([(0, U.tokens(cfg, 700, 92), []), (1, U.tokens(cfg, 30, 93), []), (2, U.tokens(cfg, 300, 94), [])], kv2)
    got += [m.forward(t, kv) for t in toks[20:]]
    assert U.err(got, orc.logits(toks)[10:]) < U.F32_TOL
    kv.close(); kv2.close()


def test_quantised_decoder_takes_steps_too():
    """The step call and the pool serve the framework's quantised decoders (last place of an entry only)."""
    from forge_llm_b200 import configs, runtime, synth
    from forge_llm_b200._lib import ForgeError
    c = configs.tiny(8, hd=64, nq=4, nkv=2, layers=2)
    m = runtime.Model(c, synth.make_weights_bin(c))
    toks = [int(t) for t in synth.prompt_tokens(c, 90)]
    kv = m.new_cache(max_seq=128, batch=2)
    want = [m.forward_prefill(toks[:70], kv, seq=0), m.forward(toks[70], kv, seq=0)]
    pool = m.new_cache(max_seq=128, batch=3, pool_tokens=256)
    m.step([(1, toks[:64], [])], pool)
    pool.free_seq(1)
    (a, b) = m.step([(2, toks[:70], [69]), (0, toks[:5], [])], pool)
    assert np.array_equal(a[0], want[0]) and len(b) == 0
    assert np.array_equal(m.step([(2, [toks[70]], [0])], pool)[0][0], want[1])
    with pytest.raises(ForgeError) as e:
        m.step([(1, toks[:5], [0])], pool)
    assert e.value.code == 6
    kv.close(); pool.close(); m.close()


# ------------------------------------------------------------------------------------------------ programs
def test_replay_program(root, tmp_path):
    folder, orc = U.make(root, "mixed")
    cfg = U.CONFIGS["mixed"]
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
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
        for s, rows in want.items():
            got = np.fromfile(out / f"{s}.f32", "<f4").reshape(len(rows), cfg["vocab"])
            assert U.err(got, rows) < U.tol(dtype)


def test_command_line_generation(root, capsys):
    from forge_llm_b200.__main__ import main
    folder, orc = U.make(root, "mixed")
    cfg = U.CONFIGS["mixed"]
    prompts = [U.tokens(cfg, n, 97 + n) for n in (5, 50)]
    args = ["generate", "--model", folder, "--dtype", "float32", "--max-new", "6", "--repeat-penalty", "1.0"]
    for p in prompts:
        args += ["--prompt", ",".join(map(str, p))]
    assert main(args) == 0
    lines = capsys.readouterr().out.strip().splitlines()
    assert [[int(x) for x in l.split()] for l in lines] == [orc.generate_greedy(p, 6) for p in prompts]
