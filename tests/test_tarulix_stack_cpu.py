"""The Tarulix design without a GPU: the plain restatement by hand, planted mistakes, configurations and their errors."""
import copy
import math
from fractions import Fraction

import numpy as np
import pytest

import stack_util as U
from oracle import layer_stack as LS


# ------------------------------------------------------------------------------------------------ the restatement
@pytest.mark.parametrize("count,longest", ((16, 128), (32, 256), (16, 240), (2, 9), (5, 50), (12, 6 * 3 ** 6), (8, 4)))
def test_buckets_begin_where_the_logarithms_say(count, longest):
    """Against whole numbers: bucket half + k begins at the least n with (n / half)^(count - half) >= (longest / half)^k."""
    half = count // 2
    for n in range(1, min(longest, 2000) + 40):
        want = n if n < half else count - 1
        if n >= half and longest > half:
            k = 0
            while k < count - half and Fraction(n, half) ** (count - half) >= Fraction(longest, half) ** (k + 1):
                k += 1
            want = min(count - 1, half + k)
        if longest > half or n < half:
            assert LS.distance_bucket(n, count, longest) == want, n


def test_blocks_and_windows():
    assert [LS.blocks_seen(i, 4, 3) for i in range(12)] == [0, 0, 0, 0, 0, 0, 1, 1, 1, 2, 2, 2]    # the block 0 .. 2 leaves the window of 4 at 6
    assert [LS.blocks_seen(i, 1, 1) for i in range(4)] == [0, 1, 2, 3] and LS.blocks_seen(50, None, 3) == 0
    assert LS.windowed(5, 2).tolist() == [False] * 4 + [True] * 2 and LS.windowed(3).all()


def test_a_block_is_one_key():
    q, k = np.zeros((7, 1, 2)), np.zeros((7, 1, 2))
    v = np.arange(7.0).reshape(7, 1, 1)
    o = LS.pooled_attention(q, k, v, 1.0, None, 4, 3, np.eye(1))
    assert np.allclose(o[:, 0, 0], [0, 0.5, 1, 1.5, 2.5, 3.5, (1 + 3 + 4 + 5 + 6) / 5])    # position 5 sees neither token 0, 1 nor a block
    k[0, 0, 0], q[6, 0, 0] = 3.0, 3.0      # its mean key is what counts, and the cap
    w = np.exp(5.0 * math.tanh(3.0 / 5.0))
    o = LS.pooled_attention(q, k, v, 1.0, 5.0, 4, 3, np.eye(1))
    assert np.isclose(o[6, 0, 0], (w * 1 + 18) / (w + 4))


def test_mixed_heads_meet_their_own_values():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((5, 4, 3)), rng.standard_normal((5, 2, 3)), rng.standard_normal((5, 2, 2))
    T = rng.standard_normal((4, 4))
    o = LS.pooled_attention(q, k, v, 0.7, None, None, None, T)
    for i in range(5):
        p = np.stack([LS.soft_weights(q[i, h] @ k[:i + 1, h // 2].T * 0.7) for h in range(4)])
        for h in range(4):
            assert np.allclose(o[i, h], sum(T[h, g] * p[g] for g in range(4)) @ v[:i + 1, h // 2])


def test_a_sink_and_a_bias():
    q, k, v = np.zeros((3, 2, 4)), np.zeros((3, 1, 4)), np.arange(1.0, 4.0).reshape(3, 1, 1)
    rel = np.log(np.array([[1.0, 1.0], [2.0, 1.0], [1.0, 1.0], [4.0, 1.0]]))
    o = LS.biased_attention(q, k, v, 1.0, rel, 4, np.array([0.0, math.log(5.0)]), None)
    assert np.allclose(o[:, 0, 0], [1 / 2, (2 * 1 + 2) / 4, (1 * 1 + 2 * 2 + 3) / 5]) and np.allclose(o[:, 1, 0], [1 / 6, 3 / 7, 6 / 8])


def test_selective_scan_by_hand():
    x, dt = np.array([[1.0], [2.0]]), np.array([[0.5], [0.25]])
    y, S = LS.selective_scan(x, dt, np.array([[-1.0, -2.0]]), np.array([[1.0, 3.0], [2.0, 1.0]]), np.array([[1.0, 1.0], [2.0, 0.5]]), np.array([10.0]))
    s0 = np.array([0.5, 1.5])
    s1 = np.exp(0.25 * np.array([-1.0, -2.0])) * s0 + 0.5 * np.array([2.0, 1.0])
    assert np.allclose(S[0], s1) and np.allclose(y[:, 0], [2.0 + 10, s1 @ [2.0, 0.5] + 20])


def test_routing():
    z, c = np.log(np.array([[1.0, 2.0, 3.0, 4.0]])), np.array([0.35, 0.0, 0.0, 0.0])
    chosen, w = LS.route_corrected(z, c, 2)
    assert chosen.tolist() == [[0, 3]] and np.allclose(w, [[0.1, 0.4]])
    t = {"router": np.zeros((3, 2)), "correction": np.array([0.0, 0.0, 1.0]), "shared.gate": np.zeros((1, 2)), "shared.up": np.zeros((1, 2)), "shared.down": np.zeros((2, 1))}
    h = np.array([[3.0, -6.0]])
    out = LS.shared_mixture_ff(h, t.__getitem__, {"router": {"experts": 2, "identity": 1, "top": 1}})
    assert np.allclose(out, h / 3)      # what is passed on, times its weight


def test_values_are_blended_with_the_first_layers():
    cfg = U.TARULIX["all"]
    m = LS.LayerStack(cfg, LS.random_tensors(cfg, 0))
    toks, seen, keep = U.tokens(cfg, 9), [], LS.blended_values

    def watch(v, first, lam):
        seen.append((first, float(lam)))
        return keep(v, first, lam)

    LS.blended_values = watch
    try:
        r = m.residuals(toks)
    finally:
        LS.blended_values = keep
    own = (r[0] @ m.t["l1.mix.v"].T + m.t["l1.mix.v.b"]).reshape(9, 2, 40)
    assert len(seen) == 2 and all(np.allclose(f, own) for f, _ in seen) and [x for _, x in seen] == [float(m.t["l3.mix.vmix"]), float(m.t["l5.mix.vmix"])]


def test_planted_mistakes_show():
    """None of these would pass the tolerances of the GPU tests."""
    cfg = U.TARULIX["all"]
    m = LS.LayerStack(cfg, LS.random_tensors(cfg, 1))
    toks = U.tokens(cfg, 130)
    want = m.logits(toks)
    names = ("windowed", "blocks_seen", "distance_bucket", "biased_attention", "pooled_attention", "blended_values", "selective_scan", "selective_mixer", "short_convolution", "route_corrected", "shared_mixture_ff",
             "rotate_half", "unit_rms", "attention_beside_scan")
    keep = {n: getattr(LS, n) for n in names}

    def err(**kw):
        for n, f in kw.items():
            setattr(LS, n, f)
        try:
            return U.err(m.logits(toks), want)
        finally:
            for n, f in keep.items():
                setattr(LS, n, f)

    pooled, biased, scan, routed = keep["pooled_attention"], keep["biased_attention"], keep["selective_scan"], keep["route_corrected"]
    assert err() == 0.0
    wrong = {
        "window one more": err(windowed=lambda i, s=None: keep["windowed"](i, s + 1 if s else None)),
        "window one less": err(windowed=lambda i, s=None: keep["windowed"](i, s - 1 if s else None)),
        "a block early": err(blocks_seen=lambda i, s, p: keep["blocks_seen"](i + 1, s, p)),
        "a block late": err(blocks_seen=lambda i, s, p: keep["blocks_seen"](i - 1, s, p)),
        "no blocks": err(blocks_seen=lambda i, s, p: 0),
        "the bias scaled": err(biased_attention=lambda q, k, v, s, rel, *a: biased(q, k, v, s, rel * s, *a)),
        "a bias one distance off": err(distance_bucket=lambda n, b, d: keep["distance_bucket"](n + 1, b, d)),
        "no sink": err(biased_attention=lambda q, k, v, s, rel, d, sink, w: biased(q, k, v, s, rel, d, sink - 1e9, w)),
        "scaled sink": err(biased_attention=lambda q, k, v, s, rel, d, sink, w: biased(q, k, v, s, rel, d, sink * s, w)),
        "no cap": err(pooled_attention=lambda q, k, v, s, cap, *a: pooled(q, k, v, s, None, *a)),
        "heads mixed the other way": err(pooled_attention=lambda q, k, v, s, c, w, p, t: pooled(q, k, v, s, c, w, p, t.T)),
        "heads not mixed": err(pooled_attention=lambda q, k, v, s, c, w, p, t: pooled(q, k, v, s, c, w, p, np.eye(len(t)))),
        "not blended": err(blended_values=lambda v, f, lam: v),
        "blended the other way": err(blended_values=lambda v, f, lam: lam * v + (1 - lam) * f),
        "positions one off after a break": err(rotate_half=lambda x, p, b, d: keep["rotate_half"](x, p + (p > 60), b, d)),
        "state lost once": err(selective_scan=lambda x, dt, A, B, C, D: (np.concatenate([scan(x[:64], dt[:64], A, B[:64], C[:64], D)[0], scan(x[64:], dt[64:], A, B[64:], C[64:], D)[0]]), None)),
        "read before the write": err(selective_scan=lambda x, dt, A, B, C, D: (scan(x, dt, A, B, np.concatenate([0 * C[:1], C[:-1]]), D)[0], None)),
        "no skip": err(selective_scan=lambda x, dt, A, B, C, D: scan(x, dt, A, B, C, 0 * D)),
        "one tap lost": err(short_convolution=lambda x, t: keep["short_convolution"](x, np.concatenate([0 * t[:, :1], t[:, 1:]], 1))),
        "weights corrected": err(route_corrected=lambda z, c, top: ((r := routed(z, c, top))[0], r[1] + c[r[0]])),
        "weights renormalised": err(route_corrected=lambda z, c, top: ((r := routed(z, c, top))[0], r[1] / r[1].sum(1, keepdims=True))),
        "no correction": err(route_corrected=lambda z, c, top: routed(z, 0 * c, top)),
        "sides swapped": err(attention_beside_scan=lambda h, w, mx, e: keep["attention_beside_scan"](h, w, {**mx, "left_scale": mx["right_scale"], "right_scale": mx["left_scale"]}, e)),
    }
    small = {k: v for k, v in wrong.items() if v < 20 * U.F32_TOL}
    assert not small, wrong


def test_routers_of_the_test_models_are_clear():
    """In the models that run in bfloat16 no choice of an expert is close."""
    for name, cfg in U.TARULIX.items():
        m = LS.LayerStack(cfg, LS.random_tensors(cfg, 0))
        gaps, keep = [], LS.route_corrected

        def watch(z, c, top):
            e = np.exp(z - z.max(1, keepdims=True))
            s = np.sort(e / e.sum(1, keepdims=True) + c, axis=1)[:, ::-1]
            if top < z.shape[1]:
                gaps.append((s[:, top - 1] - s[:, top]).min())
            return keep(z, c, top)

        LS.route_corrected = watch
        try:
            m.residuals(U.tokens(cfg, 80))
        finally:
            LS.route_corrected = keep
        assert min(gaps, default=1) > 0.02, (name, min(gaps))


# ------------------------------------------------------------------------------------------------ configurations
def _folder(tmp_path, change=lambda c: None, tensors=lambda t: None):
    cfg = copy.deepcopy(U.TARULIX["all"])
    t = LS.random_tensors(cfg, 0)
    change(cfg)
    tensors(t)
    LS.write_model(str(tmp_path), cfg, t)
    return str(tmp_path)


def _info(folder):
    from forge_llm_b200 import runtime
    return runtime.checkpoint_info(folder)


def test_checkpoint_info(tmp_path):
    i = _info(_folder(tmp_path))
    assert i["architecture"] == "Tarulix" and (i["num_layers"], i["num_weight_layers"]) == (6, 6)
    assert i["cache_values_per_token"] == 128 * (2 + 2 + 4 + 2 + 1 + 2)
    assert i["state_values_per_sequence"] == 72 * 16 + 4 * 72 + 40 * 6 + 3 * 40


@pytest.mark.parametrize("change,code,text", [
    (lambda c: c["layers"][0].update(type="gla"), 6, "mixer"),
    (lambda c: c["layers"][0].update(type="attention"), 2, "heads"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), 2, "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), 2, "size"),
    (lambda c: c["layers"][1]["mixer"].pop("bias_max"), 2, "bias_max"),
    (lambda c: c["layers"][1]["mixer"].update(dim=600), 6, "600"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].pop("pool"), 2, "pool"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(pool=0), 2, "pool"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1), 2, "softcap"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=26), 2, "rot"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), 2, "left"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), 2, "left_scale"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), 2, "inner"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("dt_rank"), 2, "dt_rank"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(state=300), 6, "300 states"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(conv=3), 2, "conv"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), 2, "top 8 of 7"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=3), 2, "router"),
    (lambda c: c["layers"][0]["mlp"]["router"].pop("identity"), 2, "identity"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(experts=600), 6, "602 experts"),
    (lambda c: c["layers"][0]["mlp"].pop("shared"), 2, "ff"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense", ff=24), 6, "feed-forward"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=32), 2, "blended"),
    (lambda c: c["norm"].pop("eps"), 2, "eps"),
])
def test_configuration_errors(tmp_path, change, code, text):
    from forge_llm_b200._lib import ForgeError
    with pytest.raises(ForgeError) as e:
        _info(_folder(tmp_path, change))
    assert e.value.code == code and text in str(e.value), e.value


def test_tensor_errors(tmp_path):
    from forge_llm_b200._lib import ForgeError
    for i, (name, value, text) in enumerate([("l1.mix.sink", None, "l1.mix.sink is missing"), ("l1.mix.k.b", None, "l1.mix.k.b is missing"), ("l1.mix.rel", None, "rel"), ("l1.mix.rel", np.ones((16, 5)), "l1.mix.rel has shape"),
                                             ("l3.mix.vmix", None, "l3.mix.vmix is missing"), ("l0.mix.left.talk", np.ones((6, 5)), "l0.mix.left.talk has shape"), ("l0.mix.left.o.b", None, "l0.mix.left.o.b is missing"),
                                             ("l0.mix.right.conv.b", None, "l0.mix.right.conv.b is missing"), ("l0.mix.right.x", np.ones((43, 72)), "l0.mix.right.x has shape"), ("l0.mlp.e4.down", None, "l0.mlp.e4.down is missing"),
                                             ("l0.mlp.shared.up", None, "l0.mlp.shared.up is missing"), ("l0.mlp.correction", None, "l0.mlp.correction is missing"), ("l0.norm1", np.ones(136), "l0.norm1 has shape"),
                                             ("l0.norm2", None, "l0.norm2 is missing")]):
        def edit(t):
            t.pop(name) if value is None else t.update({name: np.asarray(value, np.float32)})
        with pytest.raises(ForgeError) as e:
            _info(_folder(tmp_path / str(i), tensors=edit))
        assert text in str(e.value), e.value


def test_shapes_of_the_synthetic_writer_agree(tmp_path):
    from forge_llm_b200 import synth
    cfg = synth.tarulix_config(128, 6, 4, 48, 77, dim=32, window=32)
    synth.write_stack(str(tmp_path), cfg)
    i = _info(str(tmp_path))
    assert i["num_layers"] == 6
    t = LS.read_safetensors(str(tmp_path / "model.safetensors"))
    assert t["l0.mlp.e7.gate"].std() > 0.05 and t["l0.mix.left.talk"].shape == (4, 4)
