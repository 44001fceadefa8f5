"""The Robazen design without a GPU: the plain restatement against itself, planted mistakes, configurations and their errors."""
import copy
import os

import numpy as np
import pytest

import stack_util as U
from oracle import layer_stack as LS


# ------------------------------------------------------------------------------------------------ the restatement
def test_short_convolution():
    x = np.arange(12.0).reshape(6, 2)
    w = np.array([[0.5, 2.0, 1.0], [0.0, 0.0, 1.0]])
    y = LS.short_convolution(x, w)
    assert np.allclose(y[:, 1], x[:, 1])
    assert np.isclose(y[0, 0], x[0, 0]) and np.isclose(y[1, 0], x[1, 0] + 2 * x[0, 0]) and np.isclose(y[5, 0], x[5, 0] + 2 * x[4, 0] + 0.5 * x[3, 0])


def test_delta_rule_replaces_what_a_key_holds():
    """beta = 1 and no decay: reading a key gives the value written last under it; orthogonal keys do not disturb each other."""
    k = np.eye(3)[[0, 1, 0, 2]][:, None, :]
    v = np.arange(8.0).reshape(4, 1, 2) + 1
    one = np.ones((4, 1))
    o, S = LS.delta_rule(k, k, v, one, np.ones((4, 1, 3)))
    assert np.allclose(o, v) and np.allclose(S[0][0], v[2, 0]) and np.allclose(S[0][1], v[1, 0])
    # the decay acts before the correction, on the rows of key channels
    g = np.ones((4, 1, 3))
    g[2, 0, 1] = 0.25
    _, S = LS.delta_rule(k, k, v, one, g)
    assert np.allclose(S[0][1], 0.25 * v[1, 0]) and np.allclose(S[0][0], v[2, 0])


def test_chunked_attention_sees_its_chunk_only():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((11, 4, 5)), rng.standard_normal((11, 2, 5)), rng.standard_normal((11, 2, 3))
    a = LS.chunked_attention(q, k, v, 0.7, 5.0, 4)
    k2, v2 = k.copy(), v.copy()
    k2[:4], v2[:4] = 7.0, -7.0
    b = LS.chunked_attention(q, k2, v2, 0.7, 5.0, 4)
    assert np.allclose(a[4:], b[4:]) and not np.allclose(a[:4], b[:4])
    assert np.allclose(a[8], np.repeat(v[8], 2, axis=0))       # the first of a chunk sees itself
    whole = LS.chunked_attention(q, k, v, 0.7, 1e9, 100)
    for h in range(4):
        s = q[10, h] @ k[:, h // 2].T * 0.7
        e = np.exp(s - s.max())
        assert np.allclose(whole[10, h], e @ v[:, h // 2] / e.sum())


def test_time_mixing_bonus_and_decay():
    m = {"heads": 1, "dim": 2}
    W = 2
    t = {"mu." + s: np.zeros(2) for s in "rkvgw"}
    t.update({s: np.eye(2) for s in "rkvg"})
    t.update({"w1": np.zeros((1, 2)), "w2": np.zeros((2, 1)), "w0": np.log(-np.log(np.array([0.5, 0.25]))), "u": np.array([[2.0, 3.0]])})
    h = np.array([[1.0, 0.0], [1.0, 0.0], [1.0, 1.0]])
    o, S = LS.time_mix_states(h, lambda n: t[n], m)
    assert np.allclose(o[0, 0], 2.0 * h[0])                    # the bonus alone
    assert np.allclose(o[1, 0], h[0] + 2.0 * h[1])             # the token before is not decayed yet
    assert np.allclose(S[0], np.diag([0.5, 0.25]) @ (np.diag([0.5, 0.25]) @ np.outer(h[0], h[0]) + np.outer(h[1], h[1])) + np.outer(h[2], h[2]))


def test_runs_of_a_loop():
    cfg = U.ROBAZEN["all"]
    assert LS.layer_runs(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert LS.layer_runs(U.ROBAZEN["loop_all"]) == [(0, 0), (1, None), (0, 1), (1, None), (0, 2), (1, None)]
    assert LS.layer_runs(U.ROBAZEN["wide"]) == [(0, None), (1, None), (2, None)]


def _attempt(m, toks, **kw):
    keep = {n: getattr(LS, n) for n in kw}
    for n, f in kw.items():
        setattr(LS, n, f)
    try:
        return m.logits(toks)
    finally:
        for n, f in keep.items():
            setattr(LS, n, f)


def test_planted_mistakes_show():
    """None of these would pass the tolerances of the GPU tests."""
    cfg = U.ROBAZEN["all"]
    m = LS.LayerStack(cfg, LS.random_tensors(cfg, 1))
    toks = U.tokens(cfg, 110)
    want = m.logits(toks)
    keep = LS.chunked_attention, LS.token_shift, LS.short_convolution, LS.delta_rule, LS.unit, LS.layer_runs, LS.softplus

    def err(**kw):
        return U.err(_attempt(m, toks, **kw), want)

    assert err() == 0.0
    wrong = {
        "chunk one off": err(chunked_attention=lambda q, k, v, s, c, n: keep[0](q, k, v, s, c, n + 1)),
        "no cap": err(chunked_attention=lambda q, k, v, s, c, n: keep[0](q, k, v, s, 1e9, n)),
        "no shift": err(token_shift=lambda h, mu: h),
        "one tap lost": err(short_convolution=lambda x, w: keep[2](x, np.concatenate([0 * w[:, :1], w[:, 1:]], 1))),
        "taps reversed": err(short_convolution=lambda x, w: keep[2](x, w[:, ::-1])),
        "no decay": err(delta_rule=lambda q, k, v, b, g: keep[3](q, k, v, b, np.ones_like(g))),
        "read before the write": err(delta_rule=lambda q, k, v, b, g: (np.concatenate([0 * v[:1], keep[3](q, k, v, b, g)[0][:-1]]), None)),
        "unit with the mean": err(unit=lambda x: x / np.sqrt((x * x).mean(-1, keepdims=True) + 1e-6)),
        "the loop's entry skipped": err(layer_runs=lambda c: [(i, None) for i, _ in keep[5](c)]),
        "the passes swapped": err(layer_runs=lambda c: [(i, None if t is None else 1 - t) for i, t in keep[5](c)]),
        "softplus without the bias of zero": err(softplus=lambda z: keep[6](z + 0.05)),
    }
    small = {k: v for k, v in wrong.items() if v < 20 * U.F32_TOL}
    assert not small, wrong

    lost = list(toks)
    lost[0] = (lost[0] + 1) % cfg["vocab"]
    assert U.err(m.logits(lost)[-1:], want[-1:]) > 10 * U.F32_TOL     # the first token is remembered over two chunks' borders


# ------------------------------------------------------------------------------------------------ configurations
def _folder(tmp_path, change=lambda c: None, tensors=lambda t: None):
    cfg = copy.deepcopy(U.ROBAZEN["all"])
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
    assert i["architecture"] == "Robazen" and (i["num_layers"], i["num_weight_layers"]) == (6, 4)
    assert i["cache_values_per_token"] == 2 * (64 + 64)
    d0, c1 = 4 * 24 * 40 + 4 * (2 * 48 + 160), 6 * 16 * 24 + 3 * (2 * 48 + 144)
    assert i["state_values_per_sequence"] == 3 * 40 * 40 + 136 + 2 * d0 + 2 * c1 + 4 * 24 * 40 + 2 * (2 * 48 + 160)


@pytest.mark.parametrize("change,code,text", [
    (lambda c: c.update(architecture="Bolenex"), 6, "mixer"),
    (lambda c: c["layers"][1].update(type="window"), 6, "mixer"),
    (lambda c: c["layers"][1].update(mixer=None), 2, "mixer"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), 2, "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), 2, "conv"),
    (lambda c: c["layers"][1]["mixer"].update(conv=40), 6, "taps"),
    (lambda c: c["layers"][1]["mixer"].update(dim=300), 6, "300"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=0), 2, "vdim"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1.0), 2, "softcap"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), 2, "size"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), 2, "heads"),
    (lambda c: c["layers"][0]["mlp"].update(kind="routed"), 6, "feed-forward"),
    (lambda c: c["loop"].update(stop=5), 2, "loop"),
    (lambda c: c["loop"].update(start=3), 2, "loop"),
    (lambda c: c["loop"].pop("times"), 2, "times"),
    (lambda c: c["loop"].update(times=3), 2, "loop.step"),
    (lambda c: c["layers"][3].update(weights_of=1), 2, "weights_of"),
])
def test_configuration_errors(tmp_path, change, code, text):
    from forge_llm_b200._lib import ForgeError
    with pytest.raises(ForgeError) as e:
        _info(_folder(tmp_path, change))
    assert e.value.code == code and text in str(e.value), e.value


def test_tensor_errors(tmp_path):
    from forge_llm_b200._lib import ForgeError
    for i, (name, value, text) in enumerate([("l1.mix.A_log", None, "l1.mix.A_log is missing"), ("l2.mix.a1", None, "l2.mix.a1"), ("l2.mix.a2", np.ones((96, 19)), "l2.mix.a2 has shape"),
                                             ("l0.mix.right.w1", np.ones(20), "no matrix"), ("l3.norm2.alpha", None, "l3.norm2.alpha is missing"), ("loop.in", np.ones((136, 136)), "loop.in has shape")]):
        def edit(t):
            t.pop(name) if value is None else t.update({name: np.asarray(value, np.float32)})
        with pytest.raises(ForgeError) as e:
            _info(_folder(tmp_path / str(i), tensors=edit))
        assert text in str(e.value), e.value


def test_shapes_of_the_synthetic_writer_agree(tmp_path):
    from forge_llm_b200 import synth
    cfg = synth.robazen_config(128, 8, 2, 48, 77, dim=64, chunk=32)
    synth.write_stack(str(tmp_path), cfg)
    i = _info(str(tmp_path))
    assert i["num_layers"] == 8 and i["num_weight_layers"] == 4
    t = LS.read_safetensors(os.path.join(str(tmp_path), "model.safetensors"))
    assert np.array_equal(t["l1.mix.q"], t["l3.mix.q"]) and t["l1.mix.q"].std() > 0.05
