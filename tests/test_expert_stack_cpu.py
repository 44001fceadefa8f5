"""The Mokatar design without a GPU: the plain restatement against itself, planted mistakes, configurations and their errors."""
import copy
import math

import numpy as np
import pytest

import stack_util as U
from oracle import layer_stack as LS


# ------------------------------------------------------------------------------------------------ the restatement
def test_visible_keys():
    assert LS.visible(9, 4, 2).tolist() == [True, True, False, False, False, False, True, True, True, True]
    assert LS.visible(3, 4, 2).all() and LS.visible(4, 4, 0).tolist() == [False, True, True, True, True]
    assert LS.visible(5).all() and LS.visible(5, 2, 9).all()


def test_a_sink_takes_its_share():
    q, k, v = np.zeros((3, 2, 4)), np.zeros((3, 1, 4)), np.arange(1.0, 4.0).reshape(3, 1, 1)
    o = LS.sink_attention(q, k, v, 1.0, np.array([0.0, math.log(5.0)]))
    assert np.allclose(o[:, 0, 0], [1 / 2, 3 / 3, 6 / 4]) and np.allclose(o[:, 1, 0], [1 / 6, 3 / 7, 6 / 8])
    gone = LS.sink_attention(q, k, v, 1.0, np.array([-1e9, 800.0]))
    assert np.allclose(gone[:, 0, 0], [1, 1.5, 2]) and np.allclose(gone[:, 1], 0)


def test_rotations():
    rng = np.random.default_rng(0)
    x, pos = rng.standard_normal((7, 2, 10)), np.arange(7) + 3
    f, c = LS.rotation(LS.rotation_of(6, 50.0), "yarn")
    assert c == 1.0 and np.allclose(f, [1, 50 ** (-1 / 3), 50 ** (-2 / 3)])
    inter, halves = LS.rotate(x, pos, f, c, True), LS.rotate(x, pos, f, c, False)
    z = (x[..., 0:6:2] + 1j * x[..., 1:6:2]) * np.exp(1j * pos[:, None, None] * f)
    assert np.allclose(inter[..., 0:6:2], z.real) and np.allclose(inter[..., 1:6:2], z.imag) and np.array_equal(inter[..., 6:], x[..., 6:])
    order = [0, 2, 4, 1, 3, 5, 6, 7, 8, 9]
    back = np.argsort(order)
    assert np.allclose(halves, LS.rotate(x[..., back], pos, f, c, True)[..., order])
    assert np.allclose(LS.rotation(LS.rotation_of(6, 50.0, factor=4.0), "linear")[0], f / 4)


def test_a_ramp_between_kept_and_divided_frequencies():
    rot = LS.rotation_of(32, 10000.0, factor=8.0, fast=4.0, original=512, slow=1.0)
    f, c = LS.rotation(rot, "yarn")
    plain, _ = LS.rotation(LS.rotation_of(32, 10000.0), "yarn")
    turns = 512 * plain / (2 * math.pi)
    r = plain / f
    assert np.allclose(r[turns > 8], 1) and np.allclose(r[turns < 0.5], 8) and (np.diff(r) > -1e-12).all() and ((r > 1.01) & (r < 7.9)).any()
    assert abs(c - (0.1 * math.log(8) + 1)) < 1e-15


def test_linear_attention_by_hand():
    m = {"heads": 1, "dim": 2, "vdim": 1, "tau": 2.0}
    t = {"q": np.eye(2), "k": np.eye(2), "v": np.array([[1.0, 1.0]]), "a1": np.zeros((1, 2)), "a2": np.zeros((2, 1)), "a2.b": np.log(np.array([0.25, 0.5]) / np.array([0.75, 0.5]))}
    h = np.array([[1.0, 0.0], [0.0, 2.0], [1.0, 1.0]])
    o, S = LS.linear_attention_states(h, lambda n: t[n], m)
    g = np.array([0.25, 0.5]) ** 0.5
    s = np.zeros(2)
    for i in range(3):
        s = g * s + h[i] * h[i].sum()
        assert np.isclose(o[i, 0, 0], s @ h[i] / math.sqrt(2))
    assert np.allclose(S[0][:, 0], s)


def test_routing():
    chosen, w = LS.route(np.array([[0.0, 3.0, 1.0, 3.0 + math.log(2)], [5.0, 4.0, 3.0, 2.0]]), 2)
    assert chosen.tolist() == [[3, 1], [0, 1]] and np.allclose(w[0], [2 / 3, 1 / 3]) and np.allclose(w.sum(1), 1)
    cfg = LS.make_mokatar(20, 11, [("gla", LS.linear_mixer(1, 4, 4), (4, 4, 6))])
    t = {k[3:]: v for k, v in LS.random_mokatar(cfg, 1).items() if k.startswith("l0.")}
    h = np.random.default_rng(2).standard_normal((3, 20))
    z = h @ t["mlp.router"].T + t["mlp.router.b"]
    e = np.exp(z) / np.exp(z).sum(1, keepdims=True)
    want = sum(e[:, i:i + 1] * LS.silu_glu_ff(h, lambda n: t[f"mlp.e{i}.{n}"]) for i in range(4))
    assert np.allclose(LS.mixture_ff(h, lambda n: t["mlp." + n], cfg["layers"][0]["mlp"]), want)


def test_bigram_rows():
    assert LS.bigram_rows([4, 9, 2], {"buckets": 10, "mul_prev": 7, "mul_cur": 3}) == [10, (28 + 27) % 10, (63 + 6) % 10]


def test_loop_adds_the_embedding_before_later_passes():
    cfg = copy.deepcopy(U.MOKATAR["loop_all"])
    t = LS.random_tensors(cfg, 3)
    for n in t:
        if n.endswith(("mix.o", ".down")):
            t[n] = t[n] * 0
    m = LS.LayerStack(cfg, t)
    toks = U.tokens(cfg, 5)
    r, s = m.residuals(toks), m.t["loop.step"]
    x0 = r[0] - s[0]
    assert np.allclose(r[2], 2 * x0 + s[0] + s[1]) and np.allclose(r[4], 3 * x0 + s.sum(0))
    b = cfg["embedding"]
    assert np.allclose(x0[0], b["scale"] * m.t["embed"][toks[0]] + m.t["bigram"][-1])


def test_planted_mistakes_show():
    """None of these would pass the tolerances of the GPU tests."""
    cfg = U.MOKATAR["all"]
    m = LS.LayerStack(cfg, LS.random_tensors(cfg, 1))
    toks = U.tokens(cfg, 110)
    want = m.logits(toks)
    keep = {n: getattr(LS, n) for n in ("visible", "rotation", "rotate", "sink_attention", "linear_attention_states", "route", "bigram_rows", "layer_runs", "rms_norm")}

    def err(**kw):
        for n, f in kw.items():
            setattr(LS, n, f)
        try:
            return U.err(m.logits(toks), want)
        finally:
            for n, f in keep.items():
                setattr(LS, n, f)

    def decays(h, w, mx, f):
        return keep["linear_attention_states"](h, w, {**mx, "tau": f(mx["tau"])})

    assert err() == 0.0
    wrong = {
        "window one more": err(visible=lambda i, size=None, k=0: keep["visible"](i, size + 1 if size else None, k)),
        "window one less": err(visible=lambda i, size=None, k=0: keep["visible"](i, size - 1 if size else None, k)),
        "a kept token less": err(visible=lambda i, size=None, k=0: keep["visible"](i, size, k - 1)),
        "a kept token more": err(visible=lambda i, size=None, k=0: keep["visible"](i, size, k + 1)),
        "no sink": err(sink_attention=lambda q, k, v, s, sink, *a: keep["sink_attention"](q, k, v, s, sink - 1e9, *a)),
        "scaled sink": err(sink_attention=lambda q, k, v, s, sink, *a: keep["sink_attention"](q, k, v, s, sink * s, *a)),
        "layouts swapped": err(rotate=lambda x, p, f, c, i: keep["rotate"](x, p, f, c, not i)),
        "positions one off after a break": err(rotate=lambda x, p, f, c, i: keep["rotate"](x, p + (p > 60), f, c, i)),
        "no scaling": err(rotation=lambda r, k: keep["rotation"]({**r, "scaling": None}, k)),
        "cos and sin not scaled": err(rotation=lambda r, k: (keep["rotation"](r, k)[0], 1.0)),
        "tau left out": err(linear_attention_states=lambda h, w, mx: decays(h, w, mx, lambda t: 1.0)),
        "read before the write": err(linear_attention_states=lambda h, w, mx: (np.concatenate([0 * (o := keep["linear_attention_states"](h, w, mx)[0])[:1], o[:-1]]), None)),
        "softmax over all experts": err(route=lambda z, top: (keep["route"](z, top)[0], np.take_along_axis(np.exp(z) / np.exp(z).sum(1, keepdims=True), keep["route"](z, top)[0], 1))),
        "one expert less": err(route=lambda z, top: keep["route"](z, top - 1)),
        "first token's row": err(bigram_rows=lambda t, b: [0 if i == 0 else r for i, r in enumerate(keep["bigram_rows"](t, b))]),
        "the token before lost once": err(bigram_rows=lambda t, b: [b["buckets"] if i == 64 else r for i, r in enumerate(keep["bigram_rows"](t, b))]),
        "the passes swapped": err(layer_runs=lambda c: [(i, None if t is None else 1 - t) for i, t in keep["layer_runs"](c)]),
    }
    small = {k: v for k, v in wrong.items() if v < 20 * U.F32_TOL}
    assert not small, wrong


def test_routers_of_the_test_models_are_clear():
    """In the models that run in bfloat16 no choice of an expert is close."""
    for name, cfg in U.MOKATAR.items():
        m = LS.LayerStack(cfg, LS.random_tensors(cfg, 0))
        gaps = []
        keep = LS.route

        def watch(z, top):
            s = np.sort(z, axis=1)[:, ::-1]
            if top < z.shape[1]:
                gaps.append((s[:, top - 1] - s[:, top]).min())
            return keep(z, top)

        LS.route = watch
        try:
            m.residuals(U.tokens(cfg, 80))
        finally:
            LS.route = keep
        assert min(gaps, default=1) > 0.02, (name, min(gaps))


# ------------------------------------------------------------------------------------------------ configurations
def _folder(tmp_path, change=lambda c: None, tensors=lambda t: None):
    cfg = copy.deepcopy(U.MOKATAR["all"])
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
    assert i["architecture"] == "Mokatar" and (i["num_layers"], i["num_weight_layers"]) == (6, 4)
    assert i["cache_values_per_token"] == 2 * (2 * (64 + 64) + 4 * (64 + 64))
    assert i["state_values_per_sequence"] == 3 * 24 * 40 + 2 * 16 * 24 + 1


@pytest.mark.parametrize("change,code,text", [
    (lambda c: c.update(architecture="Robazen"), 6, "mixer"),
    (lambda c: c["layers"][0].update(type="delta"), 6, "mixer"),
    (lambda c: c["layers"][0].update(type="latent_attention"), 6, "mixer"),
    (lambda c: c.pop("embedding"), 2, "scale"),
    (lambda c: c["embedding"]["bigram"].pop("mul_prev"), 2, "mul_prev"),
    (lambda c: c["embedding"]["bigram"].update(buckets=60), 2, "bigram"),
    (lambda c: c.pop("logit_scale"), 2, "logit_scale"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), 2, "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["mask"].pop("keep_first"), 2, "keep_first"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), 2, "size"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), 2, "rot"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), 2, "rot"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), 2, "slow"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(factor=0), 2, "rot"),
    (lambda c: c["layers"][2]["mixer"].pop("rot"), 2, "dims"),
    (lambda c: c["layers"][2]["mixer"].update(dim=600), 6, "600"),
    (lambda c: c["layers"][0]["mixer"].update(tau=0), 2, "tau"),
    (lambda c: c["layers"][0]["mixer"].update(dim=300), 6, "300"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), 2, "top 6 of 5"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(experts=600), 6, "600 experts"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(experts=6), 2, "e5"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), 2, "ff"),
    (lambda c: c["layers"][1]["mlp"].update(kind="routed"), 6, "feed-forward"),
    (lambda c: c["loop"].update(times=3), 2, "loop.step"),
])
def test_configuration_errors(tmp_path, change, code, text):
    from forge_llm_b200._lib import ForgeError
    with pytest.raises(ForgeError) as e:
        _info(_folder(tmp_path, change))
    assert e.value.code == code and text in str(e.value), e.value


def test_tensor_errors(tmp_path):
    from forge_llm_b200._lib import ForgeError
    for i, (name, value, text) in enumerate([("l1.mix.sink", None, "l1.mix.sink is missing"), ("l2.mix.k.b", None, "l2.mix.k.b is missing"), ("l2.mix.q.norm", np.ones(32), "l2.mix.q.norm has shape"),
                                             ("l1.mix.q.norm", np.ones(144), "l1.mix.q.norm has shape"), ("l0.mix.a2.b", None, "l0.mix.a2.b is missing"), ("l0.mix.a2", np.ones((72, 9)), "l0.mix.a2 has shape"),
                                             ("l1.mlp.e4.down", None, "l1.mlp.e4.down is missing"), ("l1.mlp.router.b", None, "l1.mlp.router.b is missing"), ("l0.norm2", None, "l0.norm2 is missing"),
                                             ("bigram", np.ones((61, 136)), "bigram has shape")]):
        def edit(t):
            t.pop(name) if value is None else t.update({name: np.asarray(value, np.float32)})
        with pytest.raises(ForgeError) as e:
            _info(_folder(tmp_path / str(i), tensors=edit))
        assert text in str(e.value), e.value


def test_shapes_of_the_synthetic_writer_agree(tmp_path):
    from forge_llm_b200 import synth
    cfg = synth.mokatar_config(128, 8, 2, 48, 77, dim=64, window=32)
    synth.write_stack(str(tmp_path), cfg)
    i = _info(str(tmp_path))
    assert i["num_layers"] == 8 and i["num_weight_layers"] == 4
    t = LS.read_safetensors(str(tmp_path / "model.safetensors"))
    assert np.array_equal(t["l1.mix.q"], t["l3.mix.q"]) and t["l1.mlp.e7.gate"].std() > 0.05
