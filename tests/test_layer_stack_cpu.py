"""Layer-list models without a GPU: the plain restatement against itself, the checkpoint reader and its errors, the scheduler,
and the replay program's file format."""
import copy
import json
import os
import struct

import numpy as np
import pytest

import stack_util as U
from oracle import layer_stack as LS


# ------------------------------------------------------------------------------------------------ the restatement
def test_rotation_keeps_pairs_and_depends_on_distance_only():
    rng = np.random.default_rng(0)
    x = rng.standard_normal((5, 2, 12))
    pos = np.array([0, 1, 7, 63, 64])
    y = LS.rotate_half(x, pos, 100.0, 8)
    assert np.array_equal(y[..., 8:], x[..., 8:]) and np.allclose(y[0], x[0])
    for i in range(4):   # entry i turns with entry i + 4
        a = np.hypot(x[..., i], x[..., i + 4])
        assert np.allclose(a, np.hypot(y[..., i], y[..., i + 4]))
        ang = pos * 100.0 ** (-2 * i / 8)
        assert np.allclose(y[:, 0, i], x[:, 0, i] * np.cos(ang) - x[:, 0, i + 4] * np.sin(ang))
    q, k = rng.standard_normal((2, 1, 12))
    dots = [float((LS.rotate_half(q, [a], 50.0, 12) @ LS.rotate_half(k, [a - 9], 50.0, 12).T).item()) for a in (9, 40, 1000)]
    assert np.allclose(dots, dots[0])


def test_attention_is_causal_and_normalised():
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal((2, 6, 2, 5))
    v = np.ones((6, 2, 3))
    assert np.allclose(LS.causal_softmax_attention(q, k, v, 0.4), 1.0)
    v = rng.standard_normal((6, 2, 3))
    a = LS.causal_softmax_attention(q, k, v, 0.4)
    v2, k2 = v.copy(), k.copy()
    v2[4:] = 9.0
    k2[4:] = -9.0
    b = LS.causal_softmax_attention(q, k2, v2, 0.4)
    assert np.allclose(a[:4], b[:4]) and not np.allclose(a[4:], b[4:])
    assert np.allclose(a[0], v[0])


def test_pointwise_mechanisms():
    x = np.array([-30.0, -2.0, -0.5, 0.0, 0.5, 2.0, 30.0])
    lim = 0.7
    y = LS.clamped_glu(x, x, lim)
    assert y[3] == 0.0 and np.isclose(y[-1], y[-2])                      # gate and up are both held at the limit
    assert np.isclose(y[-1], lim / (1 + np.exp(-1.702 * lim)) * (lim + 1))
    assert np.isclose(y[1], -2.0 / (1 + np.exp(3.404)) * (1 - lim))      # the gate has no lower limit
    n = LS.dynamic_tanh(x, 0.5, 2.0, 0.25)
    assert np.isclose(n[3], 0.25) and np.isclose(n[-1], 2.25) and np.isclose(n[5], np.tanh(1.0) * 2 + 0.25)
    r = LS.rms_norm(np.array([[3.0, 4.0]]), np.array([1.0, 2.0]), 0.5)
    assert np.allclose(r, np.array([[3.0, 8.0]]) / np.sqrt(13.0))


def test_planted_mistakes_show():
    """The tolerances of the GPU tests would not hide a lost key, a wrong rotation or a dropped term on the sharpened models."""
    cfg = U.CONFIGS["mixed"]
    t = U.sharp(LS.random_tensors(cfg, 3), cfg)
    m = LS.LayerStack(cfg, t)
    toks = U.tokens(cfg, 150)
    want = m.logits(toks)
    keep = LS.causal_softmax_attention, LS.rotate_half, LS.clamped_glu, LS.rms_norm

    def lose(n_back):
        def f(q, k, v, scale):
            out = keep[0](q, k, v, scale)
            i = len(q) - 1
            ok = [j for j in range(i + 1) if j != i - n_back]
            for h in range(q.shape[1]):
                s = k[ok, h] @ q[i, h] * scale
                w = np.exp(s - s.max())
                out[i, h] = (w / w.sum()) @ v[ok, h]
            return out
        return f

    def attempt(**kw):
        for name, fn in kw.items():
            setattr(LS, name, fn)
        try:
            return U.err(m.logits(toks)[-1:], want[-1:])
        finally:
            LS.causal_softmax_attention, LS.rotate_half, LS.clamped_glu, LS.rms_norm = keep

    assert attempt() == 0.0
    far = [attempt(causal_softmax_attention=lose(b)) for b in (0, 1, 20, 22, 85, 86, 149)]
    assert sorted(far)[len(far) // 2] > 10 * U.F32_TOL, far
    assert attempt(rotate_half=lambda x, p, b, d: keep[1](x, np.asarray(p) + np.arange(len(p)) % 2, b, d)) > U.BF16_TOL
    assert attempt(clamped_glu=lambda g, u, l: keep[2](g, u, l * 1.2)) > U.BF16_TOL
    assert attempt(clamped_glu=lambda g, u, l: keep[2](g, u, l) / (u.clip(-l, l) + 1) * u.clip(-l, l)) > U.BF16_TOL
    assert attempt(rms_norm=lambda x, w, e: keep[3](x, np.ones_like(w), e)) > U.BF16_TOL


# ------------------------------------------------------------------------------------------------ checkpoints
def _info(folder):
    from forge_llm_b200 import runtime
    return runtime.checkpoint_info(folder)


def test_checkpoint_info(tmp_path):
    folder, m = U.make(tmp_path, "mixed")
    i = _info(folder)
    assert i["architecture"] == "Bolenex" and i["hidden_size"] == 136 and i["vocab_size"] == 203
    assert i["num_layers"] == 3 and i["num_weight_layers"] == 2
    assert i["parameters"] == sum(v.size for v in m.t.values())
    assert i["cache_values_per_token"] == (64 + 64) + (128 + 64) + (64 + 64)


def _broken(tmp_path, change, tensors=None):
    cfg = copy.deepcopy(U.CONFIGS["mixed"])
    t = LS.random_tensors(cfg, 0)
    change(cfg)
    if tensors:
        tensors(t)
    LS.write_model(str(tmp_path), cfg, t)
    return str(tmp_path)


@pytest.mark.parametrize("change,code,text", [
    (lambda c: c.update(architecture="Other"), 6, "not registered"),
    (lambda c: c["layers"][0].update(type="conv"), 6, "mixer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="routed"), 6, "feed-forward"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), 2, "scale"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), 2, "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].update(heads=0), 2, "heads"),
    (lambda c: c.pop("norm"), 2, "eps"),
    (lambda c: c.update(layers=[]), 2, "layers"),
    (lambda c: c["layers"][2].update(weights_of=1), 2, "weights_of"),
    (lambda c: c["layers"][2].update(weights_of=7), 2, "weights_of"),
    (lambda c: c.update(width=144), 2, "shape"),
    (lambda c: c["layers"][2].pop("weights_of"), 2, "l2.norm1"),
])
def test_configuration_errors(tmp_path, change, code, text):
    from forge_llm_b200._lib import ForgeError
    with pytest.raises(ForgeError) as e:
        _info(_broken(tmp_path, change))
    assert e.value.code == code and text in str(e.value), e.value


def test_missing_and_misshapen_tensors(tmp_path):
    from forge_llm_b200._lib import ForgeError
    with pytest.raises(ForgeError, match="l0.mix.uk is missing"):
        _info(_broken(tmp_path / "a", lambda c: None, lambda t: t.pop("l0.mix.uk")))
    with pytest.raises(ForgeError, match="l1.mix.dkv.norm has shape"):
        _info(_broken(tmp_path / "b", lambda c: None, lambda t: t.update({"l1.mix.dkv.norm": np.ones(73, np.float32)})))


def test_truncated_files(tmp_path):
    from forge_llm_b200._lib import ForgeError
    folder = _broken(tmp_path, lambda c: None)
    st = os.path.join(folder, "model.safetensors")
    data = open(st, "rb").read()
    for cut in (0, 7, 8, 100, len(data) - 2):
        open(st, "wb").write(data[:cut])
        with pytest.raises(ForgeError):
            _info(folder)
    open(st, "wb").write(struct.pack("<Q", 1 << 60) + data[8:])
    with pytest.raises(ForgeError, match="longer than the file"):
        _info(folder)
    open(st, "wb").write(data)
    _info(folder)
    cfg = open(os.path.join(folder, "config.json")).read()
    for bad in (cfg[:-2], cfg + "x", "[1, 2]", "{\"a\": tru}", "", "{" * 100):
        open(os.path.join(folder, "config.json"), "w").write(bad)
        with pytest.raises(ForgeError):
            _info(folder)
    os.remove(os.path.join(folder, "config.json"))
    with pytest.raises(ForgeError, match="cannot open"):
        _info(folder)


def test_json_escapes_and_numbers(tmp_path):
    folder = _broken(tmp_path, lambda c: c.update(note="a\"\\€\U0001F600\n", eps2=-1.5e-3, flags=[True, False, None, {}, []]))
    assert _info(folder)["num_layers"] == 3


def test_without_a_device_loading_reports_it(tmp_path):
    from forge_llm_b200 import runtime
    from forge_llm_b200._lib import ForgeError, lib
    if lib.forge_device_count():
        pytest.skip("a device is present")
    folder, _ = U.make(tmp_path, "one_head")
    with pytest.raises(ForgeError) as e:
        runtime.Model.open(folder)
    assert e.value.code == 4


# ------------------------------------------------------------------------------------------------ scheduler
class FakeEngine:
    """The engine's surface over a counting model: the next token is (sum of all tokens so far) % vocab."""

    def __init__(self, slots, pages, vocab=50):
        self.slots, self.vocab, self.live_, self.pages = slots, vocab, {}, pages
        self.cache = self
        self.steps = []

    def free_tokens(self):
        return self.pages * 64

    def free_slots(self):
        return self.slots - len(self.live_)

    def admit(self, rid):
        assert rid not in self.live_ and self.free_slots() > 0
        self.live_[rid] = []

    def release(self, rid):
        del self.live_[rid]

    def step(self, entries):
        self.steps.append([(r, len(t)) for r, t, _ in entries])
        out = []
        for rid, toks, want in entries:
            seq = self.live_[rid]
            n0 = len(seq)
            seq += toks
            rows = np.zeros((len(want), self.vocab), np.float32)
            for i, w in enumerate(want):
                rows[i, sum(seq[: n0 + w + 1]) % self.vocab] = 1.0
            out.append(rows)
        assert sum(-(-len(s) // 64) for s in self.live_.values()) <= self.pages
        return out


def _expected(prompt, n, vocab=50):
    seq = list(prompt)
    for _ in range(n):
        seq.append(sum(seq) % vocab)
    return seq[len(prompt):]


def test_scheduler_serves_unequal_requests():
    from forge_llm_b200.engine import Scheduler
    eng = FakeEngine(slots=3, pages=8)
    s = Scheduler(eng, step_tokens=40)
    rng = np.random.default_rng(4)
    want = {}
    for i in range(9):
        p = [int(x) for x in rng.integers(0, 50, int(rng.integers(1, 130)))]
        n = int(rng.integers(1, 30))
        s.submit(i, p, n)
        want[i] = _expected(p, n)
    assert s.run() == want
    assert max(sum(n for _, n in st) for st in eng.steps) <= 40
    assert any(1 in [n for _, n in st] and max(n for _, n in st) > 1 for st in eng.steps)   # portions beside decoded tokens
    assert not eng.live_ and s._reserved == 0
    with pytest.raises(ValueError):
        s.submit("big", list(range(600)), 10)


def test_scheduler_stops_at_eos():
    from forge_llm_b200.engine import Scheduler
    eng = FakeEngine(slots=1, pages=4)
    s = Scheduler(eng)
    out = _expected([3, 4], 20)
    s.submit("a", [3, 4], 20, eos=[out[5]])
    first = out.index(out[5])
    assert s.run()["a"] == out[:first]


# ------------------------------------------------------------------------------------------------ command line
def test_command_line_info(tmp_path, capsys):
    from forge_llm_b200.__main__ import main
    folder, _ = U.make(tmp_path, "mixed", seed=1)
    assert main(["info", "--model", folder]) == 0
    assert json.loads(capsys.readouterr().out)["num_weight_layers"] == 2


def test_shapes_of_the_synthetic_writer_agree(tmp_path):
    from forge_llm_b200 import synth
    cfg = synth.bolenex_config(64, 2, 3, 48, 77, dim=16, rot_dim=8, vdim=24, kv_rank=32)
    synth.write_stack(str(tmp_path), cfg)
    i = _info(str(tmp_path))
    assert i["num_layers"] == 2 and i["vocab_size"] == 77
    t = LS.read_safetensors(os.path.join(str(tmp_path), "model.safetensors"))
    assert np.array_equal(t["l0.mix.q"], t["l1.mix.q"]) and t["l0.mix.q"].std() > 0.05
