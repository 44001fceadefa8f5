"""Small layer-list models shared by the tests: configurations of many shapes, seeded weights, comparison of logits."""
import numpy as np

from oracle import layer_stack as LS

F32_TOL, BF16_TOL = 3e-5, 3e-2


def _l(mixer, ff, limit=1.0, of=None):
    return (mixer, ff, limit, of)


SMALL = dict(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=56, base=5000.0)
CONFIGS = {
    # odd sizes everywhere, two layers of different sizes, tensors used again by a later layer
    "mixed": LS.make_config(136, 203, [_l(LS.mixer(**SMALL), 72, 0.7), _l(LS.mixer(heads=5, dim=40, rot_dim=24, vdim=16, kv_rank=72, base=300.0, scale=0.21), 120, 2.5),
                                       _l(LS.mixer(**SMALL), 72, 0.7, 0)], eps=1e-3),
    # no feed-forward, and one weight layer run three times
    "no_mlp": LS.make_config(96, 131, [_l(LS.mixer(heads=2, dim=16, rot_dim=32, vdim=24, kv_rank=40), None), _l(LS.mixer(heads=4, dim=8, rot_dim=16, vdim=8, kv_rank=24), 64, 0.9),
                                       _l(LS.mixer(heads=4, dim=8, rot_dim=16, vdim=8, kv_rank=24), 64, 0.9, 1), _l(LS.mixer(heads=4, dim=8, rot_dim=16, vdim=8, kv_rank=24), 64, 0.9, 1)]),
    # one head, sizes no multiple of anything
    "one_head": LS.make_config(70, 67, [_l(LS.mixer(heads=1, dim=9, rot_dim=6, vdim=11, kv_rank=13, base=77.0), 21, 1.3)] * 2),
    # more heads than one tensor-core tile, wide rotated part
    "many_heads": LS.make_config(192, 259, [_l(LS.mixer(heads=21, dim=16, rot_dim=80, vdim=16, kv_rank=136), 96, 1.1)]),
    # a real model's latent: nine column chunks per cache row
    "wide_latent": LS.make_config(128, 150, [_l(LS.mixer(heads=6, dim=128, rot_dim=64, vdim=128, kv_rank=512, base=10000.0), 64, 1.0)]),
    # wide values (512 columns of tensor memory), two stages of the key ring
    "wide_values": LS.make_config(128, 150, [_l(LS.mixer(heads=2, dim=120, rot_dim=72, vdim=200, kv_rank=200), 64, 1.0)]),
    # beyond the tensor-core kernels: rows and prompts on the CUDA cores
    "beyond": LS.make_config(64, 90, [_l(LS.mixer(heads=2, dim=300, rot_dim=16, vdim=24, kv_rank=600), 40, 1.0)]),
}


_delta, _pair = LS.delta_mixer, LS.pair_mixer
ROBAZEN = {
    # every mixer, with and without a feed-forward, the middle layers twice
    "all": LS.make_robazen(136, 203, [("parallel", _pair(), 72), ("delta", _delta(), None), ("channel_delta", _delta(heads=6, kv_heads=3, dim=16, vdim=24, conv=3), 56), ("delta", _delta(conv=2), 40)],
                           (1, 3, 2), eps=1e-3),
    # the loop is the whole model, three passes; one head; no history in the convolution
    "loop_all": LS.make_robazen(72, 67, [("channel_delta", _delta(1, 1, 8, 8, 1), 24), ("parallel", _pair(1, 1, 8, 16, 7, 5.0, 0.9, 1, 8), None)], (0, 2, 3), eps=1e-2),
    # one pass only, at the end; sizes no multiple of eight (token by token everywhere)
    "odd": LS.make_robazen(70, 91, [("parallel", _pair(3, 1, 9, 13, 33, 11.0, None, 2, 11), 21), ("delta", _delta(3, 1, 13, 11, 5), 30), ("channel_delta", _delta(2, 2, 10, 7, 6), None)], (2, 3, 1)),
    # no loop; a real model's head sizes
    "wide": LS.make_robazen(128, 150, [("delta", _delta(2, 1, 128, 128, 4), 64), ("parallel", _pair(8, 2, 128, 128, 80, 30.0, None, 2, 64), None), ("channel_delta", _delta(2, 2, 128, 64, 4), 64)]),
    # wide heads and values beyond the chunked kernels, many query heads on one key head, a chunk larger than the prompt
    "beyond": LS.make_robazen(96, 110, [("delta", _delta(2, 2, 160, 200, 4), None), ("parallel", _pair(10, 1, 72, 136, 1000, 50.0, None, 1, 136), 40), ("channel_delta", _delta(1, 1, 136, 40, 7), None)]),
}
_yarn = LS.rotation_of
MOKATAR = {
    # every mixer and feed-forward, the middle layers twice
    "all": LS.make_mokatar(136, 203, [("gla", LS.linear_mixer(), 72), ("attention", LS.head_normed_mixer(), (5, 2, 24)), ("attention_2", LS.row_normed_mixer(), 56), ("gla", LS.linear_mixer(2, 16, 24, 3.0), None)],
                           (1, 3, 2), eps=1e-3),
    # the loop is the whole model, three passes; one head; every expert used; no kept tokens; a rotation without scaling
    "loop_all": LS.make_mokatar(72, 67, [("attention", LS.head_normed_mixer(1, 1, 16, 8, 9, 0, _yarn(16, 50.0), 0.4), (3, 3, 70)), ("gla", LS.linear_mixer(1, 8, 8, 1.0), (4, 1, 16))], (0, 2, 3), eps=1e-2,
                                scale=1.0, bigram=(7, 1, 0), logit_scale=1.0),
    # one pass only, at the end; sizes no multiple of eight; layers without a feed-forward
    "odd": LS.make_mokatar(70, 91, [("attention_2", LS.row_normed_mixer(3, 1, 9, 13, _yarn(6, 77.0, factor=2.5)), 21), ("attention", LS.head_normed_mixer(6, 3, 13, 11, 33, 3, _yarn(10, 90.0, factor=2.0, fast=2.0, original=40, slow=0.5)), (7, 3, 21)),
                                    ("gla", LS.linear_mixer(2, 11, 9, 5.0), None), ("attention", LS.head_normed_mixer(2, 1, 10, 7, 64, 1, _yarn(4, 20.0)), None)], (3, 4, 1)),
    # no loop; a real model's head sizes, many experts, several row tiles per expert
    "wide": LS.make_mokatar(192, 150, [("attention", LS.head_normed_mixer(8, 2, 128, 128, 80, 4, _yarn(64, 10000.0, factor=8.0, fast=32.0, original=256, slow=1.0)), (40, 4, 100)), ("attention_2", LS.row_normed_mixer(4, 2, 128, 64, _yarn(128, 1e6, factor=4.0)), 64),
                                       ("gla", LS.linear_mixer(2, 128, 128, 16.0), (70, 6, 40))]),
    # wide heads and values beyond the tensor-core kernels, many query heads on one key head, a window larger than the prompt, more kept tokens than the window holds
    "beyond": LS.make_mokatar(96, 110, [("attention", LS.head_normed_mixer(10, 1, 72, 272, 1000, 100), (3, 2, 40)), ("gla", LS.linear_mixer(1, 136, 200, 2.0), None), ("attention_2", LS.row_normed_mixer(2, 2, 300, 136), 40),
                                        ("attention", LS.head_normed_mixer(3, 3, 24, 24, 20, 70), None)]),
}
_far, _scan = LS.distance_mixer, LS.scan_pair
TARULIX = {
    # every mechanism: windows shorter and longer than the biases reach, blocks that divide a page and blocks that do not, a layer without a feed-forward, values
    # blended twice (between heads of different sizes) and not at all
    "all": LS.make_tarulix(136, 203, [("parallel", _scan(), (5, 2, 24, 2, 40)), ("attention", _far(), None), ("parallel", _scan(4, 4, 16, 24, 33, 24, 10, 50.0, 8.0, 0.6, 40, 6, 9, 3, (1.3, 0.6)), (4, 3, 40, 0, 72)),
                                      ("attention", _far(8, 2, 32, 40, 50, 20), (3, 4, 16, 3, 24)), ("attention", _far(3, 1, 16, 24, 20, 100, None, False), (6, 1, 24, 1, 16)), ("attention", _far(2, 2, 16, 40, 64, 64), None)], eps=1e-3),
    # one of everything: a window of one token, blocks of one, two and sixty-four, no history in the convolution, every choice taken
    "ones": LS.make_tarulix(72, 67, [("parallel", _scan(1, 1, 8, 8, 1, 2, 8, 9.0, 5.0, 0.9, 8, 1, 1, 1, (1.0, 1.0)), (1, 2, 16, 1, 8)), ("parallel", _scan(2, 1, 16, 16, 7, 1, 2, 90.0, 50.0, 0.3, 24, 4, 2, 2), None),
                                     ("parallel", _scan(2, 2, 8, 16, 20, 64, 0, 90.0, 50.0, 0.5, 16, 8, 5, 2, (0.5, 2.0)), (2, 1, 40, 2, 8)), ("attention", _far(1, 1, 8, 8, 1, 2), (1, 1, 8, 0, 40))], eps=1e-2),
    # sizes no multiple of eight
    "odd": LS.make_tarulix(70, 91, [("attention", _far(6, 3, 13, 11, 33, 37), (7, 3, 21, 2, 13)), ("parallel", _scan(3, 1, 9, 13, 45, 5, 6, 77.0, 11.0, 0.4, 37, 5, 3, 5, (0.9, -0.8)), (3, 2, 9, 4, 21)), ("attention", _far(9, 3, 7, 11, None, 30), None),
                                    ("parallel", _scan(4, 2, 10, 7, 70, 48, 4, 20.0, 40.0, 0.5, 50, 20, 33, 2), (4, 2, 30, 1, 9))]),
    # a real model's head sizes, many experts, several row tiles per expert
    "wide": LS.make_tarulix(192, 150, [("parallel", _scan(8, 2, 128, 128, 80, 16, 64, 10000.0, 30.0, None, 256, 16, 64, 4), (40, 4, 100, 8, 136)), ("attention", _far(8, 2, 128, 64, 70, 300), (70, 6, 40, 10, 64)),
                                       ("parallel", _scan(6, 6, 64, 64, 100, 32, 64, 1e6, 30.0, None, 192, 64, 72, 4), None)]),
    # beyond the tensor-core kernels: wide heads and values, many query heads on a key head, blocks longer than a page, many states and taps, the whole past
    "beyond": LS.make_tarulix(96, 110, [("parallel", _scan(20, 1, 72, 272, 60, 70, 40, 500.0, 25.0, None, 40, 200, 20, 6), (3, 2, 40, 1, 24)), ("attention", _far(10, 1, 300, 24, 1000, 500), None),
                                        ("parallel", _scan(34, 2, 24, 24, None, 0, 24, 500.0, 25.0, None, 24, 33, 6, 4), None)]),
}
CONFIGS.update({"tarulix_" + k: v for k, v in TARULIX.items()})
CONFIGS.update({"mokatar_" + k: v for k, v in MOKATAR.items()})
CONFIGS.update({"robazen_" + k: v for k, v in ROBAZEN.items()})
ROBAZEN_NAMES = ["robazen_" + k for k in ROBAZEN]
BOLENEX_NAMES = [k for k in CONFIGS if not k.startswith(("robazen_", "mokatar_", "tarulix_"))]


def sharp(tensors, cfg, gain=5.0):
    """Query weights scaled up, so that single keys decide the attention."""
    return {k: (LS.bf16_round(v * gain) if k.endswith(".mix.q") else v) for k, v in tensors.items()}


_made = {}


def make(tmp_root, name, seed=0, gain=1.0):
    """(folder, oracle) of a configuration; the folder is written once per session."""
    key = (name, seed, gain)
    if key not in _made:
        cfg = CONFIGS[name]
        t = LS.random_tensors(cfg, seed)
        if gain != 1.0:
            t = sharp(t, cfg, gain)
        folder = str(tmp_root / f"{name}-{seed}-{gain}")
        LS.write_model(folder, cfg, t)
        _made[key] = (folder, LS.LayerStack(cfg, t))
    return _made[key]


def tokens(cfg, n, seed=1):
    return [int(x) for x in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


def err(got, want):
    """Root mean square of the difference of logits (mean taken off) over that of the reference, worst row."""
    d = np.asarray(got, np.float64) - np.asarray(want, np.float64)
    d -= d.mean(-1, keepdims=True)
    w = np.asarray(want, np.float64)
    w = w - w.mean(-1, keepdims=True)
    return float(np.sqrt((d * d).mean(-1) / (w * w).mean()).max())


def tol(dtype):
    return F32_TOL if dtype == "float32" else BF16_TOL
