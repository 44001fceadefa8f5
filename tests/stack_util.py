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
