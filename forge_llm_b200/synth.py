"""Seeded synthetic models in the reference's ``weights.bin`` layout.

The layout is the one the reference's exporter writes and its generated loader reads
(crates/forgellm-cli/src/main.rs:2714-2757, crates/forgellm-codegen-cpu/src/project.rs:341-407):
``embed_tokens`` f32 ``[V, h]``; per layer ``attn_norm`` f32, ``q``, ``k``, ``v`` raw blocks,
optional f32 ``q_bias, k_bias, v_bias``, ``o``, ``ffn_norm`` f32, ``gate``, ``up``, ``down``;
``final_norm`` f32; ``lm_head`` raw blocks.  Projection bytes are GGUF Q8_0 (34 B per 32 values)
or Q4_0 (18 B per 32 values), rows of ``K/32`` blocks, ``N`` rows.

Values: every linear weight ~ N(0, 0.02) f32 from ``numpy.random.default_rng(seed)`` (PCG64),
drawn in file order and quantised at once; norm weights 1.0; biases N(0, 0.02).  For a tied
model the embedding is the dequantised lm_head, which is what the reference's exporter
produces from a tied quantised checkpoint (main.rs:2655-2693).
"""
from __future__ import annotations

import numpy as np


def _f16_round(x: np.ndarray) -> np.ndarray:
    return x.astype(np.float16)  # IEEE round-to-nearest-even, as weight_loader.rs:1361-1442


def _round_half_away(x: np.ndarray) -> np.ndarray:
    return np.copysign(np.floor(np.abs(x) + np.float32(0.5)), x)  # Rust f32::round


def quantize_q8_0(x: np.ndarray) -> np.ndarray:
    """weight_loader.rs:1454-1486: d = amax/127 (stored f16), q = round(x * (1/d_f32)), clamp +-127."""
    b = np.ascontiguousarray(x, np.float32).reshape(-1, 32)
    amax = np.abs(b).max(axis=1)
    scale = np.where(amax == 0, np.float32(0), amax / np.float32(127.0)).astype(np.float32)
    with np.errstate(divide="ignore"):
        inv = np.where(scale != 0, np.float32(1.0) / scale, np.float32(0)).astype(np.float32)
    q = np.clip(_round_half_away(b * inv[:, None]), -127, 127).astype(np.int8)
    out = np.empty((b.shape[0], 34), np.uint8)
    out[:, :2] = _f16_round(scale).view(np.uint8).reshape(-1, 2)
    out[:, 2:] = q.view(np.uint8)
    return out.reshape(-1)


def quantize_q4_0(x: np.ndarray) -> np.ndarray:
    """Signed-max rule of the benchmark configurations: d = (largest-magnitude value) / -8 stored
    as f16, nibble = clamp(round(x * (1/d_f32)) + 8, 0, 15); element j in the low nibble of byte j,
    element j+16 in the high nibble (weight_loader.rs:1494-1544 packs the same way)."""
    b = np.ascontiguousarray(x, np.float32).reshape(-1, 32)
    idx = np.abs(b).argmax(axis=1)
    vmax = b[np.arange(b.shape[0]), idx]
    d = np.where(vmax == 0, np.float32(0), vmax / np.float32(-8.0)).astype(np.float32)
    with np.errstate(divide="ignore"):
        inv = np.where(d != 0, np.float32(1.0) / d, np.float32(0)).astype(np.float32)
    q = np.clip(_round_half_away(b * inv[:, None]).astype(np.int32) + 8, 0, 15).astype(np.uint8)
    out = np.empty((b.shape[0], 18), np.uint8)
    out[:, :2] = _f16_round(d).view(np.uint8).reshape(-1, 2)
    out[:, 2:] = q[:, :16] | (q[:, 16:] << 4)
    return out.reshape(-1)


def dequantize(quant: int, raw: np.ndarray, n: int) -> np.ndarray:
    """weight_loader.rs:860-926."""
    if quant == 8:
        b = raw.reshape(-1, 34)
        d = b[:, :2].copy().view(np.float16).astype(np.float32)
        return (b[:, 2:].view(np.int8).astype(np.float32) * d).reshape(-1)[:n]
    b = raw.reshape(-1, 18)
    d = b[:, :2].copy().view(np.float16).astype(np.float32)
    lo = (b[:, 2:] & 0x0F).astype(np.int32) - 8
    hi = (b[:, 2:] >> 4).astype(np.int32) - 8
    return (np.concatenate([lo, hi], axis=1).astype(np.float32) * d).reshape(-1)[:n]


_native = None


def quantize(quant: int, x: np.ndarray) -> np.ndarray:
    """Quantise with the library's host quantisers (multithreaded C++) when the shared object is
    built, else with the numpy statements above; the two are bit-identical (tests/)."""
    global _native
    if _native is None:
        try:
            from . import runtime
            _native = runtime
        except Exception:
            _native = False
    if _native:
        return _native.quantize_q8_0(x) if quant == 8 else _native.quantize_q4_0(x, True)
    return quantize_q8_0(x) if quant == 8 else quantize_q4_0(x)


def random_kquant(quant: int, rng: np.random.Generator, n: int, k: int, std: float) -> np.ndarray:
    """n rows of K-quant super-blocks drawn field by field (no quantiser is involved: every bit pattern of the
    scale and quant fields is a legal block); the f16 super-block scales are sized so that the dequantised weights
    have about the magnitude ``std``.  Q4_K: 144 bytes {d, dmin, 12 scale bytes, 128 nibble bytes}; Q6_K: 210 bytes
    {128 low-nibble bytes, 64 two-bit bytes, 16 int8 scales, d} (emit.rs:2962-2969, :3542-3546)."""
    nsb = n * (k // 256)
    if quant == 12:
        blk = rng.integers(0, 256, (nsb, 144), dtype=np.uint8)
        blk[:, 0:2] = (std / 256 * (0.5 + rng.random(nsb))).astype(np.float16).view(np.uint8).reshape(nsb, 2)
        blk[:, 2:4] = (std / 256 * (0.5 + rng.random(nsb))).astype(np.float16).view(np.uint8).reshape(nsb, 2)
    else:
        blk = rng.integers(0, 256, (nsb, 210), dtype=np.uint8)
        blk[:, 208:210] = (std / 1024 * (0.5 + rng.random(nsb))).astype(np.float16).view(np.uint8).reshape(nsb, 2)
    return blk.reshape(-1)


def weights_bin_size(c: dict) -> int:
    from .configs import proj_quants, raw_row_bytes
    h, qk, kv = c["hidden_size"], c["num_heads"] * c["head_dim"], c["num_kv_heads"] * c["head_dim"]
    ff, V = c["intermediate_size"], c["vocab_size"]
    pq = proj_quants(c)
    mb = lambda cat, n, k: n * raw_row_bytes(pq[cat], k)
    per = h * 4 + mb(0, qk, h) + mb(1, kv, h) + mb(2, kv, h) + ((qk + 2 * kv) * 4 if c.get("qkv_bias") else 0) + mb(3, h, qk) + h * 4 \
        + mb(4, ff, h) + mb(5, ff, h) + mb(6, h, ff)
    return V * h * 4 + per * c["num_layers"] + h * 4 + mb(7, V, h)


def make_weights_bin(c: dict, seed: int = 0, std: float = 0.02, chunk_rows: int = 8192, quantize_fn=None,
                     repeat_layers: bool = False) -> np.ndarray:
    """Return the whole ``weights.bin`` image as a uint8 array.

    ``quantize_fn(quant, f32 array) -> uint8 array`` replaces the default quantiser (callers that must not load the
    CUDA library pass their own).  ``repeat_layers``: layer 0 is drawn from the generator and its bytes are repeated
    for the other layers - same shapes, sizes and value distribution at a fraction of the host time (timing runs of
    the multi-billion-parameter shapes, and the full-depth parity runs of those two shapes; every other test draws every layer)."""
    rng = np.random.default_rng(seed)
    qfn = quantize_fn or quantize
    h, qk, kv = c["hidden_size"], c["num_heads"] * c["head_dim"], c["num_kv_heads"] * c["head_dim"]
    from .configs import proj_quants
    ff, V = c["intermediate_size"], c["vocab_size"]
    pq = proj_quants(c)
    out = np.empty(weights_bin_size(c), np.uint8)
    off = 0

    def put(a: np.ndarray):
        nonlocal off
        b = a.view(np.uint8).reshape(-1)
        out[off:off + b.size] = b
        off += b.size

    def draw_quant(n: int, k: int, cat: int) -> np.ndarray:
        quant = pq[cat]
        if quant in (12, 14):
            return random_kquant(quant, rng, n, k, std)
        parts = []
        for r0 in range(0, n, chunk_rows):
            r = min(chunk_rows, n - r0)
            w = rng.standard_normal((r, k), dtype=np.float32) * np.float32(std)
            parts.append(qfn(quant, w))
        return np.concatenate(parts) if len(parts) > 1 else parts[0]

    embed_off = off
    off += V * h * 4  # filled below (tied: from lm_head; untied: drawn first)
    if not c.get("tied"):
        save = off
        off = embed_off
        for r0 in range(0, V, chunk_rows):
            r = min(chunk_rows, V - r0)
            put(rng.standard_normal((r, h), dtype=np.float32) * np.float32(std))
        off = save
    ones = np.ones(h, np.float32)
    layer0 = off
    for li in range(c["num_layers"]):
        if repeat_layers and li > 0:
            n = off - layer0 if li == 1 else layer_bytes
            if li == 1:
                layer_bytes = n
            out[off:off + layer_bytes] = out[layer0:layer0 + layer_bytes]
            off += layer_bytes
            continue
        put(ones)
        put(draw_quant(qk, h, 0))
        put(draw_quant(kv, h, 1))
        put(draw_quant(kv, h, 2))
        if c.get("qkv_bias"):
            put(rng.standard_normal(qk, dtype=np.float32) * np.float32(std))
            put(rng.standard_normal(kv, dtype=np.float32) * np.float32(std))
            put(rng.standard_normal(kv, dtype=np.float32) * np.float32(std))
        put(draw_quant(h, qk, 3))
        put(ones)
        put(draw_quant(ff, h, 4))
        put(draw_quant(ff, h, 5))
        put(draw_quant(h, ff, 6))
    put(ones)
    lm = draw_quant(V, h, 7)
    put(lm)
    assert off == out.size
    if c.get("tied"):
        assert pq[7] in (8, 4), "tied synthetic models need a Q8_0 / Q4_0 head"
        emb = dequantize(pq[7], lm, V * h)
        out[embed_off:embed_off + V * h * 4] = emb.view(np.uint8)
    return out


def prompt_tokens(c: dict, n: int, seed: int = 1) -> np.ndarray:
    """Uniform token ids, ``numpy.random.default_rng(seed).integers(0, V)``."""
    return np.random.default_rng(seed).integers(0, c["vocab_size"], size=n).astype(np.uint32)


# ------------------------------------------------------------------------------------------------ layer-list models
def bolenex_config(width: int, layers: int, heads: int, ff: int, vocab: int, dim: int = 128, rot_dim: int = 64, vdim: int = 128, kv_rank: int = 512) -> dict:
    """config.json of a uniform Bolenex stack."""
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": {"base": 10000.0, "dims": rot_dim},
             "scale": float((dim + rot_dim) ** -0.5)}
    entry = {"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff, "limit": 7.0}}
    return {"architecture": "Bolenex", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "layers": [dict(entry) for _ in range(layers)]}


def bolenex_shapes(cfg: dict, layer: int) -> dict:
    """Tensor shapes of one layer, without its prefix."""
    W, L = cfg["width"], cfg["layers"][layer]
    m, f = L["mixer"], L.get("mlp")
    hv = m["heads"] * m["vdim"]
    s = {"norm1": (W,), "norm1.b": (W,), "norm1.alpha": (), "mix.q": (m["heads"] * (m["dim"] + m["rot_dim"]), W),
         "mix.dkv": (m["kv_rank"] + m["rot_dim"], W), "mix.dkv.norm": (m["kv_rank"],), "mix.uk": (m["heads"] * m["dim"], m["kv_rank"]),
         "mix.uv": (hv, m["kv_rank"]), "mix.g": (hv, W), "mix.o": (W, hv)}
    if f:
        s.update({"mlp.gate": (f["ff"], W), "mlp.up": (f["ff"], W), "mlp.down": (W, f["ff"])})
    return s


def robazen_config(width: int, layers: int, heads: int, ff: int, vocab: int, dim: int = 128, chunk: int = 1024, loop: bool = True) -> dict:
    """config.json of a Robazen stack of ``layers`` layer runs (a multiple of four): groups of (attention beside time mixing, delta, channel
    delta, delta), each with a feed-forward.  With ``loop`` a quarter of the groups (at least one) runs twice with the same weights."""
    pair = {"left": {"heads": heads, "kv_heads": max(1, heads // 4), "dim": dim, "vdim": dim, "scale": float(dim ** -0.5), "softcap": 50.0, "mask": {"size": chunk}},
            "right": {"heads": heads * dim // 64, "dim": 64}}
    rec = {"heads": heads, "kv_heads": heads, "dim": dim, "vdim": dim, "conv": 4}
    mlp = {"kind": "dense", "ff": ff}
    group = [("parallel", pair), ("delta", rec), ("channel_delta", rec), ("delta", rec)]
    n = layers // 4
    twice = max(1, n // 4) if loop and n >= 2 else 0
    out = [{"type": t, "mixer": dict(m), "mlp": dict(mlp)} for _ in range(n - twice) for t, m in group]
    cfg = {"architecture": "Robazen", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "layers": out, "loop": None}
    if twice:
        cfg["loop"] = {"start": len(out) - 4 * twice, "stop": len(out), "times": 2}
    return cfg


def robazen_shapes(cfg: dict, layer: int, rank: int = 64) -> dict:
    """Tensor shapes of one layer, without its prefix; ``rank``: inner size of the two-step projections."""
    W, L = cfg["width"], cfg["layers"][layer]
    m, f = L["mixer"], L.get("mlp")

    def norm(n):
        return {n: (W,), n + ".b": (W,), n + ".alpha": ()}

    s = norm("norm1")
    if L["type"] == "parallel":
        a, r = m["left"], m["right"]
        d = r["heads"] * r["dim"]
        s.update({"mix.left.q": (a["heads"] * a["dim"], W), "mix.left.k": (a["kv_heads"] * a["dim"], W), "mix.left.v": (a["kv_heads"] * a["vdim"], W),
                  "mix.left.g": (a["heads"], W), "mix.left.o": (W, a["heads"] * a["vdim"]), "mix.left.out": (W,), "mix.right.out": (W,)})
        s.update({"mix.right." + x: (d, W) for x in "rkvg"})
        s.update({"mix.right.mu." + x: (W,) for x in "rkvgw"})
        s.update({"mix.right.w1": (rank, W), "mix.right.w2": (d, rank), "mix.right.w0": (d,), "mix.right.u": (r["heads"], r["dim"]),
                  "mix.right.norm": (d,), "mix.right.o": (W, d)})
    else:
        H, D, hv = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
        for x, n in (("q", m["kv_heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", hv)):
            s.update({"mix." + x: (n, W), f"mix.{x}.conv": (n, m["conv"])})
        s.update({"mix.b": (H, W), "mix.A_log": (H,), "mix.norm": (m["vdim"],), "mix.o": (W, hv)})
        if L["type"] == "delta":
            s.update({"mix.a": (H, W), "mix.dt_bias": (H,), "mix.g": (hv, W)})
        else:
            s.update({"mix.a1": (rank, W), "mix.a2": (D, rank), "mix.dt_bias": (D,), "mix.g1": (rank, W), "mix.g2": (hv, rank)})
    if f:
        s.update(norm("norm2"))
        s.update({"mlp.gate": (f["ff"], W), "mlp.up": (f["ff"], W), "mlp.down": (W, f["ff"])})
    return s


def mokatar_config(width: int, layers: int, heads: int, ff: int, vocab: int, dim: int = 128, window: int = 1024, experts: int = 8, top: int = 2, loop: bool = True) -> dict:
    """config.json of a Mokatar stack of ``layers`` layer runs (a multiple of four): groups of (gated linear attention, windowed attention,
    attention, windowed attention), the windowed ones with a mixture of experts whose used ones have ``ff`` rows together, the others with
    a dense feed-forward.  With ``loop`` a quarter of the groups (at least one) runs twice with the same weights."""
    def rot(**scaling):
        return {"base": 10000.0, "dims": dim, "scaling": scaling}

    kv = max(1, heads // 4)
    near = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": float(dim ** -0.5), "mask": {"size": window, "keep_first": 16},
            "rot": rot(factor=4.0, fast=32.0, original=4096, slow=1.0)}
    far = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": float(dim ** -0.5), "rot": rot(factor=4.0)}
    lin = {"heads": heads, "dim": dim, "vdim": dim, "tau": 16.0}
    dense, moe = {"kind": "dense", "ff": ff}, {"kind": "moe", "expert": {"ff": ff // top}, "router": {"experts": experts, "top": top}}
    group = [("gla", lin, dense), ("attention", near, moe), ("attention_2", far, dense), ("attention", near, moe)]
    n = layers // 4
    twice = max(1, n // 4) if loop and n >= 2 else 0
    out = [{"type": t, "mixer": dict(m), "mlp": dict(f)} for _ in range(n - twice) for t, m, f in group]
    cfg = {"architecture": "Mokatar", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "layers": out, "loop": None, "logit_scale": 1.0,
           "embedding": {"scale": 1.0, "bigram": {"buckets": 4093, "mul_prev": 31, "mul_cur": 7}}}
    if twice:
        cfg["loop"] = {"start": len(out) - 4 * twice, "stop": len(out), "times": 2}
    return cfg


def mokatar_shapes(cfg: dict, layer: int, rank: int = 64) -> dict:
    """Tensor shapes of one layer, without its prefix; ``rank``: inner size of the two-step projections."""
    W, L = cfg["width"], cfg["layers"][layer]
    m, f = L["mixer"], L.get("mlp")
    H, hv = m["heads"], m["heads"] * m["vdim"]
    s = {"norm1": (W,), "mix.o": (W, hv)}
    if L["type"] == "gla":
        D = H * m["dim"]
        s.update({"mix.q": (D, W), "mix.k": (D, W), "mix.v": (hv, W), "mix.g": (hv, W), "mix.a1": (rank, W), "mix.a2": (D, rank), "mix.a2.b": (D,), "mix.norm": (m["vdim"],)})
    else:
        q, k, v = H * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        s.update({"mix.q": (q, W), "mix.k": (k, W), "mix.v": (v, W)})
        if L["type"] == "attention":
            s.update({"mix.q.norm": (m["dim"],), "mix.k.norm": (m["dim"],), "mix.sink": (H,)})
        else:
            s.update({"mix.q.b": (q,), "mix.k.b": (k,), "mix.v.b": (v,), "mix.q.norm": (q,), "mix.k.norm": (k,)})
    if f:
        s["norm2"] = (W,)
        if f["kind"] == "dense":
            s.update({"mlp.gate": (f["ff"], W), "mlp.up": (f["ff"], W), "mlp.down": (W, f["ff"])})
        else:
            E, n = f["router"]["experts"], f["expert"]["ff"]
            for e in range(E):
                s.update({f"mlp.e{e}.gate": (n, W), f"mlp.e{e}.up": (n, W), f"mlp.e{e}.down": (W, n)})
            s.update({"mlp.router": (E, W), "mlp.router.b": (E,)})
    return s


def tarulix_config(width: int, layers: int, heads: int, ff: int, vocab: int, dim: int = 128, window: int = 1024, pool: int = 16, state: int = 16, experts: int = 8, identity: int = 2, top: int = 2) -> dict:
    """config.json of a Tarulix stack: attention over a window and blocks beside a selective scan of twice the width, and windowed attention, in turn; a
    mixture whose used experts and shared expert have ``ff`` rows together."""
    kv = max(1, heads // 4)
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": float(dim ** -0.5), "softcap": 30.0, "mask": {"size": window, "pool": pool}, "rot": {"base": 10000.0, "dims": dim}}
    pair = {"left": left, "left_scale": 0.9, "right": {"inner": 2 * width, "state": state, "dt_rank": max(1, width // 16), "conv": 4}, "right_scale": 1.1}
    near = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": float(dim ** -0.5), "bias_max": 4 * window, "mask": {"size": window}, "v_mix": True}
    moe = {"kind": "moe", "expert": {"ff": ff // 2 // top}, "shared": {"ff": ff // 2}, "router": {"experts": experts, "identity": identity, "top": top}}
    return {"architecture": "Tarulix", "width": width, "vocab": vocab, "norm": {"eps": 1e-5},
            "layers": [{"type": "attention" if i % 2 else "parallel", "mixer": dict(near if i % 2 else pair), "mlp": dict(moe)} for i in range(layers)]}


def tarulix_shapes(cfg: dict, layer: int, buckets: int = 32) -> dict:
    """Tensor shapes of one layer, without its prefix; ``buckets``: of the biases by distance."""
    W, L = cfg["width"], cfg["layers"][layer]
    m, f = L["mixer"], L.get("mlp")
    a, p = (m["left"], "mix.left.") if L["type"] == "parallel" else (m, "mix.")
    q, k, v, hv = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"], a["heads"] * a["vdim"]
    s = {"norm1": (), p + "q": (q, W), p + "q.b": (q,), p + "k": (k, W), p + "k.b": (k,), p + "v": (v, W), p + "v.b": (v,), p + "o": (W, hv), p + "o.b": (W,)}
    if L["type"] == "parallel":
        r = m["right"]
        n, st, k = r["inner"], r["state"], r["dt_rank"]
        s[p + "talk"] = (a["heads"], a["heads"])
        s.update({"mix.right." + x: y for x, y in (("in", (2 * n, W)), ("conv", (n, r["conv"])), ("conv.b", (n,)), ("x", (k + 2 * st, n)), ("dt", (n, k)), ("dt.b", (n,)), ("A_log", (n, st)), ("D", (n,)), ("o", (W, n)))})
    else:
        s.update({"mix.rel": (buckets, a["heads"]), "mix.sink": (a["heads"],)})
        if a.get("v_mix"):
            s["mix.vmix"] = ()
    if f:
        E, n, sh = f["router"]["experts"], f["expert"]["ff"], f["shared"]["ff"]
        s["norm2"] = ()
        for e, c in [(f"e{e}", n) for e in range(E)] + [("shared", sh)]:
            s.update({f"mlp.{e}.gate": (c, W), f"mlp.{e}.up": (c, W), f"mlp.{e}.down": (W, c)})
        s.update({"mlp.router": (E + f["router"]["identity"], W), "mlp.correction": (E + f["router"]["identity"],)})
    return s


LAYER_SHAPES = {"Bolenex": bolenex_shapes, "Robazen": robazen_shapes, "Mokatar": mokatar_shapes, "Tarulix": tarulix_shapes}


def stack_shapes(cfg: dict) -> dict:
    """Tensor shapes of a layer-list model."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "head": (V, W), "final.norm": () if cfg["architecture"] == "Tarulix" else (W,)}
    if cfg["architecture"] == "Tarulix":
        pass
    elif cfg["architecture"] == "Mokatar":
        out["bigram"] = (cfg["embedding"]["bigram"]["buckets"] + 1, W)
    else:
        out.update({"final.norm.b": (W,), "final.norm.alpha": ()})
        if cfg.get("loop"):
            out["loop.in"] = (W, 2 * W)
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], W)
    for i, L in enumerate(cfg["layers"]):
        if "weights_of" not in L:
            out.update({f"l{i}.{n}": s for n, s in LAYER_SHAPES[cfg["architecture"]](cfg, i).items()})
    return out


def write_stack(folder: str, cfg: dict, seed: int = 0, repeat_layers: bool = True) -> None:
    """config.json and model.safetensors (bfloat16): matrices ~ N(0, 1/inputs), norm weights 1, biases and mixes 0, alpha 0.5.  With
    ``repeat_layers`` a layer's values are stored again for later tensors of the same name and shape."""
    import json
    import os
    import struct
    rng = np.random.default_rng(seed)

    def draw(name, shape):
        if name.endswith("alpha"):
            x = np.full(shape, 0.5, np.float32)
        elif len(shape) < 2:
            x = np.zeros(shape, np.float32) if name.endswith((".b", "A_log", "dt_bias", ".w0")) or ".mu." in name else np.ones(shape, np.float32)
        else:
            x = rng.standard_normal(shape, np.float32) * np.float32(shape[1] ** -0.5)
        return (np.ascontiguousarray(x).view(np.uint32) >> 16).astype(np.uint16)

    parts = list(stack_shapes(cfg).items())
    head, off = {}, 0
    for n, s in parts:
        size = 2 * int(np.prod(s, dtype=np.int64))
        head[n] = {"dtype": "BF16", "shape": list(s), "data_offsets": [off, off + size]}
        off += size
    os.makedirs(folder, exist_ok=True)
    text = json.dumps(head).encode()
    kept: dict = {}
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text)
        for n, s in parts:
            key = (n.split(".", 1)[1], s) if n.startswith("l") and not n.startswith("loop") and repeat_layers else None
            data = kept.get(key) if key else None
            if data is None:
                data = draw(n, s).tobytes()
                if key:
                    kept[key] = data
            f.write(data)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
