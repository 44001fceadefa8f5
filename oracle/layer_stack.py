"""Plain restatement of the layer-list models (a ``config.json`` whose "layers" entry lists mixers and feed-forwards):
one function per mechanism, numpy, written from the equations, slow on purpose.

Bolenex: latent attention and a clamped gated feed-forward in parallel behind one Dynamic Tanh norm.
Robazen: mixer and feed-forward one after the other, each behind its own Dynamic Tanh norm; mixers are gated delta rules (one
decay per head or per key channel) and a pair of chunked attention and time mixing; some layers run several times.
Mokatar: mixer and feed-forward side by side, each behind its own RMS norm of the same stream; mixers are softmax attentions with
normed and rotated queries and keys (a window with kept first tokens and a learned sink per head, or the whole past and a sink of
score zero) and gated linear attention; feed-forwards may be mixtures of experts; bigram embeddings; some layers run several times.
Tarulix: norms on the outputs of the sublayers only; mixers are windowed attention with learned distance biases, sinks and values
blended with an earlier layer's, and a pair of attention over a window and pooled blocks, whose heads' weights are mixed, beside a
selective scan; feed-forwards are mixtures of experts, some of which pass their input on, beside a shared expert.

TEST INFRASTRUCTURE ONLY, like the rest of this folder; it shares no code with the shipped package.  Everything is computed in
``dtype`` (float64 by default).  A sequence is evaluated as a whole: there is no cache, no page and no batch here.
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np


# ---------------------------------------------------------------------------------------------- mechanisms
def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def dynamic_tanh(x, alpha, weight, bias):
    """Element by element: tanh(alpha x) weight + bias."""
    return np.tanh(alpha * x) * weight + bias


def rotate_half(x, positions, base, dims):
    """Rotary positions on the first ``dims`` entries of the last axis; entry i turns with entry i + dims/2.
    x: [tokens, ..., n], positions: [tokens]."""
    half = dims // 2
    freq = np.array([base ** (-2.0 * i / dims) for i in range(half)], np.float64)
    ang = np.asarray(positions, np.float64)[:, None] * freq[None, :]
    shape = (len(positions),) + (1,) * (x.ndim - 2) + (half,)
    c, s = np.cos(ang).reshape(shape).astype(x.dtype), np.sin(ang).reshape(shape).astype(x.dtype)
    out = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def causal_softmax_attention(q, k, v, scale):
    """q, k: [tokens, heads, d], v: [tokens, heads, dv]; position i sees every j <= i."""
    n, heads, _ = q.shape
    out = np.zeros((n, heads, v.shape[2]), q.dtype)
    for h in range(heads):
        s = (q[:, h] @ k[:, h].T) * q.dtype.type(scale)
        for i in range(n):
            row = s[i, : i + 1]
            w = np.exp(row - row.max())
            out[i, h] = (w / w.sum()) @ v[: i + 1, h]
    return out


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def latent_attention(h, w, m, eps, positions=None):
    """h: [tokens, width]; ``w(name)`` gives a tensor of the mixer, ``m`` its sizes."""
    n = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(n) if positions is None else positions
    q = (h @ w("q").T).reshape(n, H, d + r)
    down = h @ w("dkv").T
    c = rms_norm(down[:, :rank], w("dkv.norm"), eps)
    rot = m["rot"]
    k_rot = rotate_half(down[:, rank:], pos, rot["base"], rot["dims"])
    q_rot = rotate_half(q[:, :, d:], pos, rot["base"], rot["dims"])
    k_un = (c @ w("uk").T).reshape(n, H, d)
    v = (c @ w("uv").T).reshape(n, H, dv)
    qq = np.concatenate([q[:, :, :d], q_rot], axis=2)
    kk = np.concatenate([k_un, np.broadcast_to(k_rot[:, None, :], (n, H, r))], axis=2)
    o = causal_softmax_attention(qq, kk, v, m["scale"]).reshape(n, H * dv)
    return (o * sigmoid(h @ w("g").T)) @ w("o").T


def clamped_glu(gate, up, limit):
    """g sigmoid(1.702 g) (u + 1) with g = min(gate, limit) and u = up held within +-limit."""
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, w, m):
    return clamped_glu(h @ w("gate").T, h @ w("up").T, h.dtype.type(m["limit"])) @ w("down").T


# ------------------------------------------------------------------------------------ recurrent mixers and their neighbours
def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def short_convolution(x, taps):
    """Causal, per channel: y[t, c] = sum_j taps[c, j] x[t - (n - 1 - j), c], zeros before the start.  x: [tokens, channels]."""
    n = taps.shape[1]
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            s = t - (n - 1 - j)
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def unit(x, eps=1e-6):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + eps)


def delta_rule(q, k, v, beta, g):
    """Token by token: the state decays, is corrected towards v at k, and is read at q behind the write.
    q, k: [tokens, heads, d], v: [tokens, heads, dv], beta: [tokens, heads], g: [tokens, heads, d] (rows of the state).
    Returns what is read and the last states [heads, d, dv]."""
    n, heads, d = q.shape
    out = np.zeros_like(v)
    last = []
    for h in range(heads):
        S = np.zeros((d, v.shape[2]), q.dtype)
        for t in range(n):
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + np.outer(k[t, h], u)
            out[t, h] = S.T @ q[t, h]
        last.append(S)
    return out, np.stack(last)


def _delta_inputs(h, w, m):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ w(t).T, w(t + ".conv"))) for t in "qkv")
    head = np.arange(H) // (H // G)
    q = unit(q.reshape(n, G, d))[:, head] * d ** -0.5
    k = unit(k.reshape(n, G, d))[:, head]
    return q, k, v.reshape(n, H, dv), sigmoid(h @ w("b").T)


def gated_delta_states(h, w, m):
    q, k, v, beta = _delta_inputs(h, w, m)
    n, H, dv = v.shape
    g = np.exp(-np.exp(w("A_log")) * softplus(h @ w("a").T + w("dt_bias")))
    return delta_rule(q, k, v, beta, np.broadcast_to(g[:, :, None], k.shape))


def gated_delta(h, w, m, eps):
    o, _ = gated_delta_states(h, w, m)
    n, H, dv = o.shape
    o = rms_norm(o, w("norm"), eps) * silu(h @ w("g").T).reshape(n, H, dv)
    return o.reshape(n, H * dv) @ w("o").T


def channel_delta_states(h, w, m):
    q, k, v, beta = _delta_inputs(h, w, m)
    n, H, dv = v.shape
    z = ((h @ w("a1").T) @ w("a2").T + w("dt_bias")).reshape(n, H, m["dim"])
    return delta_rule(q, k, v, beta, np.exp(-np.exp(w("A_log"))[None, :, None] * softplus(z)))


def channel_delta(h, w, m, eps):
    o, _ = channel_delta_states(h, w, m)
    n, H, dv = o.shape
    o = rms_norm(o, w("norm"), eps) * sigmoid((h @ w("g1").T) @ w("g2").T).reshape(n, H, dv)
    return o.reshape(n, H * dv) @ w("o").T


def chunked_attention(q, k, v, scale, softcap, chunk):
    """q: [tokens, heads, d], k: [tokens, kv heads, d], v: [tokens, kv heads, dv]; position i sees the keys j <= i of its own chunk."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((n, H, v.shape[2]), q.dtype)
    for h in range(H):
        kh, vh = k[:, h // (H // G)], v[:, h // (H // G)]
        for i in range(n):
            j0 = i // chunk * chunk
            s = kh[j0:i + 1] @ q[i, h] * q.dtype.type(scale)
            s = softcap * np.tanh(s / softcap)
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ vh[j0:i + 1]
    return out


def gated_attention(h, w, m):
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    o = chunked_attention((h @ w("q").T).reshape(n, H, m["dim"]), (h @ w("k").T).reshape(n, G, m["dim"]), (h @ w("v").T).reshape(n, G, m["vdim"]),
                          m["scale"], m["softcap"], m["mask"]["size"])
    o = o * sigmoid(h @ w("g").T)[:, :, None]
    return o.reshape(n, H * m["vdim"]) @ w("o").T


def token_shift(h, mu):
    """h + (h' - h) mu with h' the row before (zeros in front of the first)."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def time_mix_states(h, w, m):
    """What is read, [tokens, heads, d], and the last states [heads, d, d]."""
    n, H, d = h.shape[0], m["heads"], m["dim"]
    r, k, v = ((token_shift(h, w("mu." + s)) @ w(s).T).reshape(n, H, d) for s in "rkv")
    dec = np.exp(-np.exp(np.tanh(token_shift(h, w("mu.w")) @ w("w1").T) @ w("w2").T + w("w0"))).reshape(n, H, d)
    o, last = np.zeros_like(v), []
    for i in range(H):
        S = np.zeros((d, d), h.dtype)
        for t in range(n):
            o[t, i] = S.T @ r[t, i] + (r[t, i] * w("u")[i] * k[t, i]).sum() * v[t, i]
            S = dec[t, i][:, None] * S + np.outer(k[t, i], v[t, i])
        last.append(S)
    return o, np.stack(last)


def time_mixing(h, w, m, eps):
    o, _ = time_mix_states(h, w, m)
    gate = silu(token_shift(h, w("mu.g")) @ w("g").T)
    o = rms_norm(o, 1.0, eps).reshape(gate.shape) * w("norm") * gate
    return o @ w("o").T


def parallel_pair(h, w, m, eps):
    left = gated_attention(h, lambda t: w("left." + t), m["left"])
    right = time_mixing(h, lambda t: w("right." + t), m["right"], eps)
    return 0.5 * (rms_norm(left, w("left.out"), eps) + rms_norm(right, w("right.out"), eps))


def silu_glu_ff(h, w):
    return (silu(h @ w("gate").T) * (h @ w("up").T)) @ w("down").T


# ------------------------------------------------------------------- softmax attention with normed, rotated queries and keys
def rotation(rot, kind):
    """(angle per position of every pair, factor on cos and sin) of a rotation; kind: what "scaling" asks for."""
    d, base = rot["dims"], float(rot["base"])
    f = np.array([base ** (-2.0 * i / d) for i in range(d // 2)])
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    if kind == "linear":
        return f / s["factor"], 1.0
    turns = lambda t: d * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))   # the pair that turns t times over the original length
    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), d - 1)
    ramp = np.clip((np.arange(d // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, freq, factor, interleaved):
    """x: [tokens, heads, n]; pair i is (2i, 2i + 1) if interleaved, else (i, i + number of pairs); the rest passes."""
    n = len(freq)
    a, b = (np.arange(n) * 2, np.arange(n) * 2 + 1) if interleaved else (np.arange(n), np.arange(n) + n)
    ang = np.asarray(positions, np.float64)[:, None, None] * freq
    c, s = (np.cos(ang) * factor).astype(x.dtype), (np.sin(ang) * factor).astype(x.dtype)
    out = x.copy()
    out[:, :, a] = x[:, :, a] * c - x[:, :, b] * s
    out[:, :, b] = x[:, :, b] * c + x[:, :, a] * s
    return out


def visible(i, size=None, keep=0):
    """Which keys j = 0 .. i position i sees: its window of ``size`` positions and the first ``keep``."""
    j = np.arange(i + 1)
    return np.ones(i + 1, bool) if size is None else (i - j < size) | (j < keep)


def sink_attention(q, k, v, scale, sink, size=None, keep=0):
    """q: [tokens, heads, d], k: [tokens, kv heads, d], v: [tokens, kv heads, dv]; the denominator holds exp(sink[head]) besides the keys'."""
    n, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((n, H, v.shape[2]), q.dtype)
    for h in range(H):
        kh, vh = k[:, h // (H // G)], v[:, h // (H // G)]
        s = (q[:, h] @ kh.T) * q.dtype.type(scale)
        for i in range(n):
            see = visible(i, size, keep)
            row = s[i, :i + 1][see]
            top = max(row.max(), sink[h])
            e = np.exp(row - top)
            out[i, h] = (e / (e.sum() + np.exp(sink[h] - top))) @ vh[:i + 1][see]
    return out


def head_normed_attention(h, w, m, eps):
    """Queries and keys normed per head, interleaved rotation, a window with kept first tokens, a learned sink."""
    n, H, G, pos = h.shape[0], m["heads"], m["kv_heads"], np.arange(h.shape[0])
    f, c = rotation(m["rot"], "yarn")
    q = rotate(rms_norm((h @ w("q").T).reshape(n, H, m["dim"]), w("q.norm"), eps), pos, f, c, True)
    k = rotate(rms_norm((h @ w("k").T).reshape(n, G, m["dim"]), w("k.norm"), eps), pos, f, c, True)
    v = (h @ w("v").T).reshape(n, G, m["vdim"])
    mask = m.get("mask") or {}
    return sink_attention(q, k, v, m["scale"], w("sink"), mask.get("size"), mask.get("keep_first", 0)).reshape(n, H * m["vdim"]) @ w("o").T


def row_normed_attention(h, w, m, eps):
    """Biased projections, queries and keys normed over all heads at once, halves rotated, a sink of score zero."""
    n, H, G, pos = h.shape[0], m["heads"], m["kv_heads"], np.arange(h.shape[0])
    f, c = rotation(m["rot"], "linear")
    q = rotate(rms_norm(h @ w("q").T + w("q.b"), w("q.norm"), eps).reshape(n, H, m["dim"]), pos, f, c, False)
    k = rotate(rms_norm(h @ w("k").T + w("k.b"), w("k.norm"), eps).reshape(n, G, m["dim"]), pos, f, c, False)
    v = (h @ w("v").T + w("v.b")).reshape(n, G, m["vdim"])
    return sink_attention(q, k, v, m["scale"], np.zeros(H, h.dtype)).reshape(n, H * m["vdim"]) @ w("o").T


def linear_attention_states(h, w, m):
    """What is read, [tokens, heads, dv], and the last states [heads, d, dv]: a key channel decays, a token is written, then read."""
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w("q").T).reshape(n, H, d) * d ** -0.5, (h @ w("k").T).reshape(n, H, d), (h @ w("v").T).reshape(n, H, dv)
    z = ((h @ w("a1").T) @ w("a2").T + w("a2.b")).reshape(n, H, d)
    alpha = sigmoid(z) ** (1.0 / m["tau"])
    o, last = np.zeros_like(v), []
    for i in range(H):
        S = np.zeros((d, dv), h.dtype)
        for t in range(n):
            S = alpha[t, i][:, None] * S + np.outer(k[t, i], v[t, i])
            o[t, i] = S.T @ q[t, i]
        last.append(S)
    return o, np.stack(last)


def gated_linear_attention(h, w, m, eps):
    o, _ = linear_attention_states(h, w, m)
    n, H, dv = o.shape
    return (rms_norm(o, w("norm"), eps).reshape(n, H * dv) * silu(h @ w("g").T)) @ w("o").T


def route(z, top):
    """z: [tokens, experts] -> chosen experts [tokens, top], largest first, and their softmax weights."""
    chosen = np.argsort(-z, axis=1, kind="stable")[:, :top]
    e = np.take_along_axis(z, chosen, 1)
    e = np.exp(e - e.max(1, keepdims=True))
    return chosen, e / e.sum(1, keepdims=True)


def mixture_ff(h, w, m):
    chosen, weight = route(h @ w("router").T + w("router.b"), m["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(chosen[t], weight[t]):
            out[t] += g * silu_glu_ff(h[t:t + 1], lambda n: w(f"e{e}.{n}"))[0]
    return out


# ------------------------------------------------------- distance biases, pooled blocks, mixed heads, selective scan, shared experts
def unit_rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def distance_bucket(n, buckets, longest):
    """Bucket of the distance n: one each for the first half, then logarithmic ones up to the distance ``longest``."""
    half = buckets // 2
    if n < half:
        return n
    x = math.log(n / half) / math.log(longest / half) * (buckets - half)
    if abs(x - round(x)) < 1e-9:       # an edge: exactly there, whatever the logarithms round to
        x = round(x)
    return min(buckets - 1, half + math.floor(x))


def windowed(i, size=None):
    """Positions 0 .. i: which of them position i sees."""
    j = np.arange(i + 1)
    return np.ones(i + 1, bool) if size is None else i - j < size


def blocks_seen(i, size, pool):
    """How many blocks of ``pool`` positions lie wholly in front of position i's window."""
    return sum(1 for b in range(i // pool + 1) if b * pool + pool - 1 <= i - size) if size and pool else 0


def head_scores(q, k, group):
    """[heads, queries, keys]: query head h meets key head h / group."""
    return np.stack([q[:, h] @ k[:, h // group].T for h in range(q.shape[1])])


def soft_weights(row, sink=None):
    """Softmax of a row of scores; a sink is one more score whose weight is left out."""
    top = row.max() if sink is None else max(row.max(), sink)
    e = np.exp(row - top)
    return e / (e.sum() + (0.0 if sink is None else np.exp(sink - top)))


def biased_attention(q, k, v, scale, rel, longest, sink, size):
    """A window, a learned bias per distance bucket and head, a sink per head."""
    n, H, _ = q.shape
    group = H // k.shape[1]
    s = head_scores(q, k, group) * scale
    bucket = np.array([distance_bucket(d, len(rel), longest) for d in range(n)])
    out = np.zeros((n, H, v.shape[2]), q.dtype)
    for h in range(H):
        for i in range(n):
            j = np.flatnonzero(windowed(i, size))
            out[i, h] = soft_weights(s[h, i, j] + rel[bucket[i - j], h], sink[h]) @ v[j, h // group]
    return out


def pooled_attention(q, k, v, scale, softcap, size, pool, talk):
    """A window of tokens and the blocks in front of it, each as the mean of its keys and values, under one softmax with capped scores; the
    heads' weights are mixed before they meet the values of each head's own key / value head."""
    n, H, _ = q.shape
    group = H // k.shape[1]
    nb = n // pool if pool else 0
    mean = lambda x: x[:nb * pool].reshape((nb, pool) + x.shape[1:]).mean(1) if nb else x[:0]
    kk, vv = np.concatenate([mean(k), k]), np.concatenate([mean(v), v])      # blocks, then tokens
    s = head_scores(q, kk, group) * scale
    if softcap:
        s = softcap * np.tanh(s / softcap)
    out = np.zeros((n, H, v.shape[2]), q.dtype)
    for i in range(n):
        j = np.concatenate([np.arange(blocks_seen(i, size, pool)), nb + np.flatnonzero(windowed(i, size))])
        w = talk @ np.stack([soft_weights(s[h, i, j]) for h in range(H)])
        for h in range(H):
            out[i, h] = w[h] @ vv[j, h // group]
    return out


def biased_qkv(h, w, m):
    n = h.shape[0]
    shape = {"q": (n, m["heads"], m["dim"]), "k": (n, m["kv_heads"], m["dim"]), "v": (n, m["kv_heads"], m["vdim"])}
    return [(h @ w(x).T + w(x + ".b")).reshape(shape[x]) for x in "qkv"]


def blended_values(v, first, lam):
    return (1 - lam) * v + lam * first


def distance_attention(h, w, m, eps, first=None):
    """(output, values in front of blending).  first: an earlier layer's values, blended in."""
    q, k, own = biased_qkv(h, w, m)
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    v = own if first is None else blended_values(own, first, w("vmix"))
    o = biased_attention(q, k, v, m["scale"], w("rel"), m["bias_max"], w("sink"), (m.get("mask") or {}).get("size"))
    return o.reshape(len(h), -1) @ w("o").T + w("o.b"), own


def talking_attention(h, w, m, eps):
    q, k, v = biased_qkv(h, w, m)
    rot = m["rot"]
    q, k = (unit_rms(rotate_half(x, np.arange(len(h)), rot["base"], rot["dims"]), eps) for x in (q, k))
    mask = m.get("mask") or {}
    o = pooled_attention(q, k, v, m["scale"], m.get("softcap"), mask.get("size"), mask.get("pool"), w("talk"))
    return o.reshape(len(h), -1) @ w("o").T + w("o.b")


def selective_inputs(h, w, m):
    """(x behind the convolution, step sizes, B, C, z)"""
    n = m["inner"]
    xz = h @ w("in").T
    x = silu(short_convolution(xz[:, :n], w("conv")) + w("conv.b"))
    p = x @ w("x").T
    r, s = m["dt_rank"], m["state"]
    return x, softplus(p[:, :r] @ w("dt").T + w("dt.b")), p[:, r:r + s], p[:, r + s:], xz[:, n:]


def selective_scan(x, dt, A, B, C, D):
    """(y [tokens, channels], last state [channels, states])"""
    S, y = np.zeros(A.shape, x.dtype), np.zeros_like(x)
    for t in range(len(x)):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def selective_mixer(h, w, m):
    x, dt, B, C, z = selective_inputs(h, w, m)
    y, _ = selective_scan(x, dt, -np.exp(w("A_log")), B, C, w("D"))
    return (y * silu(z)) @ w("o").T


def attention_beside_scan(h, w, m, eps):
    return m["left_scale"] * talking_attention(h, lambda n: w("left." + n), m["left"], eps) + m["right_scale"] * selective_mixer(h, lambda n: w("right." + n), m["right"])


def route_corrected(z, correction, top):
    """The ``top`` largest of softmax(z) + correction, and their softmax values as they are."""
    e = np.exp(z - z.max(1, keepdims=True))
    s = e / e.sum(1, keepdims=True)
    chosen = np.argsort(-(s + correction), axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, 1)


def shared_mixture_ff(h, w, m):
    """Experts, the last ``identity`` choices passing their input on, beside a shared expert."""
    r = m["router"]
    chosen, weight = route_corrected(h @ w("router").T, w("correction"), r["top"])
    out = silu_glu_ff(h, lambda n: w("shared." + n))
    for t in range(h.shape[0]):
        for e, g in zip(chosen[t], weight[t]):
            out[t] += g * (h[t] if e >= r["experts"] else silu_glu_ff(h[t:t + 1], lambda n: w(f"e{e}.{n}"))[0])
    return out


def bigram_rows(tokens, b):
    """Row of the bigram table for every token; the last row for the first token."""
    return [b["buckets"] if i == 0 else (int(tokens[i - 1]) * b["mul_prev"] + int(t) * b["mul_cur"]) % b["buckets"] for i, t in enumerate(tokens)]


def mixer_of(kind, h, w, m, eps):
    if kind == "latent_attention":
        return latent_attention(h, w, m, eps)
    if kind in ("attention", "attention_2", "gla"):
        return {"attention": head_normed_attention, "attention_2": row_normed_attention, "gla": gated_linear_attention}[kind](h, w, m, eps)
    return {"delta": gated_delta, "channel_delta": channel_delta, "parallel": parallel_pair}[kind](h, w, m, eps)


def layer_runs(cfg):
    """[(layer, pass that starts in front of it or None)] in the order of running."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + body + [(i, None) for i in range(b, n)]


# ---------------------------------------------------------------------------------------------- the model
class LayerStack:
    """``config``: the parsed config.json; ``tensors``: name -> array."""

    def __init__(self, config: dict, tensors: dict, dtype=np.float64):
        self.cfg = config
        self.t = {k: np.asarray(v, dtype) for k, v in tensors.items()}
        self.dtype = dtype
        self.side_by_side = config["architecture"] == "Mokatar"
        self.post_norm = config["architecture"] == "Tarulix"

    def norm(self, x, name):
        if self.post_norm:
            return unit_rms(x, self.cfg["norm"]["eps"]) * self.t[name]
        if self.side_by_side:
            return rms_norm(x, 1.0 + self.t[name], self.cfg["norm"]["eps"])
        return dynamic_tanh(x, self.t[name + ".alpha"], self.t[name], self.t[name + ".b"])

    def layer(self, x, i):
        L = self.cfg["layers"][i]
        p = f"l{L.get('weights_of', i)}."
        mix, mlp = (lambda n: self.t[p + "mix." + n]), (lambda n: self.t[p + "mlp." + n])
        if self.post_norm:
            m, eps = L["mixer"], self.cfg["norm"]["eps"]
            if L["type"] == "parallel":
                y = attention_beside_scan(x, mix, m, eps)
            else:
                y, own = distance_attention(x, mix, m, eps, self.first_values if m.get("v_mix") else None)
                if m.get("v_mix") and self.first_values is None:
                    self.first_values = own
            x = x + self.norm(y, p + "norm1")
            return x + self.norm(shared_mixture_ff(x, mlp, L["mlp"]), p + "norm2") if L.get("mlp") else x
        h = self.norm(x, p + "norm1")
        y = mixer_of(L["type"], h, mix, L["mixer"], self.cfg["norm"]["eps"])
        if self.side_by_side:
            if L.get("mlp"):
                h = self.norm(x, p + "norm2")
                y = y + (mixture_ff(h, mlp, L["mlp"]) if L["mlp"]["kind"] == "moe" else silu_glu_ff(h, mlp))
            return x + y
        if self.cfg["architecture"] == "Bolenex":
            if L.get("mlp"):
                y = y + dense_ff(h, mlp, L["mlp"])
            return x + y
        x = x + y
        return x + silu_glu_ff(self.norm(x, p + "norm2"), mlp) if L.get("mlp") else x

    def residuals(self, tokens):
        """The residual stream after every layer run: [runs, tokens, width]."""
        x = self.t["embed"][np.asarray(tokens, np.int64)]
        if self.side_by_side:
            x = x * self.dtype(self.cfg["embedding"]["scale"]) + self.t["bigram"][bigram_rows(tokens, self.cfg["embedding"]["bigram"])]
        x0 = x
        self.first_values = None
        out = []
        for i, start in layer_runs(self.cfg):
            if start is not None and self.side_by_side:
                x = (x + x0 if start else x) + self.t["loop.step"][start]
            elif start is not None:
                x = np.concatenate([x, x0], axis=1) @ self.t["loop.in"].T + self.t["loop.step"][start]
            x = self.layer(x, i)
            out.append(x)
        return np.stack(out)

    def logits(self, tokens):
        """[tokens, vocab]: the logits behind every position."""
        return self.norm(self.residuals(tokens)[-1], "final.norm") @ self.t["head"].T * self.cfg.get("logit_scale", 1.0)

    def generate_greedy(self, prompt, n_new):
        """The next n_new tokens, the last index winning a tie."""
        toks = [int(t) for t in prompt]
        for _ in range(n_new):
            row = self.logits(toks)[-1]
            toks.append(int(np.flatnonzero(row == row.max())[-1]))
        return toks[len(prompt):]


# ---------------------------------------------------------------------------------------------- files
def bf16_bits(x):
    """float32 -> bfloat16 bit patterns, round to nearest even."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16).reshape(np.shape(x))


def bf16_round(x):
    return (bf16_bits(x).astype(np.uint32) << 16).view(np.float32)


def read_safetensors(path):
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, d in head.items():
        if name == "__metadata__":
            continue
        a, b = d["data_offsets"]
        raw = data[a:b]
        if d["dtype"] == "BF16":
            arr = (np.frombuffer(raw, np.uint16).astype(np.uint32) << 16).view(np.float32)
        else:
            arr = np.frombuffer(raw, {"F32": np.float32, "F16": np.float16, "I32": np.int32}[d["dtype"]])
        out[name] = arr.reshape(d["shape"])
    return out


def write_model(folder, config, tensors):
    """config.json and model.safetensors (bfloat16, the tensors as they are given)."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    head, blobs, off = {}, [], 0
    for name, arr in tensors.items():
        b = bf16_bits(arr).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(arr)), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    h = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)))
        f.write(h)
        for b in blobs:
            f.write(b)


def load(folder, dtype=np.float64):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return LayerStack(cfg, read_safetensors(os.path.join(folder, "model.safetensors")), dtype)


# ---------------------------------------------------------------------------------------------- seeded models
def mixer(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=56, base=5000.0, scale=None):
    return {"dim": dim, "heads": heads, "kv_rank": kv_rank, "rot": {"base": float(base), "dims": rot_dim}, "rot_dim": rot_dim,
            "scale": float(scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim)), "vdim": vdim}


def make_config(width=136, vocab=203, layers=(), eps=1e-5):
    """``layers``: (mixer, ff size or None, limit, weights_of or None) per layer."""
    out = []
    for mx, ff, limit, of in layers:
        e = {"mixer": mx, "mlp": None if ff is None else {"ff": ff, "kind": "dense", "limit": float(limit)}, "type": "latent_attention"}
        if of is not None:
            e["weights_of"] = of
        out.append(e)
    return {"architecture": "Bolenex", "layers": out, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def delta_mixer(heads=4, kv_heads=2, dim=24, vdim=40, conv=4):
    return {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim}


def pair_mixer(heads=6, kv_heads=2, dim=24, vdim=40, chunk=48, softcap=20.0, scale=None, heads_r=3, dim_r=40):
    return {"left": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": chunk}, "scale": float(scale if scale is not None else dim ** -0.5),
                     "softcap": float(softcap), "vdim": vdim}, "right": {"dim": dim_r, "heads": heads_r}}


def make_robazen(width=136, vocab=203, layers=(), loop=None, eps=1e-5):
    """``layers``: (type, mixer, ff size or None) per layer; ``loop``: (start, stop, times)."""
    out = [{"mixer": mx, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}, "type": t} for t, mx, ff in layers]
    return {"architecture": "Robazen", "layers": out, "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "norm": {"eps": eps}, "vocab": vocab, "width": width}


def random_robazen(cfg, seed=0, rank=20):
    """Seeded weights of a Robazen model, rounded to bfloat16: decays between almost none and almost all, every factor away from 1 and 0."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    t = {}

    def mat(name, out, inp, gain=1.0):
        t[name] = bf16_round(rng.standard_normal((out, inp)) * (gain / math.sqrt(inp)))

    def vec(name, n, mean, dev):
        t[name] = bf16_round(mean + dev * rng.standard_normal(n))

    def norm(name):
        vec(name, W, 1.0, 0.3)
        vec(name + ".b", W, 0.0, 0.2)
        t[name + ".alpha"] = bf16_round(np.asarray(0.5 + 0.4 * rng.random()))

    t["embed"] = bf16_round(rng.standard_normal((cfg["vocab"], W)))
    if cfg.get("loop"):
        mat("loop.in", W, 2 * W, 1.3)
        t["loop.step"] = bf16_round(0.5 * rng.standard_normal((cfg["loop"]["times"], W)))
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1")
        x = p + "mix."
        if L["type"] == "parallel":
            a, r = m["left"], m["right"]
            D = r["heads"] * r["dim"]
            mat(x + "left.q", a["heads"] * a["dim"], W, 1.5)
            mat(x + "left.k", a["kv_heads"] * a["dim"], W, 1.5)
            mat(x + "left.v", a["kv_heads"] * a["vdim"], W)
            mat(x + "left.g", a["heads"], W, 2.0)
            mat(x + "left.o", W, a["heads"] * a["vdim"], 2.0)
            for n in "rkvgw":
                t[x + "right.mu." + n] = bf16_round(rng.random(W))
            for n in "rkvg":
                mat(x + "right." + n, D, W)
            mat(x + "right.w1", rank, W)
            mat(x + "right.w2", D, rank, 1.5)
            vec(x + "right.w0", D, -2.0, 1.5)
            t[x + "right.u"] = bf16_round(rng.standard_normal((r["heads"], r["dim"])))
            vec(x + "right.norm", D, 1.0, 0.3)
            mat(x + "right.o", W, D)
            vec(x + "left.out", W, 0.8, 0.3)
            vec(x + "right.out", W, 1.2, 0.3)
        else:
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, c in (("q", G * d), ("k", G * d), ("v", H * dv)):
                mat(x + n, c, W, 1.5)
                t[x + n + ".conv"] = bf16_round(0.6 * rng.standard_normal((c, m["conv"])))
            mat(x + "b", H, W, 2.0)
            vec(x + "A_log", H, -1.0, 1.5)
            vec(x + "norm", dv, 1.0, 0.3)
            mat(x + "o", W, H * dv, 1.5)
            if L["type"] == "delta":
                mat(x + "a", H, W, 2.0)
                vec(x + "dt_bias", H, -1.0, 1.0)
                mat(x + "g", H * dv, W, 1.5)
            else:
                mat(x + "a1", rank, W)
                mat(x + "a2", H * d, rank, 2.0)
                vec(x + "dt_bias", H * d, -1.0, 1.5)
                mat(x + "g1", rank + 4, W)
                mat(x + "g2", H * dv, rank + 4, 2.0)
        if L.get("mlp"):
            norm(p + "norm2")
            mat(p + "mlp.gate", L["mlp"]["ff"], W, 1.5)
            mat(p + "mlp.up", L["mlp"]["ff"], W, 1.5)
            mat(p + "mlp.down", W, L["mlp"]["ff"])
    norm("final.norm")
    mat("head", cfg["vocab"], W)
    return t


def rotation_of(dims, base=1000.0, **scaling):
    return {"base": float(base), "dims": dims, "scaling": scaling or None}


def head_normed_mixer(heads=6, kv_heads=2, dim=24, vdim=40, window=40, keep=5, rot=None, scale=None):
    return {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"keep_first": keep, "size": window}, "rot": rot or rotation_of(16, 3000.0, factor=4.0, fast=8.0, original=64, slow=1.0),
            "scale": float(scale if scale is not None else dim ** -0.5), "vdim": vdim}


def row_normed_mixer(heads=4, kv_heads=4, dim=32, vdim=16, rot=None, scale=None):
    return {"dim": dim, "heads": heads, "kv_heads": kv_heads, "rot": rot or rotation_of(20, 700.0, factor=3.0), "scale": float(scale if scale is not None else dim ** -0.5), "vdim": vdim}


def linear_mixer(heads=3, dim=24, vdim=40, tau=8.0):
    return {"dim": dim, "heads": heads, "tau": float(tau), "vdim": vdim}


def make_mokatar(width=136, vocab=203, layers=(), loop=None, eps=1e-5, scale=3.0, bigram=(61, 5, 3), logit_scale=0.7):
    """``layers``: (type, mixer, feed-forward) per layer, the feed-forward None, a size, or (experts, top, size); ``loop``: (start, stop, times); ``bigram``:
    (buckets, factor of the token before, factor of the token)."""
    def ff(f):
        if f is None:
            return None
        return {"ff": f, "kind": "dense"} if isinstance(f, int) else {"expert": {"ff": f[2]}, "kind": "moe", "router": {"experts": f[0], "top": f[1]}}
    return {"architecture": "Mokatar", "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram)), "scale": float(scale)},
            "layers": [{"mixer": mx, "mlp": ff(f), "type": t} for t, mx, f in layers], "logit_scale": float(logit_scale),
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "norm": {"eps": eps}, "vocab": vocab, "width": width}


MARKERS = 4


def random_mokatar(cfg, seed=0, rank=12, clear=True):
    """Seeded weights of a Mokatar model, rounded to bfloat16.  clear: routers read MARKERS columns of the stream alone, in which the embedding
    holds signs and nobody else writes, so that rounding does not change a choice."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    t = {}

    def mat(name, out, inp, gain=1.0):
        t[name] = bf16_round(rng.standard_normal((out, inp)) * (gain / math.sqrt(inp)))

    def vec(name, n, mean, dev):
        t[name] = bf16_round(mean + dev * rng.standard_normal(n))

    t["embed"] = bf16_round(rng.standard_normal((cfg["vocab"], W)))
    t["bigram"] = bf16_round(2.0 * rng.standard_normal((cfg["embedding"]["bigram"]["buckets"] + 1, W)))
    if cfg.get("loop"):
        t["loop.step"] = bf16_round(1.5 * rng.standard_normal((cfg["loop"]["times"], W)))
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x = p + "mix."
        vec(p + "norm1", W, 0.1, 0.3)
        H, dv = m["heads"], m["vdim"]
        if L["type"] == "gla":
            D = H * m["dim"]
            mat(x + "q", D, W, 1.5)
            mat(x + "k", D, W)
            mat(x + "v", H * dv, W)
            mat(x + "g", H * dv, W, 1.5)
            mat(x + "a1", rank, W)
            mat(x + "a2", D, rank, 2.0)
            vec(x + "a2.b", D, 0.5, 2.0)
            vec(x + "norm", dv, 1.0, 0.3)
        else:
            q, k, v = H * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * dv
            mat(x + "q", q, W)
            mat(x + "k", k, W)
            mat(x + "v", v, W)
            if L["type"] == "attention":
                vec(x + "q.norm", m["dim"], 1.2, 0.4)
                vec(x + "k.norm", m["dim"], 1.2, 0.4)
                vec(x + "sink", H, 0.5, 1.5)
            else:
                for n, c in (("q", q), ("k", k), ("v", v)):
                    vec(x + n + ".b", c, 0.0, 0.5)
                vec(x + "q.norm", q, 1.2, 0.4)
                vec(x + "k.norm", k, 1.2, 0.4)
        mat(x + "o", W, H * dv, 2.0)
        f = L.get("mlp")
        if f:
            vec(p + "norm2", W, -0.1, 0.3)
            if f["kind"] == "dense":
                mat(p + "mlp.gate", f["ff"], W, 1.5)
                mat(p + "mlp.up", f["ff"], W, 1.5)
                mat(p + "mlp.down", W, f["ff"], 1.5)
            else:
                E, n = f["router"]["experts"], f["expert"]["ff"]
                for e in range(E):
                    mat(p + f"mlp.e{e}.gate", n, W, 1.5)
                    mat(p + f"mlp.e{e}.up", n, W, 1.5)
                    mat(p + f"mlp.e{e}.down", W, n, 2.0)
                mat(p + "mlp.router", E, W, 2.0)
                vec(p + "mlp.router.b", E, 0.0, 0.5)
    vec("final.norm", W, 0.0, 0.3)
    mat("head", cfg["vocab"], W)
    if clear:
        signs = np.sign(rng.standard_normal((cfg["vocab"], MARKERS)))
        t["embed"][:, :MARKERS] = signs
        t["bigram"][:, :MARKERS] = 0
        if "loop.step" in t:
            t["loop.step"][:, :MARKERS] = 0
        patterns = np.array([[1.0 if i >> c & 1 else -1.0 for c in range(MARKERS)] for i in range(1 << MARKERS)])
        for name in t:
            if name.endswith(("mix.o", ".down")):
                t[name][:MARKERS] = 0
            if name.endswith((".norm1", ".norm2")):
                t[name][:MARKERS] = 0.5
            if name.endswith("mlp.router"):
                best = None
                for _ in range(200):     # of some routers the one whose closest call is least close
                    r = np.zeros_like(t[name])
                    r[:, :MARKERS] = bf16_round(2.0 * rng.standard_normal((len(r), MARKERS)))
                    z = np.sort(patterns @ r[:, :MARKERS].T, axis=1)[:, ::-1]
                    top = cfg["layers"][int(name[1:name.index(".")])]["mlp"]["router"]["top"]
                    gap = (z[:, top - 1] - z[:, top]).min() if top < len(r) else 1e9
                    if best is None or gap > best[0]:
                        best = (gap, r)
                t[name] = best[1]
                t[name + ".b"] = bf16_round(0.02 * rng.standard_normal(len(best[1])))
    return t


def distance_mixer(heads=6, kv_heads=2, dim=24, vdim=40, window=40, bias_max=64, scale=None, v_mix=True):
    m = {"bias_max": bias_max, "dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": None if window is None else {"size": window}, "scale": float(scale if scale is not None else dim ** -0.5), "vdim": vdim}
    return {**m, "v_mix": True} if v_mix else m


def scan_pair(heads=6, kv_heads=2, dim=24, vdim=40, window=40, pool=8, rot=16, base=3000.0, softcap=20.0, scale=None, inner=72, state=16, rank=12, conv=4, scales=(0.7, 1.2)):
    left = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": None if window is None else {"pool": pool, "size": window}, "rot": {"base": float(base), "dims": rot},
            "scale": float(scale if scale is not None else 1.5 * dim ** -0.5), "softcap": float(softcap), "vdim": vdim}
    return {"left": left, "left_scale": scales[0], "right": {"conv": conv, "dt_rank": rank, "inner": inner, "state": state}, "right_scale": scales[1]}


def make_tarulix(width=136, vocab=203, layers=(), eps=1e-5):
    """``layers``: (type, mixer, feed-forward) per layer, the feed-forward None or (experts, top, size, identity choices, size of the shared expert)."""
    def ff(f):
        return f and {"expert": {"ff": f[2]}, "kind": "moe", "router": {"experts": f[0], "identity": f[3], "top": f[1]}, "shared": {"ff": f[4]}}
    return {"architecture": "Tarulix", "layers": [{"mixer": m, "mlp": ff(f), "type": t} for t, m, f in layers], "norm": {"eps": eps}, "vocab": vocab, "width": width}


def random_tarulix(cfg, seed=0, clear=True, buckets=16):
    """Seeded weights of a Tarulix model, rounded to bfloat16.  clear: as for Mokatar; what is passed on scales the marked columns up, so routers are
    drawn for a range of scales."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    t = {}

    def mat(name, out, inp, gain=1.0):
        t[name] = bf16_round(rng.standard_normal((out, inp)) * (gain / math.sqrt(inp)))

    def vec(name, n, mean, dev):
        t[name] = bf16_round(mean + dev * rng.standard_normal(n))

    def scalar(name, lo, hi):
        t[name] = bf16_round(np.asarray(lo + (hi - lo) * rng.random()))

    def attention(x, m):
        H, q, k, v = m["heads"], m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        for n, c in (("q", q), ("k", k), ("v", v)):
            mat(x + n, c, W)
            vec(x + n + ".b", c, 0.0, 1.0 if n == "k" and x.endswith("left.") else 0.5)     # keys of a block have something in common
        mat(x + "o", W, H * m["vdim"], 4.0 if x.endswith("left.") else 2.0)
        vec(x + "o.b", W, 0.0, 0.2)
        return H

    t["embed"] = bf16_round(rng.standard_normal((cfg["vocab"], W)))
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x = p + "mix."
        scalar(p + "norm1", 0.6, 1.4)
        if L["type"] == "parallel":
            H = attention(x + "left.", m["left"])
            t[x + "left.talk"] = bf16_round(np.eye(H) + 0.4 * rng.standard_normal((H, H)))
            r = m["right"]
            n, s, k = r["inner"], r["state"], r["dt_rank"]
            x += "right."
            mat(x + "in", 2 * n, W, 0.7)
            t[x + "conv"] = bf16_round(0.6 * rng.standard_normal((n, r["conv"])))
            vec(x + "conv.b", n, 0.0, 0.3)
            mat(x + "x", k + 2 * s, n, 0.7)
            mat(x + "dt", n, k, 1.5)
            vec(x + "dt.b", n, -2.5, 1.5)
            t[x + "A_log"] = bf16_round(-1.0 + 1.5 * rng.standard_normal((n, s)))
            vec(x + "D", n, 0.8, 0.3)
            mat(x + "o", W, n, 2.0)
        else:
            H = attention(x, m)
            t[x + "rel"] = bf16_round(rng.standard_normal((buckets, H)))
            vec(x + "sink", H, 1.0, 1.5)
            if m.get("v_mix"):
                scalar(x + "vmix", 0.2, 0.8)
        f = L.get("mlp")
        if f:
            scalar(p + "norm2", 0.6, 1.4)
            E, C, n, sh = f["router"]["experts"], f["router"]["experts"] + f["router"]["identity"], f["expert"]["ff"], f["shared"]["ff"]
            for e, c in [(f"e{e}", n) for e in range(E)] + [("shared", sh)]:
                mat(p + f"mlp.{e}.gate", c, W, 1.5)
                mat(p + f"mlp.{e}.up", c, W, 1.5)
                mat(p + f"mlp.{e}.down", W, c, 2.0)
            mat(p + "mlp.router", C, W, 2.0)
            vec(p + "mlp.correction", C, 0.3, 0.3)
    scalar("final.norm", 0.6, 1.4)
    mat("head", cfg["vocab"], W)
    if clear:
        t["embed"][:, :MARKERS] = np.sign(rng.standard_normal((cfg["vocab"], MARKERS)))
        patterns = np.array([[1.0 if i >> c & 1 else -1.0 for c in range(MARKERS)] for i in range(1 << MARKERS)])
        patterns = np.concatenate([s * patterns for s in np.linspace(1.0, 2.5, 16)])
        for name in t:
            if name.endswith((".o", ".down", ".o.b")):
                t[name][:MARKERS] = 0
            if name.endswith("mlp.router"):
                top, best = cfg["layers"][int(name[1:name.index(".")])]["mlp"]["router"]["top"], None
                for _ in range(300):     # of some routers the one whose closest call is least close
                    r = np.zeros_like(t[name])
                    r[:, :MARKERS] = bf16_round(2.0 * rng.standard_normal((len(r), MARKERS)))
                    corr = bf16_round(0.3 + (0.3 if len(r) < 20 else 0.6) * rng.standard_normal(len(r)))
                    e = np.exp(patterns @ r[:, :MARKERS].T)
                    z = np.sort(e / e.sum(1, keepdims=True) + corr, axis=1)[:, ::-1]
                    gap = (z[:, top - 1] - z[:, top]).min() if top < len(r) else 1e9
                    if best is None or gap > best[0]:
                        best = (gap, r, corr)
                _, t[name], t[name[:-6] + "correction"] = best
    return t


def random_tensors(cfg, seed=0):
    """Seeded weights, rounded to bfloat16, in which every factor matters (norm weights and biases away from 1 and 0)."""
    if cfg["architecture"] == "Tarulix":
        return random_tarulix(cfg, seed)
    if cfg["architecture"] == "Mokatar":
        return random_mokatar(cfg, seed)
    if cfg["architecture"] == "Robazen":
        return random_robazen(cfg, seed)
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    t = {}

    def mat(name, out, inp, gain=1.0):
        t[name] = bf16_round(rng.standard_normal((out, inp)) * (gain / math.sqrt(inp)))

    def norm(name):
        t[name] = bf16_round(1.0 + 0.3 * rng.standard_normal(W))
        t[name + ".b"] = bf16_round(0.2 * rng.standard_normal(W))
        t[name + ".alpha"] = bf16_round(np.asarray(0.5 + 0.4 * rng.random()))

    t["embed"] = bf16_round(rng.standard_normal((cfg["vocab"], W)))
    for i, L in enumerate(cfg["layers"]):
        if "weights_of" in L:
            continue
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1")
        mat(p + "mix.q", m["heads"] * (m["dim"] + m["rot_dim"]), W, 1.5)
        mat(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], W)
        t[p + "mix.dkv.norm"] = bf16_round(1.0 + 0.3 * rng.standard_normal(m["kv_rank"]))
        mat(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"], 1.5)
        mat(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
        mat(p + "mix.g", m["heads"] * m["vdim"], W, 2.0)
        mat(p + "mix.o", W, m["heads"] * m["vdim"], 2.0)
        if L.get("mlp"):
            mat(p + "mlp.gate", L["mlp"]["ff"], W, 1.5)
            mat(p + "mlp.up", L["mlp"]["ff"], W, 1.5)
            mat(p + "mlp.down", W, L["mlp"]["ff"], 1.0)
    norm("final.norm")
    mat("head", cfg["vocab"], W)
    return t
