"""A plain, slow implementation of the Fupapel design in float64 numpy: one function per mechanism, whole sequences at a
time, no cache, no batching.  The tests hold the engine against it.  It shares no code with the package.

A model is (cfg, w): cfg the contents of config.json, w a dict name -> float64 array.

    layer             x += m (mixer(shift(norm1 x)) + ff(norm2 x)), both sides of the same x; norms are x / rms(x) * (1 + weight)
    shift             a row mixed with the row before it, element by element: h_t + (h_(t-1) - h_t) * mu
    attention         grouped heads, an RMS norm over the whole q and the whole k, partial rotate-half rotation, keys of the
                      query's own chunk, softmax with one more in the denominator, a sigmoid gate per output element
    attention_2       the same masks and norms behind short convolutions of q, k and v; stretched frequencies; a factor per
                      head on the scores, a learned sink per head; a layer may read another layer's keys and values
    latent_attention  queries through a normed latent, keys and values from one normed latent per position beside a rotated
                      key part that all heads share; a learned sink and a sigmoid gate per head
    feed-forward      softmax over all experts and identities; choice by score + correction within the best groups; the scores
                      themselves weigh the chosen units; an identity returns its input
    output            final norm, output matrix
"""
from __future__ import annotations

import math

import numpy as np


def operand(a):
    """Every operand of a matrix product passes here.  The identity; a test that wants to know what 16-bit operands alone do
    to a model's logits replaces it by a rounding."""
    return a


def rms_unit(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_plain(x, weight, eps):
    return rms_unit(x, eps) * weight


def norm_one_plus(x, weight, eps):
    return rms_unit(x, eps) * (1.0 + weight)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def token_shift(h, mu, before=None):
    """h [T, n]; `before` [n]: the row ahead of the first (zeros at a sequence's start)."""
    first = np.zeros((1, h.shape[1])) if before is None else before[None, :]
    previous = np.concatenate([first, h[:-1]], axis=0)
    return h + (previous - h) * mu


def short_conv(u, taps, before=None):
    """u [T, C], taps [C, J] (last column: the current row); `before` [J - 1, C]: the rows ahead of the first (zeros)."""
    T, C = u.shape
    J = taps.shape[1]
    pad = np.zeros((J - 1, C)) if before is None else before
    full = np.concatenate([pad, u], axis=0)
    out = np.zeros((T, C))
    for j in range(J):
        out += full[j: j + T] * taps[:, j]
    return out


def rotary_frequencies(rot):
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc:
            length = 2.0 * math.pi / f
            factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            if length > original / low:
                f = f / factor
            elif length >= original / high:
                s = (original / length - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return np.array(out)


def rotate_half(x, positions, rot):
    """x [T, heads, dim]: element i < dims/2 of a head pairs with element i + dims/2; the elements behind dims pass."""
    half = int(rot["dims"]) // 2
    a = np.asarray(positions, dtype=np.float64)[:, None] * rotary_frequencies(rot)[None, :]
    cos, sin = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half: 2 * half]
    return np.concatenate([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half:]], axis=-1)


# ---- masks and softmax ---------------------------------------------------------------------------------------------------
def sees_chunk(i, j, size):
    return j <= i and i // size == j // size


def sees_all(i, j, size=None):
    return j <= i


def visibility(positions, rule, size=None):
    p = np.asarray(positions)
    return np.array([[rule(int(i), int(j), size) for j in p] for i in p], dtype=bool)


def softmax_with_sink(s, sink):
    """s [T, keys] with -inf where a key is not seen: weights exp(s) / (exp(sink) + sum exp(s))."""
    m = np.maximum(s.max(axis=-1, keepdims=True), sink)
    p = np.exp(s - m)
    return p / (p.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def attend(q, k, v, scale, see, sinks, temps=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; sinks [H]; temps [H] multiplies the heads' scores."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[-1]))
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * scale * (1.0 if temps is None else temps[hd])
        out[:, hd] = operand(softmax_with_sink(np.where(see, s, -np.inf), sinks[hd])) @ v[:, g]
    return out


# ---- mixers --------------------------------------------------------------------------------------------------------------
def attention(h, m, w, p, eps, positions=None, store=None, borrowed=None):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    positions = np.arange(T) if positions is None else np.asarray(positions)
    q = norm_plain(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, H, d)
    k = norm_plain(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, G, d)
    v = operand((h @ w[p + "v"].T).reshape(T, G, dv))
    q, k = operand(rotate_half(q, positions, m["rot"])), operand(rotate_half(k, positions, m["rot"]))
    see = visibility(positions, sees_chunk, int(m["mask"]["size"]))
    out = attend(q, k, v, float(m["scale"]), see, np.zeros(H)).reshape(T, H * dv)
    return operand(out * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def conv_attention(h, m, w, p, eps, positions=None, store=None, borrowed=None):
    """`store` receives (keys, values) as another layer would read them; `borrowed`: such a pair of another layer."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    positions = np.arange(T) if positions is None else np.asarray(positions)
    q = norm_plain(short_conv(h @ w[p + "q"].T, w[p + "q.conv"]), w[p + "q.norm"], eps).reshape(T, H, d)
    q = rotate_half(q, positions, m["rot"])
    if borrowed is None:
        k = norm_plain(short_conv(h @ w[p + "k"].T, w[p + "k.conv"]), w[p + "k.norm"], eps).reshape(T, G, d)
        k = operand(rotate_half(k, positions, m["rot"]))
        v = operand(short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).reshape(T, G, dv))
    else:
        k, v = borrowed
    if store is not None:
        store.append((k, v))
    see = visibility(positions, sees_chunk, int(m["mask"]["size"]))
    out = attend(operand(q), k, v, float(m["scale"]), see, w[p + "sink"], w[p + "temp"])
    return operand(out.reshape(T, H * dv)) @ w[p + "o"].T


def latent_attention(h, m, w, p, eps, positions=None, store=None, borrowed=None):
    T = h.shape[0]
    H, dn, dr, dv, R = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    positions = np.arange(T) if positions is None else np.asarray(positions)
    cq = operand(norm_plain(h @ w[p + "dq"].T, w[p + "dq.norm"], eps))
    q = (cq @ w[p + "uq"].T).reshape(T, H, dn + dr)
    low = h @ w[p + "dkv"].T
    c = operand(norm_plain(low[:, :R], w[p + "dkv.norm"], eps))
    k_rot = rotate_half(low[:, None, R:], positions, m["rot"])                          # one part for all heads
    q_rot = rotate_half(q[..., dn:], positions, m["rot"])
    k = (c @ w[p + "uk"].T).reshape(T, H, dn)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    q = operand(np.concatenate([q[..., :dn], q_rot], axis=-1))
    k = operand(np.concatenate([k, np.repeat(k_rot, H, axis=1)], axis=-1))
    out = attend(q, k, operand(v), float(m["scale"]), visibility(positions, sees_all), w[p + "sink"])
    out = out * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return operand(out.reshape(T, H * dv)) @ w[p + "o"].T


MIXERS = {"attention": attention, "attention_2": conv_attention, "latent_attention": latent_attention}


# ---- feed-forward --------------------------------------------------------------------------------------------------------
def unit(h, w, p):
    return operand(silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def router_scores(h, w, p):
    z = h @ w[p + "router"].T
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def choice_scores(s, correction, groups):
    """s [T, N] -> the scores by which experts are chosen, -inf outside the groups that are kept."""
    c = s + correction
    if not groups:
        return c
    count, keep = int(groups["count"]), int(groups["keep"])
    best = c.reshape(c.shape[0], count, -1).max(axis=-1)
    kept = np.argsort(-best, axis=-1, kind="stable")[:, :keep]
    mask = np.zeros(best.shape, dtype=bool)
    np.put_along_axis(mask, kept, True, axis=-1)
    return np.where(np.repeat(mask, c.shape[1] // count, axis=1), c, -np.inf)


def route(h, w, p, router):
    """(chosen [T, top], their weights [T, top])."""
    s = router_scores(h, w, p)
    c = choice_scores(s, w[p + "correction"], router.get("groups"))
    chosen = np.argsort(-c, axis=-1, kind="stable")[:, :int(router["top"])]
    return chosen, np.take_along_axis(s, chosen, axis=-1)


def router_margin(h, w, p, router):
    """Per row: how far its choice is from another one, of a group or of an expert (in score)."""
    s = router_scores(h, w, p)
    out = np.full(s.shape[0], np.inf)
    groups = router.get("groups")
    if groups and int(groups["keep"]) < int(groups["count"]):
        best = np.sort((s + w[p + "correction"]).reshape(s.shape[0], int(groups["count"]), -1).max(axis=-1), axis=-1)[:, ::-1]
        out = np.minimum(out, best[:, int(groups["keep"]) - 1] - best[:, int(groups["keep"])])
    c = np.sort(choice_scores(s, w[p + "correction"], groups), axis=-1)[:, ::-1]
    top = int(router["top"])
    if c.shape[1] > top:
        gap = c[:, top - 1] - c[:, top]
        out = np.minimum(out, np.where(np.isfinite(gap), gap, np.inf))
    return out


def experts_ff(h, mlp, w, p, margins=None):
    router = mlp["router"]
    chosen, weight = route(h, w, p, router)
    if margins is not None:
        margins.append(router_margin(h, w, p, router))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], weight[t]):
            row = h[t: t + 1]
            out[t] += s * (unit(row, w, f"{p}e{int(e)}.")[0] if e < int(router["experts"]) else row[0])
    return out


# ---- the model -----------------------------------------------------------------------------------------------------------
def layer(x, spec, w, p, cfg, margins=None, store=None, borrowed=None):
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    h = operand(token_shift(norm_one_plus(x, w[p + "norm1"], eps), w[p + "shift"]))
    out = MIXERS[spec["type"]](h, spec["mixer"], w, p + "mix.", eps, store=store, borrowed=borrowed)
    if spec.get("mlp") is not None:
        out = out + experts_ff(operand(norm_one_plus(x, w[p + "norm2"], eps)), spec["mlp"], w, p + "mlp.", margins)
    return x + m * out


def forward(cfg, w, tokens, streams=None, margins=None):
    """Logits [T, vocab] of one whole sequence.  `streams`: a list that receives the stream after every layer."""
    x = w["embed"][np.asarray(tokens)]
    kept = {}
    for i, spec in enumerate(cfg["layers"]):
        source = spec["mixer"].get("kv_from")
        store = []
        x = layer(x, spec, w, f"l{i}.", cfg, margins, store, None if source is None else kept[int(source)])
        if store:
            kept[i] = store[0]
        if streams is not None:
            streams.append(x.copy())
    return operand(norm_one_plus(x, w["final.norm"], float(cfg["norm"]["eps"]))) @ w["head"].T
