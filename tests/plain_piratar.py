"""A plain, slow implementation of the Piratar design in float64 numpy: one function per mechanism, whole sequences at a
time, no cache, no batching.  The tests hold the engine against it.  It shares no code with the package.

A model is (cfg, w): cfg the contents of config.json, w a dict name -> float64 array.

    embedding     rms_norm(scale E[token] + B[hash(previous token, token)]), the norm's weight stored around zero
    layer         x += mixer(norm1 x) + ff(norm2 x), both of the same x; then the token's own side vector e of the layer:
                  y = P (gelu(G x) * e), x += y / rms(y) * w
    parallel      half of softmax attention (short convolutions, rotation in halves, grouped heads, a gate per output element)
                  plus half of retention (a constant decay per head, rotated queries and keys), each RMS-normed over the width
    rglru         a gated branch beside a convolved branch that runs through a real-gated linear recurrence per channel
    feed-forward  a gated silu unit, or experts chosen by softmax with renormalised and scaled weights beside a gated shared one
    output        final norm, output matrix
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


def norm_one_plus(x, weight, eps):
    return rms_unit(x, eps) * (1.0 + weight)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


# ---- embedding -----------------------------------------------------------------------------------------------------------
def bigram_rows(tokens, bigram, before=None):
    """The row of the pair table of every token; `before`: the token ahead of the first (None: the sequence starts here)."""
    buckets, out, last = int(bigram["buckets"]), [], before
    for t in tokens:
        out.append(buckets if last is None else (int(last) * int(bigram["mul_prev"]) + int(t) * int(bigram["mul_cur"])) % buckets)
        last = t
    return np.array(out)


def embedding(tokens, cfg, w, before=None):
    emb = cfg["embedding"]
    x = w["embed"][np.asarray(tokens)] * float(emb["scale"])
    if emb.get("bigram"):
        x = x + w["bigram"][bigram_rows(tokens, emb["bigram"], before)]
    return norm_one_plus(x, w["embed.norm"], float(cfg["norm"]["eps"]))


# ---- mechanisms of the mixers ----------------------------------------------------------------------------------------------
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


def rotate_half(x, positions, rot):
    """x [T, heads, dim]: element i < dims/2 of a head pairs with element i + dims/2; the elements behind dims pass."""
    if not rot or not int(rot.get("dims") or 0):
        return x
    dims = int(rot["dims"])
    half = dims // 2
    f = np.array([float(rot["base"]) ** (-2.0 * i / dims) for i in range(half)])
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    cos, sin = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half: dims]
    return np.concatenate([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], axis=-1)


def causal_softmax(s):
    """s [T, T] scores: row i's weights over the keys 0 .. i."""
    T = s.shape[0]
    s = np.where(np.tril(np.ones((T, T), dtype=bool)), s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return p / p.sum(axis=-1, keepdims=True)


def attention(h, m, w, p, positions=None):
    """Grouped heads behind short convolutions; every earlier key; a sigmoid gate per output element."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    positions = np.arange(T) if positions is None else positions
    conv = lambda n: short_conv(h @ w[p + n].T, w[p + n + ".conv"])
    q = operand(rotate_half(conv("q").reshape(T, H, d), positions, m.get("rot")))
    k = operand(rotate_half(conv("k").reshape(T, G, d), positions, m.get("rot")))
    v = operand(conv("v").reshape(T, G, dv))
    out = np.zeros((T, H, dv))
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = operand(causal_softmax((q[:, hd] @ k[:, g].T) * float(m["scale"]))) @ v[:, g]
    return operand(out.reshape(T, H * dv) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def retention_scan(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, dv], decay [H]: S = decay S + k v^T, o = S^T q per head; (o [T, H, dv], the last state)."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[-1])) if state is None else state.copy()
    out = np.zeros((T, H, v.shape[-1]))
    for t in range(T):
        S = S * np.asarray(decay)[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S, q[t])
    return out, S


def retention(h, m, w, p, eps, positions=None):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    positions = np.arange(T) if positions is None else positions
    q = rotate_half((h @ w[p + "q"].T).reshape(T, H, d), positions, m.get("rot"))
    k = rotate_half((h @ w[p + "k"].T).reshape(T, H, d), positions, m.get("rot")) * d ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    o, _ = retention_scan(q, k, v, m["decay"])
    return operand(rms_unit(o, eps).reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, m, w, p, eps):
    left = attention(h, m["left"], w, p + "left.")
    right = retention(h, m["right"], w, p + "right.", eps)
    return 0.5 * (rms_unit(left, eps) * w[p + "left.out"] + rms_unit(right, eps) * w[p + "right.out"])


def block_maps(u, matrices, bias):
    """u [T, C] in equal parts, each through its own square matrix: matrices [B, C/B, C/B] (out, in), bias [B, C/B]."""
    B, n, _ = matrices.shape
    return (np.einsum("tbi,boi->tbo", u.reshape(-1, B, n), matrices) + bias).reshape(u.shape[0], -1)


def gated_linear_scan(u, r, i, lam, state=None):
    """S = a S + sqrt(1 - a^2) i u with log a = -8 r softplus(lam), per channel; (S of every row, the last one)."""
    T, C = u.shape
    S = np.zeros(C) if state is None else state.copy()
    out = np.zeros((T, C))
    for t in range(T):
        a = np.exp(-8.0 * r[t] * softplus(lam))
        S = a * S + np.sqrt(1.0 - a * a) * i[t] * u[t]
        out[t] = S
    return out, S


def rglru(h, m, w, p, eps=None):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = short_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"]) + w[p + "conv.b"]
    r = sigmoid(block_maps(u, w[p + "ra"], w[p + "ra.b"]))
    i = sigmoid(block_maps(u, w[p + "ri"], w[p + "ri.b"]))
    S, _ = gated_linear_scan(u, r, i, w[p + "lam"])
    return operand(S * y) @ w[p + "o"].T


MIXERS = {"parallel": parallel, "rglru": rglru}


# ---- feed-forward --------------------------------------------------------------------------------------------------------
def unit(h, w, p):
    return operand(silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def router_scores(h, w, p):
    z = h @ w[p + "router"].T
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def route(h, w, p, router):
    """(chosen [T, top], their weights [T, top])."""
    s = router_scores(h, w, p)
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :int(router["top"])]
    picked = np.take_along_axis(s, chosen, axis=-1)
    scale = router.get("scale")
    return chosen, picked / (picked.sum(axis=-1, keepdims=True) + 1e-20) * (1.0 if scale is None else float(scale))


def router_margin(h, w, p, router):
    """Per row: how far its choice of experts is from another one (in score)."""
    s = np.sort(router_scores(h, w, p), axis=-1)[:, ::-1]
    top = int(router["top"])
    return s[:, top - 1] - s[:, top] if s.shape[1] > top else np.full(s.shape[0], np.inf)


def experts_ff(h, mlp, w, p, margins=None):
    chosen, weight = route(h, w, p, mlp["router"])
    if margins is not None:
        margins.append(router_margin(h, w, p, mlp["router"]))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], weight[t]):
            out[t] += s * unit(h[t: t + 1], w, f"{p}e{int(e)}.")[0]
    if mlp.get("shared") is not None:
        out = out + unit(h, w, p + "shared.") * sigmoid(h @ w[p + "shared.sg"].T)
    return out


# ---- the model -----------------------------------------------------------------------------------------------------------
def token_side(x, tokens, index, dim, w, p, eps):
    e = w["side.embed"][np.asarray(tokens)][:, index * dim: (index + 1) * dim]
    y = operand(gelu_tanh(operand(x) @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return x + rms_unit(y, eps) * w[p + "norm"]


def layer(x, tokens, index, cfg, w, margins=None):
    spec, p, eps = cfg["layers"][index], f"l{index}.", float(cfg["norm"]["eps"])
    out = MIXERS[spec["type"]](operand(norm_one_plus(x, w[p + "norm1"], eps)), spec["mixer"], w, p + "mix.", eps)
    mlp = spec.get("mlp")
    if mlp is not None:
        h2 = operand(norm_one_plus(x, w[p + "norm2"], eps))
        out = out + (unit(h2, w, p + "mlp.") if mlp["kind"] == "dense" else experts_ff(h2, mlp, w, p + "mlp.", margins))
    x = x + out
    if cfg.get("token_side"):
        x = token_side(x, tokens, index, int(cfg["token_side"]["dim"]), w, p + "side.", eps)
    return x


def forward(cfg, w, tokens, streams=None, margins=None):
    """Logits [T, vocab] of one whole sequence.  `streams`: a list that receives the stream after every layer."""
    x = embedding(tokens, cfg, w)
    for i in range(len(cfg["layers"])):
        x = layer(x, tokens, i, cfg, w, margins)
        if streams is not None:
            streams.append(x.copy())
    return operand(norm_one_plus(x, w["final.norm"], float(cfg["norm"]["eps"]))) @ w["head"].T
