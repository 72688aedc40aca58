"""Plain, slow implementation of the Sebudra decoder design (numpy, float64): the oracle of tests/test_gpu_sebudra.py.

One function per mechanism, written from the design's equations; nothing here is shared with the engine.  A model is a configuration
dictionary (the keys of config.json) and a dictionary name -> float array.  A sequence is evaluated from its first token on in one
piece; keys, values and states are those of the whole sequence, so the answer at a position does not depend on any batching.

  residual        one norm a layer: h = norm(x), x <- x + mixer(h) + ff(h); the start is embed[token] * a constant
  norm            y = x / sqrt(mean(x^2) + eps) * w
  attention       grouped heads; q and k normed per head with one weight vector for all heads, THEN turned (half-split pairs); weights are
                  a softmax over the visible keys, or sigmoid(capped score + per-head number) without any normalisation
  state space     one input projection [z | x | B | C | dt]; causal depth-wise convolution + silu on x, B, C; per head
                  S <- exp(-exp(A) dt) S + dt B x^T, y = S^T C + D x; times silu(z), normed in equal parts, output projection
  gla             S <- diag(a) S + k v^T, o = S^T q with a decay per key channel; per-head norm, silu gate, output projection
  side by side    left_scale * attention(h) + right_scale * state_space(h)
  dense ff        down(g sigmoid(1.702 g) (u + 1)) with g, u cut at a limit
  routed ff       sigmoid scores, choice by corrected scores inside the best groups, weights without the correction
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


# ---- rotation -----------------------------------------------------------------------------------------------------------------
def frequencies(rot):
    """-> (frequency of every pair, factor on cos and sin)"""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_with_turns(t):   # the (real-valued) pair index whose angle makes t turns over the original context
        return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_with_turns(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_with_turns(float(sc["slow"]))), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(v, pos, rot):
    """v [n, heads, d], pos [n]: coordinate i of the first rot.dims pairs with i + dims / 2."""
    f, amp = frequencies(rot)
    half = len(f)
    ang = pos[:, None] * f[None, :]
    c, s = (np.cos(ang) * amp)[:, None, :], (np.sin(ang) * amp)[:, None, :]
    out = np.array(v, np.float64, copy=True)
    a, b = v[..., :half], v[..., half:2 * half]
    out[..., :half] = a * c - b * s
    out[..., half:2 * half] = b * c + a * s
    return out


# ---- attention ----------------------------------------------------------------------------------------------------------------
def sees(i, j, window):
    """window 0: everything before and itself"""
    return 0 <= i - j and (window <= 0 or i - j < window)


def visible(n, window):
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (d >= 0) & ((d < window) if window > 0 else True)


def softmax_weights(score, mask):
    score = np.where(mask, score, -np.inf)
    e = np.exp(score - score.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def sigmoid_weights(score, pb, mask):
    """score [H, n, n]"""
    return np.where(mask, sigmoid(score + pb[:, None, None]), 0.0)


def attention(W, p, mx, eps, h, biased, mask=None):
    """h [n, width] -> [n, width].  mask (tests): [n, n] instead of the design's own."""
    n = len(h)
    H, G, d, dv = (int(mx[k]) for k in ("heads", "kv_heads", "dim", "vdim"))

    def project(name, heads, size):
        y = h @ W[p + name].T
        return (y + W[p + name + ".b"] if biased else y).reshape(n, heads, size)

    q, k, v = project("q", H, d), project("k", G, d), project("v", G, dv)
    pos = np.arange(n, dtype=np.float64)
    q = rotate(norm(q, W[p + "q.norm"], eps), pos, mx["rot"])
    k = rotate(norm(k, W[p + "k.norm"], eps), pos, mx["rot"])
    k, v = np.repeat(k, H // G, axis=1), np.repeat(v, H // G, axis=1)
    score = np.einsum("ihd,jhd->hij", q, k) * float(mx["scale"])
    if mx.get("softcap"):
        score = float(mx["softcap"]) * np.tanh(score / float(mx["softcap"]))
    if mask is None:
        mask = visible(n, int(mx["mask"]["size"]) if mx.get("mask") else 0)
    wgt = softmax_weights(score, mask) if (p + "pb") not in W else sigmoid_weights(score, W[p + "pb"], mask)
    return np.einsum("hij,jhv->ihv", wgt, v).reshape(n, H * dv) @ W[p + "o"].T


# ---- recurrences --------------------------------------------------------------------------------------------------------------
def short_conv(x, w, b):
    """x [n, channels], w [channels, taps] with the newest input's weight last, zeros before the start"""
    n, taps = len(x), w.shape[1]
    y = np.tile(b, (n, 1))
    for t in range(n):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y


def ssm_scan(x, B, C, dt, A_log, D):
    """x [n, heads, dv], B and C [n, groups, N], dt [n, heads] (positive)"""
    n, H, dv = x.shape
    per = H // B.shape[1]
    S = np.zeros((H, B.shape[2], dv))
    y = np.zeros_like(x)
    for t in range(n):
        Bh, Ch = np.repeat(B[t], per, axis=0), np.repeat(C[t], per, axis=0)
        S = np.exp(-np.exp(A_log) * dt[t])[:, None, None] * S + (dt[t][:, None] * Bh)[:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnv,hn->hv", S, Ch) + D[:, None] * x[t]
    return y


def norm_in_parts(y, w, parts, eps):
    n, size = y.shape
    z = y.reshape(n, parts, size // parts)
    return (z / np.sqrt(np.mean(z * z, axis=-1, keepdims=True) + eps)).reshape(n, size) * w


def state_space(W, p, mx, eps, h):
    n = len(h)
    H, dv, N, G = (int(mx[k]) for k in ("heads", "vdim", "state", "groups"))
    inner = H * dv
    u = h @ W[p + "in"].T
    z, xBC, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xBC = silu(short_conv(xBC, W[p + "conv"], W[p + "conv.b"]))
    x = xBC[:, :inner].reshape(n, H, dv)
    B, C = xBC[:, inner:inner + G * N].reshape(n, G, N), xBC[:, inner + G * N:].reshape(n, G, N)
    y = ssm_scan(x, B, C, softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"])
    y = norm_in_parts(y.reshape(n, inner) * silu(z), W[p + "norm"], int(mx["norm_groups"]), eps)
    return y @ W[p + "o"].T


def gla_decay(W, p, tau, h):
    return sigmoid(h @ W[p + "a1"].T @ W[p + "a2"].T + W[p + "a2.b"]) ** (1.0 / tau)


def gla(W, p, mx, eps, h):
    n = len(h)
    H, d, dv = (int(mx[k]) for k in ("heads", "dim", "vdim"))
    q = (h @ W[p + "q"].T).reshape(n, H, d) * d ** -0.5
    k, v = (h @ W[p + "k"].T).reshape(n, H, d), (h @ W[p + "v"].T).reshape(n, H, dv)
    a = gla_decay(W, p, float(mx["tau"]), h).reshape(n, H, d)
    S = np.zeros((H, d, dv))
    o = np.zeros((n, H, dv))
    for t in range(n):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S, q[t])
    o = norm(o, W[p + "norm"], eps).reshape(n, H * dv) * silu(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def mixer(W, p, L, eps, h, mask=None):
    mx = L["mixer"]
    if L["type"] == "parallel":
        left = attention(W, p + "left.", mx["left"], eps, h, True, mask)
        return float(mx["left_scale"]) * left + float(mx["right_scale"]) * state_space(W, p + "right.", mx["right"], eps, h)
    if L["type"] == "attention":
        return attention(W, p, mx, eps, h, False, mask)
    if L["type"] == "gla":
        return gla(W, p, mx, eps, h)
    raise ValueError(L["type"])


# ---- feed-forward -------------------------------------------------------------------------------------------------------------
def dense_ff(W, p, limit, h):
    g = np.minimum(h @ W[p + "gate"].T, limit)
    u = np.clip(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def relu2_expert(W, p, h):
    return np.maximum(h @ W[p + "up"].T, 0.0) ** 2 @ W[p + "down"].T


def route(W, p, r, h):
    """one token -> [(expert, weight)]"""
    n, top = int(r["experts"]), int(r["top"])
    g = r.get("groups") or {"count": 1, "keep": 1}
    count, keep = int(g["count"]), int(g["keep"])
    s = sigmoid(W[p + "router"] @ h)
    choice = s + W[p + "correction"]
    size = n // count
    best = [sum(sorted(choice[i * size:(i + 1) * size])[-2:]) for i in range(count)]
    kept = sorted(range(count), key=lambda i: -best[i])[:keep]
    allowed = [e for i in kept for e in range(i * size, (i + 1) * size)]
    picked = sorted(allowed, key=lambda e: -choice[e])[:top]
    tot = sum(s[e] for e in picked) + 1e-20
    return [(e, s[e] / tot * float(r.get("scale", 1.0))) for e in picked]


def routed_ff(W, p, mlp, h):
    y = np.zeros_like(h)
    for t in range(len(h)):
        for e, w in route(W, p, mlp["router"], h[t]):
            y[t] += w * relu2_expert(W, p + "e%d." % e, h[t])
    if mlp.get("shared"):
        y += sigmoid(h @ W[p + "shared.sg"].T) * relu2_expert(W, p + "shared.", h)
    return y


def feed_forward(W, p, mlp, h):
    return dense_ff(W, p, float(mlp["limit"]), h) if mlp["kind"] == "dense" else routed_ff(W, p, mlp, h)


# ---- the model ----------------------------------------------------------------------------------------------------------------
def owner(cfg, i):
    """the layer whose tensors layer i uses"""
    while cfg["layers"][i].get("weights_of") is not None:
        i = int(cfg["layers"][i]["weights_of"])
    return i


def run(cfg, weights, tokens, masks=None):
    """-> (logits [n, vocab], residual stream after every layer [layers, n, width]); masks (tests): layer index -> [n, n]"""
    W = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][np.asarray(tokens, int)] * float(cfg["embedding"]["scale"])
    after = []
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % owner(cfg, i)
        h = norm(x, W[p + "norm1"], eps)
        y = mixer(W, p + "mix.", L, eps, h, (masks or {}).get(i))
        if L.get("mlp"):
            y = y + feed_forward(W, p + "mlp.", L["mlp"], h)
        x = x + y
        after.append(x)
    return norm(x, W["final.norm"], eps) @ W["head"].T, np.stack(after)
