"""Plain, slow implementation of the Nubipel decoder design (numpy, float64): the oracle of tests/test_gpu_nubipel.py.

One function per mechanism, written from the design's equations; nothing here is shared with the engine.  A model is a configuration
dictionary (the keys of config.json) and a dictionary name -> float array.  A sequence is evaluated from its first token on in one
piece; keys, values and states are those of the whole sequence, so the answer at a position does not depend on any batching.

  residual        one norm a layer: h = norm(x), x <- x + mixer(h) + ff(h); the start is embed[token] * a constant
  attention       grouped heads, q and k normed per head with one weight vector for all heads, no rotation; a row sees the keys of its own
                  chunk of positions; the softmax has one more term exp(sink) per head in its denominator
  latent          q = Uq norm(Dq h), c = norm(Dkv h), per head k = Uk c and v = Uv c; causal softmax; the heads' outputs times sigmoid(G h)
  delta           q, k, v behind causal depth-wise convolutions and silu; unit q and k; per head S <- g S, u = beta (v - S^T k),
                  S <- S + k u^T, o = S^T q; per-head norm with a weight, times silu(G h)
  feed-forward    down(gelu(up h)) with the error-function gelu
  output          logits = cap * tanh(scale * (embed norm(x)) / cap)
"""
from __future__ import annotations

import math

import numpy as np

_erf = np.vectorize(math.erf, otypes=[float])


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


# ---- attention ----------------------------------------------------------------------------------------------------------------
def sees(i, j, chunk):
    """chunk 0: everything before and itself"""
    return j <= i and (chunk <= 0 or i // chunk == j // chunk)


def visible(n, chunk):
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i // chunk == j // chunk) if chunk > 0 else True)


def softmax_weights(score, mask, sink=None):
    """score [H, n, n]; sink [H]: a term without key or value in the denominator"""
    score = np.where(mask, score, -np.inf)
    top = score.max(-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink[:, None, None])
    e = np.exp(score - top)
    den = e.sum(-1, keepdims=True)
    if sink is not None:
        den = den + np.exp(sink[:, None, None] - top)
    return e / den


def attention(W, p, mx, eps, h, mask=None):
    """h [n, width] -> [n, width].  mask (tests): [n, n] instead of the design's own."""
    n = len(h)
    H, G, d, dv = (int(mx[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    q = norm((h @ W[p + "q"].T).reshape(n, H, d), W[p + "q.norm"], eps)
    k = norm((h @ W[p + "k"].T).reshape(n, G, d), W[p + "k.norm"], eps)
    v = (h @ W[p + "v"].T).reshape(n, G, dv)
    k, v = np.repeat(k, H // G, axis=1), np.repeat(v, H // G, axis=1)
    score = np.einsum("ihd,jhd->hij", q, k) * float(mx["scale"])
    if mask is None:
        mask = visible(n, int(mx["mask"]["size"]) if mx.get("mask") else 0)
    wgt = softmax_weights(score, mask, W[p + "sink"])
    return np.einsum("hij,jhv->ihv", wgt, v).reshape(n, H * dv) @ W[p + "o"].T


def latent_attention(W, p, mx, eps, h, mask=None):
    n = len(h)
    H, d, dv = (int(mx[k]) for k in ("heads", "dim", "vdim"))
    q = (norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).reshape(n, H, d)
    c = norm(h @ W[p + "dkv"].T, W[p + "dkv.norm"], eps)
    k, v = (c @ W[p + "uk"].T).reshape(n, H, d), (c @ W[p + "uv"].T).reshape(n, H, dv)
    score = np.einsum("ihd,jhd->hij", q, k) * float(mx["scale"])
    wgt = softmax_weights(score, visible(n, 0) if mask is None else mask)
    o = np.einsum("hij,jhv->ihv", wgt, v).reshape(n, H * dv)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---- delta rule ---------------------------------------------------------------------------------------------------------------
def short_conv(x, w):
    """x [n, channels], w [channels, taps] with the newest input's weight last, zeros before the start"""
    n, taps = len(x), w.shape[1]
    y = np.zeros_like(x)
    for t in range(n):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y


def delta_scan(q, k, v, g, beta):
    """q, k [n, H, dk] (k of unit length), v [n, H, dv], g and beta [n, H] -> o [n, H, dv]"""
    n, H, dk = q.shape
    S = np.zeros((H, dk, v.shape[2]))
    o = np.zeros_like(v)
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S, q[t])
    return o


def delta_decay(W, p, h):
    return np.exp(-np.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))


def delta(W, p, mx, eps, h):
    n = len(h)
    H, G, d, dv = (int(mx[k]) for k in ("heads", "kv_heads", "dim", "vdim"))

    def branch(name, heads, size):
        return silu(short_conv(h @ W[p + name].T, W[p + name + ".conv"])).reshape(n, heads, size)

    q, k, v = branch("q", G, d), branch("k", G, d), branch("v", H, dv)
    q, k = np.repeat(unit(q) * d ** -0.5, H // G, axis=1), np.repeat(unit(k), H // G, axis=1)
    o = delta_scan(q, k, v, delta_decay(W, p, h), sigmoid(h @ W[p + "b"].T))
    o = norm(o, W[p + "norm"], eps).reshape(n, H * dv) * silu(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def mixer(W, p, L, eps, h, mask=None):
    mx = L["mixer"]
    if L["type"] == "attention":
        return attention(W, p, mx, eps, h, mask)
    if L["type"] == "latent_attention":
        return latent_attention(W, p, mx, eps, h, mask)
    if L["type"] == "delta":
        return delta(W, p, mx, eps, h)
    raise ValueError(L["type"])


def feed_forward(W, p, h):
    return gelu(h @ W[p + "up"].T) @ W[p + "down"].T


# ---- the model ----------------------------------------------------------------------------------------------------------------
def logits(cfg, W, x):
    z = norm(x, W["final.norm"], float(cfg["norm"]["eps"])) @ W["embed"].T * float(cfg["logit_scale"])
    cap = float(cfg["logit_softcap"])
    return cap * np.tanh(z / cap)


def run(cfg, weights, tokens, masks=None):
    """-> (logits [n, vocab], residual stream after every layer [layers, n, width]); masks (tests): layer index -> [n, n]"""
    W = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][np.asarray(tokens, int)] * float(cfg["embedding"]["scale"])
    after = []
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % i
        h = norm(x, W[p + "norm1"], eps)
        y = mixer(W, p + "mix.", L, eps, h, (masks or {}).get(i))
        if L.get("mlp"):
            y = y + feed_forward(W, p + "mlp.", h)
        x = x + y
        after.append(x)
    return logits(cfg, W, x), np.stack(after)
