"""Small Nubipel configurations with random weights for the tests, and helpers that run them through the engine.

Weights are rounded to bfloat16-representable values, so the bf16 and the fp32 engine and the plain implementation all see
exactly the same numbers."""
from __future__ import annotations

import math

import numpy as np

from binusun_cases import rel_err, run_schedule, to_bf16_values  # noqa: F401  (re-exported for the tests)
from tudasun_cases import row_errs  # noqa: F401


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def attn(heads=4, kv_heads=2, dim=12, vdim=20, chunk=24, scale=None, mlp=None):
    mx = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    if chunk:
        mx["mask"] = {"size": chunk}
    return {"type": "attention", "mlp": mlp, "mixer": mx}


def latent(heads=3, dim=12, vdim=16, kv_rank=28, q_rank=20, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}}


def delta(heads=4, kv_heads=2, dim=12, vdim=20, conv=3, mlp=None):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def make_config(layers, vocab=131, width=48, eps=1e-5, scale=1.5, logit_scale=0.7, softcap=9.0):
    return {"architecture": "Nubipel", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "logit_scale": logit_scale, "logit_softcap": softcap}


def random_weights(cfg, seed=0, out_amp=0.7, memory=0.0):
    """out_amp: size of the output matrices; memory shifts the delta rule's decays (larger: closer to 1)."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    W = {}

    def mat(o, i, amp=1.0):
        return to_bf16_values(rng.standard_normal((o, i)).astype(np.float32) * (amp / math.sqrt(i)))

    def vec(n, lo, hi):
        return to_bf16_values(rng.uniform(lo, hi, n).astype(np.float32))

    W["embed"] = to_bf16_values(rng.standard_normal((V, D)).astype(np.float32) / math.sqrt(D) * 4.0)
    for i, L in enumerate(cfg["layers"]):
        p, mx = "l%d." % i, L["mixer"]
        q = p + "mix."
        H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
        W[p + "norm1"] = vec(D, 0.5, 1.5)
        if L["type"] == "attention":
            G = mx["kv_heads"]
            W[q + "q"], W[q + "k"], W[q + "v"] = mat(H * d, D), mat(G * d, D), mat(G * dv, D)
            W[q + "q.norm"], W[q + "k.norm"], W[q + "sink"] = vec(d, 0.5, 1.8), vec(d, 0.5, 1.8), vec(H, -1.0, 2.0)
        elif L["type"] == "latent_attention":
            R, Q = mx["kv_rank"], mx["q_rank"]
            W[q + "dq"], W[q + "dq.norm"], W[q + "uq"] = mat(Q, D), vec(Q, 0.5, 1.5), mat(H * d, Q)
            W[q + "dkv"], W[q + "dkv.norm"] = mat(R, D), vec(R, 0.5, 1.5)
            W[q + "uk"], W[q + "uv"], W[q + "g"] = mat(H * d, R), mat(H * dv, R), mat(H * dv, D, 1.5)
        else:
            G, taps = mx["kv_heads"], mx["conv"]
            for nm, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
                W[q + nm] = mat(n, D)
                W[q + nm + ".conv"] = to_bf16_values((rng.standard_normal((n, taps)) * 0.6).astype(np.float32))
            W[q + "b"], W[q + "a"], W[q + "g"] = mat(H, D, 1.5), mat(H, D), mat(H * dv, D)
            W[q + "A_log"], W[q + "dt_bias"], W[q + "norm"] = vec(H, -1.5 - memory, 0.5 - memory), vec(H, -2.0, 0.5), vec(dv, 0.5, 1.5)
        W[q + "o"] = mat(D, H * dv, out_amp)
        if L.get("mlp"):
            F = L["mlp"]["ff"]
            W[p + "mlp.up"], W[p + "mlp.down"] = mat(F, D, 1.5), mat(D, F, out_amp)
    W["final.norm"] = vec(D, 0.5, 1.5)
    return W


def build_engine(cfg, W, dtype="float32", max_tokens=1024, max_seqs=4):
    from turboinfer_b200 import models
    return models.REGISTRY["Nubipel"](cfg, W, dtype, max_tokens, max_seqs)


def plant_pair(cfg, W, a, b, gain=12.0):
    """Makes token `a` (as a key) and token `b` (as a query) stand out against each other in head 0 of layer 0: both get a large embedding
    along one coordinate of their own that no other token uses; head 0's queries read b's coordinate only and its keys a's coordinate only,
    along the same vector r, so that every other (query, key) pair of this head scores zero."""
    W = {k: np.array(v, np.float32, copy=True) for k, v in W.items()}
    L = cfg["layers"][0]
    p, mx = "l0.mix.", L["mixer"]
    d, dv = mx["dim"], mx["vdim"]
    u, v = 0, 1   # the coordinates the two tokens own
    E = W["embed"]
    E[:, [u, v]] = 0.0
    E[[a, b]] = 0.0
    E[b, u] = gain
    E[a, v] = gain
    W["l0.norm1"][[u, v]] = 1.0
    r = np.random.default_rng(99).choice([-1.0, 1.0], d).astype(np.float32) * 1.5
    if L["type"] == "attention":
        W[p + "q"][:, [u, v]] = 0.0
        W[p + "k"][:, [u, v]] = 0.0
        W[p + "q"][:d] = 0.0
        W[p + "k"][:d] = 0.0
        W[p + "q"][:d, u] = r
        W[p + "k"][:d, v] = r
        W[p + "q.norm"][:] = 2.5
        W[p + "k.norm"][:] = 2.5
    else:   # the low-rank vectors' first coordinates carry the pair
        for down, coord in (("dq", u), ("dkv", v)):
            W[p + down][0] = 0.0
            W[p + down][1:, [u, v]] = 0.0
            W[p + down][0, coord] = 3.0
            W[p + down + ".norm"][0] = 1.0
        for up in ("uq", "uk"):
            W[p + up][:d] = 0.0
            W[p + up][:, 0] = 0.0
            W[p + up][:d, 0] = r * 0.5
    W[p + "o"][:, :dv] *= 4.0
    return {k: to_bf16_values(x) for k, x in W.items()}
