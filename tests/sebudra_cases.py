"""Small Sebudra configurations with random weights for the tests, and helpers that run them through the engine.

Weights are rounded to bfloat16-representable values, so the bf16 and the fp32 engine and the plain implementation all see
exactly the same numbers."""
from __future__ import annotations

import math

import numpy as np

from binusun_cases import rel_err, run_schedule, to_bf16_values  # noqa: F401  (re-exported for the tests)
from tudasun_cases import row_errs  # noqa: F401

YARN = {"factor": 8.0, "fast": 16.0, "slow": 2.0, "original": 512}


def dense(ff=40, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff=12, experts=6, top=2, groups=(3, 2), scale=1.75, shared=20):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r, "shared": {"ff": shared} if shared else None}


def _heads(heads, kv_heads, dim, vdim, rot_dims, base, scaling, scale):
    mx = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims},
          "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    if scaling:
        mx["rot"]["scaling"] = scaling
    return mx


def attn(heads=4, kv_heads=2, dim=12, vdim=20, rot_dims=8, base=3000.0, softcap=6.0, scale=None, scaling=None, window=None, mlp=None):
    mx = _heads(heads, kv_heads, dim, vdim, rot_dims, base, scaling, scale)
    if softcap:
        mx["softcap"] = softcap
    if window:
        mx["mask"] = {"size": window}
    return {"type": "attention", "mlp": mlp, "mixer": mx}


def ssm(heads=4, vdim=8, state=12, groups=2, conv=3, parts=2):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": parts}


def par(heads=4, kv_heads=2, dim=12, vdim=16, rot_dims=8, base=20000.0, scaling=YARN, window=24, scale=None, right=None, left_scale=0.7, right_scale=1.3,
        softcap=None, mlp=None):
    left = _heads(heads, kv_heads, dim, vdim, rot_dims, base, scaling, scale)
    if window:
        left["mask"] = {"size": window}
    if softcap:
        left["softcap"] = softcap
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "left_scale": left_scale, "right": right or ssm(), "right_scale": right_scale}}


def gla(heads=3, dim=8, vdim=12, tau=8.0, rank=5, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "_rank": rank}


def again(cfg_layers, j):
    """layer j once more, on layer j's tensors"""
    return dict(cfg_layers[j], weights_of=j)


def make_config(layers, vocab=131, width=48, eps=1e-5, scale=1.5):
    return {"architecture": "Sebudra", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def public_config(cfg):
    """The configuration as a checkpoint folder carries it (test-only keys removed)."""
    return dict(cfg, layers=[{k: v for k, v in L.items() if not k.startswith("_")} for L in cfg["layers"]])


def random_weights(cfg, seed=0, out_amp=0.7, memory=0.0):
    """out_amp: size of the output matrices; memory shifts the recurrences' decays (larger: closer to 1)."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    W = {}

    def mat(o, i, amp=1.0):
        return to_bf16_values(rng.standard_normal((o, i)).astype(np.float32) * (amp / math.sqrt(i)))

    def vec(n, lo, hi):
        return to_bf16_values(rng.uniform(lo, hi, n).astype(np.float32))

    def noise(n, amp):
        return to_bf16_values((rng.standard_normal(n) * amp).astype(np.float32))

    def attention(p, mx, biased):
        H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        for nm, n in (("q", H * d), ("k", G * d), ("v", G * dv)):
            W[p + nm] = mat(n, D)
            if biased:
                W[p + nm + ".b"] = noise(n, 0.4)
        W[p + "q.norm"], W[p + "k.norm"] = vec(d, 0.5, 1.8), vec(d, 0.5, 1.8)
        W[p + "o"] = mat(D, H * dv, out_amp)

    W["embed"] = to_bf16_values(rng.standard_normal((V, D)).astype(np.float32))
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, mx = "l%d." % i, L["mixer"]
        W[p + "norm1"] = vec(D, 0.5, 1.5)
        if L["type"] == "parallel":
            attention(p + "mix.left.", mx["left"], True)
            r, q = mx["right"], p + "mix.right."
            inner, ch = r["heads"] * r["vdim"], r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"]
            W[q + "in"] = mat(inner + ch + r["heads"], D, 1.3)
            W[q + "conv"], W[q + "conv.b"] = noise((ch, r["conv"]), 0.6), noise(ch, 0.3)
            W[q + "dt_bias"], W[q + "A_log"], W[q + "D"] = vec(r["heads"], -2.0, 0.5), vec(r["heads"], -1.0 - memory, 1.0 - memory), vec(r["heads"], -1.0, 1.5)
            W[q + "norm"], W[q + "o"] = vec(inner, 0.5, 1.5), mat(D, inner, out_amp)
        elif L["type"] == "attention":
            attention(p + "mix.", mx, False)
            W[p + "mix.pb"] = vec(mx["heads"], -3.5, -1.0)
        else:
            H, d, dv, R = mx["heads"], mx["dim"], mx["vdim"], L.get("_rank", 5)
            W[p + "mix.q"], W[p + "mix.k"], W[p + "mix.v"], W[p + "mix.g"] = mat(H * d, D), mat(H * d, D), mat(H * dv, D), mat(H * dv, D)
            W[p + "mix.a1"], W[p + "mix.a2"], W[p + "mix.a2.b"] = mat(R, D), mat(H * d, R), vec(H * d, -1.0 + memory, 2.0 + memory)
            W[p + "mix.norm"], W[p + "mix.o"] = vec(dv, 0.5, 1.5), mat(D, H * dv, out_amp)
        mlp = L.get("mlp")
        if mlp and mlp["kind"] == "dense":
            F = mlp["ff"]
            W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"] = mat(F, D, 1.5), mat(F, D, 1.5), mat(D, F, out_amp)
        elif mlp:
            n, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            for e in range(n):
                W[p + "mlp.e%d.up" % e], W[p + "mlp.e%d.down" % e] = mat(F, D), mat(D, F, out_amp)
            W[p + "mlp.router"], W[p + "mlp.correction"] = mat(n, D), vec(n, -0.6, 0.2)
            if mlp.get("shared"):
                S = mlp["shared"]["ff"]
                W[p + "mlp.shared.up"], W[p + "mlp.shared.down"], W[p + "mlp.shared.sg"] = mat(S, D), mat(D, S, out_amp), mat(1, D, 2.0)
    W["final.norm"] = vec(D, 0.5, 1.5)
    W["head"] = mat(V, D)
    return W


def fixed_choice(cfg, W):
    """The routers' choice decided by the corrections alone (bf16 comparisons: a rounding difference in front of a router would otherwise
    flip a close choice)."""
    W = dict(W)
    for i, L in enumerate(cfg["layers"]):
        if L.get("mlp") and L["mlp"]["kind"] == "moe" and L.get("weights_of") is None:
            n = L["mlp"]["router"]["experts"]
            W["l%d.mlp.correction" % i] = to_bf16_values((3.0 * np.random.default_rng(100 + i).permutation(n) - 2.0 * n).astype(np.float32))
    return W


def build_engine(cfg, W, dtype="float32", max_tokens=1024, max_seqs=4):
    from turboinfer_b200 import models
    return models.REGISTRY["Sebudra"](public_config(cfg), W, dtype, max_tokens, max_seqs)


def plant_pair(cfg, W, a, b, gain=12.0, bias=-9.0):
    """Makes token `a` (as a key) and token `b` (as a query) stand out against each other in head 0 of layer 0, whatever their
    positions: both get a large embedding along one coordinate of their own that no other token uses; the query of head 0 reads b's
    coordinate and the key of its key/value head reads a's coordinate with the same vector r, placed on coordinates that are NOT
    rotated.  The other tokens' queries and keys of these heads have nothing there."""
    W = {k: np.array(v, np.float32, copy=True) for k, v in W.items()}
    L = cfg["layers"][0]
    p, mx = ("l0.mix.left.", L["mixer"]["left"]) if L["type"] == "parallel" else ("l0.mix.", L["mixer"])
    d, rd = mx["dim"], mx["rot"]["dims"]
    assert rd < d, "the planted direction lives on the coordinates that do not turn"
    rng = np.random.default_rng(99)
    u, v = 0, 1   # the coordinates the two tokens own
    E = W["embed"]
    E[:, [u, v]] = 0.0
    E[[a, b]] = 0.0
    E[b, u] = gain
    E[a, v] = gain
    W["l0.norm1"][[u, v]] = 1.0
    r = np.zeros(d, np.float32)
    r[rd:] = rng.choice([-1.0, 1.0], d - rd) * 1.5
    W[p + "q"][:, [u, v]] = 0.0
    W[p + "k"][:, [u, v]] = 0.0
    W[p + "q"][rd:d] = 0.0
    W[p + "k"][rd:d] = 0.0
    W[p + "q"][:d, u] = r
    W[p + "k"][:d, v] = r
    W[p + "q.norm"][rd:] = 2.5
    W[p + "k.norm"][rd:] = 2.5
    if (p + "q.b") in W:
        W[p + "q.b"][:d] = 0.0
        W[p + "k.b"][:d] = 0.0
    if (p + "pb") in W:
        W[p + "pb"][0] = bias
    W[p + "o"][:, :mx["vdim"]] *= 4.0
    return {k: to_bf16_values(x) for k, x in W.items()}
