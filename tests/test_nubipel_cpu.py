"""CPU-side checks around the Nubipel model: the plain implementation's own invariants (each mechanism against a second, direct
formula), the configuration reader and the checkpoint reader.  No GPU, no engine library."""
import math

import numpy as np
import pytest

import nubipel_plain as plain
from nubipel_cases import attn, delta, dense, latent, make_config, random_weights, rel_err


def toks(n, vocab, seed=0):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def f64(W):
    return {k: np.asarray(v, np.float64) for k, v in W.items()}


def test_prefix_property():
    cfg = make_config([latent(mlp=dense(16)), delta(), attn(chunk=5, mlp=dense(9))])
    W = random_weights(cfg, seed=1)
    t = toks(30, cfg["vocab"])
    assert rel_err(plain.run(cfg, W, t)[0][:17], plain.run(cfg, W, t[:17])[0]) < 1e-12


def test_chunks_count_from_position_zero():
    m = plain.visible(14, 5)
    assert [j for j in range(14) if m[9, j]] == [5, 6, 7, 8, 9]
    assert [j for j in range(14) if m[10, j]] == [10]
    assert [j for j in range(14) if m[12, j]] == [10, 11, 12]
    assert all(m[i, j] == plain.sees(i, j, 5) for i in range(14) for j in range(14))
    assert [j for j in range(14) if plain.visible(14, 0)[9, j]] == list(range(10))
    assert (plain.visible(6, 1) == np.eye(6, dtype=bool)).all()


def test_sink_takes_its_share_once_and_unscaled():
    s = np.random.default_rng(1).standard_normal((2, 4, 4)) * 3
    sink = np.array([0.3, -50.0])
    w = plain.softmax_weights(s, plain.visible(4, 0), sink)
    e = np.exp(s[0, 2, :3])
    assert np.allclose(w[0, 2, :3], e / (e.sum() + math.exp(0.3))) and w[0, 2, 3] == 0.0
    assert np.allclose(w[1], plain.softmax_weights(s, plain.visible(4, 0))[1])   # a sink of nothing: an ordinary softmax
    big = plain.softmax_weights(s * 400.0, plain.visible(4, 0), np.array([900.0, 1000.0]))
    assert np.isfinite(big).all()


def test_attention_against_loops():
    cfg = make_config([attn(heads=4, kv_heads=2, dim=3, vdim=2, chunk=3, scale=0.9)], width=8)
    W = f64(random_weights(cfg, seed=3))
    W["l0.mix.o"] = np.eye(8)
    h = np.random.default_rng(3).standard_normal((7, 8))
    mx, eps = cfg["layers"][0]["mixer"], 1e-5
    out = plain.attention(W, "l0.mix.", mx, eps, h)
    for i in range(7):
        for hd in range(4):
            g = hd // 2
            q = h[i] @ W["l0.mix.q"][3 * hd:3 * hd + 3].T
            q = q / math.sqrt((q * q).mean() + eps) * W["l0.mix.q.norm"]
            num, den = np.zeros(2), math.exp(W["l0.mix.sink"][hd])
            for j in range(i // 3 * 3, i + 1):
                k = h[j] @ W["l0.mix.k"][3 * g:3 * g + 3].T
                k = k / math.sqrt((k * k).mean() + eps) * W["l0.mix.k.norm"]
                e = math.exp(0.9 * (q @ k))
                num, den = num + e * (h[j] @ W["l0.mix.v"][2 * g:2 * g + 2].T), den + e
            assert np.allclose(out[i, 2 * hd:2 * hd + 2], num / den)


def test_latent_attention_equals_its_absorbed_form():
    """Moving Uk to the query and Uv behind the weighted sum is the same arithmetic; the gate per coordinate comes behind Uv."""
    cfg = make_config([latent(heads=2, dim=5, vdim=3, kv_rank=7, q_rank=4)], width=9)
    W = f64(random_weights(cfg, seed=4))
    h = np.random.default_rng(4).standard_normal((6, 9))
    mx, eps, p = cfg["layers"][0]["mixer"], 1e-5, "l0.mix."
    out = plain.latent_attention(W, p, mx, eps, h)
    c = h @ W[p + "dkv"].T
    c = c / np.sqrt((c * c).mean(-1, keepdims=True) + eps) * W[p + "dkv.norm"]
    cq = h @ W[p + "dq"].T
    cq = cq / np.sqrt((cq * cq).mean(-1, keepdims=True) + eps) * W[p + "dq.norm"]
    heads = []
    for hd in range(2):
        qa = cq @ W[p + "uq"][5 * hd:5 * hd + 5].T @ W[p + "uk"][5 * hd:5 * hd + 5]
        s = np.where(np.tri(6) > 0, qa @ c.T * mx["scale"], -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        heads.append(e / e.sum(-1, keepdims=True) @ c @ W[p + "uv"][3 * hd:3 * hd + 3].T)
    gate = 1.0 / (1.0 + np.exp(-(h @ W[p + "g"].T)))
    assert np.allclose(out, (np.concatenate(heads, 1) * gate) @ W[p + "o"].T)


def test_short_conv_is_a_causal_filter():
    rng = np.random.default_rng(2)
    x, w = rng.standard_normal((9, 5)), rng.standard_normal((5, 4))
    y = plain.short_conv(x, w)
    for c in range(5):
        assert np.allclose(y[:, c], np.convolve(x[:, c], w[c, ::-1])[:9])   # the last column meets the newest input
    assert np.allclose(plain.short_conv(x, w[:, :1]), x * w[:, 0])


def test_delta_rule_writes_what_the_state_does_not_answer():
    rng = np.random.default_rng(5)
    n, dk, dv = 4, 4, 3
    k = np.eye(dk)[:, None, :]
    v = rng.standard_normal((n, 1, dv))
    one, half = np.ones((n, 1)), np.full((n, 1), 0.5)
    # orthonormal keys, no decay, full step: every value is read back exactly at once
    assert np.allclose(plain.delta_scan(k, k, v, one, one), v)
    # the same key again with a full step replaces its value, whatever was there
    same = np.repeat(k[:1], n, axis=0)
    assert np.allclose(plain.delta_scan(same, same, v, one, one), v)
    # half a step: a running average; decay comes before the read of the old answer
    want, s = [], np.zeros(dv)
    for t in range(n):
        s = 0.5 * s
        s = s + 0.5 * (v[t, 0] - s)
        want.append(s)
    assert np.allclose(plain.delta_scan(same, same, v, half, half)[:, 0], want)


def test_delta_scan_equals_the_product_of_its_transitions():
    """S_t = g (I - beta k k^T) S_(t-1) + beta k v^T for unit keys, written out with matrices."""
    rng = np.random.default_rng(6)
    n, H, dk, dv = 6, 2, 5, 3
    q, k, v = rng.standard_normal((n, H, dk)), plain.unit(rng.standard_normal((n, H, dk))), rng.standard_normal((n, H, dv))
    g, b = rng.uniform(0.3, 1.0, (n, H)), rng.uniform(0.0, 1.0, (n, H))
    o = plain.delta_scan(q, k, v, g, b)
    for h in range(H):
        for t in range(n):
            S = np.zeros((dk, dv))
            for s in range(t + 1):
                A = np.eye(dk)
                for r in range(s + 1, t + 1):
                    A = g[r, h] * (np.eye(dk) - b[r, h] * np.outer(k[r, h], k[r, h])) @ A
                S += A @ (b[s, h] * np.outer(k[s, h], v[s, h]))
            assert np.allclose(o[t, h], q[t, h] @ S)


def test_delta_mixer_against_loops():
    cfg = make_config([delta(heads=4, kv_heads=2, dim=3, vdim=2, conv=2)], width=8)
    W = f64(random_weights(cfg, seed=7))
    W["l0.mix.o"] = np.eye(8)
    h = np.random.default_rng(7).standard_normal((5, 8))
    mx, eps, p = cfg["layers"][0]["mixer"], 1e-5, "l0.mix."
    out = plain.delta(W, p, mx, eps, h)

    def branch(nm, t):
        x = [h[t] @ W[p + nm].T, h[t - 1] @ W[p + nm].T if t else 0.0]
        z = x[0] * W[p + nm + ".conv"][:, 1] + x[1] * W[p + nm + ".conv"][:, 0]
        return z / (1 + np.exp(-z))
    for hd in range(4):
        S = np.zeros((3, 2))
        for t in range(5):
            q, k = branch("q", t)[3 * (hd // 2):][:3], branch("k", t)[3 * (hd // 2):][:3]
            v = branch("v", t)[2 * hd:][:2]
            q, k = q / math.sqrt(q @ q + 1e-6) / math.sqrt(3), k / math.sqrt(k @ k + 1e-6)
            a = h[t] @ W[p + "a"][hd] + W[p + "dt_bias"][hd]
            S = math.exp(-math.exp(W[p + "A_log"][hd]) * math.log1p(math.exp(a))) * S
            S = S + np.outer(k, (v - k @ S) / (1 + math.exp(-(h[t] @ W[p + "b"][hd]))))
            o = q @ S
            z = h[t] @ W[p + "g"][2 * hd:2 * hd + 2].T
            assert np.allclose(out[t, 2 * hd:2 * hd + 2], o / math.sqrt((o * o).mean() + eps) * W[p + "norm"] * z / (1 + np.exp(-z)))


def test_gelu_is_the_error_function_form():
    assert np.allclose(plain.gelu(np.array([0.0, 1.0, -1.0])), [0.0, 0.8413447460685429, -0.15865525393145707])
    z = np.linspace(-4, 4, 101)
    tanh_form = 0.5 * z * (1 + np.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))
    assert np.abs(plain.gelu(z) - tanh_form).max() > 1e-4


def test_logits_are_scaled_then_capped():
    cfg = make_config([attn()], logit_scale=0.3, softcap=2.0)
    W = f64(random_weights(cfg, seed=8))
    x = np.random.default_rng(8).standard_normal((3, cfg["width"]))
    z = plain.norm(x, W["final.norm"], 1e-5) @ W["embed"].T
    assert np.allclose(plain.logits(cfg, W, x), 2.0 * np.tanh(0.3 * z / 2.0))


def test_config_reader_takes_every_constant_from_the_configuration():
    from turboinfer_b200 import models, seq
    layers = [latent(heads=5, dim=10, vdim=14, kv_rank=36, q_rank=22, scale=0.21, mlp=dense(72)), delta(heads=6, kv_heads=3, dim=7, vdim=9, conv=5),
              attn(heads=6, kv_heads=2, dim=8, vdim=11, chunk=77, scale=0.4, mlp=dense(33))]
    cfg = make_config(layers, vocab=77, width=36, eps=3e-4, scale=0.25, logit_scale=0.125, softcap=21.0)
    m, L = models.nubipel_descs(cfg, seq.F32, 640, 3)
    assert (m.vocab, m.width, m.n_layers, m.max_tokens, m.max_seqs, m.mode) == (77, 36, 3, 640, 3, seq.F32)
    assert abs(m.norm_eps - 3e-4) < 1e-9 and m.norm_kind == seq.NORM_VECTOR and m.norm_place == seq.NORMS_SHARED
    assert (m.embed_scale, m.logit_scale, m.logit_softcap, m.tied_head, m.streams) == (0.25, 0.125, 21.0, 1, 0)
    a, b, c = L
    assert (a.mixer, a.heads, a.dim, a.vdim, a.kv_rank, a.q_rank, a.rot_dims, a.kv_from) == (seq.MIXER_LATENT, 5, 10, 14, 36, 22, 0, -1)
    assert (a.out_gate, a.sink, a.window, a.chunk) == (seq.GATE_ELEMENT, seq.SINK_NONE, 0, 0) and abs(a.scale - 0.21) < 1e-7
    assert (a.ff_kind, a.ff_act, a.ff) == (seq.FF_DENSE, seq.ACT_GELU, 72)
    assert (b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.mix_taps, b.ff) == (seq.MIXER_DELTA, 6, 3, 7, 9, 5, 0)
    assert (c.mixer, c.heads, c.kv_heads, c.dim, c.vdim, c.chunk, c.window, c.rot_dims) == (seq.MIXER_ATTENTION, 6, 2, 8, 11, 77, 0, 0)
    assert (c.qk_norm, c.sink, c.out_gate, c.ff) == (seq.QK_NORM_HEAD_GAIN, seq.SINK_LEARNED, seq.GATE_NONE, 33) and abs(c.scale - 0.4) < 1e-7
    assert models.nubipel_descs(make_config([attn(chunk=None)]), seq.F32, 64, 1)[1][0].chunk == 0
    for bad in (dict(attn(), type="wkv"), attn(mlp={"kind": "sparse", "ff": 8}), attn(chunk=-3)):
        with pytest.raises(ValueError):
            models.nubipel_descs(make_config([bad]), seq.F32, 64, 1)
    for gone in ("embedding", "norm", "layers", "logit_scale", "logit_softcap", "vocab"):
        with pytest.raises(ValueError):
            models.nubipel_descs({k: v for k, v in cfg.items() if k != gone}, seq.F32, 64, 1)
    for L0, key in ((latent(), "kv_rank"), (latent(), "q_rank"), (delta(), "conv"), (delta(), "kv_heads"), (attn(), "scale")):
        with pytest.raises(ValueError):
            models.nubipel_descs(make_config([dict(L0, mixer={k: v for k, v in L0["mixer"].items() if k != key})]), seq.F32, 64, 1)
    assert "Nubipel" in models.REGISTRY


def test_checkpoint_round_trip(tmp_path):
    from turboinfer_b200.safetensors_io import read_safetensors, write_safetensors
    cfg = make_config([latent(mlp=dense(8)), attn(), delta()])
    W = random_weights(cfg, seed=4)
    path = str(tmp_path / "model.safetensors")
    write_safetensors(path, W)
    back = read_safetensors(path)
    assert set(back) == set(W)
    for k, v in W.items():
        assert np.array_equal(back[k].to_f32(), np.asarray(v, np.float32)), k
