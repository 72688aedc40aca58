"""CPU-side checks around the Sebudra model: the plain implementation's own invariants (each mechanism against a second, direct
formula), the configuration reader and the checkpoint reader.  No GPU, no engine library."""
import math

import numpy as np
import pytest

import sebudra_plain as plain
from sebudra_cases import again, attn, dense, gla, make_config, moe, par, public_config, random_weights, rel_err, ssm


def toks(n, vocab, seed=0):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def f64(W):
    return {k: np.asarray(v, np.float64) for k, v in W.items()}


def test_prefix_property():
    layers = [par(window=5, mlp=dense(16)), attn(mlp=moe()), gla(mlp=dense(8))]
    cfg = make_config(layers + [again(layers, 0)])
    W = random_weights(cfg, seed=1)
    t = toks(30, cfg["vocab"])
    assert rel_err(plain.run(cfg, W, t)[0][:17], plain.run(cfg, W, t[:17])[0]) < 1e-12


def test_rotation_pairs_the_two_halves_and_depends_on_the_distance_only():
    rot = {"base": 100.0, "dims": 6}
    rng = np.random.default_rng(3)
    v = rng.standard_normal((1, 1, 9))
    r = plain.rotate(v, np.array([5.0]), rot)[0, 0]
    assert np.allclose(r[6:], v[0, 0, 6:])                      # behind rot.dims nothing turns
    for i in range(3):
        a = 5 * 100.0 ** (-2.0 * i / 6)
        x, y = v[0, 0, i], v[0, 0, i + 3]
        assert np.allclose([r[i], r[i + 3]], [x * math.cos(a) - y * math.sin(a), y * math.cos(a) + x * math.sin(a)])
    q, k = rng.standard_normal((1, 1, 9)), rng.standard_normal((1, 1, 9))

    def score(pq, pk):
        return float((plain.rotate(q, np.array([pq]), rot) * plain.rotate(k, np.array([pk]), rot)).sum())
    assert abs(score(40.0, 33.0) - score(7.0, 0.0)) < 1e-12


def test_frequencies_by_turns():
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 4.0, "fast": 16.0, "slow": 2.0, "original": 1024}}
    f, amp = plain.frequencies(rot)
    full = np.array([10000.0 ** (-2.0 * i / 32) for i in range(16)])
    turns = 1024 * full / (2 * math.pi)              # how often pair i turns over the original context
    assert np.allclose(f[turns > 32], full[turns > 32])             # fast pairs stay
    assert np.allclose(f[turns < 1], full[turns < 1] / 4.0)         # slow pairs are stretched
    mid = (turns < 15) & (turns > 3)
    assert mid.any() and (f[mid] < full[mid]).all() and (f[mid] > full[mid] / 4.0).all()
    assert abs(amp - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    assert plain.frequencies({"base": 10.0, "dims": 4})[1] == 1.0
    # the two borders fall together: a ramp of (almost) no width, no division by zero
    g, _ = plain.frequencies({"base": 10000.0, "dims": 4, "scaling": {"factor": 2.0, "fast": 1.0, "slow": 1.0, "original": 6}})
    assert np.isfinite(g).all()


def test_windows_and_weights():
    m = plain.visible(12, 4)
    assert [j for j in range(12) if m[9, j]] == [6, 7, 8, 9]
    assert all(m[i, j] == plain.sees(i, j, 4) for i in range(12) for j in range(12))
    assert [j for j in range(12) if plain.visible(12, 0)[9, j]] == list(range(10))
    s = np.random.default_rng(1).standard_normal((2, 5, 5)) * 3
    w = plain.sigmoid_weights(s, np.array([-1.0, 0.5]), plain.visible(5, 0))
    assert np.allclose(w[1, 3, 2], 1 / (1 + math.exp(-(s[1, 3, 2] + 0.5)))) and w[0, 1, 3] == 0.0
    assert not np.allclose(w.sum(-1), 1.0)           # nothing is normalised
    assert np.allclose(plain.softmax_weights(s, plain.visible(5, 2)).sum(-1), 1.0)


def test_query_norm_comes_before_the_rotation():
    """With uneven gains the two orders differ; the plain one is: divide by the RMS, gain, turn."""
    cfg = make_config([attn(heads=1, kv_heads=1, dim=4, vdim=4, rot_dims=4, softcap=None)], width=8)
    W = f64(random_weights(cfg, seed=3))
    W["l0.mix.o"] = np.eye(8)[:, :4]
    h = np.random.default_rng(3).standard_normal((3, 8))
    mx, eps = cfg["layers"][0]["mixer"], 1e-5
    out = plain.attention(W, "l0.mix.", mx, eps, h, False)
    q, k, v = (h @ W["l0.mix." + n].T for n in "qkv")
    want = np.zeros((3, 4))

    def turned(x, g, pos):
        x = x / math.sqrt((x * x).mean() + eps) * g
        c = [math.cos(pos * mx["rot"]["base"] ** (-i / 2)) for i in range(2)]
        s = [math.sin(pos * mx["rot"]["base"] ** (-i / 2)) for i in range(2)]
        return np.array([x[0] * c[0] - x[2] * s[0], x[1] * c[1] - x[3] * s[1], x[2] * c[0] + x[0] * s[0], x[3] * c[1] + x[1] * s[1]])
    for i in range(3):
        for j in range(i + 1):
            sc = turned(q[i], W["l0.mix.q.norm"], i) @ turned(k[j], W["l0.mix.k.norm"], j) * mx["scale"]
            want[i] += v[j] / (1 + math.exp(-(sc + W["l0.mix.pb"][0])))
    assert np.allclose(out[:, :4], want)


def test_short_conv_is_a_causal_filter():
    rng = np.random.default_rng(2)
    x, w, b = rng.standard_normal((9, 5)), rng.standard_normal((5, 4)), rng.standard_normal(5)
    y = plain.short_conv(x, w, b)
    for c in range(5):
        full = np.convolve(x[:, c], w[c, ::-1])[:9]   # the last column meets the newest input
        assert np.allclose(y[:, c], full + b[c])
    assert np.allclose(plain.short_conv(x, w[:, :1], b), x * w[:, 0] + b)


def test_ssm_scan_equals_the_unrolled_sum():
    rng = np.random.default_rng(4)
    n, H, G, N, dv = 7, 4, 2, 3, 5
    x, B, C = rng.standard_normal((n, H, dv)), rng.standard_normal((n, G, N)), rng.standard_normal((n, G, N))
    dt, A, D = rng.uniform(0.1, 1.0, (n, H)), rng.standard_normal(H), rng.standard_normal(H)
    y = plain.ssm_scan(x, B, C, dt, A, D)
    for h in range(H):
        g = h // 2
        for t in range(n):
            want = D[h] * x[t, h]
            for s in range(t + 1):
                want = want + math.exp(-math.exp(A[h]) * dt[s + 1:t + 1, h].sum()) * dt[s, h] * (C[t, g] @ B[s, g]) * x[s, h]
            assert np.allclose(y[t, h], want)


def test_norm_in_parts():
    y = np.random.default_rng(5).standard_normal((2, 12)) * 4
    out = plain.norm_in_parts(y, np.ones(12), 3, 0.0)
    for part in range(3):
        assert np.allclose((out[:, 4 * part:4 * part + 4] ** 2).mean(-1), 1.0)
    assert np.allclose(plain.norm_in_parts(y, np.full(12, 2.0), 1, 1e-5), plain.norm(y, 2.0, 1e-5))


def test_gla_decay_is_a_root_of_a_sigmoid():
    cfg = make_config([gla(tau=4.0)])
    W = f64(random_weights(cfg, seed=6))
    h = np.random.default_rng(6).standard_normal((2, cfg["width"]))
    a = plain.gla_decay(W, "l0.mix.", 4.0, h)
    z = h @ W["l0.mix.a1"].T @ W["l0.mix.a2"].T + W["l0.mix.a2.b"]
    assert np.allclose(a ** 4, 1 / (1 + np.exp(-z))) and ((a > 0) & (a < 1)).all()


def test_dense_ff_cuts_gate_and_up():
    W = {"gate": np.array([[1.0], [1.0], [-1.0]]), "up": np.array([[1.0], [-1.0], [0.1]]), "down": np.eye(3)}
    out = plain.dense_ff(W, "", 2.0, np.array([[5.0]]))[0]

    def s(z):
        return 1 / (1 + math.exp(-z))
    # gate 5 -> 2 and up 5 -> 2; gate 5 -> 2 and up -5 -> -2; gate -5 stays (only its top is cut), up 0.5 stays
    assert np.allclose(out, [2 * s(3.404) * 3, 2 * s(3.404) * -1, -5 * s(-8.51) * 1.5])


def test_router_groups_corrections_and_weights():
    W = {"router": np.eye(6), "correction": np.zeros(6)}
    z = np.array([2.0, -3.0, 1.0, 0.9, -1.0, 0.0])
    s = 1 / (1 + np.exp(-z))
    r = {"experts": 6, "top": 2, "scale": 2.5, "groups": {"count": 3, "keep": 1}}
    # the best single expert is 0, but its group's two largest add up to less than those of experts 2 and 3
    assert s[0] + s[1] < s[2] + s[3]
    got = dict(plain.route(W, "", r, z))
    assert set(got) == {2, 3} and np.allclose(got[2], 2.5 * s[2] / (s[2] + s[3]))
    assert abs(sum(got.values()) - 2.5) < 1e-12
    # corrections move the choice but not the weights; choice scores may be negative and a group that is out stays out
    W["correction"] = np.array([-3.0, -3.0, -4.0, -4.0, -5.0, -5.0])
    got = dict(plain.route(W, "", r, z))
    assert set(got) == {0, 1} and np.allclose(got[0], 2.5 * s[0] / (s[0] + s[1]))
    # groups of one expert: a group is worth that expert
    one = {"experts": 6, "top": 2, "groups": {"count": 6, "keep": 3}}
    W["correction"] = np.zeros(6)
    assert set(dict(plain.route(W, "", one, z))) == {0, 2}
    assert set(dict(plain.route(W, "", {"experts": 6, "top": 3}, z))) == {0, 2, 3}


def test_shared_tensors_and_chains():
    layers = [par(), gla()]
    layers += [again(layers, 0)]
    layers += [dict(layers[2], weights_of=2)]
    cfg = make_config(layers)
    assert [plain.owner(cfg, i) for i in range(4)] == [0, 1, 0, 0]
    W = random_weights(cfg, seed=2)
    assert not any(k.startswith(("l2.", "l3.")) for k in W)
    assert plain.run(cfg, W, toks(5, 131))[1].shape[0] == 4


def test_config_reader_takes_every_constant_from_the_configuration():
    from turboinfer_b200 import models, seq
    layers = [par(heads=6, kv_heads=3, dim=10, vdim=14, rot_dims=6, base=777.0, scale=0.21, window=17, left_scale=0.3, right_scale=-1.7,
                  scaling={"factor": 3.0, "fast": 9.0, "slow": 0.5, "original": 300}, right=ssm(heads=6, vdim=10, state=7, groups=3, conv=5, parts=4),
                  mlp=dense(72, limit=3.25)),
              attn(heads=5, kv_heads=1, dim=8, vdim=9, rot_dims=4, base=55.0, softcap=12.5, scale=0.4, mlp=moe(ff=11, experts=12, top=5, groups=(4, 3), scale=0.9, shared=33)),
              gla(heads=2, dim=6, vdim=5, tau=3.0, rank=9, mlp=moe(groups=None, shared=0))]
    layers.append(again(layers, 2))
    layers.append(dict(layers[3], weights_of=3))
    cfg = public_config(make_config(layers, vocab=77, width=36, eps=3e-4, scale=0.25))
    m, L = models.sebudra_descs(cfg, seq.F32, 640, 3, {"l2.mix.a1": (9, 36)})
    assert (m.vocab, m.width, m.n_layers, m.max_tokens, m.max_seqs, m.mode) == (77, 36, 5, 640, 3, seq.F32)
    assert abs(m.norm_eps - 3e-4) < 1e-9 and m.norm_kind == seq.NORM_VECTOR and m.norm_place == seq.NORMS_SHARED
    assert abs(m.embed_scale - 0.25) < 1e-9 and m.streams == 0 and m.tied_head == 0
    a = L[0]
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.window) == (seq.MIXER_ATTENTION, 6, 3, 10, 14, 17)
    assert (a.rot_dims, a.rot_half, a.rot_scaled, a.proj_bias, a.qk_norm, a.weights_kind) == (6, 1, seq.ROT_BY_TURNS, seq.BIAS_QKV, seq.QK_NORM_HEAD_GAIN, seq.WEIGHTS_SOFTMAX)
    assert abs(a.scale - 0.21) < 1e-7 and abs(a.rot_base - 777.0) < 1e-3 and abs(a.rot_amp - (0.1 * math.log(3.0) + 1.0)) < 1e-6
    assert (a.rot_factor, a.rot_high, a.rot_low, a.rot_original) == (3.0, 9.0, 0.5, 300.0)
    assert (a.ssm_heads, a.ssm_vdim, a.ssm_state, a.ssm_groups, a.ssm_taps, a.ssm_parts) == (6, 10, 7, 3, 5, 4)
    assert abs(a.left_scale - 0.3) < 1e-7 and abs(a.right_scale + 1.7) < 1e-6
    assert (a.ff_kind, a.ff, a.ff_act, a.ff_limit, a.weights_of) == (seq.FF_GLU, 72, seq.ACT_CLAMPED_SWISH, 3.25, 0)
    b = L[1]
    assert (b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.window) == (seq.MIXER_ATTENTION, 5, 1, 8, 9, 0)
    assert (b.weights_kind, b.softcap, b.rot_scaled, b.rot_amp, b.proj_bias, b.ssm_heads) == (seq.WEIGHTS_SIGMOID, 12.5, 0, 0.0, seq.BIAS_NONE, 0)
    assert (b.ff_kind, b.ff, b.experts, b.top, b.groups, b.groups_keep, b.shared_ff) == (seq.FF_EXPERTS, 11, 12, 5, 4, 3, 33)
    assert (b.expert_form, b.route_kind) == (seq.EXPERT_RELU2, seq.ROUTE_SIGMOID) and abs(b.route_scale - 0.9) < 1e-7
    c = L[2]
    assert (c.mixer, c.heads, c.dim, c.vdim, c.decay_tau, c.decay_rank, c.groups, c.groups_keep, c.shared_ff) == (seq.MIXER_GLA, 2, 6, 5, 3.0, 9, 1, 1, 0)
    assert [x.weights_of for x in L] == [0, 0, 0, 3, 3] and L[4].decay_rank == 9
    with pytest.raises(ValueError):
        models.sebudra_descs(make_config([dict(attn(), type="wkv")]), seq.F32, 64, 1)
    with pytest.raises(ValueError):
        models.sebudra_descs(make_config([attn(mlp={"kind": "sparse", "ff": 8})]), seq.F32, 64, 1)
    with pytest.raises(ValueError):   # no layer with tensors of its own at the end of the chain
        models.sebudra_descs(make_config([dict(attn(), weights_of=1), dict(attn(), weights_of=0)]), seq.F32, 64, 1)
    with pytest.raises(ValueError):
        models.sebudra_descs(make_config([attn(window=None, mlp=None), dict(attn(), weights_of=7)]), seq.F32, 64, 1)
    for gone in ("embedding", "norm", "layers"):
        with pytest.raises(ValueError):
            models.sebudra_descs({k: v for k, v in cfg.items() if k != gone}, seq.F32, 64, 1, {"l2.mix.a1": (9, 36)})
    assert "Sebudra" in models.REGISTRY


def test_checkpoint_round_trip(tmp_path):
    from turboinfer_b200.safetensors_io import read_safetensors, write_safetensors
    cfg = make_config([par(mlp=dense(8)), attn(mlp=moe())])
    W = random_weights(cfg, seed=4)
    path = str(tmp_path / "model.safetensors")
    write_safetensors(path, W)
    back = read_safetensors(path)
    assert set(back) == set(W)
    for k, v in W.items():
        assert np.array_equal(back[k].to_f32(), np.asarray(v, np.float32)), k
