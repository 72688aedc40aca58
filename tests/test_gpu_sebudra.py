"""The layered sequence engine on Sebudra models against the plain implementation (tests/sebudra_plain.py): every mechanism alone,
prompts against token-by-token decoding, portions, ragged batches, reuse of pages and state slots, one key that stands out far back, at
page borders and at the window's edges, states across every cut, the router's choice, shared tensors, the first tokens, long decoding,
odd sizes, and greedy generation through the engine's own generation loop and command line."""
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import sebudra_plain as plain
from sebudra_cases import (again, attn, build_engine, dense, fixed_choice, gla, make_config, moe, par, plant_pair, public_config, random_weights, rel_err, row_errs,
                           run_schedule, ssm, to_bf16_values)

pytestmark = pytest.mark.gpu

# bf16 mode: products round their inputs to bf16 (relative 4e-3 each; a row whose state-space output is close to zero in front of its norm
# carries ten times as much, so most rows are held to a tighter bound than the worst one); fp32 mode is fp32 arithmetic against float64
TOL = {"float32": 2e-4, "bfloat16": 0.15}
MOST = {"float32": 2e-4, "bfloat16": 0.025}


def tokens(n, vocab, seed=1):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def whole(m, toks):
    return run_schedule(m, {"a": toks}, [[("a", len(toks))]])["a"]


def check_logits(got, want, dtype):
    e = row_errs(got, want)
    assert e.max() < TOL[dtype] and np.quantile(e, 0.9) < MOST[dtype]


# ---- each mechanism alone: the residual stream after every layer, and the logits ------------------------------------------------
def _shared(layers, *again_of):
    return layers + [again(layers, j) for j in again_of]


MECHANISMS = {
    "parallel_only": make_config([par()]),
    "attention_only": make_config([attn()]),
    "gla_only": make_config([gla()]),
    "parallel_with_ff": make_config([par(mlp=dense(24))]),
    "attention_with_ff": make_config([attn(mlp=dense(56, limit=0.5))]),
    "gla_with_ff": make_config([gla(mlp=dense(33))]),
    "parallel_with_experts": make_config([par(mlp=moe())]),
    "attention_with_experts": make_config([attn(mlp=moe(experts=8, top=3, groups=(4, 2)))]),
    "gla_with_experts": make_config([gla(mlp=moe(groups=None))]),
    "no_shared_expert": make_config([attn(mlp=moe(shared=0))]),
    "one_expert_group_kept": make_config([gla(mlp=moe(experts=8, top=2, groups=(2, 1), scale=0.5))]),
    "groups_of_one_expert": make_config([attn(mlp=moe(experts=5, top=2, groups=(5, 3)))]),
    "every_allowed_expert_is_used": make_config([attn(mlp=moe(experts=6, top=4, groups=(3, 2)))]),
    "one_expert": make_config([gla(mlp=moe(experts=1, top=1, groups=(1, 1), scale=3.0))]),
    "many_experts_many_picks": make_config([attn(mlp=moe(ff=5, experts=40, top=11, groups=(8, 5), shared=7))]),
    "large_limit": make_config([gla(mlp=dense(24, limit=50.0))]),
    "small_limit_odd_ff": make_config([par(mlp=dense(13, limit=0.2))]),
    "odd_width": make_config([par(heads=3, kv_heads=3, dim=10, vdim=7, rot_dims=6, right=ssm(heads=3, vdim=5, state=7, groups=1, conv=2, parts=3), mlp=dense(11)),
                              attn(heads=3, kv_heads=1, dim=6, vdim=5, rot_dims=4, mlp=moe(ff=7, shared=9)), gla(heads=1, dim=5, vdim=9, rank=3)], width=37, eps=1e-3),
    "every_coordinate_turns": make_config([attn(dim=16, rot_dims=16), par(dim=16, rot_dims=16)]),
    "two_coordinates_turn": make_config([attn(dim=16, rot_dims=2, base=50.0), par(dim=16, rot_dims=2)]),
    "left_without_frequency_scaling": make_config([par(scaling=None)]),
    "sigmoid_attention_with_frequency_scaling": make_config([attn(rot_dims=12, scaling={"factor": 3.0, "fast": 8.0, "slow": 1.0, "original": 128})]),
    "ramp_of_no_width": make_config([par(rot_dims=4, base=10000.0, scaling={"factor": 2.0, "fast": 1.0, "slow": 1.0, "original": 6})]),
    "small_cap": make_config([attn(softcap=0.7, scale=1.5)]),
    "no_cap": make_config([attn(softcap=None)]),
    "capped_left": make_config([par(softcap=0.8, scale=1.5)]),
    "windowed_sigmoid_attention": make_config([attn(window=9)]),
    "one_head": make_config([attn(heads=1, kv_heads=1), par(heads=1, kv_heads=1, right=ssm(heads=1, vdim=6, state=4, groups=1, conv=4, parts=1)), gla(heads=1)]),
    "one_key_value_head": make_config([attn(heads=5, kv_heads=1), par(heads=6, kv_heads=1)]),
    "as_many_key_value_heads": make_config([attn(heads=3, kv_heads=3), par(heads=3, kv_heads=3)]),
    "window_one": make_config([par(window=1)]),
    "window_two": make_config([par(window=2)]),
    "window_beyond_the_sequence": make_config([par(window=700)]),
    "left_without_window": make_config([par(window=None)]),
    "sides_scaled_apart": make_config([par(left_scale=-2.0, right_scale=0.25)]),
    "wide_heads": make_config([attn(heads=2, kv_heads=1, dim=72, vdim=136, rot_dims=40), par(heads=2, kv_heads=2, dim=136, vdim=24, rot_dims=20)], width=64),
    "heads_40_and_100_on_tensor_cores": make_config([attn(heads=4, kv_heads=2, dim=40, vdim=100, rot_dims=24), par(heads=2, kv_heads=1, dim=100, vdim=40, rot_dims=64)], width=64),
    "heads_64_and_128_on_tensor_cores": make_config([attn(heads=4, kv_heads=2, dim=64, vdim=64, rot_dims=64, mlp=dense(96)), par(heads=2, kv_heads=1, dim=128, vdim=128, rot_dims=32),
                                                     attn(heads=2, kv_heads=2, dim=64, vdim=128, rot_dims=32)], width=128),
    "one_tap": make_config([par(right=ssm(conv=1))]),
    "nine_taps": make_config([par(right=ssm(conv=9))]),
    "one_group_many_heads": make_config([par(right=ssm(heads=6, vdim=4, state=20, groups=1, parts=1))]),
    "a_group_per_head": make_config([par(right=ssm(heads=4, vdim=8, state=9, groups=4, parts=4))]),
    "norm_parts_across_heads": make_config([par(right=ssm(heads=3, vdim=8, state=6, groups=3, parts=2))]),
    "state_of_one": make_config([par(right=ssm(heads=2, vdim=3, state=1, groups=1, parts=1))]),
    "state_40": make_config([par(right=ssm(heads=2, vdim=40, state=40, groups=2))]),
    "state_64_columns_64": make_config([par(right=ssm(heads=2, vdim=64, state=64, groups=1))]),
    "state_128_columns_33": make_config([par(right=ssm(heads=2, vdim=33, state=128, groups=2, parts=1))]),
    "state_200": make_config([par(right=ssm(heads=2, vdim=8, state=200, groups=1))]),
    "state_300": make_config([par(right=ssm(heads=2, vdim=8, state=300, groups=2))]),
    "gla_channels_32_64": make_config([gla(heads=2, dim=32, vdim=64), gla(heads=2, dim=64, vdim=32)], width=64),
    "gla_channels_48_136": make_config([gla(heads=2, dim=48, vdim=40), gla(heads=1, dim=136, vdim=150, rank=17)], width=64),
    "gla_slow_and_fast_decay": make_config([gla(tau=1.0), gla(tau=40.0)]),
    "embedding_scale_one": make_config([attn(mlp=dense(16))], scale=1.0),
    "shared_tensors": make_config(_shared([par(mlp=dense(24)), attn(mlp=moe()), gla(mlp=dense(16))], 0, 2, 1, 0)),
    "layers_that_differ": make_config([gla(mlp=moe()), par(mlp=dense(40)), attn(heads=6, kv_heads=3, dim=8, vdim=8, rot_dims=8, mlp=dense(24, limit=3.0)),
                                       par(heads=2, dim=16, vdim=8, window=7, right=ssm(heads=8, vdim=4, state=16, groups=4, conv=4, parts=4), mlp=moe(experts=9, top=4, groups=(3, 2))),
                                       gla(heads=4, dim=16, vdim=8, tau=2.0)], vocab=101, width=56, scale=4.0),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_layers_and_logits(name, dtype):
    cfg = MECHANISMS[name]
    W = random_weights(cfg, seed=3)
    if dtype == "bfloat16":
        W = fixed_choice(cfg, W)
    toks = tokens(75, cfg["vocab"])
    want, layers = plain.run(cfg, W, toks)
    m = build_engine(cfg, W, dtype)
    m.debug_layers(True)
    got = whole(m, toks)
    got_layers = m.read_layers(len(toks))
    few = run_schedule(m, {"a": toks}, [[("a", 70)]] + [[("a", 1)]] * 5)["a"]   # decode rows of the same model
    m.free()
    assert got_layers.shape == layers.shape
    for i in range(layers.shape[0]):
        scale = np.sqrt((layers[i] ** 2).mean())
        assert np.abs(got_layers[i] - layers[i]).max() / scale < (1e-3 if dtype == "float32" else 0.3), f"layer run {i}"
    check_logits(got, want, dtype)
    check_logits(few, want, dtype)


# ---- prompts against decoding, portions, batches ---------------------------------------------------------------------------------
HYBRID = make_config(_shared([par(window=70, mlp=dense(40)), attn(mlp=moe()), gla(mlp=dense(24)),
                              par(heads=2, window=9, right=ssm(heads=2, vdim=16, state=20, groups=1, conv=5, parts=1), mlp=moe(experts=4, top=2, groups=None))], 0, 2))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_equals_token_by_token(dtype):
    W = random_weights(HYBRID, seed=5)
    if dtype == "bfloat16":
        W = fixed_choice(HYBRID, W)
    toks = tokens(150, HYBRID["vocab"], 2)
    want, _ = plain.run(HYBRID, W, toks)
    m = build_engine(HYBRID, W, dtype)
    a = whole(m, toks)
    b = run_schedule(m, {"a": toks}, [[("a", 1)] for _ in toks])["a"]
    m.free()
    check_logits(a, want, dtype)
    check_logits(b, want, dtype)
    check_logits(b, a, dtype)


@pytest.mark.parametrize("sizes", [[2] * 40, [3, 61, 2, 64, 5, 65, 1, 63, 2], [64, 64, 64], [1, 127, 2, 2, 100], [129, 2, 33], [7, 1, 1, 8, 9, 1, 2, 31], [200, 17, 130]])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions(sizes, dtype):
    """Portions down to two tokens and single tokens in between: the convolution's and both recurrences' states, the caches and the
    window all cross the cuts (portions of fewer than 8 rows take the row kernels, longer ones the tile kernels)."""
    toks = tokens(sum(sizes), HYBRID["vocab"], 7)
    W = random_weights(HYBRID, seed=6)
    if dtype == "bfloat16":
        W = fixed_choice(HYBRID, W)
    want, _ = plain.run(HYBRID, W, toks)
    m = build_engine(HYBRID, W, dtype)
    got = run_schedule(m, {"a": toks}, [[("a", n)] for n in sizes])["a"]
    m.free()
    check_logits(got, want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_ragged_batch_equals_each_alone(dtype):
    cfg = HYBRID
    W = random_weights(cfg, seed=8)
    if dtype == "bfloat16":
        W = fixed_choice(cfg, W)
    reqs = {"a": tokens(90, cfg["vocab"], 11), "b": tokens(17, cfg["vocab"], 12), "c": tokens(130, cfg["vocab"], 13), "d": tokens(1, cfg["vocab"], 14)}
    m = build_engine(cfg, W, dtype, max_tokens=448)
    alone = {k: whole(m, v) for k, v in reqs.items()}
    sched = [[("a", 30), ("b", 2)], [("a", 1), ("b", 9), ("c", 64)], [("c", 2), ("a", 1), ("d", 1)], [("b", 6), ("a", 58), ("c", 64)]]
    got = run_schedule(m, reqs, sched)
    m.free()
    for k, v in reqs.items():
        check_logits(got[k], alone[k], dtype)
        check_logits(got[k], plain.run(cfg, W, v)[0], dtype)


def test_pages_and_slots_are_reused():
    """Two slots and three pages for five requests: later requests run in the slots and pages earlier ones gave back, and a stale
    convolution state, recurrent state or cache row would show in their logits (long memories, large convolution weights)."""
    cfg = HYBRID
    W = random_weights(cfg, seed=9, memory=2.0)
    m = build_engine(cfg, W, "float32", max_tokens=192, max_seqs=2)
    seen_pages, seen_slots = [], []
    for i, n in enumerate([100, 70, 128, 5, 64]):
        toks = tokens(n, cfg["vocab"], 20 + i)
        s = m.open()
        other = m.open()   # a second live sequence holds the other slot and a page while this one runs
        m.step([(other, tokens(3, cfg["vocab"], 40 + i))], [[]])
        got = np.concatenate([m.step([(s, toks[:n // 2])], [list(range(n // 2))]), m.step([(s, toks[n // 2:])], [list(range(n - n // 2))])])
        seen_pages.append(tuple(m.pages(s)))
        seen_slots.append(s)
        assert rel_err(got, plain.run(cfg, W, toks)[0]) < TOL["float32"], i
        m.close(s)
        m.close(other)
    assert m.pool_info()["free_pages"] == 3 and m.pool_info()["free_slots"] == 2
    m.free()
    assert len(set(seen_slots)) <= 2
    assert len(set(p for ps in seen_pages for p in ps)) <= 3 and len(seen_pages) == 5


# ---- a key that stands out: far back, at page borders, at position 0, at the window's edges ----------------------------------------
@functools.lru_cache(maxsize=None)
def planted_case(kind, window, place, n):
    """Token A sits at `place` among n - 1 other tokens, token B is last; head 0 of layer 0 gives B's query a large score against
    A's key (and, without a softmax, next to nothing against any other).  Returns the model, the tokens, the true logits and how far
    the last row moves when the mask is off by that one key."""
    if kind == "sigmoid":
        cfg = make_config([attn(heads=4, kv_heads=2, dim=16, vdim=16, rot_dims=8, scale=0.5, softcap=20.0, window=window or None), gla()], width=64)
    else:
        cfg = make_config([par(heads=4, kv_heads=2, dim=16, vdim=16, rot_dims=8, scale=0.5, window=window or None), gla()], width=64)
    A, B = 7, 11
    W = plant_pair(cfg, random_weights(cfg, seed=13), A, B)
    rng = np.random.default_rng(place * 7 + n)
    fill = [t for t in range(cfg["vocab"]) if t not in (A, B)]
    toks = [fill[int(i)] for i in rng.integers(0, len(fill), n)]
    toks[place], toks[-1] = A, B
    true = plain.visible(n, window)
    shown, hidden = true.copy(), true.copy()
    shown[-1, place], hidden[-1, place] = True, False
    a, b = plain.run(cfg, W, toks, {0: shown})[0], plain.run(cfg, W, toks, {0: hidden})[0]
    want = a if true[-1, place] else b
    return cfg, W, toks, want, row_errs(b[-1:], a[-1:])[0]


def standing_out(kind, window, place, n, decode, dtype="float32", tol=None):
    """Whether B sees A decides its logits (the plain implementation with a mask that is off by that one key differs by far more
    than the tolerance), so an engine whose window or page walk is one key off, or that loses a far key, cannot pass."""
    cfg, W, toks, want, moved = planted_case(kind, window, place, n)
    tol = tol or TOL[dtype]
    assert moved > 3 * tol and moved > 0.1, "the planted key does not decide the last logits"
    m = build_engine(cfg, W, dtype)
    if decode:
        got = run_schedule(m, {"a": toks}, [[("a", n - 4)]] + [[("a", 1)]] * 4)["a"]
    else:
        got = whole(m, toks)
    m.free()
    assert rel_err(got, want) < tol


EDGES = [  # (attention of layer 0, window, place of the key, tokens)
    ("sigmoid", 0, 0, 400),          # position 0, hundreds of keys back
    ("sigmoid", 0, 63, 330),         # the end of the first page
    ("sigmoid", 0, 64, 330),         # the start of the second
    ("sigmoid", 0, 17, 600),         # far back among hundreds
    ("sigmoid", 0, 198, 200),        # the key right before the row
    ("sigmoid", 33, 99 - 32, 100),   # a window on the unnormalised weights: inside ...
    ("sigmoid", 33, 99 - 33, 100),   # ... and outside
    ("left", 20, 99 - 19, 100),      # the last key inside the window
    ("left", 20, 99 - 20, 100),      # the first key outside it
    ("left", 64, 199 - 63, 200),     # a window of exactly one page: inside ...
    ("left", 64, 199 - 64, 200),     # ... and outside
    ("left", 65, 192 - 64, 193),     # the window's edge on a page border, the row the first of its page
    ("left", 65, 192 - 65, 193),
    ("left", 300, 329 - 299, 330),   # the far edge of a long window among hundreds of keys
    ("left", 300, 329 - 300, 330),
    ("left", 300, 63, 330),          # inside a long window, at a page's end
    ("left", 500, 0, 330),           # a window beyond the sequence: position 0
    ("left", 1, 98, 100),            # a window of one: the key right before the row is already outside
    ("left", 0, 5, 500),             # no window
]


@pytest.mark.parametrize("kind,window,place,n", EDGES)
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_stands_out(kind, window, place, n, decode):
    standing_out(kind, window, place, n, decode)


@pytest.mark.parametrize("kind,window,place,n", [e for e in EDGES if e[1:] in ((0, 64, 330), (0, 17, 600), (33, 67, 100), (33, 66, 100), (20, 80, 100), (20, 79, 100), (65, 128, 193), (65, 127, 193))])
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_stands_out_bf16(kind, window, place, n, decode):
    standing_out(kind, window, place, n, decode, dtype="bfloat16", tol=0.05)


def test_sigmoid_weights_are_not_normalised():
    """Hundreds of keys with weights around one half: the attention's output grows with the number of keys, and the per-head number
    decides its size -- a softmax, a missing number or a mean over the keys differs by far."""
    cfg = make_config([attn(heads=3, kv_heads=3, softcap=1.0)])
    W = random_weights(cfg, seed=14, out_amp=0.05)
    W["l0.mix.pb"] = to_bf16_values(np.array([0.5, -0.5, -4.0], np.float32))
    toks = tokens(260, cfg["vocab"], 3)
    want, layers = plain.run(cfg, W, toks)
    W0 = dict(W)
    W0["l0.mix.pb"] = np.zeros(3, np.float32)
    assert row_errs(plain.run(cfg, W0, toks)[0], want).max() > 50 * TOL["float32"]
    Ws = {k: v for k, v in W.items() if not k.endswith(".pb")}
    assert row_errs(plain.run(cfg, Ws, toks)[0], want).max() > 50 * TOL["float32"]   # (a softmax)
    m = build_engine(cfg, W, "float32")
    a = whole(m, toks)
    b = run_schedule(m, {"a": toks}, [[("a", 200)]] + [[("a", 1)]] * 60)["a"]
    m.free()
    check_logits(a, want, "float32")
    check_logits(b, want, "float32")


def test_states_cross_every_cut():
    """Long memories and large convolution weights: a row depends on rows in the same portion, the portion before, two portions back and
    before the sequence's start; a layer that runs twice on the same tensors has states of its own."""
    layers = [par(window=3, right=ssm(conv=5, heads=2, vdim=8, state=10, groups=1)), gla()]
    cfg = make_config(_shared(layers, 0, 1))
    W = random_weights(cfg, seed=16, memory=3.0)
    W["l0.mix.right.conv"] = to_bf16_values(np.random.default_rng(1).standard_normal(W["l0.mix.right.conv"].shape).astype(np.float32))
    toks = tokens(40, cfg["vocab"], 8)
    want, _ = plain.run(cfg, W, toks)
    W0 = dict(W)
    W0["l0.mix.right.conv"] = np.array(W["l0.mix.right.conv"], copy=True)
    W0["l0.mix.right.conv"][:, 0] = 0
    assert row_errs(plain.run(cfg, W0, toks)[0][4:], want[4:]).min() > 20 * TOL["float32"]
    # the first token still shows in the last logits
    assert row_errs(plain.run(cfg, W, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])[0][-1:], want[-1:]).max() > 20 * TOL["float32"]
    m = build_engine(cfg, W, "float32")
    for sizes in ([1] * 40, [2, 1, 1, 3, 1, 2, 2, 9, 1, 1, 1, 1, 1, 14], [40], [3, 37]):
        got = run_schedule(m, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert rel_err(got, want) < TOL["float32"], sizes
    m.free()


def test_a_layer_on_shared_tensors_has_its_own_cache_and_states():
    cfg = make_config(_shared([par(mlp=dense(16)), attn(), gla()], 0, 1, 2))
    W = random_weights(cfg, seed=23)
    toks = tokens(60, cfg["vocab"], 9)
    want, layers = plain.run(cfg, W, toks)
    assert layers.shape[0] == 6
    m = build_engine(cfg, W, "float32")
    by = m.bytes()
    got = run_schedule(m, {"a": toks}, [[("a", 30)]] + [[("a", 1)]] * 30)["a"]
    m.free()
    check_logits(got, want, "float32")
    one = build_engine(make_config(cfg["layers"][:3]), W, "float32")
    assert by["kv_per_token"] == 2 * one.bytes()["kv_per_token"] and by["state_per_seq"] == 2 * one.bytes()["state_per_seq"]
    one.free()


def test_biases_gains_and_mixing_scales_matter_and_match():
    """Dropping a bias, a gain, the D term, the convolution's bias or swapping the two sides' scales moves the logits by far."""
    cfg = make_config([par(left_scale=1.5, right_scale=0.5), attn()])
    W = random_weights(cfg, seed=21)
    rng = np.random.default_rng(2)
    for nm in ("q.b", "k.b", "v.b"):
        W["l0.mix.left." + nm] = to_bf16_values(rng.standard_normal(W["l0.mix.left." + nm].shape).astype(np.float32) * 2.0)
    toks = tokens(50, cfg["vocab"], 4)
    want, _ = plain.run(cfg, W, toks)
    for nm in ("l0.mix.left.q.b", "l0.mix.left.k.b", "l0.mix.left.v.b", "l0.mix.left.q.norm", "l1.mix.k.norm", "l0.mix.right.D", "l0.mix.right.conv.b", "l0.mix.right.dt_bias",
               "l0.mix.right.A_log", "l0.mix.right.norm"):
        W0 = dict(W)
        W0[nm] = np.ones_like(W[nm]) if nm.endswith("norm") else np.zeros_like(W[nm])
        assert row_errs(plain.run(cfg, W0, toks)[0], want).max() > 50 * TOL["float32"], nm
    swapped = make_config([par(left_scale=0.5, right_scale=1.5), attn()])
    assert row_errs(plain.run(swapped, W, toks)[0], want).max() > 50 * TOL["float32"]
    m = build_engine(cfg, W, "float32")
    a = whole(m, toks)
    b = run_schedule(m, {"a": toks}, [[("a", 20)]] + [[("a", 1)]] * 30)["a"]
    m.free()
    assert rel_err(a, want) < TOL["float32"] and rel_err(b, want) < TOL["float32"]


def test_router_choice_weights_and_scale():
    """Corrections that bring groups with negative choice scores to the top, and a router scale: choosing without the groups, by the best
    single expert of a group, with the correction in the weights or without the scale differs by far."""
    cfg = make_config([gla(mlp=moe(ff=16, experts=9, top=3, groups=(3, 1), scale=2.25))])
    W = random_weights(cfg, seed=24)
    W["l0.mlp.correction"] = to_bf16_values(np.array([-0.9, -3.0, -3.0, -1.2, -1.25, -1.3, -1.5, -1.1, -2.5], np.float32))
    toks = tokens(80, cfg["vocab"], 6)
    want, _ = plain.run(cfg, W, toks)
    for change in ({"groups": None}, {"scale": 1.0}, {"groups": {"count": 3, "keep": 2}}, {"top": 2}):
        other = make_config([gla(mlp=dict(cfg["layers"][0]["mlp"], router=dict(cfg["layers"][0]["mlp"]["router"], **change)))])
        assert row_errs(plain.run(other, W, toks)[0], want).max() > 50 * TOL["float32"], change
    m = build_engine(cfg, W, "float32")
    a = whole(m, toks)
    b = run_schedule(m, {"a": toks}, [[("a", 20)]] + [[("a", 1)]] * 60)["a"]
    m.free()
    check_logits(a, want, "float32")
    check_logits(b, want, "float32")


def test_limits_cut_both_branches():
    cfg = make_config([attn(mlp=dense(32, limit=0.6))])
    W = random_weights(cfg, seed=25)
    toks = tokens(40, cfg["vocab"], 4)
    want, _ = plain.run(cfg, W, toks)
    wide = make_config([attn(mlp=dense(32, limit=60.0))])
    assert row_errs(plain.run(wide, W, toks)[0], want).max() > 50 * TOL["float32"]
    for dtype in ("float32", "bfloat16"):
        m = build_engine(cfg, W, dtype)
        check_logits(whole(m, toks), want, dtype)
        check_logits(run_schedule(m, {"a": toks}, [[("a", 1)]] * 40)["a"], want, dtype)
        m.free()


def test_rotation_far_into_a_sequence():
    """Positions in the hundreds, angle = position x frequency in fp32: a scaling factor or a border of the ramp that is off moves the
    late logits by far more than the tolerance, so the engine's frequencies, angles and amplitude are the design's."""
    def config(factor=4.0, fast=20.0, slow=1.5):
        return make_config([par(dim=16, rot_dims=16, window=300, base=500.0, scaling={"factor": factor, "fast": fast, "slow": slow, "original": 256}),
                            attn(dim=16, rot_dims=12, base=10000.0)])
    cfg = config()
    W = random_weights(cfg, seed=4)
    toks = tokens(700, cfg["vocab"], 12)
    want, _ = plain.run(cfg, W, toks)
    for off in (config(factor=4.1), config(fast=12.0), config(slow=3.0)):
        assert row_errs(plain.run(off, W, toks)[0][600:], want[600:]).max() > 10 * TOL["float32"]
    m = build_engine(cfg, W, "float32")
    got = run_schedule(m, {"a": toks}, [[("a", 690)]] + [[("a", 1)]] * 10)["a"]
    m.free()
    check_logits(got, want, "float32")


def test_first_tokens_and_single_token_requests():
    W = random_weights(HYBRID, seed=16)
    m = build_engine(HYBRID, W, "float32")
    for n in (1, 2, 3):
        toks = tokens(n, HYBRID["vocab"], 30 + n)
        assert rel_err(whole(m, toks), plain.run(HYBRID, W, toks)[0]) < TOL["float32"]
        assert rel_err(run_schedule(m, {"a": toks}, [[("a", 1)]] * n)["a"], plain.run(HYBRID, W, toks)[0]) < TOL["float32"]
    m.free()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    """The windows (70 and 9) pass over decoded tokens; 320 single-token steps."""
    cfg = HYBRID
    W = random_weights(cfg, seed=17, out_amp=0.4)
    if dtype == "bfloat16":
        W = fixed_choice(cfg, W)
    toks = tokens(330, cfg["vocab"], 5)
    want, _ = plain.run(cfg, W, toks)
    m = build_engine(cfg, W, dtype)
    got = run_schedule(m, {"a": toks}, [[("a", 10)]] + [[("a", 1)]] * 320)["a"]
    m.free()
    check_logits(got, want, dtype)


@pytest.mark.parametrize("rows", [1, 3, 8])
def test_wide_model_decode_rows_and_tiles(rows):
    """Widths in whole 32-element chunks (bf16 mode: the decode rows' products run on the tensor-core few-row kernel with the gated
    columns behind plain ones and unchosen experts left out, prompt products on tcgen05), attention heads of 64 and 128."""
    cfg = make_config(_shared([par(heads=8, kv_heads=2, dim=64, vdim=64, rot_dims=32, window=50, right=ssm(heads=8, vdim=32, state=64, groups=2, conv=4, parts=2), mlp=dense(264)),
                               attn(heads=4, kv_heads=2, dim=128, vdim=128, rot_dims=128, mlp=moe(ff=96, experts=8, top=2, groups=(2, 1), shared=160)),
                               gla(heads=4, dim=64, vdim=64, rank=16, mlp=moe(ff=64, experts=16, top=3, groups=(4, 2), shared=0))], 0), vocab=203, width=256)
    W = fixed_choice(cfg, random_weights(cfg, seed=31))
    lens = [150, 9, 33, 70, 21, 7, 12, 40][:rows]
    reqs = {"r%d" % i: tokens(n, 203, 60 + i) for i, n in enumerate(lens)}
    m = build_engine(cfg, W, "bfloat16", max_tokens=sum((n + 63) // 64 * 64 for n in lens), max_seqs=rows)
    alone = {k: whole(m, v) for k, v in reqs.items()}
    tail = 6
    got = run_schedule(m, reqs, [[(k, len(v) - tail) for k, v in reqs.items()]] + [[(k, 1) for k in reqs]] * tail)
    m.free()
    for k, v in reqs.items():
        check_logits(got[k], alone[k], "bfloat16")
        check_logits(alone[k], plain.run(cfg, W, v)[0], "bfloat16")


def test_experts_that_rows_choose_apart():
    """Decode rows whose routers choose different experts (the choice follows the token): the few-row path reads the union of the chosen
    experts, and every row must still get its own."""
    cfg = make_config([gla(heads=2, dim=32, vdim=32, mlp=moe(ff=64, experts=16, top=2, groups=(4, 2), shared=32))], vocab=64, width=256)
    W = random_weights(cfg, seed=33)
    W["l0.mlp.correction"] = np.zeros(16, np.float32)
    # token t carries a large coordinate that only expert (5 t) mod 16 and its neighbour's routers read
    E, R = W["embed"], np.zeros((16, 256), np.float32)
    E[:, :16] = 0
    for t in range(64):
        E[t, (5 * t) % 16] = 6.0
    for e in range(16):
        R[e, e], R[e, e ^ 1] = 4.0, 2.0
        R[e, [c for c in range(16) if c // 4 != e // 4]] = -1.0
    W["l0.mlp.router"], W["embed"] = to_bf16_values(R), to_bf16_values(E)
    W["l0.norm1"][:16] = 1.0
    toks = {"r%d" % i: tokens(6, 64, 80 + i) for i in range(7)}
    m = build_engine(cfg, W, "bfloat16", max_seqs=7)
    got = run_schedule(m, toks, [[(k, 1) for k in toks]] * 6)
    m.free()
    for k, v in toks.items():
        check_logits(got[k], plain.run(cfg, W, v)[0], "bfloat16")


# ---- generation through the engine's own loop, and the command line ---------------------------------------------------------------
def plain_greedy(cfg, W, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(np.argmax(plain.run(cfg, W, toks)[0][-1])))
    return toks[len(prompt):]


def test_greedy_generation_continuous_batching():
    """Six requests through two slots and a pool that holds about two of them: admission, portions of prompts beside decoded
    tokens, and slots / pages handed on, all inside the engine's generation loop."""
    W = random_weights(HYBRID, seed=18)
    prompts = [tokens(n, HYBRID["vocab"], 70 + i) for i, n in enumerate([5, 40, 90, 1, 64, 23])]
    want = [plain_greedy(HYBRID, W, p, 10) for p in prompts]
    m = build_engine(HYBRID, W, "float32", max_tokens=256, max_seqs=2)
    got = m.generate(prompts, 10, step_tokens=48)
    m.free()
    assert got == want


def test_command_line_generate_and_trace_replay(tmp_path):
    from turboinfer_b200.safetensors_io import write_safetensors
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = make_config(_shared([par(mlp=dense(24)), attn(heads=2, kv_heads=1, mlp=moe()), gla()], 0), vocab=53)
    W = random_weights(cfg, seed=19)
    folder = os.path.join(tmp_path, "model")
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(public_config(cfg), f)
    write_safetensors(os.path.join(folder, "model.safetensors"), W)
    prompts = [tokens(7, 53, 3), tokens(30, 53, 4)]
    want = [plain_greedy(cfg, W, p, 6) for p in prompts]
    cmd = [sys.executable, os.path.join(root, "bin", "generate"), "--model", folder, "--dtype", "float32", "--max-new", "6"]
    for p in prompts:
        cmd += ["--prompt-ids", ",".join(str(t) for t in p)]
    res = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr
    assert [json.loads(line)["tokens"] for line in res.stdout.splitlines() if line.startswith("{")] == want
    out = os.path.join(tmp_path, "out")
    os.makedirs(out)
    p = prompts[1]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": p[:11], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": p[11:13], "want": []}, {"id": "b", "tokens": prompts[0], "want": [6]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": p[13:], "want": [0, len(p) - 14]}], "end": ["a"]}]
    res = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", out,
                          "--max-tokens", "128"], input="".join(json.dumps(x) + "\n" for x in steps), capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr
    assert [ln for ln in res.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not os.path.exists(os.path.join(out, "0.f32"))
    ref_a, ref_b = plain.run(cfg, W, p)[0], plain.run(cfg, W, prompts[0])[0]
    l1 = np.fromfile(os.path.join(out, "1.f32"), "<f4").reshape(1, 53)
    l2 = np.fromfile(os.path.join(out, "2.f32"), "<f4").reshape(2, 53)
    assert rel_err(l1, ref_b[[6]]) < TOL["float32"]
    assert rel_err(l2, ref_a[[13, len(p) - 1]]) < TOL["float32"]


def test_state_space_mixer_alone_through_the_description():
    """The state-space mixer as a layer's only mixer (tensors under mix.*): what a layer with a zero left side computes."""
    from turboinfer_b200 import models, seq
    cfg = make_config([par(left_scale=0.0, right_scale=1.0, mlp=dense(16))])
    W = random_weights(cfg, seed=27)
    toks = tokens(70, cfg["vocab"], 5)
    want, _ = plain.run(cfg, W, toks)
    desc, layers = models.sebudra_descs(cfg, seq.F32, 1024, 2)
    layers[0].mixer = seq.MIXER_SSM
    m = seq.SeqModel(desc, layers).load({k.replace("mix.right.", "mix."): v for k, v in W.items() if ".left." not in k})
    check_logits(whole(m, toks), want, "float32")
    check_logits(run_schedule(m, {"a": toks}, [[("a", 1)]] * 70)["a"], want, "float32")
    m.free()


def test_errors_are_reported():
    cfg = make_config([par(mlp=dense(16)), attn(mlp=moe()), gla()])
    W = random_weights(cfg, seed=20)
    bad = dict(W)
    bad["l0.mix.right.conv"] = W["l0.mix.right.conv"][:-1]
    with pytest.raises(Exception):
        build_engine(cfg, bad)
    for gone in ("l0.mix.left.q.b", "l0.mix.right.dt_bias", "l1.mix.pb", "l1.mlp.correction", "l1.mlp.shared.sg", "l2.mix.a2.b", "l0.norm1"):
        with pytest.raises(Exception):
            build_engine(cfg, {k: v for k, v in W.items() if k != gone})
    for layer in (attn(heads=3, kv_heads=2), par(right=ssm(heads=3, groups=2)), par(right=ssm(parts=7)), par(right=ssm(state=2000)), attn(mlp=moe(experts=7, groups=(3, 1))),
                  attn(mlp=moe(top=9)), gla(mlp=dense(16, limit=0.0))):
        with pytest.raises(Exception):
            c = make_config([layer])
            try:
                w = random_weights(c)
            except Exception:
                w = W
            build_engine(c, w)
