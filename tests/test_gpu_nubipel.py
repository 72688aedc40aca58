"""The layered sequence engine on Nubipel models against the plain implementation (tests/nubipel_plain.py): every mechanism alone,
prompts against token-by-token decoding, portions, ragged batches, reuse of pages and state slots, one key that stands out far back, at
page borders and at both sides of every chunk's edge, states across every cut, the sink, the gates, the first tokens, long decoding, odd
sizes, and greedy generation through the engine's own generation loop and command line."""
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import nubipel_plain as plain
from nubipel_cases import attn, build_engine, delta, dense, latent, make_config, plant_pair, random_weights, rel_err, row_errs, run_schedule, to_bf16_values

pytestmark = pytest.mark.gpu

# bf16 mode: products round their inputs to bf16 (relative 4e-3 each; a row whose delta output is close to zero in front of its norm carries
# more, so most rows are held to a tighter bound than the worst one); fp32 mode is fp32 arithmetic against float64
TOL = {"float32": 1e-4, "bfloat16": 0.15}
MOST = {"float32": 1e-4, "bfloat16": 0.025}


def tokens(n, vocab, seed=1):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def whole(m, toks):
    return run_schedule(m, {"a": toks}, [[("a", len(toks))]])["a"]


def check_logits(got, want, dtype):
    e = row_errs(got, want)
    assert e.max() < TOL[dtype] and np.quantile(e, 0.9) < MOST[dtype]


# ---- each mechanism alone: the residual stream after every layer, and the logits ------------------------------------------------
MECHANISMS = {
    "attention_only": make_config([attn()]),
    "latent_only": make_config([latent()]),
    "delta_only": make_config([delta()]),
    "attention_with_ff": make_config([attn(mlp=dense(24))]),
    "latent_with_ff": make_config([latent(mlp=dense(56))]),
    "delta_with_ff": make_config([delta(mlp=dense(33))]),
    "odd_width_odd_sizes": make_config([attn(heads=3, kv_heads=1, dim=7, vdim=5, chunk=11, mlp=dense(13)), latent(heads=3, dim=5, vdim=7, kv_rank=9, q_rank=11, mlp=dense(11)),
                                        delta(heads=3, kv_heads=3, dim=5, vdim=7, conv=2, mlp=dense(17))], width=37, eps=1e-3),
    "one_head": make_config([attn(heads=1, kv_heads=1), latent(heads=1), delta(heads=1, kv_heads=1)]),
    "one_key_value_head": make_config([attn(heads=5, kv_heads=1), delta(heads=6, kv_heads=1)]),
    "as_many_key_value_heads": make_config([attn(heads=3, kv_heads=3), delta(heads=3, kv_heads=3)]),
    "chunk_of_one": make_config([attn(chunk=1)]),
    "chunk_of_two": make_config([attn(chunk=2)]),
    "chunk_of_a_page": make_config([attn(chunk=64)]),
    "chunk_beyond_the_sequence": make_config([attn(chunk=700)]),
    "no_chunks": make_config([attn(chunk=None)]),
    "large_scale": make_config([attn(scale=2.0), latent(scale=1.5)]),
    "small_eps_large_eps": make_config([attn(), latent(), delta()], eps=0.3),
    "attention_sizes_40_100": make_config([attn(heads=4, kv_heads=2, dim=40, vdim=100, chunk=30), attn(heads=2, kv_heads=1, dim=100, vdim=40, chunk=50)], width=64),
    "attention_sizes_64_128": make_config([attn(heads=4, kv_heads=2, dim=64, vdim=64, chunk=33, mlp=dense(96)), attn(heads=2, kv_heads=1, dim=128, vdim=128, chunk=20),
                                           attn(heads=2, kv_heads=2, dim=64, vdim=128)], width=128),
    "attention_sizes_136_200": make_config([attn(heads=2, kv_heads=1, dim=136, vdim=24, chunk=40), attn(heads=2, kv_heads=2, dim=24, vdim=200)], width=64),
    "latent_rank_128": make_config([latent(heads=2, dim=24, vdim=40, kv_rank=128, q_rank=50)], width=96),
    "latent_rank_100": make_config([latent(heads=4, dim=16, vdim=24, kv_rank=100, q_rank=7)], width=96),
    "latent_rank_256": make_config([latent(heads=2, dim=40, vdim=24, kv_rank=256, q_rank=33)], width=96),
    "latent_rank_180": make_config([latent(heads=2, dim=64, vdim=64, kv_rank=180, q_rank=64)], width=96),
    "latent_rank_512": make_config([latent(heads=2, dim=16, vdim=32, kv_rank=512, q_rank=24)], width=64),
    "latent_rank_300": make_config([latent(heads=3, dim=20, vdim=12, kv_rank=300, q_rank=24)], width=64),
    "latent_rank_600": make_config([latent(heads=2, dim=8, vdim=8, kv_rank=600, q_rank=24)], width=64),
    "latent_rank_128_large_heads": make_config([latent(heads=2, dim=120, vdim=140, kv_rank=128, q_rank=32)], width=64),   # (not worth expanding: on the cached rows themselves)
    "latent_rank_256_large_heads": make_config([latent(heads=2, dim=136, vdim=24, kv_rank=256, q_rank=32)], width=64),
    "latent_rank_512_large_heads": make_config([latent(heads=2, dim=16, vdim=132, kv_rank=512, q_rank=32)], width=64),
    "latent_heads_wider_than_the_rank": make_config([latent(heads=2, dim=128, vdim=128, kv_rank=96, q_rank=32)], width=64),
    "latent_rank_one": make_config([latent(heads=2, dim=3, vdim=2, kv_rank=1, q_rank=1)]),
    "delta_one_tap": make_config([delta(conv=1)]),
    "delta_nine_taps": make_config([delta(conv=9)]),
    "delta_key_one_value_one": make_config([delta(heads=2, kv_heads=1, dim=1, vdim=1)]),
    "delta_32_by_48": make_config([delta(heads=4, kv_heads=2, dim=32, vdim=48, conv=4)], width=64),
    "delta_64_by_17": make_config([delta(heads=4, kv_heads=1, dim=64, vdim=17)], width=64),
    "delta_128_by_64": make_config([delta(heads=2, kv_heads=1, dim=128, vdim=64, conv=4)], width=64),
    "delta_128_by_128": make_config([delta(heads=2, kv_heads=2, dim=128, vdim=128, conv=4)], width=64),
    "delta_96_by_80": make_config([delta(heads=2, kv_heads=2, dim=96, vdim=80)], width=64),
    "delta_200_by_40": make_config([delta(heads=1, kv_heads=1, dim=200, vdim=40)], width=64),
    "delta_500_by_16": make_config([delta(heads=1, kv_heads=1, dim=500, vdim=16)], width=64),
    "delta_66_by_33": make_config([delta(heads=2, kv_heads=1, dim=66, vdim=33)], width=64),
    "embedding_scale_one": make_config([attn(mlp=dense(16))], scale=1.0),
    "logits_neither_scaled_nor_close_to_the_cap": make_config([latent(mlp=dense(16))], logit_scale=1.0, softcap=500.0),
    "layers_that_differ": make_config([delta(mlp=dense(24)), attn(heads=6, kv_heads=3, dim=8, vdim=8, chunk=7), latent(heads=2, dim=16, vdim=8, kv_rank=20, q_rank=40, mlp=dense(40)),
                                       attn(heads=2, kv_heads=1, dim=20, vdim=12, chunk=31, mlp=dense(8)), delta(heads=6, kv_heads=2, dim=16, vdim=8, conv=5),
                                       latent(heads=5, dim=8, vdim=20, kv_rank=44, q_rank=12)], vocab=101, width=56, scale=4.0),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_layers_and_logits(name, dtype):
    cfg = MECHANISMS[name]
    W = random_weights(cfg, seed=3)
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
        assert np.abs(got_layers[i] - layers[i]).max() / scale < (1e-3 if dtype == "float32" else 0.3), f"layer {i}"
    check_logits(got, want, dtype)
    check_logits(few, want, dtype)


# ---- prompts against decoding, portions, batches ---------------------------------------------------------------------------------
HYBRID = make_config([latent(mlp=dense(40)), delta(mlp=dense(24)), attn(chunk=70), delta(heads=2, kv_heads=1, dim=16, vdim=24, conv=5), attn(heads=2, kv_heads=2, chunk=9, mlp=dense(16)),
                      latent(heads=2, dim=20, vdim=8, kv_rank=16, q_rank=8)])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_equals_token_by_token(dtype):
    W = random_weights(HYBRID, seed=5, memory=1.0)
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
    """Portions down to two tokens and single tokens in between: the convolutions' and the recurrences' states, the caches and the chunks
    all cross the cuts (portions of fewer than 8 rows take the row kernels, longer ones the tile kernels)."""
    toks = tokens(sum(sizes), HYBRID["vocab"], 7)
    W = random_weights(HYBRID, seed=6, memory=1.0)
    want, _ = plain.run(HYBRID, W, toks)
    m = build_engine(HYBRID, W, dtype)
    got = run_schedule(m, {"a": toks}, [[("a", n)] for n in sizes])["a"]
    m.free()
    check_logits(got, want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_ragged_batch_equals_each_alone(dtype):
    cfg = HYBRID
    W = random_weights(cfg, seed=8, memory=1.0)
    reqs = {"a": tokens(90, cfg["vocab"], 11), "b": tokens(17, cfg["vocab"], 12), "c": tokens(130, cfg["vocab"], 13), "d": tokens(1, cfg["vocab"], 14)}
    m = build_engine(cfg, W, dtype, max_tokens=448)
    alone = {k: whole(m, v) for k, v in reqs.items()}
    sched = [[("a", 30), ("b", 2)], [("a", 1), ("b", 9), ("c", 64)], [("c", 2), ("a", 1), ("d", 1)], [("b", 6), ("a", 58), ("c", 64)]]
    got = run_schedule(m, reqs, sched)
    m.free()
    for k, v in reqs.items():
        check_logits(got[k], alone[k], dtype)
        check_logits(got[k], plain.run(cfg, W, v)[0], dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_and_slots_are_reused(dtype):
    """Two slots and three pages for five requests: later requests run in the slots and pages earlier ones gave back, and a stale
    convolution state, recurrent state or cache row would show in their logits (long memories)."""
    cfg = HYBRID
    W = random_weights(cfg, seed=9, memory=4.0)
    m = build_engine(cfg, W, dtype, max_tokens=192, max_seqs=2)
    seen_pages, seen_slots = [], []
    for i, n in enumerate([100, 70, 128, 5, 64]):
        toks = tokens(n, cfg["vocab"], 20 + i)
        s = m.open()
        other = m.open()   # a second live sequence holds the other slot and a page while this one runs
        m.step([(other, tokens(3, cfg["vocab"], 40 + i))], [[]])
        got = np.concatenate([m.step([(s, toks[:n // 2])], [list(range(n // 2))]), m.step([(s, toks[n // 2:])], [list(range(n - n // 2))])])
        seen_pages.append(tuple(m.pages(s)))
        seen_slots.append(s)
        check_logits(got, plain.run(cfg, W, toks)[0], dtype)
        m.close(s)
        m.close(other)
    assert m.pool_info()["free_pages"] == 3 and m.pool_info()["free_slots"] == 2
    m.free()
    assert len(set(seen_slots)) <= 2
    assert len(set(p for ps in seen_pages for p in ps)) <= 3 and len(seen_pages) == 5


# ---- a key that stands out: far back, at page borders, at position 0, on both sides of a chunk's edge ------------------------------
@functools.lru_cache(maxsize=None)
def planted_case(kind, chunk, place, n, rank=28, dim=16):
    """Token A sits at `place` among n - 1 other tokens, token B is last; head 0 of layer 0 gives B's query a large score against
    A's key and zero against any other.  Returns the model, the tokens, the true logits and how far the last row moves when the mask is
    off by that one key."""
    if kind == "chunked":
        cfg = make_config([attn(heads=4, kv_heads=2, dim=dim, vdim=dim, scale=0.5, chunk=chunk or None), delta()], width=64)
    else:
        cfg = make_config([latent(heads=3, dim=dim, vdim=24, kv_rank=rank, q_rank=20, scale=0.5), delta()], width=64)
    A, B = 7, 11
    W = plant_pair(cfg, random_weights(cfg, seed=13), A, B)
    rng = np.random.default_rng(place * 7 + n)
    fill = [t for t in range(cfg["vocab"]) if t not in (A, B)]
    toks = [fill[int(i)] for i in rng.integers(0, len(fill), n)]
    toks[place], toks[-1] = A, B
    true = plain.visible(n, chunk)
    shown, hidden = true.copy(), true.copy()
    shown[-1, place], hidden[-1, place] = True, False
    a, b = plain.run(cfg, W, toks, {0: shown})[0], plain.run(cfg, W, toks, {0: hidden})[0]
    want = a if true[-1, place] else b
    return cfg, W, toks, want, row_errs(b[-1:], a[-1:])[0]


def standing_out(kind, chunk, place, n, decode, dtype="float32", tol=None, **sizes):
    """Whether B sees A decides its logits (the plain implementation with a mask that is off by that one key differs by far more
    than the tolerance), so an engine whose chunk or page walk is one key off, or that loses a far key, cannot pass."""
    cfg, W, toks, want, moved = planted_case(kind, chunk, place, n, **sizes)
    tol = tol or TOL[dtype]
    assert moved > 3 * tol and moved > 0.1, "the planted key does not decide the last logits"
    m = build_engine(cfg, W, dtype)
    if decode:
        got = run_schedule(m, {"a": toks}, [[("a", n - 4)]] + [[("a", 1)]] * 4)["a"]
    else:
        got = whole(m, toks)
    m.free()
    check_logits(got, want, dtype)
    assert row_errs(got[-1:], want[-1:])[0] < tol


EDGES = [  # (attention of layer 0, chunk, place of the key, tokens): the row is the last token
    ("latent", 0, 0, 400),           # position 0, hundreds of keys back
    ("latent", 0, 63, 330),          # the end of the first page
    ("latent", 0, 64, 330),          # the start of the second
    ("latent", 0, 17, 600),          # far back among hundreds
    ("latent", 0, 198, 200),         # the key right before the row
    ("chunked", 20, 80, 100),        # the row ends its chunk: the chunk's first key is inside ...
    ("chunked", 20, 79, 100),        # ... and the last key of the chunk before is outside
    ("chunked", 33, 99, 101),        # the second row of a chunk: first key inside,
    ("chunked", 33, 98, 101),        # the key in front of the edge outside
    ("chunked", 33, 98, 100),        # the first row of a chunk: the key right before it is outside
    ("chunked", 64, 128, 192),       # a chunk of exactly one page
    ("chunked", 64, 127, 192),
    ("chunked", 64, 127, 129),
    ("chunked", 65, 130, 193),       # an edge two keys behind a page border
    ("chunked", 65, 129, 193),
    ("chunked", 300, 300, 420),      # a long chunk over several pages
    ("chunked", 300, 299, 420),
    ("chunked", 300, 0, 300),        # position 0 seen from the end of the first chunk
    ("chunked", 300, 63, 290),       # inside the first chunk, at a page's end
    ("chunked", 500, 0, 330),        # a chunk beyond the sequence
    ("chunked", 1, 98, 100),         # a chunk of one: nothing but itself
    ("chunked", 0, 5, 500),          # no chunks
]


@pytest.mark.parametrize("kind,chunk,place,n", EDGES)
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_stands_out(kind, chunk, place, n, decode):
    standing_out(kind, chunk, place, n, decode)


@pytest.mark.parametrize("kind,chunk,place,n", [e for e in EDGES if e[1] in (0, 33, 64, 65, 300) and e[3] != 600])
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_stands_out_bf16(kind, chunk, place, n, decode):
    standing_out(kind, chunk, place, n, decode, dtype="bfloat16", tol=0.05)


@pytest.mark.parametrize("rank", [100, 128, 200, 256, 512])
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_stands_out_in_wide_latents(rank, decode):
    standing_out("latent", 0, 65, 210, decode, dtype="bfloat16", tol=0.06, rank=rank, dim=32)


@pytest.mark.parametrize("decode", [False, True])
def test_chunk_edges_inside_a_tile_of_rows(decode):
    """Chunks of 5 positions: every tile of rows holds many edges, and a page many chunks."""
    cfg = make_config([attn(chunk=5), attn(heads=2, kv_heads=1, dim=64, vdim=64, chunk=13)])
    W = random_weights(cfg, seed=15)
    toks = tokens(200, cfg["vocab"], 3)
    want, _ = plain.run(cfg, W, toks)
    for off in (4, 6):
        other = dict(cfg, layers=[dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], mask={"size": off})), cfg["layers"][1]])
        assert row_errs(plain.run(other, W, toks)[0], want).max() > 0.1
    for dtype in ("float32", "bfloat16"):
        m = build_engine(cfg, W, dtype)
        got = run_schedule(m, {"a": toks}, [[("a", 150)]] + [[("a", 1)]] * 50)["a"] if decode else whole(m, toks)
        m.free()
        check_logits(got, want, dtype)


# ---- what each number does ---------------------------------------------------------------------------------------------------------
def test_sinks_gains_gates_and_decays_matter_and_match():
    """A sink, a gain, a gate or a decay that is left out moves the logits by far more than the tolerance."""
    cfg = make_config([attn(mlp=dense(24)), latent(), delta()])
    W = random_weights(cfg, seed=21)
    W["l0.mix.sink"] = to_bf16_values(np.array([3.0, 1.5, -0.5, 2.0], np.float32))
    toks = tokens(60, cfg["vocab"], 4)
    want, _ = plain.run(cfg, W, toks)
    fill = {"sink": -1e4, "norm": 1.0, "g": 0.0}
    for nm in ("l0.mix.sink", "l0.mix.q.norm", "l0.mix.k.norm", "l1.mix.dq.norm", "l1.mix.dkv.norm", "l1.mix.g", "l2.mix.norm", "l2.mix.A_log", "l2.mix.dt_bias", "l2.mix.b", "l2.mix.a",
               "l2.mix.q.conv", "l2.mix.k.conv", "l2.mix.v.conv", "l0.mlp.up"):
        W0 = dict(W)
        if nm.endswith(".conv"):   # the newest tap alone
            W0[nm] = np.array(W[nm], copy=True)
            W0[nm][:, :-1] = 0
        else:
            W0[nm] = np.full_like(W[nm], fill.get(nm.split(".")[-1], 0.0))
        assert row_errs(plain.run(cfg, W0, toks)[0], want).max() > 50 * TOL["float32"], nm
    m = build_engine(cfg, W, "float32")
    a = whole(m, toks)
    b = run_schedule(m, {"a": toks}, [[("a", 20)]] + [[("a", 1)]] * 40)["a"]
    m.free()
    check_logits(a, want, "float32")
    check_logits(b, want, "float32")


@pytest.mark.parametrize("decode", [False, True])
def test_sink_against_hundreds_of_keys(decode):
    """A sink as heavy as all keys together: it counts once whatever the number of key splits or tiles a row's keys are cut into."""
    cfg = make_config([attn(heads=2, kv_heads=1, dim=16, vdim=16, chunk=None), attn(heads=2, kv_heads=2, dim=64, vdim=64, chunk=200)], width=64)
    W = random_weights(cfg, seed=22)
    for i in range(2):
        W["l%d.mix.sink" % i] = to_bf16_values(np.array([6.0, 5.0], np.float32))
    toks = tokens(500, cfg["vocab"], 6)
    want, _ = plain.run(cfg, W, toks)
    W0 = {k: v + np.float32(np.log(2.0)) if k.endswith("sink") else v for k, v in W.items()}   # counted twice
    assert row_errs(plain.run(cfg, W0, toks)[0][-5:], want[-5:]).min() > 0.02
    for dtype in ("float32", "bfloat16"):
        m = build_engine(cfg, W, dtype)
        got = run_schedule(m, {"a": toks}, [[("a", 490)]] + [[("a", 1)]] * 10)["a"] if decode else whole(m, toks)
        m.free()
        assert rel_err(got, want) < (TOL["float32"] if dtype == "float32" else 0.015)


def test_gelu_is_the_error_function_form():
    """The tanh form differs by a few 1e-4 of the activation: more than fp32 rounding by two orders."""
    cfg = make_config([attn(mlp=dense(64))])
    W = random_weights(cfg, seed=25, out_amp=2.0)
    toks = tokens(40, cfg["vocab"], 4)
    want, _ = plain.run(cfg, W, toks)
    exact = plain.gelu
    try:
        plain.gelu = lambda z: 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))
        off = row_errs(plain.run(cfg, W, toks)[0], want).max()
    finally:
        plain.gelu = exact
    assert off > 1e-4
    m = build_engine(cfg, W, "float32")
    assert rel_err(whole(m, toks), want) < 0.1 * off
    assert rel_err(run_schedule(m, {"a": toks}, [[("a", 1)]] * 40)["a"], want) < 0.1 * off
    m.free()


def test_logit_scale_and_cap():
    base = make_config([latent()], logit_scale=0.8, softcap=3.0)
    W = random_weights(base, seed=26)
    toks = tokens(30, base["vocab"], 4)
    want, _ = plain.run(base, W, toks)
    assert 1.5 < np.abs(want).max() < 3.0
    for other in (dict(base, logit_scale=1.0), dict(base, logit_softcap=4.0)):
        assert row_errs(plain.run(other, W, toks)[0], want).max() > 0.02
    for dtype in ("float32", "bfloat16"):
        m = build_engine(base, W, dtype)
        got = whole(m, toks)
        few = run_schedule(m, {"a": toks}, [[("a", 1)]] * 30)["a"]
        m.free()
        assert np.abs(got - want).max() < (1e-4 if dtype == "float32" else 0.1)
        assert np.abs(few - want).max() < (1e-4 if dtype == "float32" else 0.1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_delta_state_recalls_a_far_write(dtype):
    """Almost no decay, and the key of token A (written once, hundreds of tokens back) is the query of token B while the other tokens' keys and
    queries have nothing there: B's output is A's value, and a state that is lost, decayed or overwritten anywhere in between shows."""
    cfg = make_config([delta(heads=2, kv_heads=1, dim=32, vdim=32, conv=2)], width=64)
    W = {k: np.array(v, copy=True) for k, v in random_weights(cfg, seed=28, memory=12.0).items()}
    A, B, u, v = 7, 11, 0, 1
    E, q = W["embed"], "l0.mix."
    E[:, [u, v]] = 0.0
    E[[A, B]] = 0.0
    E[A, v], E[B, u] = 12.0, 12.0
    for nm, coord in (("k", v), ("q", u)):   # channel 0 belongs to the pair, the others to the rest
        W[q + nm][0] = 0.0
        W[q + nm][1:, [u, v]] = 0.0
        W[q + nm][0, coord] = 3.0
        W[q + nm + ".conv"][0] = [0.0, 1.0]
    W[q + "b"][:, v] = 3.0     # a full write for A
    W[q + "v.conv"][:, 0] = 0.0
    W[q + "o"] *= 8.0
    W = {k: to_bf16_values(x) for k, x in W.items()}
    rng = np.random.default_rng(5)
    fill = [t for t in range(cfg["vocab"]) if t not in (A, B)]
    toks = [fill[int(i)] for i in rng.integers(0, len(fill), 400)]
    toks[70], toks[-1] = A, B
    want, _ = plain.run(cfg, W, toks)
    gone = list(toks)
    gone[70] = fill[0]
    assert row_errs(plain.run(cfg, W, gone)[0][-1:], want[-1:])[0] > 0.5
    m = build_engine(cfg, W, dtype)
    for sizes in ([400], [69, 2, 200, 128, 1], [396, 1, 1, 1, 1], [64] * 6 + [16]):
        got = run_schedule(m, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        check_logits(got, want, dtype)
        assert row_errs(got[-1:], want[-1:])[0] < (1e-4 if dtype == "float32" else 0.03)
    m.free()


def test_keys_that_repeat_and_keys_that_barely_exist():
    """The same token over and over (its key is written on itself each time: the recurrence's transition is as far from a plain sum as it
    gets), and projections so small that the unit norms divide by almost nothing."""
    cfg = make_config([delta(heads=2, kv_heads=2, dim=24, vdim=16, conv=3), delta(heads=4, kv_heads=2, dim=64, vdim=32, conv=4)], width=64)
    W = random_weights(cfg, seed=29, memory=6.0)
    W["l0.mix.b"] = W["l0.mix.b"] * 4
    toks = [5] * 70 + tokens(20, cfg["vocab"], 3) + [5, 9] * 40
    want, _ = plain.run(cfg, W, toks)
    tiny = dict(W)
    for nm in ("q", "k"):
        tiny["l0.mix." + nm] = to_bf16_values(W["l0.mix." + nm] * 1e-2)
    want_tiny, _ = plain.run(cfg, tiny, toks)
    assert row_errs(want_tiny, want).max() > 0.01   # (the constant under the unit norm's root shows)
    for dtype in ("float32", "bfloat16"):
        for w, ref in ((W, want), (tiny, want_tiny)):
            m = build_engine(cfg, w, dtype)
            check_logits(whole(m, toks), ref, dtype)
            check_logits(run_schedule(m, {"a": toks}, [[("a", 100)]] + [[("a", 1)]] * 70)["a"], ref, dtype)
            m.free()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decays_from_none_to_everything(dtype):
    """Logarithms of the decay between -0.001 and -1000 a token in the same head: sums over a portion are large, differences between
    neighbouring tokens small, and a state survives the one and not the other."""
    cfg = make_config([delta(heads=4, kv_heads=2, dim=32, vdim=24, conv=2), delta(heads=2, kv_heads=1, dim=128, vdim=16, conv=4)], width=64)
    W = random_weights(cfg, seed=30)
    W["l0.mix.A_log"] = to_bf16_values(np.array([-8.0, 0.0, 3.0, 5.0], np.float32))
    W["l1.mix.A_log"] = to_bf16_values(np.array([4.0, -3.0], np.float32))
    for i in range(2):
        W["l%d.mix.a" % i] = to_bf16_values(W["l%d.mix.a" % i] * 6.0)
        W["l%d.mix.dt_bias" % i] = to_bf16_values(np.full_like(W["l%d.mix.dt_bias" % i], -6.0))
    lg = np.log(np.maximum(plain.delta_decay({k: np.asarray(v, np.float64) for k, v in W.items()}, "l0.mix.", plain.norm(W["embed"].astype(np.float64), W["l0.norm1"], 1e-5)), 1e-300))
    assert lg[:, 3].min() < -300 and lg[:, 3].max() > -0.5
    toks = tokens(300, cfg["vocab"], 5)
    want, _ = plain.run(cfg, W, toks)
    m = build_engine(cfg, W, dtype)
    for sizes in ([300], [100, 7, 193], [250] + [1] * 50):
        check_logits(run_schedule(m, {"a": toks}, [[("a", n)] for n in sizes])["a"], want, dtype)
    m.free()


def test_states_cross_every_cut():
    """Long memories and large convolution weights: a row depends on rows in the same portion, the portion before, two portions back and
    before the sequence's start."""
    cfg = make_config([delta(conv=5), attn(chunk=3), delta(heads=2, kv_heads=1, dim=8, vdim=8, conv=2)])
    W = random_weights(cfg, seed=16, memory=4.0)
    toks = tokens(40, cfg["vocab"], 8)
    want, _ = plain.run(cfg, W, toks)
    W0 = dict(W)
    W0["l0.mix.v.conv"] = np.array(W["l0.mix.v.conv"], copy=True)
    W0["l0.mix.v.conv"][:, 0] = 0
    assert row_errs(plain.run(cfg, W0, toks)[0][4:], want[4:]).min() > 20 * TOL["float32"]
    # the first token still shows in the last logits
    assert row_errs(plain.run(cfg, W, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])[0][-1:], want[-1:]).max() > 20 * TOL["float32"]
    m = build_engine(cfg, W, "float32")
    for sizes in ([1] * 40, [2, 1, 1, 3, 1, 2, 2, 9, 1, 1, 1, 1, 1, 14], [40], [3, 37]):
        got = run_schedule(m, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert rel_err(got, want) < TOL["float32"], sizes
    m.free()


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
    """The chunks (70 and 9) pass over decoded tokens; 320 single-token steps."""
    cfg = HYBRID
    W = random_weights(cfg, seed=17, out_amp=0.4, memory=3.0)
    toks = tokens(330, cfg["vocab"], 5)
    want, _ = plain.run(cfg, W, toks)
    m = build_engine(cfg, W, dtype)
    got = run_schedule(m, {"a": toks}, [[("a", 10)]] + [[("a", 1)]] * 320)["a"]
    m.free()
    check_logits(got, want, dtype)


@pytest.mark.parametrize("rows", [1, 3, 8])
def test_wide_model_decode_rows_and_tiles(rows):
    """Widths in whole 32-element chunks (bf16 mode: the decode rows' products run on the tensor-core few-row kernel with the activated
    columns behind plain ones, prompt products on tcgen05 with the activation in their epilogue)."""
    cfg = make_config([latent(heads=4, dim=64, vdim=32, kv_rank=128, q_rank=96, mlp=dense(264)), delta(heads=4, kv_heads=2, dim=64, vdim=64, conv=4, mlp=dense(100)),
                       attn(heads=4, kv_heads=2, dim=128, vdim=128, chunk=50, mlp=dense(300)), delta(heads=2, kv_heads=2, dim=128, vdim=64, conv=4)], vocab=203, width=256)
    W = random_weights(cfg, seed=31, memory=2.0)
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


# ---- generation through the engine's own loop, and the command line ---------------------------------------------------------------
def plain_greedy(cfg, W, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(np.argmax(plain.run(cfg, W, toks)[0][-1])))
    return toks[len(prompt):]


def test_greedy_generation_continuous_batching():
    """Six requests through two slots and a pool that holds about two of them: admission, portions of prompts beside decoded
    tokens, and slots / pages handed on, all inside the engine's generation loop."""
    W = random_weights(HYBRID, seed=18, memory=2.0)
    prompts = [tokens(n, HYBRID["vocab"], 70 + i) for i, n in enumerate([5, 40, 90, 1, 64, 23])]
    want = [plain_greedy(HYBRID, W, p, 10) for p in prompts]
    m = build_engine(HYBRID, W, "float32", max_tokens=256, max_seqs=2)
    got = m.generate(prompts, 10, step_tokens=48)
    m.free()
    assert got == want


def test_command_line_generate_and_trace_replay(tmp_path):
    from turboinfer_b200.safetensors_io import write_safetensors
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = make_config([delta(mlp=dense(24)), attn(heads=2, kv_heads=1, chunk=9), latent(mlp=dense(10))], vocab=53)
    W = random_weights(cfg, seed=19)
    folder = os.path.join(tmp_path, "model")
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
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


def test_errors_are_reported():
    cfg = make_config([attn(mlp=dense(16)), latent(), delta()])
    W = random_weights(cfg, seed=20)
    bad = dict(W)
    bad["l2.mix.v.conv"] = W["l2.mix.v.conv"][:-1]
    with pytest.raises(Exception):
        build_engine(cfg, bad)
    for gone in ("l0.mix.sink", "l0.mix.q.norm", "l1.mix.g", "l1.mix.dq.norm", "l1.mix.uk", "l2.mix.dt_bias", "l2.mix.k.conv", "l2.mix.b", "l0.mlp.down", "l0.norm1"):
        with pytest.raises(Exception):
            build_engine(cfg, {k: v for k, v in W.items() if k != gone})
    for layer in (attn(heads=3, kv_heads=2), delta(heads=3, kv_heads=2), delta(conv=0), delta(dim=600), latent(kv_rank=0), latent(kv_rank=700)):
        with pytest.raises(Exception):
            c = make_config([layer])
            try:
                w = random_weights(c)
            except Exception:
                w = W
            build_engine(c, w)
