"""Bolapel folder models on the GPU against the slow float64 implementation of tests/bolapel_oracle.py.

Small random models (bf16-representable weights, so both operand modes load the same numbers) are written to a temporary
folder and opened through lmrs_b200.Transformer.open -- the entry point trace replay, forward, forward_argmax and
generate_greedy share.  float32 mode is held to 1e-4 of the logits' root mean square, bfloat16 mode to 4e-2."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import bolapel_oracle as O

pytestmark = pytest.mark.gpu

TOL = {"float32": 1e-4, "bfloat16": 4e-2}
D, A = O.delta_layer, O.attention_layer
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def mixed_cfg(**kw):
    """both mixers, two layers that borrow keys and values, layers without a feed-forward, grouped and ungrouped heads, blocks
    shorter and longer than a key tile, sizes that are no powers of two and differ from each other"""
    return O.make_config([
        D(),
        A(size=9),
        D(heads=2, dim=20, rank=3, mlp=None),
        A(heads=6, kv_heads=3, dim=8, vdim=12, size=70, rot_dims=8, scale=0.3, mlp=O.dense(ff=30)),
        A(heads=4, kv_heads=2, size=13, kv_from=1, scale=0.6, mlp=None),
        D(heads=1, dim=36, rank=8, mlp=O.dense(ff=24)),
        A(heads=3, kv_heads=3, dim=8, vdim=12, size=40, rot_dims=8, kv_from=3),
    ], **kw)


def open_model(gpu_lib, tmp_path, cfg, W, dtype, max_tokens=256, name="m"):
    return gpu_lib.Transformer.open(O.write_model(str(tmp_path / name), cfg, W), dtype=dtype, max_tokens=max_tokens)


def tokens_for(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt_logits_and_every_layer(gpu_lib, tmp_path, dtype):
    cfg = mixed_cfg()
    n = 85
    toks = tokens_for(cfg, n)
    W = O.random_weights(cfg, seed=1)
    want, outs = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, dtype)
    assert m.args.model_type == gpu_lib.ModelType.BOLAPEL and m.args.vocab_size == cfg["vocab"] and m.args.n_layers == 7
    m.set_option("keep_layers", 1)
    got = m.forward_tokens(toks, 0, list(range(n)))
    lo = m.layer_outputs(n)
    for li in range(7):   # the first layer that differs names the broken mechanism
        assert O.rel_rms(lo[li], outs[li]) < TOL[dtype], f"residual stream after layer {li}"
    assert O.rel_rms(got, want) < TOL[dtype]
    assert m.kernel_launches() > 0
    m.close()


# each mechanism alone: a one-layer model in which only that mechanism is not trivial, in shapes that take different branches
ALONE = {
    "delta": dict(layers=[D(mlp=None)]),
    "delta_one_head_one_channel": dict(layers=[D(heads=1, dim=1, rank=1, mlp=None)]),
    "delta_odd_sizes": dict(layers=[D(heads=3, dim=7, rank=3, mlp=None)]),
    "delta_head_64": dict(layers=[D(heads=2, dim=64, rank=16, mlp=None)]),
    "delta_just_above_64": dict(layers=[D(heads=2, dim=65, rank=16, mlp=None)]),
    "delta_head_100": dict(layers=[D(heads=2, dim=100, rank=4, mlp=None)]),
    "delta_head_136": dict(layers=[D(heads=1, dim=136, rank=8, mlp=None)]),
    "delta_head_264": dict(layers=[D(heads=1, dim=264, rank=8, mlp=None)]),
    "delta_many_heads": dict(layers=[D(heads=21, dim=4, rank=2, mlp=None)]),
    "delta_rank_wider_than_a_head": dict(layers=[D(heads=2, dim=8, rank=72, mlp=None)]),
    "attention": dict(layers=[A(mlp=None)]),
    "attention_no_blocks": dict(layers=[A(size=0, mlp=None)]),
    "attention_block_of_one": dict(layers=[A(size=1, mlp=None)]),
    "attention_block_one_tile": dict(layers=[A(size=64, mlp=None)]),
    "attention_block_tile_plus_one": dict(layers=[A(size=65, mlp=None)]),
    "attention_block_longer_than_the_prompt": dict(layers=[A(size=500, mlp=None)]),
    "attention_no_rotation": dict(layers=[A(rot_dims=0, mlp=None)]),
    "attention_whole_head_rotated": dict(layers=[A(rot_dims=12, mlp=None)]),
    "attention_one_kv_head": dict(layers=[A(heads=5, kv_heads=1, size=33, mlp=None)]),
    "attention_ungrouped": dict(layers=[A(heads=3, kv_heads=3, dim=8, vdim=8, rot_dims=8, mlp=None)]),
    "attention_many_heads_per_kv_head": dict(layers=[A(heads=20, kv_heads=1, dim=8, vdim=8, rot_dims=4, mlp=None)]),
    "attention_wide_values": dict(layers=[A(heads=2, kv_heads=1, dim=8, vdim=136, size=40, rot_dims=2, mlp=None)]),
    "attention_odd_head_sizes": dict(layers=[A(heads=3, kv_heads=1, dim=7, vdim=5, rot_dims=4, mlp=None)]),
    "attention_large_scores": dict(layers=[A(scale=8.0, mlp=None)]),
    "borrowed_keys": dict(layers=[A(mlp=None), A(heads=8, size=5, kv_from=0, scale=1.1, mlp=None), A(size=50, kv_from=0, mlp=None)]),
    "dense_ff": dict(layers=[D(mlp=O.dense(ff=72))]),
    "no_logit_cap": dict(layers=[D()], softcap=None),
    "logit_cap_that_bites": dict(layers=[D()], softcap=0.7),
    "large_eps": dict(layers=[D(), A()], eps=0.3),
    "odd_width": dict(layers=[D(heads=3, dim=10), A(dim=10, vdim=6, rot_dims=6)], width=27, vocab=33),
    # rows too long for the norm kernels to hold in registers between their passes (one row: 4 x 1024, many: 12 x 256 columns)
    "very_wide_rows": dict(layers=[D(heads=1, dim=8, mlp=O.dense(ff=8)), A(heads=1, kv_heads=1, dim=8, vdim=8, mlp=None)], width=4104, vocab=20),
}


@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(gpu_lib, tmp_path, name):
    kw = dict(ALONE[name])
    cfg = O.make_config(kw.pop("layers"), **kw)
    toks = tokens_for(cfg, 70, seed=2)   # crosses one key-tile border; no multiple of the scan's block
    W = O.random_weights(cfg, seed=5, gain=2.0)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    got = m.forward_tokens(toks, 0, list(range(70)))
    assert O.rel_rms(got, want) < TOL["float32"]
    # and token by token through the decode step
    for i, t in enumerate(toks):
        lg = m.forward(t, i)
        if i in (0, 1, 2, 3, 8, 9, 10, 63, 64, 65, 66, 67, 69):
            assert O.rel_rms(lg, want[i]) < TOL["float32"], f"decoded position {i}"
    # and token by token through the kernels of longer steps
    m.set_option("step_fused", 0)
    for i, t in enumerate(toks[:12]):
        assert O.rel_rms(m.forward(t, i), want[i]) < TOL["float32"], f"position {i}, one-token steps of the many-token kernels"
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_of_every_size_and_decoding_agree_with_the_whole_prompt(gpu_lib, tmp_path, dtype):
    cfg = mixed_cfg()
    n = 150
    toks = tokens_for(cfg, n, seed=3)
    W = O.random_weights(cfg, seed=2, gain=1.5)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, dtype)
    for cuts in ([n], [2] * 8 + [3, 61, 2, 64, 1, 1, 1, 1], [63, 1, 64, 2, 20], [1] * 6 + [129, 2, 13], [127, 23], [4, 5, 6, 7, 8, 9, 10, 11, 12, 78], [9] * 16 + [6]):
        assert sum(cuts) == n
        at, rows = 0, []
        for c in cuts:   # the same handle again and again: what an earlier schedule left in cache and state must not matter
            rows.append(m.forward_tokens(toks[at:at + c], at, list(range(c))))
            at += c
        assert O.rel_rms(np.concatenate(rows), want) < TOL[dtype], cuts
    # a long portion split by the library itself; a last internal piece of one row
    for rows in (37, 149):
        m.set_option("chunk_rows", rows)
        assert O.rel_rms(m.forward_tokens(toks, 0, list(range(n))), want) < TOL[dtype]
    m.close()


def test_portions_do_not_change_the_numbers_beyond_rounding(gpu_lib, tmp_path):
    """a position's logits from a whole prompt, from two-token portions and from single tokens differ by summation order only"""
    cfg = mixed_cfg()
    toks = tokens_for(cfg, 90, seed=4)
    W = O.random_weights(cfg, seed=3)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    whole = m.forward_tokens(toks, 0, list(range(90)))
    pairs = np.concatenate([m.forward_tokens(toks[i:i + 2], i, [0, 1]) for i in range(0, 90, 2)])
    triples = np.concatenate([m.forward_tokens(toks[i:i + 3], i, [0, 1, 2]) for i in range(0, 90, 3)])
    singles = np.stack([m.forward(t, i).copy() for i, t in enumerate(toks)])
    for other in (pairs, triples, singles):
        assert O.rel_rms(other, whole) < 2e-5
    m.close()


def test_wanted_rows_in_any_order(gpu_lib, tmp_path):
    cfg = mixed_cfg()
    toks = tokens_for(cfg, 40)
    W = O.random_weights(cfg, seed=4)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    idx = [39, 0, 17, 17, 5]
    assert O.rel_rms(m.forward_tokens(toks, 0, idx), want[idx]) < TOL["float32"]
    assert m.forward_tokens(toks, 0, []).shape == (0, cfg["vocab"])
    m.set_option("chunk_rows", 16)
    assert O.rel_rms(m.forward_tokens(toks, 0, idx), want[idx]) < TOL["float32"]
    m.close()


@pytest.mark.parametrize("shape", [1, 2])
@pytest.mark.parametrize("dim", [12, 64, 72, 128])
def test_other_thread_layouts_of_the_scan(gpu_lib, tmp_path, dim, shape):
    cfg = O.make_config([D(heads=2, dim=dim, mlp=None)])
    toks = tokens_for(cfg, 61, seed=6)
    W = O.random_weights(cfg, seed=7)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    m.set_option("scan_shape", shape)
    got = np.concatenate([m.forward_tokens(toks[:30], 0, list(range(30))), m.forward_tokens(toks[30:], 30, list(range(31)))])
    assert O.rel_rms(got, want) < TOL["float32"]
    m.close()


# ---- one token that matters ----------------------------------------------------------------------------------------------
def private_channel(W, toks, dim=0):
    """an input dimension becomes private to some tokens: their embedding is large there, every other token's is zero (an RMS
    norm keeps a zero a zero)"""
    W["embed"][:, dim] = 0.0
    W["embed"][toks, dim] = 8.0
    W["l0.norm1"][dim] = 1.0


def check_one_token_matters(gpu_lib, tmp_path, cfg, W, n, places, a_tok, b_tok, seen, teeth=100):
    """The last token (b) asks for what one earlier token (a) left behind.  Where `seen(place)` says it can be reached, taking
    token a away must move the slow implementation's answer a lot (the case has teeth); where it cannot, the answer must not
    depend on it.  The library must agree in a prompt, in decoding, and with the prompt cut near the token."""
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32", max_tokens=n + 8)
    for far in places:
        toks = [t if t < a_tok else 0 for t in tokens_for(cfg, n, seed=far)]
        toks[far], toks[n - 1] = a_tok, b_tok
        want, _ = O.forward(cfg, W, toks)
        toks2 = list(toks)
        toks2[far] = 0
        moved = O.rel_rms(O.forward(cfg, W, toks2)[0][n - 1], want[n - 1])
        if seen(far):
            assert moved > teeth * TOL["float32"], f"token at {far}: the case has no teeth ({moved})"
        else:
            assert moved < 1e-9, f"token at {far} should be out of reach"
        got = m.forward_tokens(toks, 0, [n - 1])
        assert O.rel_rms(got[0], want[n - 1]) < TOL["float32"], f"token at {far} (prompt)"
        m.forward_tokens(toks[:n - 1], 0, [])
        assert O.rel_rms(m.forward(toks[n - 1], n - 1), want[n - 1]) < TOL["float32"], f"token at {far} (decoded)"
        for cut in (far + 1, n - 2):
            if 0 < cut < n:
                m.forward_tokens(toks[:cut], 0, [])
                assert O.rel_rms(m.forward_tokens(toks[cut:], cut, [n - 1 - cut])[0], want[n - 1]) < TOL["float32"], f"token at {far}, cut at {cut}"
    m.close()


def one_key_attention(size, seed=7, kv_from=False):
    """the query of token 49 and the key of token 48 share an unrotated dimension that no other token uses; every other weight is
    all but shut by the bias; no token shift"""
    layer = A(heads=2, kv_heads=1, dim=8, vdim=8, size=size, rot_dims=4, scale=2.0, mlp=None)
    layers = [layer] if not kv_from else [A(heads=2, kv_heads=1, dim=8, vdim=8, size=3, rot_dims=4, scale=2.0, mlp=None),
                                          A(heads=2, kv_heads=1, dim=8, vdim=8, size=size, rot_dims=4, scale=2.0, kv_from=0, mlp=None)]
    cfg = O.make_config(layers, width=16, vocab=50)
    W = O.random_weights(cfg, seed=seed)
    private_channel(W, [48, 49])
    for p in [f"l{i}." for i in range(len(layers))]:
        W[p + "shift"][:] = 0.0
        W[p + "norm1"][0] = 1.0
        W[p + "mix.pb"][:] = -6.0
        for t in ("q", "k"):
            if p + "mix." + t in W:
                W[p + "mix." + t][:, 0] = 0.0
                W[p + "mix." + t][5, 0] = 16.0      # after the norm this dimension carries nearly all of q (in head 0) and of k
                W[p + "mix." + t + ".norm"][:] = 1.0
    return cfg, W


@pytest.mark.parametrize("size", [7, 64, 65, 100])
def test_keys_just_inside_and_just_outside_the_block(gpu_lib, tmp_path, size):
    cfg, W = one_key_attention(size)
    for n in (size * 2 + 1, size * 2 + 2, size * 3, 200):     # the asking token first, second and last in its block, and anywhere
        last = n - 1
        start = last // size * size
        places = sorted({p for p in (0, start - size, start - 2, start - 1, start, start + 1, last - 1) if 0 <= p < last})
        check_one_token_matters(gpu_lib, tmp_path, cfg, W, n, places, 48, 49, seen=lambda p: p >= start)


def test_blocks_of_a_layer_on_borrowed_keys(gpu_lib, tmp_path):
    """the lender's own blocks are short; the borrower's block decides what the borrower sees.  What the lender itself adds to the
    asking token is moved by near tokens only"""
    cfg, W = one_key_attention(50, kv_from=True)
    n = 140
    check_one_token_matters(gpu_lib, tmp_path, cfg, W, n, [40, 98, 99, 100, 101, 120, 135], 48, 49, seen=lambda p: p >= 100)


def test_a_far_key_is_found_among_hundreds(gpu_lib, tmp_path):
    cfg, W = one_key_attention(0, seed=8)
    n = 330
    check_one_token_matters(gpu_lib, tmp_path, cfg, W, n, [0, 1, 63, 64, 191, 192, n - 3], 48, 49, seen=lambda p: True)


def remembering_delta(seed=9, decay=-9.0):
    """almost no decay and no removal: what token a writes under a key channel that no other token uses stays for token b"""
    cfg = O.make_config([D(heads=2, dim=8, rank=2, mlp=None)], width=16, vocab=50)
    W = O.random_weights(cfg, seed=seed)
    private_channel(W, [48], 0)             # read by the key
    private_channel(W, [49], 1)             # read by the query
    W["l0.shift"][:] = 0.0
    W["l0.mix.w0"][:] = decay
    W["l0.mix.w2"][:] = O.bf16_round(W["l0.mix.w2"] * 0.05)
    W["l0.mix.a"][:] = 0.0
    W["l0.mix.a.b"][:] = -14.0
    for name, dim in (("l0.mix.k", 0), ("l0.mix.r", 1)):
        W[name][:, dim] = 0.0
        W[name][[3, 11], :] = 0.0
        W[name][[3, 11], dim] = 4.0         # channel 3 of both heads
    return cfg, W


def test_the_state_remembers_a_write_from_far_back(gpu_lib, tmp_path):
    cfg, W = remembering_delta()
    n = 300
    check_one_token_matters(gpu_lib, tmp_path, cfg, W, n, [0, 1, 2, 3, 4, 7, 8, 150, n - 3, n - 2], 48, 49, seen=lambda p: True)


def test_a_removal_takes_a_write_away(gpu_lib, tmp_path):
    """token 47 writes nothing under token 48's key but removes what is there: its presence between the write and the question
    changes the answer, in every place of a four-token block and across portions"""
    cfg, W = remembering_delta(seed=10)
    W["embed"][47] = W["embed"][48]         # the same key ...
    W["embed"][47, 2] = 8.0
    W["embed"][:47, 2] = 0.0; W["embed"][48:, 2] = 0.0
    W["l0.norm1"][2] = 1.0
    W["l0.mix.a"][[3, 11], 2] = 40.0        # ... and a removal rate of one in channel 3
    n = 120
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32", max_tokens=n + 8)
    for wrote, gone in ((10, 11), (10, 50), (12, 15), (13, 16), (40, n - 2), (n - 3, n - 2)):
        toks = [t if t < 47 else 0 for t in tokens_for(cfg, n, seed=gone)]
        toks[wrote], toks[gone], toks[n - 1] = 48, 47, 49
        want, _ = O.forward(cfg, W, toks)
        without = O.forward(cfg, W, toks[:gone] + [0] + toks[gone + 1:])[0][n - 1]
        assert O.rel_rms(without, want[n - 1]) > 100 * TOL["float32"]
        assert O.rel_rms(m.forward_tokens(toks, 0, [n - 1])[0], want[n - 1]) < TOL["float32"]
        m.forward_tokens(toks[:gone], 0, [])
        m.forward(toks[gone], gone)
        assert O.rel_rms(m.forward_tokens(toks[gone + 1:], gone + 1, [n - 2 - gone])[0], want[n - 1]) < TOL["float32"]
    m.close()


def test_decays_a_hair_below_one_keep_their_precision(gpu_lib, tmp_path):
    """hundreds of tokens under decays of 1 - 1e-5: the float32 result stays within a few roundings of the exact one"""
    cfg, W = remembering_delta(seed=11, decay=-11.0)
    toks = tokens_for(cfg, 700, seed=1)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32", max_tokens=700)
    assert O.rel_rms(m.forward_tokens(toks, 0, [650, 699]), want[[650, 699]]) < 2e-5
    m.close()


def test_the_shift_reaches_exactly_one_token_back(gpu_lib, tmp_path):
    """a layer that sees only the previous token's row (shift of one, blocks of one position): the asking token's answer depends on
    the token before it and on no other; at a portion's start that row comes from the state"""
    layer = A(heads=2, kv_heads=1, dim=8, vdim=8, size=1, rot_dims=4, mlp=None)
    cfg = O.make_config([layer], width=16, vocab=50)
    W = O.random_weights(cfg, seed=12)
    private_channel(W, [48, 49])
    W["l0.shift"][:] = 1.0
    for n in (9, 40):
        check_one_token_matters(gpu_lib, tmp_path, cfg, W, n, [0, n - 4, n - 3, n - 2], 48, 49, seen=lambda p: p == n - 2, teeth=50)


# ---- cache, state, generation, errors --------------------------------------------------------------------------------------
def test_cache_and_state_are_reused_by_the_next_sequence(gpu_lib, tmp_path):
    cfg = mixed_cfg()
    a, b = tokens_for(cfg, 90, seed=1), tokens_for(cfg, 33, seed=2)
    W = O.random_weights(cfg, seed=6)
    wa, _ = O.forward(cfg, W, a)
    wb, _ = O.forward(cfg, W, b)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    assert O.rel_rms(m.forward_tokens(a, 0, [89]), wa[[89]]) < TOL["float32"]
    # a shorter sequence over the same positions: nothing of `a` (keys beyond position 32, its states, its shift rows) may show
    assert O.rel_rms(m.forward_tokens(b[:20], 0, [0, 19]), wb[[0, 19]]) < TOL["float32"]
    for i in range(20, 33):
        assert O.rel_rms(m.forward(b[i], i), wb[i]) < TOL["float32"]
    assert O.rel_rms(m.forward_tokens(a, 0, [0, 50]), wa[[0, 50]]) < TOL["float32"]
    # a new sequence that starts with single tokens (the first tokens of a sequence, decoded)
    for i in range(5):
        assert O.rel_rms(m.forward(b[i], i), wb[i]) < TOL["float32"]
    # the state stands at one position: a step elsewhere is refused, a restart is not
    with pytest.raises(gpu_lib.LmrsError, match="position"):
        m.forward_tokens(b[:3], 17, [])
    assert O.rel_rms(m.forward_tokens(b, 0, [32]), wb[[32]]) < TOL["float32"]
    m.close()


def test_first_tokens_and_a_prompt_of_one(gpu_lib, tmp_path):
    cfg = mixed_cfg()
    W = O.random_weights(cfg, seed=8)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    for toks in ([7], [7, 7], [0, 1, 2], [5, 4, 3, 2, 1]):
        want, _ = O.forward(cfg, W, toks)
        assert O.rel_rms(m.forward_tokens(toks, 0, list(range(len(toks)))), want) < TOL["float32"]
        assert O.rel_rms(m.forward(toks[0], 0), want[0]) < TOL["float32"]
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_greedy_generation_through_the_generate_loop(gpu_lib, tmp_path, dtype):
    cfg = mixed_cfg()
    W = O.random_weights(cfg, seed=9)
    prompt = tokens_for(cfg, 21, seed=4)
    n_new = 150   # decodes across key-tile borders, through several key splits, and many block borders
    m = open_model(gpu_lib, tmp_path, cfg, W, dtype, max_tokens=21 + n_new)
    m.forward_tokens(prompt[:-1], 0, [])
    ids = m.generate_greedy(prompt[-1], len(prompt) - 1, n_new).tolist()
    assert len(ids) == n_new
    # replay the produced sequence through the slow implementation: every pick must be its argmax or within a hair of it
    want, _ = O.forward(cfg, W, prompt + ids)
    hair = 1e-3 if dtype == "float32" else 0.15
    for i, t in enumerate(ids):
        row = want[len(prompt) - 1 + i]
        assert row[t] >= row.max() - hair * (row.max() - row.min()), f"generated token {i}"
    # forward_argmax is the same pick
    m.forward_tokens(prompt[:-1], 0, [])
    assert m.forward_argmax(prompt[-1], len(prompt) - 1) == ids[0]
    # decode steps replayed from CUDA graphs and launched one by one are the same arithmetic
    m.set_option("graphs", 0)
    m.forward_tokens(prompt[:-1], 0, [])
    assert m.generate_greedy(prompt[-1], len(prompt) - 1, n_new).tolist() == ids
    # ... and so are steps whose kernels are chained with programmatic dependent launch, replayed or not
    for graphs in (1, 0):
        m.set_option("graphs", graphs)
        m.set_option("pdl", 1)
        m.forward_tokens(prompt[:-1], 0, [])
        assert m.generate_greedy(prompt[-1], len(prompt) - 1, n_new).tolist() == ids
    with pytest.raises(gpu_lib.LmrsError):
        m.forward(1, 21 + n_new)   # beyond the cache
    m.close()


def test_long_decoding_stays_with_the_slow_implementation(gpu_lib, tmp_path):
    cfg = O.make_config([D(), A(size=100), D(heads=2, dim=20), A(size=300, kv_from=1)])
    toks = tokens_for(cfg, 420, seed=5)
    W = O.random_weights(cfg, seed=14)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32", max_tokens=420)
    m.forward_tokens(toks[:20], 0, [])
    for i in range(20, 420):
        lg = m.forward(toks[i], i)
        if i % 7 == 0 or i in (99, 100, 101, 199, 200, 299, 300, 301, 399, 400, 419):
            assert O.rel_rms(lg, want[i]) < TOL["float32"], f"decoded position {i}"
    m.close()


def test_tensor_core_products_equal_the_cuda_core_products(gpu_lib, tmp_path):
    """bf16 mode, shapes that are no multiples of the 128 x 128 x 64 tile: rows, outputs and K tails are masked or zero-filled"""
    cfg = O.make_config([
        D(heads=5, dim=24, rank=8, mlp=O.dense(ff=200)),
        A(heads=6, kv_heads=2, dim=32, vdim=20, size=50, rot_dims=16, mlp=None),
        D(heads=4, dim=40, rank=16, mlp=O.dense(ff=72)),
        A(heads=4, kv_heads=2, dim=32, vdim=20, size=90, rot_dims=16, kv_from=1),
    ], width=72, vocab=203)
    toks = tokens_for(cfg, 300)
    W = O.random_weights(cfg, seed=10)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "bfloat16", max_tokens=320)
    a = m.forward_tokens(toks, 0, list(range(300)))
    m.set_option("tensor_cores", 0)
    b = m.forward_tokens(toks, 0, list(range(300)))
    assert O.rel_rms(a, b) < 2e-2 and not np.array_equal(a, b)   # different kernels, same numbers up to summation order
    assert O.rel_rms(a, want) < TOL["bfloat16"] and O.rel_rms(b, want) < TOL["bfloat16"]
    m.close()


def test_configuration_errors_are_reported(gpu_lib, tmp_path):
    cfg = mixed_cfg()
    W = O.random_weights(cfg)
    opened = lambda c, w, name: gpu_lib.Transformer.open(O.write_model(str(tmp_path / name), c, w))
    for missing in ("l0.mix.w1", "l0.shift", "l3.mix.k.norm", "l6.mix.pb", "l1.norm2b", "head"):
        with pytest.raises(gpu_lib.LmrsError, match=missing.replace(".", r"\.")):
            opened(cfg, {k: v for k, v in W.items() if k != missing}, "miss")
    W2 = dict(W)
    W2["l2.mix.w2"] = W["l2.mix.w2"][:, :-1]
    with pytest.raises(gpu_lib.LmrsError, match="l2.mix.w2"):
        opened(cfg, W2, "shape")
    for bad, match in ((dict(D(), type="no_such_mixer"), "no_such_mixer"), (dict(D(), mlp={"kind": "moe", "ff": 8}), "moe"), (A(kv_from=0), "kv_from"),
                       (A(kv_from=2), "kv_from"), (A(rot_dims=7), "rot"), (A(heads=3, kv_heads=2), "head")):
        with pytest.raises(gpu_lib.LmrsError, match=match):
            opened(O.make_config([D(), bad]), O.random_weights(O.make_config([D(), D()])), "bad")
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32", max_tokens=16)
    with pytest.raises(gpu_lib.LmrsError):
        m.forward_tokens([1] * 17, 0, [])
    with pytest.raises(gpu_lib.LmrsError, match="token"):
        m.forward_tokens([cfg["vocab"]], 0, [])
    m.close()


def test_cached_rows_can_be_read_back(gpu_lib, tmp_path):
    cfg = O.make_config([D(mlp=None), A(mlp=None), A(kv_from=1, mlp=None)])
    W = O.random_weights(cfg, seed=3)
    toks = tokens_for(cfg, 12)
    st = O.StepOracle(cfg, W)
    st.step(toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    m.forward_tokens(toks, 0, [])
    for layer in (1, 2):   # a borrower shows the lender's rows
        k, v = m.read_kv(layer, 0, 12, k_cols=2 * 12, v_cols=2 * 20)
        assert np.allclose(k.reshape(12, -1), st.state[1]["k"].reshape(12, -1), atol=1e-4)
        assert np.allclose(v.reshape(12, -1), st.state[1]["v"].reshape(12, -1), atol=1e-4)
    with pytest.raises(gpu_lib.LmrsError, match="state"):
        m.read_kv(0, 0, 12, k_cols=4, v_cols=4)
    m.close()


def test_the_command_line_generates_from_a_folder(gpu_lib, tmp_path):
    """lm.rs_b200/examples/generate on a model folder prints the ids that generate_greedy picks"""
    subprocess.check_call(["make", "-C", os.path.join(ROOT, "lm.rs_b200"), "-s", "examples"])
    cfg = mixed_cfg()
    W = O.random_weights(cfg, seed=11)
    d = O.write_model(str(tmp_path / "cli"), cfg, W)
    prompt = [3, 9, 27, 20]
    env = dict(os.environ, GENERATE_DTYPE="float32")
    r = subprocess.run([os.path.join(ROOT, "lm.rs_b200", "examples", "generate"), d, "10"] + [str(t) for t in prompt],
                       capture_output=True, text=True, env=env)
    assert r.returncode == 0, r.stderr
    m = gpu_lib.Transformer.open(d, dtype="float32", max_tokens=32)
    m.forward_tokens(prompt[:-1], 0, [])
    assert [int(x) for x in r.stdout.split()] == m.generate_greedy(prompt[-1], 3, 10).tolist()
    m.close()


def test_trace_replay_writes_the_logits_asked_for(gpu_lib, tmp_path):
    """bin/trace_run: a prompt in portions, then single tokens, then a second request over the same cache and state"""
    cfg = mixed_cfg()
    a, b = tokens_for(cfg, 75, seed=5), tokens_for(cfg, 9, seed=6)
    W = O.random_weights(cfg, seed=12)
    d = O.write_model(str(tmp_path / "tr"), cfg, W)
    wa, _ = O.forward(cfg, W, a)
    wb, _ = O.forward(cfg, W, b)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:66], "want": [0, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[66:73], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[73:74], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "x", "tokens": a[74:75], "want": [0]}], "end": ["x"]},
             {"step": 4, "entries": [{"id": "y", "tokens": b, "want": [8, 2]}], "end": ["y"]}]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "80"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done %d" % i for i in range(5)]
    assert not (out / "1.f32").exists()
    V = cfg["vocab"]
    for step, want in ((0, wa[[0, 65]]), (2, wa[[73]]), (3, wa[[74]]), (4, wb[[8, 2]])):
        got = np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(-1, V)
        assert O.rel_rms(got, want) < TOL["float32"], f"step {step}"
