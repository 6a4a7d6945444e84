"""Lutesun folder models on the GPU against the slow float64 implementation of tests/lutesun_oracle.py.

Small random models (bf16-representable weights, so both operand modes load the same numbers) are written to a temporary
folder and opened through lmrs_b200.Transformer.open -- the entry point trace replay, forward, forward_argmax and
generate_greedy share.  float32 mode is held to 2e-4 of the logits' root mean square, bfloat16 mode to 4e-2.  For float32
the weights are drawn until no routing decision of the run (of groups or of experts) is a close call; the bfloat16
comparisons against the slow implementation use routers that choose all of their outputs -- the weights still matter, no
choice can flip -- and the one bfloat16 test with real choices holds the typical row to the tolerance."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import lutesun_oracle as O

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-4, "bfloat16": 4e-2}
GAP = 1e-4
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def mixed_cfg(dtype="float32", **kw):
    """both forms of the mixer, both feed-forwards, a layer without one, windows shorter and longer than a key tile and one longer
    than the prompts, sizes that are no powers of two and differ from each other; for bfloat16 every router chooses all of its outputs"""
    def ff(e, i, t, f, s, groups, keep, scale):
        return O.moe(e, i, t, f, s, groups, keep, scale) if dtype == "float32" else O.moe(e, i, e + i, f, s, groups, groups, scale)
    return O.make_config([
        O.direct_layer(mlp=O.dense()),
        O.gated_layer(mlp=ff(7, 2, 3, 24, 40, 3, 2, 1.75)),
        O.direct_layer(heads=2, dim=20, rot_dim=4, vdim=6, kv_rank=12, size=70, base=1e4, mlp=None),
        O.gated_layer(heads=4, dim=16, rot_dim=6, vdim=20, kv_rank=36, q_rank=10, size=64, mlp=ff(6, 0, 1, 16, 0, 2, 1, 0.8)),
        O.direct_layer(heads=6, dim=6, rot_dim=10, vdim=8, kv_rank=16, size=500, mlp=ff(3, 5, 2, 30, 12, 4, 3, 2.5)),
    ], **kw)


def open_model(gpu_lib, tmp_path, cfg, W, dtype, max_tokens=256, name="m"):
    return gpu_lib.Transformer.open(O.write_model(str(tmp_path / name), cfg, W), dtype=dtype, max_tokens=max_tokens)


def tokens_for(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def weights_for(cfg, toks, seed=0, **kw):
    for s in range(seed, seed + 400, 7):
        W = O.random_weights(cfg, seed=s, **kw)
        if O.clear_choices(cfg, W, toks, GAP):
            return W
    raise AssertionError("no seed without a close routing decision")


def typical_row_close(got, want, tol):
    """the median row within tolerance and most rows too: a few may show an expert choice that flipped on a near-tie"""
    e = np.array([O.rel_rms(g, w) for g, w in zip(got, want)])
    return np.median(e) < tol and np.mean(e > tol) <= 0.35


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt_logits_and_every_layer(gpu_lib, tmp_path, dtype):
    cfg = mixed_cfg(dtype)
    toks = tokens_for(cfg, 85)
    W = weights_for(cfg, toks, seed=1)
    want, outs = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, dtype)
    assert m.args.model_type == gpu_lib.ModelType.LUTESUN and m.args.vocab_size == cfg["vocab"] and m.args.n_layers == 5
    m.set_option("keep_layers", 1)
    got = m.forward_tokens(toks, 0, list(range(85)))
    lo = m.layer_outputs(85)
    for li in range(5):   # the first layer that differs names the broken mechanism
        assert O.rel_rms(lo[li], outs[li]) < TOL[dtype], f"residual stream after layer {li}"
    assert O.rel_rms(got, want) < TOL[dtype]
    assert m.kernel_launches() > 0
    m.close()


# each mechanism alone: a model in which only that mechanism is not trivial, in shapes that take different branches
D, G, M = O.direct_layer, O.gated_layer, O.moe
ALONE = {
    "direct": dict(layers=[D(mlp=None)]),
    "direct_no_window": dict(layers=[D(size=0, mlp=None)]),
    "direct_window_of_one": dict(layers=[D(size=1, mlp=None)]),
    "direct_window_one_tile": dict(layers=[D(size=64, mlp=None)]),
    "direct_window_tile_plus_one": dict(layers=[D(size=65, mlp=None)]),
    "direct_one_head": dict(layers=[D(heads=1, mlp=None)]),
    "direct_many_heads": dict(layers=[D(heads=20, dim=4, rot_dim=2, vdim=4, kv_rank=8, size=33, mlp=None)]),
    "direct_rotated_part_larger": dict(layers=[D(dim=4, rot_dim=24, mlp=None)]),
    "direct_sizes_all_equal": dict(layers=[D(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=16, size=16, mlp=None)], width=16),
    "direct_wide_values": dict(layers=[D(heads=2, vdim=72, size=40, mlp=None)]),
    "direct_odd_sizes": dict(layers=[D(heads=3, dim=7, rot_dim=6, vdim=9, kv_rank=13, mlp=None)]),
    "gated": dict(layers=[G(mlp=None)]),
    "gated_no_window": dict(layers=[G(size=0, mlp=None)]),
    "gated_window_longer_than_the_prompt": dict(layers=[G(size=300, mlp=None)]),
    "gated_one_head": dict(layers=[G(heads=1, mlp=None)]),
    "gated_query_latent_wider_than_the_model": dict(layers=[G(q_rank=56, mlp=None)]),
    "gated_odd_sizes": dict(layers=[G(heads=3, dim=5, rot_dim=10, vdim=7, kv_rank=11, q_rank=9, size=20, mlp=None)]),
    "gated_wide_latent": dict(layers=[G(heads=2, kv_rank=136, q_rank=24, size=50, mlp=None)]),
    "latent_over_half_the_widest_tile": dict(layers=[D(heads=3, kv_rank=300, size=30, mlp=None)]),
    "latent_too_wide_for_a_shared_head": dict(layers=[G(heads=3, kv_rank=560, size=30, mlp=None), D(heads=2, kv_rank=520, size=0, mlp=None)]),
    "dense_ff": dict(layers=[D(size=300, mlp=O.dense())]),
    "dense_ff_odd": dict(layers=[D(size=300, mlp=O.dense(ff=33))]),
    "experts": dict(layers=[D(size=300)]),
    "experts_top_one_no_identity_no_shared": dict(layers=[D(size=300, mlp=M(4, 0, 1, shared=0, groups=1, keep=1, scale=1.0))]),
    "experts_every_group_kept": dict(layers=[D(size=300, mlp=M(6, 0, 2, groups=3, keep=3))]),
    "experts_one_group_of_many": dict(layers=[D(size=300, mlp=M(14, 2, 3, ff=8, groups=4, keep=1))]),
    "experts_groups_of_one": dict(layers=[D(size=300, mlp=M(5, 1, 2, groups=6, keep=2))]),
    "experts_a_group_of_identity_experts_only": dict(layers=[D(size=300, mlp=M(4, 4, 3, groups=2, keep=1))]),
    "experts_all_chosen": dict(layers=[D(size=300, mlp=M(3, 1, 4, groups=2, keep=2))]),
    "experts_mostly_identity": dict(layers=[D(size=300, mlp=M(1, 5, 2, ff=8, shared=8, groups=2, keep=2))]),
    "experts_many": dict(layers=[D(size=300, mlp=M(45, 3, 5, ff=8, shared=16, groups=8, keep=3))]),
    "experts_shared_wider_than_the_chosen": dict(layers=[D(size=300, mlp=M(4, 0, 2, ff=8, shared=104, groups=2, keep=2))]),
    "experts_shared_odd": dict(layers=[D(size=300, mlp=M(4, 0, 2, ff=12, shared=13, groups=1, keep=1))]),
    "no_embedding_scale": dict(layers=[G(mlp=None)], embed_scale=1.0),
    "large_eps": dict(layers=[D(mlp=O.dense()), G(mlp=None)], eps=0.3),
    "odd_width": dict(layers=[D(), G(mlp=O.dense())], width=27, vocab=33),
    # rows too long for the norm kernels to hold in registers between their passes; rows that need the wider register form
    "very_wide_rows": dict(layers=[D(heads=2, size=300, mlp=M(2, 1, 2, ff=8, shared=8, groups=1, keep=1)), G(heads=2, mlp=O.dense(ff=8))], width=4104, vocab=20),
    "wide_rows": dict(layers=[D(heads=2, size=300, mlp=M(2, 1, 2, ff=8, shared=8, groups=1, keep=1))], width=2056, vocab=20),
    # one-row products whose output rows are few and long: the warps of a CTA split each row, for the shared expert too
    "long_rows_into_a_narrow_stream": dict(layers=[D(heads=16, vdim=64, size=300, mlp=O.dense(ff=1024)),
                                                   G(heads=2, mlp=M(3, 0, 2, ff=1024, shared=1032, groups=1, keep=1))], width=64, vocab=40),
    "long_chosen_rows_beside_an_odd_shared_one": dict(layers=[D(heads=2, size=300, mlp=M(3, 0, 2, ff=1024, shared=21, groups=1, keep=1))], width=64, vocab=40),
}


@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(gpu_lib, tmp_path, name):
    kw = dict(ALONE[name])
    cfg = O.make_config(kw.pop("layers"), **kw)
    toks = tokens_for(cfg, 70, seed=2)   # crosses one key-tile border
    W = weights_for(cfg, toks, seed=5, gain=1.5)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    got = m.forward_tokens(toks, 0, list(range(70)))
    assert O.rel_rms(got, want) < TOL["float32"]
    # and token by token through the decode step
    for i, t in enumerate(toks):
        lg = m.forward(t, i)
        if i in (0, 1, 2, 3, 9, 31, 63, 64, 65, 66, 67, 69):
            assert O.rel_rms(lg, want[i]) < TOL["float32"], f"decoded position {i}"
    # short portions (the latent-space form for several rows)
    rows = [m.forward_tokens(toks[i:i + 7], i, list(range(7))) for i in range(0, 70, 7)]
    assert O.rel_rms(np.concatenate(rows), want) < TOL["float32"]
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_of_every_size_and_decoding_agree_with_the_whole_prompt(gpu_lib, tmp_path, dtype):
    cfg = mixed_cfg(dtype)
    n = 150
    toks = tokens_for(cfg, n, seed=3)
    W = weights_for(cfg, toks, seed=2)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, dtype)
    for cuts in ([n], [2] * 8 + [3, 61, 2, 64, 1, 1, 1, 1], [63, 1, 64, 2, 20], [1] * 6 + [129, 2, 13], [127, 23], [70, 16, 15, 17, 32]):
        assert sum(cuts) == n
        at, rows = 0, []
        for c in cuts:   # the same handle again and again: what an earlier schedule left in the cache must not matter
            rows.append(m.forward_tokens(toks[at:at + c], at, list(range(c))))
            at += c
        assert O.rel_rms(np.concatenate(rows), want) < TOL[dtype], cuts
    # a long internal portion split by the library itself
    m.set_option("chunk_rows", 37)
    assert O.rel_rms(m.forward_tokens(toks, 0, list(range(n))), want) < TOL[dtype]
    m.close()


def test_portions_do_not_change_the_numbers_beyond_rounding(gpu_lib, tmp_path):
    """a position's logits from a whole prompt, from two-token portions and from single tokens differ by summation order only"""
    cfg = mixed_cfg()
    toks = tokens_for(cfg, 90, seed=4)
    W = weights_for(cfg, toks, seed=3)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    whole = m.forward_tokens(toks, 0, list(range(90)))
    pairs = np.concatenate([m.forward_tokens(toks[i:i + 2], i, [0, 1]) for i in range(0, 90, 2)])
    singles = np.stack([m.forward(t, i).copy() for i, t in enumerate(toks)])
    assert O.rel_rms(pairs, whole) < 2e-5 and O.rel_rms(singles, whole) < 2e-5
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_latent_space_and_the_per_head_form_agree(gpu_lib, tmp_path, dtype):
    """short steps multiply the keys' up-projection into the query, long portions up-project the cached latents inside the window:
    the same numbers either way, for whole prompts and for portions that continue a cache behind several windows"""
    cfg = O.make_config([D(mlp=None), G(heads=4, size=65, mlp=None), D(size=0, mlp=None)])
    n = 260
    toks = tokens_for(cfg, n, seed=6)
    W = O.random_weights(cfg, seed=13, gain=1.5)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, dtype, max_tokens=n + 4)
    for rows in (1000, 2):   # never per head | always per head (portions of two and more)
        m.set_option("latent_expand_rows", rows)
        assert O.rel_rms(m.forward_tokens(toks, 0, list(range(n))), want) < TOL[dtype]
        at, got = 0, []
        for c in (3, 61, 2, 33, 1, 29, 65, 2, 64):
            got.append(m.forward_tokens(toks[at:at + c], at, list(range(c))))
            at += c
        assert at == n and O.rel_rms(np.concatenate(got), want) < TOL[dtype]
    m.close()


def test_long_prompts_take_the_wide_query_tiles(gpu_lib, tmp_path):
    """portions with enough rows for eight rows per warp (the grid covers the GPU twice) equal the same prompt in small portions"""
    cfg = O.make_config([D(heads=12, dim=8, rot_dim=4, vdim=8, kv_rank=12, size=100, mlp=None), G(heads=12, dim=8, rot_dim=4, vdim=40, kv_rank=16, q_rank=16, size=0, mlp=None)],
                        width=32, vocab=60)
    n = 900
    toks = tokens_for(cfg, n, seed=7)
    W = O.random_weights(cfg, seed=3, gain=1.5)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32", max_tokens=n)
    want = [0, 63, 64, 99, 100, 101, 639, 640, 898, 899]
    whole = m.forward_tokens(toks, 0, want)
    m.set_option("chunk_rows", 50)
    assert O.rel_rms(m.forward_tokens(toks, 0, want), whole) < 2e-5
    near, _ = O.forward(cfg, W, toks[:102])
    assert O.rel_rms(whole[:6], near[want[:6]]) < TOL["float32"]
    m.close()


def test_wanted_rows_in_any_order(gpu_lib, tmp_path):
    cfg = mixed_cfg()
    toks = tokens_for(cfg, 40)
    W = weights_for(cfg, toks, seed=4)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    idx = [39, 0, 17, 17, 5]
    assert O.rel_rms(m.forward_tokens(toks, 0, idx), want[idx]) < TOL["float32"]
    assert m.forward_tokens(toks, 0, []).shape == (0, cfg["vocab"])
    m.set_option("chunk_rows", 16)
    assert O.rel_rms(m.forward_tokens(toks, 0, idx), want[idx]) < TOL["float32"]
    m.close()


def one_key_attention(kind, window, seed=7):
    """one layer in which the query of token 49 and the key of token 48 share an unrotated dimension of head 0 that no other token uses:
    input dimension 0 is private to token 49 and seen by the queries only, dimension 1 is private to token 48 and seen by one channel
    of the key/value latent only, which feeds the keys and not the values"""
    make = D if kind == "direct" else G
    cfg = O.make_config([make(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=24, size=window, scale=0.25, mlp=None)], width=16, vocab=50)
    W = O.random_weights(cfg, seed=seed)
    p = "l0.mix."
    W["embed"][:, :2] = 0.0
    W["embed"][49, 0], W["embed"][48, 1] = 8.0, 8.0
    W["final.norm"][:2] = -1.0   # the private dimensions do not reach the logits
    for name in ("dkv", "q", "dq", "g"):
        if p + name in W:
            W[p + name][:, :2] = 0.0
    W[p + "dkv"][0, 1] = 0.5
    W[p + "uk"][:, 0] = 0.0
    W[p + "uk"][3, 0] = 4.0
    W[p + "uv"][:, 0] = 0.0
    if kind == "direct":
        W[p + "q"][3, 0] = 4.0
    else:
        W[p + "dq"][0, 0] = 2.0
        W[p + "uq"][:, 0] = 0.0
        W[p + "uq"][3, 0] = 8.0
    return cfg, W


def check_one_key_matters(gpu_lib, tmp_path, cfg, W, n, places, seen):
    """The last token (49) asks for the one earlier token (48) whose key matches it.  Where `seen(place)` says the key is visible,
    taking it away must move the slow implementation's answer a lot (the case has teeth); where it is not, the answer must not
    depend on it.  The library must agree in a prompt, in decoding and in portions."""
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32", max_tokens=n + 8)
    for far in places:
        toks = [t if t < 48 else 0 for t in tokens_for(cfg, n, seed=far)]
        toks[far], toks[n - 1] = 48, 49
        want, _ = O.forward(cfg, W, toks)
        toks2 = list(toks)
        toks2[far] = 0
        moved = O.rel_rms(O.forward(cfg, W, toks2)[0][n - 1], want[n - 1])
        if seen(far):
            assert moved > 100 * TOL["float32"], f"key at {far}: the case has no teeth ({moved})"
        else:
            assert moved < 1e-9, f"key at {far} should be invisible"
        got = m.forward_tokens(toks, 0, [n - 1])
        assert O.rel_rms(got[0], want[n - 1]) < TOL["float32"], f"key at {far} (prompt)"
        m.forward_tokens(toks[:n - 1], 0, [])
        assert O.rel_rms(m.forward(toks[n - 1], n - 1), want[n - 1]) < TOL["float32"], f"key at {far} (decoded)"
        # the prompt cut right behind the key, two tokens before the end, and a last portion in the per-head form
        for cut in (far + 1, n - 2, n - 20):
            if 0 < cut < n:
                m.forward_tokens(toks[:cut], 0, [])
                assert O.rel_rms(m.forward_tokens(toks[cut:], cut, [n - 1 - cut])[0], want[n - 1]) < TOL["float32"], f"key at {far}, cut at {cut}"
        # many decoded tokens: the window passes over them
        m.forward_tokens(toks[:far + 1], 0, [])
        for i in range(far + 1, n):
            lg = m.forward(toks[i], i)
        if far < n - 1:
            assert O.rel_rms(lg, want[n - 1]) < TOL["float32"], f"key at {far}, everything behind it decoded"
    m.close()


@pytest.mark.parametrize("kind", ["direct", "gated"])
@pytest.mark.parametrize("window", [1, 7, 64, 65, 100])
def test_keys_just_inside_and_just_outside_the_window(gpu_lib, tmp_path, kind, window):
    cfg, W = one_key_attention(kind, window)
    n = 200
    last = n - 1
    places = sorted({p for p in (last - window - 1, last - window, last - window + 1, last - window + 2, last - 1) if 0 <= p < last})
    check_one_key_matters(gpu_lib, tmp_path, cfg, W, n, places, seen=lambda p: last - p < window)


@pytest.mark.parametrize("kind", ["direct", "gated"])
def test_a_far_key_is_found_among_hundreds(gpu_lib, tmp_path, kind):
    """windows of 300 and none: keys at tile borders, the very first token, the edge"""
    n = 330
    cfg, W = one_key_attention(kind, 0, seed=8)
    check_one_key_matters(gpu_lib, tmp_path, cfg, W, n, [0, 1, 63, 64, 192], seen=lambda p: True)
    cfg, W = one_key_attention(kind, 300, seed=8)
    check_one_key_matters(gpu_lib, tmp_path, cfg, W, n, [29, 30, 63, 64], seen=lambda p: p >= 30)


def test_the_cache_is_reused_by_the_next_sequence(gpu_lib, tmp_path):
    cfg = mixed_cfg()
    a, b = tokens_for(cfg, 90, seed=1), tokens_for(cfg, 33, seed=2)
    W = weights_for(cfg, a + b, seed=6)
    wa, _ = O.forward(cfg, W, a)
    wb, _ = O.forward(cfg, W, b)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    assert O.rel_rms(m.forward_tokens(a, 0, [89]), wa[[89]]) < TOL["float32"]
    # a shorter sequence over the same positions: nothing of `a` (latents beyond position 32) may show
    assert O.rel_rms(m.forward_tokens(b[:20], 0, [0, 19]), wb[[0, 19]]) < TOL["float32"]
    for i in range(20, 33):
        assert O.rel_rms(m.forward(b[i], i), wb[i]) < TOL["float32"]
    assert O.rel_rms(m.forward_tokens(a, 0, [0, 50]), wa[[0, 50]]) < TOL["float32"]
    # a new sequence that starts with single tokens (the first tokens of a sequence, decoded)
    for i in range(5):
        assert O.rel_rms(m.forward(b[i], i), wb[i]) < TOL["float32"]
    # everything is addressed by position: a step may go back and continue from there
    m.forward_tokens(a, 0, [])
    assert O.rel_rms(m.forward_tokens(a[40:60], 40, [0, 19]), wa[[40, 59]]) < TOL["float32"]
    m.close()


def test_first_tokens_and_a_prompt_of_one(gpu_lib, tmp_path):
    cfg = mixed_cfg()
    W = weights_for(cfg, [7, 7, 0, 1, 2], seed=8)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    for toks in ([7], [7, 7], [0, 1, 2]):
        want, _ = O.forward(cfg, W, toks)
        assert O.rel_rms(m.forward_tokens(toks, 0, list(range(len(toks)))), want) < TOL["float32"]
        assert O.rel_rms(m.forward(toks[0], 0), want[0]) < TOL["float32"]
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_greedy_generation_through_the_generate_loop(gpu_lib, tmp_path, dtype):
    cfg = mixed_cfg(dtype)
    W = O.random_weights(cfg, seed=9)
    prompt = tokens_for(cfg, 21, seed=4)
    n_new = 150   # decodes across two key-tile borders, through several key splits, and the windows pass over decoded tokens
    m = open_model(gpu_lib, tmp_path, cfg, W, dtype, max_tokens=21 + n_new)
    m.forward_tokens(prompt[:-1], 0, [])
    ids = m.generate_greedy(prompt[-1], len(prompt) - 1, n_new).tolist()
    assert len(ids) == n_new
    if dtype == "float32":
        # replay the produced sequence through the slow implementation: every pick must be its argmax or within a hair of it,
        # up to the first routing decision too close to call
        inc = O.StepOracle(cfg, W)
        want = inc.step(prompt)[0][-1:]
        checked = 0
        for t in ids:
            assert want[0, t] >= want[0].max() - 1e-3 * (want[0].max() - want[0].min()), f"generated token {checked}"
            checked += 1
            del O.CHOICE_GAPS[:]
            want = inc.step([t])[0]
            if any(g < 1e-6 for g in O.CHOICE_GAPS):
                break
        assert checked > 20
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


def test_long_decoding_with_a_latent_that_is_always_up_projected(gpu_lib, tmp_path):
    """a latent too wide for the shared-head tiles: a one-row step up-projects what its 64-position bucket can see, graph-replayed"""
    cfg = O.make_config([G(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=528, q_rank=16, size=70, mlp=None), D(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=520, size=9, mlp=None)],
                        width=24, vocab=40)
    W = O.random_weights(cfg, seed=4, gain=1.5)
    toks = tokens_for(cfg, 230, seed=9)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32", max_tokens=231)
    m.forward_tokens(toks[:40], 0, [])
    for i in range(40, 230):
        lg = m.forward(toks[i], i)
        if i % 16 in (0, 15):
            assert O.rel_rms(lg, want[i]) < TOL["float32"], f"decoded position {i}"
    m.close()


TC_LAYERS = [
    D(heads=5, dim=24, rot_dim=8, vdim=24, kv_rank=40, size=50, mlp=O.dense(ff=200)),
    G(heads=6, dim=32, rot_dim=16, vdim=20, kv_rank=48, q_rank=56, size=100, mlp=M(7, 2, 2, ff=72, shared=56, groups=3, keep=2)),
    D(heads=4, dim=24, rot_dim=8, vdim=40, kv_rank=32, size=0, mlp=M(9, 0, 4, ff=40, shared=0, groups=3, keep=3)),
    G(heads=3, dim=16, rot_dim=24, vdim=24, kv_rank=24, q_rank=40, size=33, mlp=M(3, 1, 1, ff=200, shared=24, groups=2, keep=1)),
]


@pytest.mark.parametrize("layer", range(len(TC_LAYERS)))
def test_tensor_core_products_equal_the_cuda_core_products(gpu_lib, tmp_path, layer):
    """bf16 mode, shapes that are no multiples of the 128 x 128 x 64 tile, experts with very unequal loads: rows, outputs and
    K tails are masked or zero-filled, group borders fall inside tiles; biases of the dense layer in both kernels' epilogues.
    One layer at a time: a sum in another order may round an operand of the next product the other way, which deeper layers spread"""
    cfg = O.make_config([TC_LAYERS[layer]], width=72, vocab=203)
    toks = tokens_for(cfg, 300)
    W = O.random_weights(cfg, seed=10)
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "bfloat16", max_tokens=320)
    a = m.forward_tokens(toks, 0, list(range(300)))
    m.set_option("tensor_cores", 0)
    b = m.forward_tokens(toks, 0, list(range(300)))
    assert typical_row_close(a, b, 1e-3) and not np.array_equal(a, b)   # different kernels, same numbers up to summation order
    assert typical_row_close(a, want, TOL["bfloat16"]) and typical_row_close(b, want, TOL["bfloat16"])
    m.close()


def test_a_group_that_is_out_stays_out_when_all_scores_are_negative(gpu_lib, tmp_path):
    """corrections far below zero: a masked group counts as minus infinity; counting it as zero would make it win"""
    cfg = O.make_config([D(size=300, mlp=M(6, 2, 2, groups=4, keep=2))])
    toks = tokens_for(cfg, 60, seed=1)
    for seed in range(20, 60):
        W = O.random_weights(cfg, seed=seed, gain=1.5)
        W["l0.mlp.correction"] = O.bf16_round(np.array([-3.0, -2.0, -2.75, -2.25, -2.0, -3.0, -2.5, -2.25]) + 0.05 * W["l0.mlp.correction"])
        if O.clear_choices(cfg, W, toks, GAP):
            break
    else:
        raise AssertionError("no seed without a close routing decision")
    want, _ = O.forward(cfg, W, toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    assert O.rel_rms(m.forward_tokens(toks, 0, list(range(60))), want) < TOL["float32"]
    m.forward_tokens(toks[:59], 0, [])
    assert O.rel_rms(m.forward(toks[59], 59), want[59]) < TOL["float32"]
    m.close()


def test_configuration_errors_are_reported(gpu_lib, tmp_path):
    cfg = mixed_cfg()
    W = O.random_weights(cfg)
    for i, gone in enumerate(("l1.mix.g", "l0.mlp.down.b", "l1.mlp.shared.sg", "l3.mix.dq.norm")):
        with pytest.raises(gpu_lib.LmrsError, match=gone):
            gpu_lib.Transformer.open(O.write_model(str(tmp_path / f"b{i}"), cfg, {k: v for k, v in W.items() if k != gone}))
    W3 = dict(W)
    W3["l1.mlp.e3.down"] = W["l1.mlp.e3.down"][:, :-1]
    with pytest.raises(gpu_lib.LmrsError, match="l1.mlp.e3.down"):
        gpu_lib.Transformer.open(O.write_model(str(tmp_path / "c"), cfg, W3))
    for i, (layer, msg) in enumerate(((dict(D(), type="no_such_mixer"), "no_such_mixer"), (D(mlp={"kind": "sparse", "ff": 8}), "sparse"),
                                      (D(mlp=M(7, 1, 3, groups=3)), "groups"), (D(mlp=M(4, 2, 3, groups=3, keep=1)), "top"), (D(rot_dim=7), "rot"))):
        bad = O.make_config([layer])
        with pytest.raises(gpu_lib.LmrsError, match=msg):
            gpu_lib.Transformer.open(O.write_model(str(tmp_path / f"d{i}"), bad, O.random_weights(O.make_config([D()]))))
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32", max_tokens=16)
    with pytest.raises(gpu_lib.LmrsError):
        m.forward_tokens([1] * 17, 0, [])
    with pytest.raises(gpu_lib.LmrsError, match="token"):
        m.forward_tokens([cfg["vocab"]], 0, [])
    m.close()


def test_cached_rows_can_be_read_back(gpu_lib, tmp_path):
    cfg = O.make_config([D(mlp=None), G(mlp=None)])
    W = O.random_weights(cfg, seed=3)
    toks = tokens_for(cfg, 12)
    st = O.StepOracle(cfg, W)
    st.step(toks)
    m = open_model(gpu_lib, tmp_path, cfg, W, "float32")
    m.forward_tokens(toks, 0, [])
    for li, (rk, dr) in enumerate(((20, 8), (24, 12))):   # the latent and the rotated key part
        c, kr = m.read_kv(li, 0, 12, k_cols=rk, v_cols=dr)
        assert np.allclose(c, st.state[li]["c"], atol=1e-4) and np.allclose(kr, st.state[li]["kr"], atol=1e-4)
    m.close()


def test_the_command_line_generates_from_a_folder(gpu_lib, tmp_path):
    """lm.rs_b200/examples/generate on a model folder prints the ids that generate_greedy picks"""
    subprocess.check_call(["make", "-C", os.path.join(ROOT, "lm.rs_b200"), "-s", "examples"])
    cfg = mixed_cfg()
    d = O.write_model(str(tmp_path / "cli"), cfg, O.random_weights(cfg, seed=11))
    prompt = [3, 9, 27, 20]
    r = subprocess.run([os.path.join(ROOT, "lm.rs_b200", "examples", "generate"), d, "10"] + [str(t) for t in prompt],
                       capture_output=True, text=True, env=dict(os.environ, GENERATE_DTYPE="float32"))
    assert r.returncode == 0, r.stderr
    m = gpu_lib.Transformer.open(d, dtype="float32", max_tokens=32)
    m.forward_tokens(prompt[:-1], 0, [])
    assert [int(x) for x in r.stdout.split()] == m.generate_greedy(prompt[-1], 3, 10).tolist()
    m.close()


def test_trace_replay_writes_the_logits_asked_for(gpu_lib, tmp_path):
    """bin/trace_run: a prompt in portions, then single tokens, then a second request over the same cache"""
    cfg = mixed_cfg()
    a, b = tokens_for(cfg, 75, seed=5), tokens_for(cfg, 9, seed=6)
    W = weights_for(cfg, a + b, seed=12)
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
