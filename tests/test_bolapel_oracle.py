"""The slow float64 implementation of the Bolapel architecture (tests/bolapel_oracle.py) pinned on cases worked out by hand,
and its incremental form against its whole-sequence form.  No GPU."""
import math

import numpy as np

import bolapel_oracle as O


def test_rms_has_eps_inside_the_root():
    assert np.allclose(O.rms(np.array([3.0, 4.0]), 0.5), np.array([3.0, 4.0]) / math.sqrt(12.5 + 0.5))


def test_token_shift_mixes_with_the_row_before_as_it_was():
    h = np.array([[2.0, 10.0], [4.0, 20.0], [8.0, 30.0]])
    out, last = O.token_shift(h, np.array([0.5, 0.0]), np.zeros(2))
    # first channel: half way to the previous row (not to its mixed version); second channel: untouched
    assert np.allclose(out, [[1.0, 10.0], [3.0, 20.0], [6.0, 30.0]]) and np.allclose(last, [8.0, 30.0])
    out2, _ = O.token_shift(h[1:], np.array([1.0, 1.0]), h[0])
    assert np.allclose(out2, h[:2])


def test_decay_lies_between_its_two_ends():
    z = np.array([-60.0, 0.0, 60.0])
    assert np.allclose(O.channel_decay(z), [1.0, math.exp(-0.5 * math.exp(-0.5)), math.exp(-math.exp(-0.5))])


def scan(r, k, v, w, a, S):
    f = lambda x: np.asarray(x, np.float64)[:, None, :]
    return O.general_delta_scan(f(r), f(k), f(v), f(w), f(a), S)[:, 0]


def test_write_decay_and_read():
    S = np.zeros((1, 2, 2))
    # no removal: two writes under different keys, channel decays 1 and 1/2, then a read of both rows
    o = scan([[0, 0], [0, 0], [1, 1]], [[1, 0], [0, 1], [0, 0]], [[2, 0], [0, 3], [0, 0]], [[1, 1], [1, 1], [1, 0.5]], np.zeros((3, 2)), S)
    assert np.allclose(S[0], [[2, 0], [0, 1.5]]) and np.allclose(o[2], [2, 1.5])


def test_removal_acts_on_the_unit_key_and_reads_the_old_state():
    S = np.array([[[8.0, 4.0], [1.0, 1.0]]])
    # key (2, 0): unit length (1, 0).  Removal rate 3/4 in its channel, decay 1/2: 8 -> 8/2 - 3/4 * 8 + 2 * v
    o = scan([[1, 0]], [[2, 0]], [[5, 0]], [[0.5, 1.0]], [[0.75, 0.3]], S)
    u2 = 4.0 / (4.0 + 1e-6)   # squared length of the unit key
    assert np.allclose(S[0, 0], [4.0 - 0.75 * 8.0 * u2 + 10.0, 2.0 - 0.75 * 4.0 * u2])
    assert np.allclose(S[0, 1], [1.0, 1.0])         # the key has nothing in channel 1: no removal there
    assert np.allclose(o[0], S[0, 0])               # the read-out sees the token's own write


def test_removal_rate_differs_by_channel():
    S = np.array([[[1.0, 0.0], [1.0, 0.0]]])
    k = np.array([1.0, 1.0])
    held = (1.0 + 1.0) / math.sqrt(2.0 + 1e-6)
    scan([[0, 0]], [k], [[0, 0]], [[1, 1]], [[1.0, 0.0]], S)
    assert np.allclose(S[0, :, 0], [1.0 - held / math.sqrt(2.0 + 1e-6), 1.0])


def test_rotation_pairs_the_two_halves():
    rot = {"dims": 4, "base": 100.0}
    x = np.zeros((2, 1, 6))
    x[:, 0] = [1.0, 0.0, 0.0, 2.0, 5.0, 6.0]
    out = O.rotate_half(x, [0, 3], rot)
    assert np.allclose(out[0], x[0])
    f1 = 100.0 ** (-2.0 / 4.0)
    assert np.allclose(out[1, 0, [0, 2]], [math.cos(3.0), math.sin(3.0)])                          # dimension 0 with 2
    assert np.allclose(out[1, 0, [1, 3]], [-2.0 * math.sin(3.0 * f1), 2.0 * math.cos(3.0 * f1)])   # dimension 1 with 3
    assert np.allclose(out[1, 0, 4:], [5.0, 6.0])


def test_blocks_are_counted_from_position_zero():
    m = {"size": 3}
    assert [j for j in range(8) if O.same_block(5, j, m)] == [3, 4, 5]
    assert [j for j in range(8) if O.same_block(6, j, m)] == [6]
    assert [j for j in range(8) if O.same_block(4, j, None)] == [0, 1, 2, 3, 4]
    assert [j for j in range(8) if O.same_block(4, j, {"size": 1})] == [4]


def test_weights_are_independent_sigmoids():
    w = O.sigmoid_weights(np.array([0.0, math.log(3.0), -80.0]), 0.0)
    assert np.allclose(w, [0.5, 0.75, 0.0])
    assert np.allclose(O.sigmoid_weights(np.array([1.0, 1.0]), -1.0), [0.5, 0.5])   # the bias adds to the score


def test_attention_by_hand():
    """one head of size 1, no rotation: q and k are +-1 after their norm, so every weight is sigmoid(scale * +-1 + bias)"""
    cfg = O.make_config([O.attention_layer(heads=1, kv_heads=1, dim=1, vdim=1, size=2, rot_dims=0, scale=2.0, mlp=None)], width=2)
    W = {k: np.zeros(s) for k, s, _ in O.tensor_table(cfg)}
    p = "l0.mix."
    W[p + "q"][:] = [[1.0, 0.0]]; W[p + "k"][:] = [[1.0, 0.0]]; W[p + "v"][:] = [[0.0, 1.0]]; W[p + "o"][:] = [[0.0], [1.0]]
    W[p + "q.norm"][:] = 1.0; W[p + "k.norm"][:] = 1.0; W[p + "pb"][:] = -0.5
    h = np.array([[1.0, 10.0], [-1.0, 20.0], [1.0, 30.0]])
    out = O.attention_mixer(h, W, p, cfg["layers"][0]["mixer"], 0.0, {}, 0)
    near, far = O.sigmoid(2.0 - 0.5), O.sigmoid(-2.0 - 0.5)
    assert np.allclose(out[:, 1], [0.5 * near * 10.0, 0.5 * (far * 10.0 + near * 20.0), 0.5 * near * 30.0])   # gate sigmoid(0) = 1/2; row 2 opens a block


def test_soft_cap():
    assert np.allclose(O.soft_cap(np.array([0.0, 1e9]), 5.0), [0.0, 5.0]) and O.soft_cap(3.0, None) == 3.0


def mixed_cfg():
    return O.make_config([
        O.delta_layer(),
        O.attention_layer(size=9),
        O.delta_layer(heads=2, dim=20, rank=3, mlp=None),
        O.attention_layer(size=7, kv_from=1, heads=6, scale=0.7),
    ])


def test_whole_sequence_portions_and_single_tokens_agree():
    cfg = mixed_cfg()
    W = O.random_weights(cfg, seed=1)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 40).tolist()
    want, outs = O.forward(cfg, W, toks)
    for cuts in ([1] * 40, [2] * 20, [7, 1, 30, 2], [39, 1]):
        st, at, rows, lay = O.StepOracle(cfg, W), 0, [], []
        for c in cuts:
            lg, lo = st.step(toks[at:at + c])
            rows.append(lg); lay.append(lo); at += c
        assert np.allclose(np.concatenate(rows), want, atol=1e-9)
        assert np.allclose(np.concatenate(lay, 1), outs, atol=1e-9)


def test_a_borrowing_layer_reads_the_lender_and_has_no_keys_of_its_own():
    cfg = mixed_cfg()
    names = {n for n, _, _ in O.tensor_table(cfg)}
    assert "l1.mix.k" in names and not {"l3.mix.k", "l3.mix.v", "l3.mix.k.norm"} & names and "l3.mix.q.norm" in names
    W = O.random_weights(cfg, seed=2)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 12).tolist()
    _, a = O.forward(cfg, W, toks)
    W["l1.mix.v"] = W["l1.mix.v"] * 2.0
    _, b = O.forward(cfg, W, toks)
    st = O.StepOracle(cfg, W)
    st.step(toks)
    assert "k" not in st.state[3] and np.abs(a[3] - b[3]).max() > 1e-3


def test_packaged_writer_and_slow_implementation_agree_on_names_and_shapes():
    from lmrs_b200 import model_dir as md
    cfg = md.bolapel_config(64, 6, 50, heads=4, kv_heads=2, head_dim=8, vdim=12, chunk=16, rot_dims=4, delta_heads=3, delta_dim=10, rank=4, ff=48,
                            pattern=("general_delta", "attention", "general_delta"))
    assert [L["mixer"].get("kv_from") for L in cfg["layers"]] == [None, None, None, None, 1, None]
    a = {n: tuple(s) for n, s, _ in md.bolapel_tensors(cfg)}
    b = {n: tuple(s) for n, s, _ in O.tensor_table(cfg)}
    assert a == b
    assert all("rank" not in L["mixer"] for L in md.written_bolapel_config(cfg)["layers"])
    assert md.bolapel_param_bytes(cfg) > 0 and md.bolapel_matmul_flops_per_token(cfg) > 0 and md.bolapel_mixer_flops(cfg, 64) > 0
