"""The slow Lutesun implementation of tests/lutesun_oracle.py against itself and against hand-made cases (no GPU): whole-sequence
arithmetic == the same fed in portions, and each mechanism on inputs whose answer is known in closed form.  The packaged model
writer is checked against this file's tensor table."""
import json
import math
import struct

import numpy as np
import pytest

import lutesun_oracle as O


def small_cfg():
    return O.make_config([
        O.direct_layer(mlp=O.dense()),
        O.gated_layer(),
        O.direct_layer(heads=2, size=30, mlp=None),
        O.gated_layer(heads=1, size=1, mlp=O.moe(experts=4, identity=0, top=2, shared=0, groups=1, keep=1)),
    ], width=24, vocab=37)


def test_whole_sequence_equals_portions_and_single_tokens():
    cfg = small_cfg()
    W = O.random_weights(cfg, seed=3)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 23).tolist()
    whole, outs = O.forward(cfg, W, toks)
    assert outs.shape == (4, 23, 24)
    for cuts in ([1] * 23, [2, 3, 5, 7, 2, 4], [22, 1]):
        inc, got, at = O.StepOracle(cfg, W), [], 0
        for c in cuts:
            got.append(inc.step(toks[at:at + c])[0])
            at += c
        assert np.allclose(np.concatenate(got), whole, rtol=0, atol=1e-9)


def test_norm_weight_is_stored_around_zero():
    x = np.array([[3.0, 4.0]])
    r = math.sqrt(12.5)
    assert np.allclose(O.offset_norm(x, np.array([0.0, 1.0]), 0.0), [[3.0 / r, 8.0 / r]])
    assert np.allclose(O.offset_norm(x, np.array([-1.0, 0.0]), 12.5), [[0.0, 4.0 / 5.0]])   # eps inside the root


def test_the_two_rotation_layouts():
    z = np.arange(1.0, 7.0).reshape(1, 6)
    rot = {"base": 100.0, "dims": 4}   # frequencies 1 and 0.1
    a, b = 3.0, 0.3
    turn = lambda u, v, t: (u * math.cos(t) - v * math.sin(t), v * math.cos(t) + u * math.sin(t))
    p = O.turned(z, [3], rot, False)[0]
    assert np.allclose(p, [*turn(1, 2, a), *turn(3, 4, b), 5, 6])
    h = O.turned(z, [3], rot, True)[0]
    u, v = turn(1, 3, a), turn(2, 4, b)
    assert np.allclose(h, [u[0], v[0], u[1], v[1], 5, 6])
    assert np.allclose(O.turned(z, [0], rot, True), z)
    # heads in between, two positions
    z3 = np.stack([z, 2 * z])
    assert np.allclose(O.turned(z3, [3, 0], rot, False), np.stack([[p], 2 * z]))


def test_window_counts_the_token_itself():
    assert [j for j in range(8) if O.visible(5, j, {"size": 3})] == [3, 4, 5]
    assert [j for j in range(8) if O.visible(5, j, {"size": 1})] == [5]
    assert [j for j in range(8) if O.visible(5, j, None)] == [0, 1, 2, 3, 4, 5]


@pytest.mark.parametrize("kind", ["latent_attention", "latent_attention_2"])
def test_latent_attention_against_explicit_heads(kind):
    make = O.direct_layer if kind == "latent_attention" else O.gated_layer
    cfg = O.make_config([make(heads=2, dim=4, rot_dim=4, vdim=6, kv_rank=5, size=3, mlp=None)], width=8, vocab=5)
    W = O.random_weights(cfg, seed=3)
    m, p = cfg["layers"][0]["mixer"], "l0.mix."
    h = np.random.default_rng(1).standard_normal((6, 8))
    st = {}
    y = O.latent_mixer(h, W, p, kind, m, 1e-5, st, 0)
    assert st["c"].shape == (6, 5) and st["kr"].shape == (6, 4)
    raw = h @ W[p + "dkv"].T
    c = raw[:, :5] / np.sqrt((raw[:, :5] ** 2).mean(1, keepdims=True) + 1e-5) * W[p + "dkv.norm"]
    kr = O.turned(raw[:, 5:], range(6), m["rot"], kind == "latent_attention_2")   # the rotated part is not normed
    if kind == "latent_attention":
        q = h[5] @ W[p + "q"].T
    else:
        cq = h[5] @ W[p + "dq"].T
        q = (cq / np.sqrt((cq ** 2).mean() + 1e-5) * W[p + "dq.norm"]) @ W[p + "uq"].T
    out = []
    for hd in range(2):
        qn, qr = q[hd * 8:hd * 8 + 4], O.turned(q[None, hd * 8 + 4:hd * 8 + 8], [5], m["rot"], kind == "latent_attention_2")[0]
        s = np.array([qn @ (W[p + "uk"][hd * 4:(hd + 1) * 4] @ c[j]) + qr @ kr[j] for j in (3, 4, 5)]) * m["scale"]
        a = np.exp(s) / np.exp(s).sum()
        o = sum(w * (W[p + "uv"][hd * 6:(hd + 1) * 6] @ c[j]) for w, j in zip(a, (3, 4, 5)))
        if kind == "latent_attention_2":
            o = o / (1.0 + math.exp(-(W[p + "g"][hd] @ h[5])))
        out.append(o)
    assert np.allclose(y[5], W[p + "o"] @ np.concatenate(out))


def test_dense_feed_forward_squares_and_has_both_biases():
    W = {"p.up": np.array([[1.0, 0.0], [0.0, 1.0]]), "p.up.b": np.array([1.0, -3.0]), "p.down": np.array([[1.0, 1.0]]), "p.down.b": np.array([0.5])}
    assert np.allclose(O.dense_ff(np.array([[2.0, 1.0]]), W, "p."), [[9.5]])      # (2 + 1)^2 + relu(1 - 3)^2 + 0.5
    assert np.allclose(O.dense_ff(np.array([[-2.0, 5.0]]), W, "p."), [[4.5]])


def test_router_groups_correction_and_weights():
    """six outputs in three groups; two groups are kept"""
    r = {"experts": 5, "identity": 1, "top": 3, "scale": 2.0, "groups": {"count": 3, "keep": 2}}
    W = {"p.router": np.eye(6), "p.correction": np.array([0.0, 0.0, -0.9, -0.9, 0.0, 0.0])}
    h = np.log(np.array([[0.1, 0.15, 0.4, 0.2, 0.06, 0.09]]))
    idx, w = O.route(h, W, "p.", r)
    # softmax scores are the numbers above; the middle group's corrected scores are -0.5 and -0.7, so it is out whatever its scores
    assert idx[0].tolist() == [1, 0, 5]
    s = np.array([0.15, 0.1, 0.09])
    assert np.allclose(w[0], s / s.sum() * 2.0)
    # all choice scores negative: a group that is out counts as minus infinity, not as zero
    W["p.correction"] = W["p.correction"] - 1.0
    assert O.route(h, W, "p.", r)[0][0].tolist() == [1, 0, 5]
    # one group: the correction decides inside it and does not enter the weights
    r1 = {"experts": 6, "top": 2, "scale": 1.0, "groups": {"count": 1, "keep": 1}}
    W["p.correction"] = np.array([0.0, 0.0, 0.0, 0.0, 5.0, 0.0])
    idx, w = O.route(h, W, "p.", r1)
    assert idx[0].tolist() == [4, 2] and np.allclose(w[0], np.array([0.06, 0.4]) / 0.46)


def test_identity_experts_and_the_gated_shared_expert():
    f = O.moe(experts=1, identity=2, top=2, ff=3, shared=2, groups=1, keep=1, scale=3.0)
    W = {"p.router": np.array([[-40.0, 0.0], [1.0, 0.0], [1.0, 0.0]]), "p.correction": np.zeros(3)}
    for e, n in (("e0", 3), ("shared", 2)):
        W.update({f"p.{e}.gate": np.ones((n, 2)), f"p.{e}.up": np.ones((n, 2)), f"p.{e}.down": np.ones((2, n))})
    W["p.shared.sg"] = np.array([[0.0, 2.0]])
    h = np.array([[1.0, 0.25]])
    z = 1.25
    shared = 2 * z * z / (1 + math.exp(-z)) / (1 + math.exp(-0.5))
    assert np.allclose(O.routed_ff(h, W, "p.", f), 3.0 * h + shared)   # both identity experts: their weights sum to the scale


def test_embedding_scale_and_tied_head():
    cfg = O.make_config([O.direct_layer(mlp=None)], width=24, vocab=11, embed_scale=0.5)
    W = O.random_weights(cfg, seed=5)
    W["l0.norm1"][:] = -1.0   # the mixer adds nothing
    lg, outs = O.forward(cfg, W, [3, 4])
    assert np.allclose(outs[0], 0.5 * W["embed"][[3, 4]])
    x = outs[0][0]
    assert np.allclose(lg[0], W["embed"] @ (x / np.sqrt((x * x).mean() + 1e-5) * (1.0 + W["final.norm"])))


def test_write_model_layout(tmp_path):
    cfg = small_cfg()
    W = O.random_weights(cfg, seed=4)
    d = O.write_model(str(tmp_path / "m"), cfg, W)
    raw = open(d + "/model.safetensors", "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    hdr = json.loads(raw[8:8 + n])
    assert n % 8 == 0 and set(hdr) == set(W)
    e = hdr["l1.mlp.shared.sg"]
    assert e["dtype"] == "BF16" and e["shape"] == [1, 24]
    bits = np.frombuffer(raw[8 + n + e["data_offsets"][0]:8 + n + e["data_offsets"][1]], np.uint16)
    assert np.array_equal((bits.astype(np.uint32) << 16).view(np.float32).reshape(1, 24), W["l1.mlp.shared.sg"].astype(np.float32))
    assert json.load(open(d + "/config.json"))["layers"][1]["type"] == "latent_attention_2"


def test_the_packaged_writer_names_the_same_tensors():
    """lmrs_b200.model_dir (random models for benchmarks) and this file's table agree on names and shapes"""
    from lmrs_b200 import model_dir as md
    cfg = md.lutesun_config(48, 4, 90, heads=3, head_dim=8, rot_dim=6, vdim=10, kv_rank=20, q_rank=28, window=12, ff=40, experts=4, identity=2, top=2,
                            groups=3, keep=2, expert_ff=24, shared_ff=16)
    assert [L["type"] for L in cfg["layers"]] == ["latent_attention", "latent_attention_2"] * 2
    assert [L["mlp"]["kind"] for L in cfg["layers"]] == ["dense", "moe", "moe", "moe"]
    a = {n: tuple(s) for n, s, _ in md.lutesun_tensors(cfg)}
    assert a == {n: tuple(s) for n, s, _ in O.tensor_table(cfg)}
    # the chosen experts' share of the expert matrices, everything else once, one more row of the table for the embedding
    rest = sum(int(np.prod(s)) for n, s in a.items() if ".mlp.e" not in n)
    experts = sum(int(np.prod(s)) for n, s in a.items() if ".mlp.e" in n)
    assert abs(md.lutesun_param_bytes(cfg) - (rest + 48 + experts * 2 / 6) * 2) <= 1
    assert md.lutesun_mixer_flops(cfg, 12) == 4 * 2 * 3 * 24 * 78 and md.lutesun_mixer_flops(cfg, 13) == 4 * 2 * 3 * 24 * 90
    logits, _ = O.forward(cfg, O.random_weights(cfg, seed=1), [1, 2, 3])
    assert logits.shape == (3, 90) and np.isfinite(logits).all()
