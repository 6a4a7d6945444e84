"""Plain, slow float64 implementation of the Lutesun architecture: test infrastructure only.

One function per mechanism, written from the equations below in numpy; it shares no code with the library.

    embedding      x = scale * E[token]
    layer          x <- x + N1(mixer(x));  x <- x + N2(ff(x))    (the sublayers read x itself; the second line only with a
                   feed-forward);  N(y) = rms(y) * (1 + w)
    rms(v)         v / sqrt(mean(v^2) + eps)
    mixers         attention through a latent, one latent row and one turned key row cached per token (latent_*):
                     [c_raw | kr] = W_dkv h;  c = rms(c_raw) * w_dkv;  kr turned by its position
                     "latent_attention"     q = W_q h, turned in neighbouring pairs (2i, 2i+1)
                     "latent_attention_2"   q = W_uq (rms(W_dq h) * w_dq), turned in halves (i, i + dims/2); every head's output
                                            times sigmoid(W_g h)_head
                     head: k_j = [W_uk c_j | kr_j],  v_j = W_uv c_j,  s_ij = scale * q_i . k_j for 0 <= i - j < size;  softmax;
                     W_o over all heads
    ff dense       W_down relu(W_up h + b_up)^2 + b_down
    ff routed      s = softmax(W_r h) over experts and identity experts;  t = s + correction;  outputs lie in `count` equal
                   neighbouring groups, a group scores its largest t, only the `keep` best groups may be chosen from;  the `top`
                   largest t are chosen;  weights = s_chosen / (sum s_chosen + 1e-20) * scale;  expert(h) = W_down (silu(W_gate h)
                   * (W_up h));  an identity expert returns h;  a shared expert of the same form, times sigmoid(w_sg . h), is added
    logits         E N_final(x)          (the embedding table without its scale)

StepOracle carries the cached rows from call to call, so whole sequences and the incremental form check each other.
make_config / random_weights / write_model build small random model folders (config.json + model.safetensors, bf16 tensors).
"""
import json
import math
import os
import struct

import numpy as np


# ---- number formats -----------------------------------------------------------------------------------------------------
def to_bf16_bits(a):
    u = np.asarray(a, np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_round(a):
    return (to_bf16_bits(a).astype(np.uint32) << 16).view(np.float32).astype(np.float64)


# ---- small functions --------------------------------------------------------------------------------------------------------
def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def offset_norm(x, w, eps):
    """the weight is stored around zero"""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ---- rotation ---------------------------------------------------------------------------------------------------------------
def turned(x, positions, rot, halves):
    """x [T, ..., n >= dims]: dimension pairs turned by position * base^(-2i/dims); pair i is (2i, 2i+1), or (i, i + dims/2) when
    `halves`; the remaining dimensions are kept"""
    d = rot["dims"]
    out = np.array(x, np.float64)
    for i in range(d // 2):
        a, b = (i, i + d // 2) if halves else (2 * i, 2 * i + 1)
        ang = np.asarray(positions, np.float64) * rot["base"] ** (-2.0 * i / d)
        ang = ang.reshape((-1,) + (1,) * (x.ndim - 2))
        c, s = np.cos(ang), np.sin(ang)
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


# ---- latent attention -----------------------------------------------------------------------------------------------------------
def visible(i, j, mask):
    """may position i look at position j?"""
    return j <= i and (not mask or i - j < mask["size"])


def softmax(s):
    e = np.exp(s - np.max(s, axis=-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def latent_queries(h, W, p, kind, eps):
    if kind == "latent_attention":
        return h @ W[p + "q"].T
    return (rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T


def latent_mixer(h, W, p, kind, m, eps, state, pos0):
    """state: 'c' [n, kv_rank] latents and 'kr' [n, rot_dim] turned key rows of the positions before pos0"""
    T = h.shape[0]
    H, dn, dr, dv, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(pos0, pos0 + T)
    halves = kind == "latent_attention_2"
    q = latent_queries(h, W, p, kind, eps).reshape(T, H, dn + dr)
    qn, qr = q[..., :dn], turned(q[..., dn:], pos, m["rot"], halves)
    kv = h @ W[p + "dkv"].T
    c = rms(kv[:, :rk], eps) * W[p + "dkv.norm"]
    kr = turned(kv[:, rk:], pos, m["rot"], halves)
    if "c" in state:
        c, kr = np.concatenate([state["c"], c]), np.concatenate([state["kr"], kr])
    state["c"], state["kr"] = c, kr
    k = (c @ W[p + "uk"].T).reshape(-1, H, dn)
    v = (c @ W[p + "uv"].T).reshape(-1, H, dv)
    gate = sigmoid(h @ W[p + "g"].T) if kind == "latent_attention_2" else np.ones((T, H))
    out = np.zeros((T, H, dv))
    for t in range(T):
        js = [j for j in range(pos0 + t + 1) if visible(pos0 + t, j, m.get("mask"))]
        for hh in range(H):
            s = (k[js, hh] @ qn[t, hh] + kr[js] @ qr[t, hh]) * m["scale"]
            out[t, hh] = softmax(s) @ v[js, hh] * gate[t, hh]
    return out.reshape(T, H * dv) @ W[p + "o"].T


# ---- feed-forward ---------------------------------------------------------------------------------------------------------------
def dense_ff(h, W, p):
    return np.maximum(h @ W[p + "up"].T + W[p + "up.b"], 0.0) ** 2 @ W[p + "down"].T + W[p + "down.b"]


CHOICE_GAPS = []   # margin between the last accepted and the first rejected score of every decision made (groups and experts)


def best(scores, n):
    """indices of the n largest scores (the lower index wins a tie), and the margin to the next"""
    order = np.argsort(-scores, kind="stable")
    if n < len(scores) and np.isfinite(scores[order[n]]):
        CHOICE_GAPS.append(scores[order[n - 1]] - scores[order[n]])
    return order[:n]


def route(h, W, p, r):
    """-> (chosen [T, top] indices into experts + identity experts, weights [T, top])"""
    s = softmax(h @ W[p + "router"].T)
    t = s + W[p + "correction"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    size = t.shape[1] // g["count"]
    idx = np.zeros((h.shape[0], r["top"]), np.int64)
    for i in range(h.shape[0]):
        kept = best(t[i].reshape(g["count"], size).max(-1), g["keep"])
        allowed = np.full(t.shape[1], -np.inf)
        for k in kept:
            allowed[k * size:(k + 1) * size] = t[i, k * size:(k + 1) * size]
        idx[i] = best(allowed, r["top"])
    sc = np.take_along_axis(s, idx, -1)
    return idx, sc / (sc.sum(-1, keepdims=True) + 1e-20) * r.get("scale", 1.0)


def expert(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def routed_ff(h, W, p, f):
    E = f["router"]["experts"]
    idx, wts = route(h, W, p, f["router"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(idx[t], wts[t]):
            out[t] += w * (h[t] if e >= E else expert(h[t:t + 1], W, f"{p}e{e}.")[0])
    if f.get("shared"):
        out += expert(h, W, p + "shared.") * sigmoid(h @ W[p + "shared.sg"].T)
    return out


# ---- the model ----------------------------------------------------------------------------------------------------------------------------
class StepOracle:
    """Feeds tokens in portions; keeps every layer's cached rows between calls."""

    def __init__(self, cfg, W):
        self.cfg, self.W = cfg, {k: np.asarray(v, np.float64) for k, v in W.items()}
        self.state = [dict() for _ in cfg["layers"]]
        self.pos = 0

    def step(self, tokens):
        """-> (logits [T, vocab], residual stream after every layer [layers, T, width])"""
        cfg, W, eps = self.cfg, self.W, self.cfg["norm"]["eps"]
        x = W["embed"][np.asarray(tokens, np.int64)] * cfg["embedding"]["scale"]
        outs = []
        for i, L in enumerate(cfg["layers"]):
            p = f"l{i}."
            y = latent_mixer(x, W, p + "mix.", L["type"], L["mixer"], eps, self.state[i], self.pos)
            x = x + offset_norm(y, W[p + "norm1"], eps)
            f = L.get("mlp")
            if f:
                y = dense_ff(x, W, p + "mlp.") if f["kind"] == "dense" else routed_ff(x, W, p + "mlp.", f)
                x = x + offset_norm(y, W[p + "norm2"], eps)
            outs.append(x.copy())
        self.pos += len(tokens)
        return offset_norm(x, W["final.norm"], eps) @ W["embed"].T, np.stack(outs)


def forward(cfg, W, tokens):
    return StepOracle(cfg, W).step(tokens)


def clear_choices(cfg, W, tokens, gap):
    """True when no routing decision of this run is closer than `gap` (a test in reduced precision must not rest on one)"""
    del CHOICE_GAPS[:]
    forward(cfg, W, tokens)
    return all(g > gap for g in CHOICE_GAPS)


def rel_rms(got, want):
    """root mean square of the difference over that of `want`, means over the last axis taken off"""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return float(np.sqrt(np.mean(d * d)) / (np.sqrt(np.mean(w * w)) + 1e-30))


# ---- small random models -----------------------------------------------------------------------------------------------------------------
def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, identity=2, top=3, ff=24, shared=40, groups=3, keep=2, scale=1.75):
    f = {"kind": "moe", "expert": {"ff": ff},
         "router": {"experts": experts, "identity": identity, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def direct_layer(heads=3, dim=12, rot_dim=8, vdim=10, kv_rank=20, size=9, base=300.0, scale=0.3, mlp="default"):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if size:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m, "mlp": moe() if mlp == "default" else mlp}


def gated_layer(heads=5, dim=8, rot_dim=12, vdim=14, kv_rank=24, q_rank=28, size=11, base=70.0, scale=0.35, mlp="default"):
    L = direct_layer(heads, dim, rot_dim, vdim, kv_rank, size, base, scale, mlp)
    L["type"] = "latent_attention_2"
    L["mixer"]["q_rank"] = q_rank
    return L


def make_config(layers, width=40, vocab=70, eps=1e-5, embed_scale=1.25):
    return {"architecture": "Lutesun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "layers": layers}


def tensor_table(cfg):
    """[(name, shape, kind)]; kind: matrix | table | gain | offset | shift | zero"""
    w = cfg["width"]
    out = [("embed", (cfg["vocab"], w), "table")]
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        q = p + "mix."
        H, dn, dr, dv, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        out.append((p + "norm1", (w,), "offset"))
        if f:
            out.append((p + "norm2", (w,), "offset"))
        if L["type"] == "latent_attention":
            out.append((q + "q", (H * (dn + dr), w), "matrix"))
        else:
            rq = m["q_rank"]
            out += [(q + "dq", (rq, w), "matrix"), (q + "dq.norm", (rq,), "gain"), (q + "uq", (H * (dn + dr), rq), "matrix"), (q + "g", (H, w), "matrix")]
        out += [(q + "dkv", (rk + dr, w), "matrix"), (q + "dkv.norm", (rk,), "gain"), (q + "uk", (H * dn, rk), "matrix"),
                (q + "uv", (H * dv, rk), "matrix"), (q + "o", (w, H * dv), "matrix")]
        if f and f["kind"] == "dense":
            out += [(p + "mlp.up", (f["ff"], w), "matrix"), (p + "mlp.up.b", (f["ff"],), "shift"), (p + "mlp.down", (w, f["ff"]), "matrix"),
                    (p + "mlp.down.b", (w,), "shift")]
        elif f:
            n = f["router"]["experts"] + f["router"].get("identity", 0)
            out += [(p + "mlp.router", (n, w), "matrix"), (p + "mlp.correction", (n,), "zero")]
            forms = [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
            if f.get("shared"):
                forms.append(("shared", f["shared"]["ff"]))
                out.append((p + "mlp.shared.sg", (1, w), "matrix"))
            for e, ff in forms:
                out += [(f"{p}mlp.{e}.gate", (ff, w), "matrix"), (f"{p}mlp.{e}.up", (ff, w), "matrix"), (f"{p}mlp.{e}.down", (w, ff), "matrix")]
    return out + [("final.norm", (w,), "offset")]


def random_weights(cfg, seed=0, gain=1.0):
    """bf16-representable float64 weights"""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape, kind in tensor_table(cfg):
        n = int(np.prod(shape))
        if kind == "matrix":
            a = rng.standard_normal(n) * gain / math.sqrt(shape[-1])
        elif kind == "table":
            a = rng.standard_normal(n)
        elif kind == "gain":
            a = 1.0 + 0.2 * rng.standard_normal(n)
        elif kind in ("offset", "shift"):
            a = 0.3 * rng.standard_normal(n)
        else:
            a = 0.1 * rng.standard_normal(n)
        W[name] = bf16_round(a).reshape(shape)
    return W


def write_model(folder, cfg, W):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, off = {}, [], 0
    for name, a in W.items():
        b = to_bf16_bits(np.asarray(a, np.float32)).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    hj = json.dumps(header).encode()
    hj += b" " * (-len(hj) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj)
        for b in blobs:
            f.write(b)
    return folder
