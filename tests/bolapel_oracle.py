"""Plain, slow float64 implementation of the Bolapel architecture: test infrastructure only.

One function per mechanism, in numpy, written from the equations below; it shares no code with the library.

    rms(v)      v / sqrt(mean(v^2) + eps)
    layer       x' = x + rms(mixer(shifted(rms(x) n1))) n1b;   x'' = x' + rms(ff(rms(x') n2)) n2b   (no second half without a
                feed-forward)
    shifted     row t of h becomes h_t + (h_{t-1} - h_t) * shift, with h_{-1} = 0; the last row of h (before this) is state
    general_delta   per head, r, k, v = W h;  w = exp(-e^{-1/2} sigmoid(W_2 tanh(W_1 h) + w0));  a = sigmoid(W_a h + b);
                u = k / sqrt(sum k^2 + 1e-6);  S_t = diag(w) S_{t-1} - (a u)(u^T S_{t-1}) + k v^T;  o = S_t^T r;
                out = W_o (rms(o) per head, joined, * norm * sigmoid(W_g h))
    attention   q, k, v = W h; q, k to rms per head * weight, then the first dims dimensions turned, dimension i with
                i + dims/2, by position * base^(-2i/dims); weight of key j for row i = sigmoid(scale q.k + pb_head), no sum to
                one, for j <= i inside the same block of `size` positions; head outputs * sigmoid(W_g h)_head; W_o.
                A layer with kv_from reads the keys and values of that layer instead of making its own.
    ff          W_down (silu(W_gate h) * (W_up h))
    logits      cap * tanh(z / cap),  z = W_head (rms(x) * w)

StepOracle keeps every layer's state between calls, so whole sequences and portions check each other.  make_config /
random_weights / write_model build small random model folders (config.json + model.safetensors with bf16 tensors).
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


# ---- small functions ----------------------------------------------------------------------------------------------------
def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


# ---- token shift --------------------------------------------------------------------------------------------------------
def token_shift(h, mu, prev):
    """-> (shifted rows, the row the next call needs as `prev`)"""
    before = np.concatenate([prev[None], h[:-1]], 0)
    return h + (before - h) * mu, h[-1].copy()


# ---- mixer: generalized delta rule --------------------------------------------------------------------------------------
def channel_decay(z):
    return np.exp(-math.exp(-0.5) * sigmoid(z))


def unit(k):
    return k / np.sqrt(np.sum(k * k, axis=-1, keepdims=True) + 1e-6)


def general_delta_scan(r, k, v, w, a, S):
    """r, k, w, a [T, H, d], v [T, H, d], S [H, d, d] (updated in place) -> o [T, H, d]"""
    o = np.zeros(v.shape)
    u = unit(k)
    for t in range(r.shape[0]):
        for h in range(r.shape[1]):
            held = u[t, h] @ S[h]                        # what the state holds under this key, before anything changes
            S[h] = w[t, h][:, None] * S[h] - np.outer(a[t, h] * u[t, h], held) + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ r[t, h]
    return o


def general_delta_mixer(h, W, p, m, eps, state):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    heads = lambda z: z.reshape(T, H, d)
    r, k, v = (heads(h @ W[p + n].T) for n in ("r", "k", "v"))
    w = heads(channel_decay(np.tanh(h @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"]))
    a = heads(sigmoid(h @ W[p + "a"].T + W[p + "a.b"]))
    if "S" not in state:
        state["S"] = np.zeros((H, d, d))
    o = rms(general_delta_scan(r, k, v, w, a, state["S"]), eps).reshape(T, H * d)
    return (o * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---- mixer: attention with independent sigmoid weights inside fixed blocks ----------------------------------------------
def rotate_half(x, positions, rot):
    """x [T, heads, n >= dims]: dimensions i and i + dims/2 (i < dims/2) turn together"""
    if not rot or not rot.get("dims"):
        return x
    n = rot["dims"]
    f = np.array([rot["base"] ** (-2.0 * i / n) for i in range(n // 2)], np.float64)
    ang = np.asarray(positions, np.float64)[:, None, None] * f
    c, s = np.cos(ang), np.sin(ang)
    out = x.copy()
    lo, hi = x[..., :n // 2], x[..., n // 2:n]
    out[..., :n // 2] = lo * c - hi * s
    out[..., n // 2:n] = hi * c + lo * s
    return out


def same_block(i, j, mask):
    """may position i look at position j?"""
    if j > i:
        return False
    return not mask or not mask.get("size") or i // mask["size"] == j // mask["size"]


def sigmoid_weights(s, bias):
    return sigmoid(s + bias)


def attention_mixer(h, W, p, m, eps, state, pos0, lender=None):
    """state: 'k' [n, G, dk] (normed and turned) and 'v' [n, G, dv] of all positions so far; a layer with a lender reads the
    lender's, which already hold this call's positions"""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(pos0, pos0 + T)
    turn = lambda z, name, n: rotate_half(rms(z.reshape(T, n, dk), eps) * W[p + name], pos, m.get("rot"))
    q = turn(h @ W[p + "q"].T, "q.norm", H)
    if lender is None:
        k = turn(h @ W[p + "k"].T, "k.norm", G)
        v = (h @ W[p + "v"].T).reshape(T, G, dv)
        state["k"] = np.concatenate([state["k"], k], 0) if "k" in state else k
        state["v"] = np.concatenate([state["v"], v], 0) if "v" in state else v
        lender = state
    gate = sigmoid(h @ W[p + "g"].T)
    out = np.zeros((T, H, dv))
    for t in range(T):
        js = [j for j in range(pos0 + t + 1) if same_block(pos0 + t, j, m.get("mask"))]
        for hh in range(H):
            g = hh // (H // G)
            wts = sigmoid_weights(lender["k"][js, g] @ q[t, hh] * m["scale"], W[p + "pb"][hh])
            out[t, hh] = gate[t, hh] * (wts @ lender["v"][js, g])
    return out.reshape(T, H * dv) @ W[p + "o"].T


# ---- feed-forward -------------------------------------------------------------------------------------------------------
def dense_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


# ---- the model ----------------------------------------------------------------------------------------------------------
class StepOracle:
    """Feeds tokens in portions; keeps every layer's state between calls."""

    def __init__(self, cfg, W):
        self.cfg, self.W = cfg, {k: np.asarray(v, np.float64) for k, v in W.items()}
        self.state = [{"prev": np.zeros(cfg["width"])} for _ in cfg["layers"]]
        self.pos = 0

    def step(self, tokens):
        """-> (logits [T, vocab], residual stream after every layer [layers, T, width])"""
        cfg, W, eps = self.cfg, self.W, self.cfg["norm"]["eps"]
        x = W["embed"][np.asarray(tokens, np.int64)]
        outs = []
        for i, L in enumerate(cfg["layers"]):
            p, m, st = f"l{i}.", L["mixer"], self.state[i]
            h, st["prev"] = token_shift(rms(x, eps) * W[p + "norm1"], W[p + "shift"], st["prev"])
            if L["type"] == "general_delta":
                y = general_delta_mixer(h, W, p + "mix.", m, eps, st)
            elif L["type"] == "attention":
                lender = self.state[m["kv_from"]] if m.get("kv_from") is not None else None
                y = attention_mixer(h, W, p + "mix.", m, eps, st, self.pos, lender)
            else:
                raise ValueError(L["type"])
            x = x + rms(y, eps) * W[p + "norm1b"]
            if L.get("mlp"):
                y = dense_ff(rms(x, eps) * W[p + "norm2"], W, p + "mlp.")
                x = x + rms(y, eps) * W[p + "norm2b"]
            outs.append(x)
        self.pos += len(tokens)
        z = (rms(x, eps) * W["final.norm"]) @ W["head"].T
        return soft_cap(z, cfg.get("logit_softcap")), np.stack(outs)


def forward(cfg, W, tokens):
    return StepOracle(cfg, W).step(tokens)


def rel_rms(got, want):
    """root mean square of the difference over that of `want`, means over the last axis taken off"""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return float(np.sqrt(np.mean(d * d)) / (np.sqrt(np.mean(w * w)) + 1e-30))


# ---- small random models ------------------------------------------------------------------------------------------------
def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def delta_layer(heads=3, dim=12, rank=5, mlp="default"):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim, "rank": rank}, "mlp": dense() if mlp == "default" else mlp}


def attention_layer(heads=4, kv_heads=2, dim=12, vdim=20, size=9, rot_dims=8, base=100.0, scale=0.4, kv_from=None, mlp="default"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": dense() if mlp == "default" else mlp}


def make_config(layers, width=40, vocab=70, eps=1e-5, softcap=9.0):
    """the low rank of the decay projection ('rank') is the shape of w1, not a configuration entry: it rides in the dictionary
    for tensor_table and is dropped from the written config.json"""
    return {"architecture": "Bolapel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": softcap, "layers": layers}


def tensor_table(cfg):
    """[(name, shape, kind)]; kind: matrix | table | gain | shift | mix | decay | bias"""
    w = cfg["width"]
    out = [("embed", (cfg["vocab"], w), "table")]
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        q = p + "mix."
        out += [(p + "norm1", (w,), "gain"), (p + "norm1b", (w,), "gain"), (p + "shift", (w,), "mix")]
        if L["type"] == "general_delta":
            n, r = m["heads"] * m["dim"], m.get("rank", 4)
            out += [(q + s, (n, w), "matrix") for s in ("r", "k", "v", "g", "a")]
            out += [(q + "a.b", (n,), "shift"), (q + "w1", (r, w), "matrix"), (q + "w2", (n, r), "matrix"), (q + "w0", (n,), "decay"),
                    (q + "norm", (n,), "gain"), (q + "o", (w, n), "matrix")]
        else:
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out += [(q + "q", (H * dk, w), "matrix"), (q + "q.norm", (dk,), "gain")]
            if m.get("kv_from") is None:
                out += [(q + "k", (G * dk, w), "matrix"), (q + "v", (G * dv, w), "matrix"), (q + "k.norm", (dk,), "gain")]
            out += [(q + "pb", (H,), "bias"), (q + "g", (H, w), "matrix"), (q + "o", (w, H * dv), "matrix")]
        if f:
            out += [(p + "norm2", (w,), "gain"), (p + "norm2b", (w,), "gain"), (p + "mlp.gate", (f["ff"], w), "matrix"),
                    (p + "mlp.up", (f["ff"], w), "matrix"), (p + "mlp.down", (w, f["ff"]), "matrix")]
    return out + [("final.norm", (w,), "gain"), ("head", (cfg["vocab"], w), "matrix")]


def random_weights(cfg, seed=0, gain=1.0):
    """bf16-representable float64 weights"""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape, kind in tensor_table(cfg):
        n = int(np.prod(shape))
        if kind == "matrix":
            a = rng.standard_normal(n) * gain / math.sqrt(shape[-1])
            if name == "head":
                a *= 2.0
        elif kind == "table":
            a = rng.standard_normal(n)
        elif kind == "gain":
            a = 1.0 + 0.2 * rng.standard_normal(n)
        elif kind == "shift":
            a = 0.5 * rng.standard_normal(n)
        elif kind == "mix":
            a = rng.random(n)
        elif kind == "decay":
            a = -1.5 + 1.5 * rng.standard_normal(n)
        elif kind == "bias":
            a = -1.0 + 0.7 * rng.standard_normal(n)
        else:
            raise ValueError(kind)
        W[name] = bf16_round(a).reshape(shape)
    return W


def written_config(cfg):
    """config.json as the library reads it: without the entries that only tensor_table uses"""
    c = json.loads(json.dumps(cfg))
    for L in c["layers"]:
        L["mixer"].pop("rank", None)
    return c


def write_model(folder, cfg, W):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(written_config(cfg), f)
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
