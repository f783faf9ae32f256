"""A plain, slow restatement of the Fokonex equations in float64 numpy, one function per mechanism, and the small
random models the tests run. It shares no code with the package.

Notation: x is the residual stream [T, W]; a layer is x' = x + m (A(n1(x)) + F(n2(x))).
"""
import json
import os
import struct

import numpy as np


# ---- number formats ----
def to_bf16_bits(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) >> np.uint32(16)).astype(np.uint16)


def from_bf16_bits(b):
    return (np.asarray(b).astype(np.uint32) << np.uint32(16)).view(np.float32)


def bf16(x):
    return from_bf16_bits(to_bf16_bits(x))


# ---- mechanisms ----
def rms_norm(x, w, eps):
    """n(x)_i = (1 + w_i) x_i / sqrt(mean_j x_j^2 + eps)."""
    x = np.asarray(x, dtype=np.float64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * (1.0 + np.asarray(w, dtype=np.float64))


def query_factor(p, coef, every):
    """tau(p) = 1 + coef ln(floor((p + 1) / every) + 1)."""
    return 1.0 + coef * np.log(np.floor((np.asarray(p) + 1) / every) + 1.0)


def cap(s, c):
    return c * np.tanh(s / c)


def relu_squared(z):
    return np.where(z > 0, z, 0.0) ** 2


def attention_weights(scores, sink):
    """Softmax over the last axis whose denominator has one more term, exp(sink)."""
    top = np.maximum(scores.max(axis=-1), sink)
    e = np.exp(scores - top[..., None])
    return e / (e.sum(axis=-1) + np.exp(sink - top))[..., None]


def attention(q, k, v, first, scale, softcap, coef, every, sinks):
    """q [T, H, d] at positions first .. first + T - 1 over keys k [L, G, d] and values v [L, G, e] of positions 0 .. L - 1.
    softcap 0 = none, every 0 = no query factor, sinks None = no sink. Returns [T, H, e]."""
    q, k, v = (np.asarray(t, dtype=np.float64) for t in (q, k, v))
    rows, heads, _ = q.shape
    length, groups, _ = k.shape
    p = first + np.arange(rows)
    if every:
        q = q * query_factor(p, coef, every)[:, None, None]
    out = np.zeros((rows, heads, v.shape[2]))
    for h in range(heads):
        g = h // (heads // groups)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap:
            s = cap(s, softcap)
        s[np.arange(length)[None, :] > p[:, None]] = -np.inf
        out[:, h] = attention_weights(s, np.full(rows, -np.inf if sinks is None else sinks[h])) @ v[:, g]
    return out


def mixer(h, cfg, w, past):
    """The attention branch of T new tokens; `past` = (keys, values) of the earlier ones, extended in place."""
    rows = h.shape[0]
    q = (h @ w["mix.q"].T).reshape(rows, cfg["heads"], cfg["dim"])
    k = (h @ w["mix.k"].T).reshape(rows, cfg["kv_heads"], cfg["dim"])
    v = (h @ w["mix.v"].T).reshape(rows, cfg["kv_heads"], cfg["vdim"])
    first = past[0].shape[0]
    past[0], past[1] = np.concatenate([past[0], k]), np.concatenate([past[1], v])
    temp = cfg["q_temp"]
    o = attention(q, past[0], past[1], first, cfg["scale"], cfg["softcap"], temp["coef"], temp["every"], w["mix.sink"])
    return o.reshape(rows, -1) @ w["mix.o"].T


def feed_forward(h, w):
    return relu_squared(h @ w["mlp.up"].T) @ w["mlp.down"].T


class Reference:
    """Runs a model token portion by token portion, from config.json's dictionary and f32 tensors."""

    def __init__(self, config, tensors):
        self.config = config
        self.t = {n: np.asarray(v, dtype=np.float64) for n, v in tensors.items()}
        self.reset()

    def reset(self):
        self.past = []
        for layer in self.config["layers"]:
            m = layer["mixer"]
            self.past.append([np.zeros((0, m["kv_heads"], m["dim"])), np.zeros((0, m["kv_heads"], m["vdim"]))])

    def forward(self, tokens):
        c = self.config
        x = self.t["embed"][np.asarray(tokens)]
        for i, layer in enumerate(c["layers"]):
            p = f"l{layer.get('weights_of', i)}."
            w = {n[len(p):]: v for n, v in self.t.items() if n.startswith(p)}
            y = mixer(rms_norm(x, w["norm1"], c["norm"]["eps"]), layer["mixer"], w, self.past[i])
            if layer["mlp"] is not None:
                y = y + feed_forward(rms_norm(x, w["norm2"], c["norm"]["eps"]), w)
            x = x + c["residual_mult"] * y
        return rms_norm(x, self.t["final.norm"], c["norm"]["eps"]) @ self.t["head"].T * c["logit_scale"]


# ---- small models ----
def layer(heads, kv_heads, dim, vdim, ff, scale=None, softcap=20.0, coef=0.3, every=16, weights_of=None):
    d = {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
         "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                   "softcap": softcap, "q_temp": {"coef": coef, "every": every}}}
    if weights_of is not None:
        d["weights_of"] = weights_of
    return d


def config(vocab, width, layers, eps=1e-5, residual_mult=0.7, logit_scale=0.6):
    return {"architecture": "Fokonex", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "residual_mult": residual_mult,
            "logit_scale": logit_scale}


CONFIGS = {
    # sizes that suit no vector width, a group of three, one layer without a feed-forward, one with its own geometry
    "odd": config(61, 52, [layer(6, 2, 20, 24, 37), layer(6, 2, 20, 24, None, every=7), layer(2, 2, 9, 33, 70, softcap=5.0)]),
    # one kv head for all, value heads wider than keys, layers out of order that share tensors
    "shared": config(130, 96, [layer(4, 1, 32, 48, 128, weights_of=1), layer(4, 1, 32, 48, 128), layer(4, 1, 32, 48, 128, weights_of=1)], eps=1e-3),
    # as many kv heads as heads, keys wider than values, unit constants
    "plain": config(96, 64, [layer(4, 4, 48, 16, 96, scale=1.0, coef=0.0, every=1), layer(2, 1, 64, 64, 64, scale=0.2, every=3)], residual_mult=1.0, logit_scale=1.0),
    # a cap too large for the fixed-range kernels
    "highcap": config(80, 64, [layer(4, 2, 32, 32, 64, softcap=90.0)]),
}


def random_tensors(cfg, seed=0, gain=1.0):
    """Weights in bf16's range of values (as f32), scaled so that every branch matters."""
    rng = np.random.default_rng(seed)
    w = cfg["width"]
    t = {"embed": rng.standard_normal((cfg["vocab"], w)), "final.norm": 0.3 * rng.standard_normal(w), "head": rng.standard_normal((cfg["vocab"], w)) / np.sqrt(w)}
    for i, l in enumerate(cfg["layers"]):
        if "weights_of" in l:
            continue
        m, p = l["mixer"], f"l{i}."
        t[p + "norm1"] = 0.3 * rng.standard_normal(w)
        for name, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
            t[p + "mix." + name] = gain * rng.standard_normal((rows, w)) / np.sqrt(w)
        t[p + "mix.sink"] = rng.standard_normal(m["heads"])
        t[p + "mix.o"] = rng.standard_normal((w, m["heads"] * m["vdim"])) / np.sqrt(m["heads"] * m["vdim"])
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            t[p + "norm2"] = 0.3 * rng.standard_normal(w)
            t[p + "mlp.up"] = rng.standard_normal((ff, w)) / np.sqrt(w)
            t[p + "mlp.down"] = rng.standard_normal((w, ff)) / np.sqrt(ff)
    return {n: bf16(v) for n, v in t.items()}


def write_safetensors(path, tensors):
    header, body, at = {}, [], 0
    for name, v in tensors.items():
        raw = to_bf16_bits(v).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [at, at + len(raw)]}
        body.append(raw)
        at += len(raw)
    h = json.dumps(header).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(body))


def write_model(folder, cfg, tensors):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return str(folder)


def row_errors(got, want):
    """Root mean square of each row's difference (its mean taken off), relative to the logits' spread."""
    d = np.asarray(got, dtype=np.float64) - want
    d = d - d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / (want - want.mean(axis=-1, keepdims=True)).std()
