"""A plain, slow restatement of the Zisevik equations in float64 numpy, one function per mechanism, and the small random
models the tests run. It shares no code with the package.

Notation: x is the residual stream [T, W], e the embedding output; a layer is x' = x + M(n1(x)), x'' = x' + F(n2(x')).
A span of layers runs several times; every pass begins with x = W_in [x; e].
"""
import numpy as np

from fokonex_reference import bf16, from_bf16_bits, row_errors, to_bf16_bits, write_model  # noqa: F401 (shared number formats and files)


# ---- mechanisms ----
def rms(x, eps):
    """x_i / sqrt(mean_j x_j^2 + eps)."""
    x = np.asarray(x, dtype=np.float64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * np.asarray(w, dtype=np.float64)


def rotate(x, positions, dims, base):
    """Turns the pairs (x_i, x_{i + dims/2}), i < dims/2, of the last axis by the angle p base^(-2i/dims); x is [T, ..., d]."""
    x = np.array(x, dtype=np.float64)
    half = dims // 2
    angle = np.asarray(positions, dtype=np.float64)[:, None] * base ** (-2.0 * np.arange(half) / dims)
    angle = angle.reshape(angle.shape[:1] + (1,) * (x.ndim - 2) + (half,))
    u, v = x[..., :half].copy(), x[..., half:dims].copy()
    x[..., :half] = u * np.cos(angle) - v * np.sin(angle)
    x[..., half:dims] = v * np.cos(angle) + u * np.sin(angle)
    return x


def attend(q, k, v, first, scale, window, sinks):
    """q [T, H, d] at positions first .. over keys k [L, G, d] and values v [L, G, e] of positions 0 .. L - 1, G groups of heads.
    Position p sees j with 0 <= p - j < window (None = all before it); the denominator of head h has one more term exp(sinks[h])."""
    q, k, v = (np.asarray(t, dtype=np.float64) for t in (q, k, v))
    rows, heads, _ = q.shape
    length, groups, _ = k.shape
    p, j = first + np.arange(rows)[:, None], np.arange(length)[None, :]
    seen = (j <= p) & (p - j < (np.inf if window is None else window))
    out = np.zeros((rows, heads, v.shape[2]))
    for h in range(heads):
        g = h // (heads // groups)
        s = np.where(seen, q[:, h] @ k[:, g].T * scale, -np.inf)
        sink = -np.inf if sinks is None else sinks[h]
        top = np.maximum(s.max(axis=1), sink)[:, None]
        e = np.exp(s - top)
        out[:, h] = e @ v[:, g] / (e.sum(axis=1, keepdims=True) + np.exp(sink - top))
    return out


def latent_attention(h, m, w, past, first, eps):
    """`past` = [latents, rotated key parts] of the earlier tokens, extended in place."""
    rows, heads, d, r, e = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    p = first + np.arange(rows)
    q = (rms_norm(h @ w["mix.dq"].T, w["mix.dq.norm"], eps) @ w["mix.uq"].T).reshape(rows, heads, d + r)
    q = np.concatenate([q[..., :d], rotate(q[..., d:], p, m["rot"]["dims"], m["rot"]["base"])], axis=-1)
    down = h @ w["mix.dkv"].T
    past[0] = np.concatenate([past[0], rms_norm(down[:, :m["kv_rank"]], w["mix.dkv.norm"], eps)])
    past[1] = np.concatenate([past[1], rotate(down[:, m["kv_rank"]:], p, m["rot"]["dims"], m["rot"]["base"])])
    length = past[0].shape[0]
    k = (past[0] @ w["mix.uk"].T).reshape(length, heads, d)
    k = np.concatenate([k, np.broadcast_to(past[1][:, None], (length, heads, r))], axis=-1)
    v = (past[0] @ w["mix.uv"].T).reshape(length, heads, e)
    o = attend(q, k, v, first, m["scale"], (m.get("mask") or {}).get("size"), w["mix.sink"])
    return o.reshape(rows, -1) @ w["mix.o"].T


def retain(q, k, v, decay, state):
    """S_t = decay_h S_{t-1} + k_t v_t^T, o_t = S_t^T q_t, token by token; q, k [T, H, d], v [T, H, e], state [H, d, e] changed in place."""
    out = np.zeros(v.shape, dtype=np.float64)
    for t in range(q.shape[0]):
        state *= np.asarray(decay, dtype=np.float64)[:, None, None]
        state += k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", state, q[t])
    return out


def silu(z):
    return z / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def retention(h, m, w, past, first, eps):
    """`past` = [state [H, d, e]], changed in place."""
    rows, heads, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    p = first + np.arange(rows)
    q = rotate((h @ w["mix.q"].T).reshape(rows, heads, d), p, m["rot"]["dims"], m["rot"]["base"])
    k = rotate((h @ w["mix.k"].T).reshape(rows, heads, d), p, m["rot"]["dims"], m["rot"]["base"]) * d ** -0.5
    v = (h @ w["mix.v"].T).reshape(rows, heads, e)
    o = rms(retain(q, k, v, m["decay"], past[0]), eps).reshape(rows, -1)
    return (o * silu(h @ w["mix.g"].T)) @ w["mix.o"].T


def route(z, top):
    """The `top` largest logits of each row and the softmax over those; ([T, top] experts, [T, top] weights)."""
    chosen = np.argsort(-z, axis=1, kind="stable")[:, :top]
    s = np.take_along_axis(z, chosen, axis=1)
    s = np.exp(s - s.max(axis=1, keepdims=True))
    return chosen, s / s.sum(axis=1, keepdims=True)


def experts(h, mlp, w):
    chosen, weight = route(h @ w["mlp.router"].T + w["mlp.router.b"], mlp["router"]["top"])
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for c, a in zip(chosen[t], weight[t]):
            y[t] += a * (silu(h[t] @ w[f"mlp.e{c}.gate"].T) * (h[t] @ w[f"mlp.e{c}.up"].T)) @ w[f"mlp.e{c}.down"].T
    return y


def feed_forward(h, mlp, w):
    if mlp["kind"] == "dense":
        return gelu_tanh(h @ w["mlp.up"].T) @ w["mlp.down"].T
    return experts(h, mlp, w)


# ---- the whole model ----
def layer_runs(config):
    """[(layer, begins a pass)] in the order they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    span = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return [(i, False) for i in range(loop["start"])] + span * loop["times"] + [(i, False) for i in range(loop["stop"], n)]


class Reference:
    """Runs a model portion by portion, from config.json's dictionary and f32 tensors; `residuals` keeps x after every layer run."""

    def __init__(self, config, tensors):
        self.config = config
        self.t = {n: np.asarray(v, dtype=np.float64) for n, v in tensors.items()}
        self.reset()

    def reset(self):
        self.past, self.length, self.residuals = [], 0, []
        for i, _ in layer_runs(self.config):
            m = self.config["layers"][i]["mixer"]
            if self.config["layers"][i]["type"] == "retention":
                self.past.append([np.zeros((m["heads"], m["dim"], m["vdim"]))])
            else:
                self.past.append([np.zeros((0, m["kv_rank"])), np.zeros((0, m["rot_dim"]))])

    def forward(self, tokens):
        c, eps = self.config, self.config["norm"]["eps"]
        e = self.t["embed"][np.asarray(tokens)]
        x, self.residuals = e, []
        for run, (i, begins) in enumerate(layer_runs(c)):
            if begins:
                x = np.concatenate([x, e], axis=1) @ self.t["loop.in"].T
            layer, p = c["layers"][i], f"l{i}."
            w = {n[len(p):]: v for n, v in self.t.items() if n.startswith(p)}
            mixer = retention if layer["type"] == "retention" else latent_attention
            x = x + mixer(rms_norm(x, w["norm1"], eps), layer["mixer"], w, self.past[run], self.length, eps)
            if layer["mlp"] is not None:
                x = x + feed_forward(rms_norm(x, w["norm2"], eps), layer["mlp"], w)
            self.residuals.append(x)
        self.length += len(tokens)
        return rms_norm(x, self.t["final.norm"], eps) @ self.t["head"].T


# ---- small models ----
def attention_layer(heads, dim, rot_dim, vdim, kv_rank, q_rank, window, mlp, base=10000.0, scale=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "rot": {"base": base, "dims": rot_dim}, "mask": {"size": window}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def retention_layer(heads, dim, vdim, rot_dims, mlp, base=10000.0, decay=None):
    decay = [1.0 - 2.0 ** -(2 + 5.0 * h / max(1, heads - 1)) for h in range(heads)] if decay is None else decay
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": rot_dims}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(count, top, ff):
    return {"kind": "moe", "router": {"experts": count, "top": top}, "expert": {"ff": ff}}


def config(vocab, width, layers, loop=None, eps=1e-5):
    c = {"architecture": "Zisevik", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


CONFIGS = {
    # sizes that suit no vector width; every kind of layer in the loop and outside it; one layer without a feed-forward
    "odd": config(61, 52, [retention_layer(3, 10, 22, 6, moe(5, 3, 19)), attention_layer(3, 20, 6, 11, 27, 23, 7, dense(37)),
                           attention_layer(5, 9, 2, 33, 18, 40, 12, None), retention_layer(2, 8, 7, 8, dense(45))], loop=(1, 3, 2), eps=1e-4),
    # the loop begins with a retention layer and takes the whole model; one expert per token
    "looped": config(130, 96, [retention_layer(4, 32, 48, 32, moe(7, 1, 40), base=500.0), attention_layer(4, 32, 16, 32, 64, 48, 33, moe(16, 4, 24), base=1e6)],
                     loop=(0, 2, 3)),
    # no loop, a window of one token, a window longer than any prompt, every expert chosen, one head
    "plain": config(96, 64, [attention_layer(4, 16, 16, 16, 32, 32, 1, dense(64), scale=0.3), attention_layer(1, 48, 8, 64, 48, 16, 4096, moe(3, 3, 32)),
                             retention_layer(1, 16, 64, 16, None, decay=[0.9])]),
    # sizes like a real model's heads: what the tensor-core kernels take
    "wide": config(200, 256, [attention_layer(8, 64, 32, 64, 128, 64, 100, moe(4, 2, 64)), retention_layer(4, 64, 128, 64, dense(128)),
                              attention_layer(4, 128, 64, 128, 256, 96, 160, dense(192))], loop=(1, 2, 2)),
}


def random_tensors(cfg, seed=0, gain=1.0):
    """Weights in bf16's range of values (as f32), scaled so that every branch matters."""
    rng = np.random.default_rng(seed)
    w, t = cfg["width"], {}

    def matrix(name, rows, cols, g=1.0):
        t[name] = g * rng.standard_normal((rows, cols)) / np.sqrt(cols)

    def vector(name, n):
        t[name] = 1.0 + 0.3 * rng.standard_normal(n)

    t["embed"] = rng.standard_normal((cfg["vocab"], w))
    if cfg.get("loop"):
        matrix("loop.in", w, 2 * w)
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        vector(p + "norm1", w)
        if l["type"] == "retention":
            for name, cols in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"]), ("g", m["vdim"])):
                matrix(p + "mix." + name, m["heads"] * cols, w, gain)
        else:
            matrix(p + "mix.dq", m["q_rank"], w)
            vector(p + "mix.dq.norm", m["q_rank"])
            matrix(p + "mix.uq", m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.5 * gain)
            matrix(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], w)
            vector(p + "mix.dkv.norm", m["kv_rank"])
            matrix(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"], 1.5 * gain)
            matrix(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
            t[p + "mix.sink"] = rng.standard_normal(m["heads"])
        matrix(p + "mix.o", w, m["heads"] * m["vdim"])
        if l["mlp"] is None:
            continue
        vector(p + "norm2", w)
        if l["mlp"]["kind"] == "dense":
            matrix(p + "mlp.up", l["mlp"]["ff"], w)
            matrix(p + "mlp.down", w, l["mlp"]["ff"])
        else:
            n, ff = l["mlp"]["router"]["experts"], l["mlp"]["expert"]["ff"]
            matrix(p + "mlp.router", n, w, 2.0)
            t[p + "mlp.router.b"] = 0.5 * rng.standard_normal(n)
            for e in range(n):
                matrix(f"{p}mlp.e{e}.gate", ff, w)
                matrix(f"{p}mlp.e{e}.up", ff, w)
                matrix(f"{p}mlp.e{e}.down", w, ff)
    vector("final.norm", w)
    matrix("head", cfg["vocab"], w)
    return {n: bf16(v) for n, v in t.items()}
