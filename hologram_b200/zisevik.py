"""Zisevik: a decoder-only design of latent attention and retention layers, dense or routed feed-forwards, and a span of
layers that runs several times, as `.holo` step archives.

The residual stream x is f32. A layer run adds mixer(norm1(x)) and then ff(norm2(x)). Every pass over the looped span begins
with x = W_in [x; embedding output] and has caches and states of its own (port `l<r>.*` belongs to layer run r). Calls of a
layer run, `rows` new tokens at a time:

  latent attention   RmsNormMulti x -> h; Linear h -> [query latent | key/value latent] (f32) and the rotated key part into the cache;
                     RmsNormParts -> query latent, cache rows; Linear -> q, its rotated part turned as it is stored; then
    few rows           HeadLinear q -> latent queries; WindowAttention over the cached latents; HeadLinear -> values
    many rows          Linear: keys and values of the visible part of the cache; WindowAttention over them
                     Linear -> x += W_o (...)
  retention          RmsNormMulti; Linear -> q, k (rotated as they are stored), v, silu gate; Retention; Linear -> x += W_o (...)
  dense              RmsNormMulti; Linear with gelu; Linear -> x += ...
  routed             RmsNormMulti; Linear -> router logits; MoePlan; (many rows: Gather by expert); grouped Linear with a silu
                     gate; grouped Linear; MoeCombine

The cache of a run is a ring of rows [latent | rotated key part] that holds the window and one portion. Rotated pairs are
stored side by side (weights are permuted when they are packed), so that a product's epilogue can turn them; head widths are
padded with zero columns to multiples of 16 and matrix widths to multiples of 8.
"""
import numpy as np

from . import holo
from . import kernel_call as kc
from .step_model import BF, F32, I32, STEP_IN_IDS, StepModel, up

LATENT, RETENTION = "latent_attention", "retention"
ABSORB_ROWS = 16       # up to here latent attention works on the latents themselves (bf16; f32 steps always do)


class Rotation:
    """Angles of the first `dims` dimensions of a vector: position * base^(-2i/dims) for pair i."""

    def __init__(self, dims, base):
        if dims % 2 or dims < 0:
            raise ValueError(f"rotation over {dims} dimensions")
        self.dims, self.base = dims, base
        self.key = (dims, base)

    @classmethod
    def from_dict(cls, d):
        return cls(int(d["dims"]), float(d["base"])) if d else cls(0, 1.0)

    def to_dict(self):
        return {"dims": self.dims, "base": self.base}

    def frequencies(self):
        """f32 [2, dims / 2]: the frequencies in turns per position, rounded, and their remainders."""
        f = self.base ** (-2.0 * np.arange(self.dims // 2, dtype=np.float64) / max(self.dims, 1)) / (2.0 * np.pi)
        hi = f.astype(np.float32)
        return np.stack([hi, (f - hi).astype(np.float32)])

    def order(self, width):
        """The stored order of a vector's dimensions: the pairs (i, i + dims / 2) side by side, then the rest."""
        half = self.dims // 2
        pairs = np.stack([np.arange(half), np.arange(half) + half], axis=1).reshape(-1)
        return np.concatenate([pairs, np.arange(self.dims, width)]).astype(np.int64)


class LatentSpec:
    kind = LATENT

    def __init__(self, heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, window, rot):
        if min(heads, dim, vdim, kv_rank, q_rank) <= 0 or rot_dim < 0 or rot.dims > rot_dim or (window is not None and window < 1):
            raise ValueError(f"latent attention: heads {heads}, dim {dim} + {rot_dim}, vdim {vdim}, ranks {q_rank} / {kv_rank}, window {window}")
        self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank, self.q_rank = heads, dim, rot_dim, vdim, kv_rank, q_rank
        self.scale, self.window, self.rot = scale, window, rot
        self.dim_p, self.rot_p, self.vdim_p = up(dim, 16), up(rot_dim, 16), up(vdim, 16)
        self.kv_p, self.q_p = up(kv_rank, 16), up(q_rank, 8)
        self.head_p, self.row_p = self.dim_p + self.rot_p, self.kv_p + self.rot_p     # columns of a query head, of a cache row

    @classmethod
    def from_dict(cls, d):
        window = (d.get("mask") or {}).get("size")
        return cls(int(d["heads"]), int(d["dim"]), int(d["rot_dim"]), int(d["vdim"]), int(d["kv_rank"]), int(d["q_rank"]), float(d["scale"]),
                   None if window is None else int(window), Rotation.from_dict(d.get("rot")))

    def to_dict(self):
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank, "q_rank": self.q_rank,
                "scale": self.scale, "mask": None if self.window is None else {"size": self.window}, "rot": self.rot.to_dict()}

    def tensor_shapes(self, w):
        return {"dq": (self.q_rank, w), "dq.norm": (self.q_rank,), "uq": (self.heads * (self.dim + self.rot_dim), self.q_rank),
                "dkv": (self.kv_rank + self.rot_dim, w), "dkv.norm": (self.kv_rank,), "uk": (self.heads * self.dim, self.kv_rank),
                "uv": (self.heads * self.vdim, self.kv_rank), "sink": (self.heads,), "o": (w, self.heads * self.vdim)}

    def in_columns(self):
        """Where the query latent, the key/value latent and the rotated key part begin in the input product, and its columns."""
        kv = up(self.q_rank, 32)
        rot = kv + up(self.kv_rank, 32)
        return (0, kv, rot), up(rot + self.rot_p, 8)

    def down_columns(self):
        """Where the key/value latent begins in a row of both latents, and the row's pitch."""
        kv = up(self.q_rank, 4)
        return kv, kv + up(self.kv_rank, 4)

    def expand_columns(self):
        """Where the values begin in the product that turns latents into keys and values, and its columns."""
        v = up(self.heads * self.dim_p, 32)
        return v, up(v + self.heads * self.vdim_p, 8)

    def cache_rows(self, capacity, portion):
        rows = capacity if self.window is None else min(capacity, self.window - 1 + portion)
        return up(rows, 128)

    def expand_rows(self, rows, capacity):
        """Rows of keys and values a step of `rows` tokens may see (the first one at a multiple of 128)."""
        return up(capacity if self.window is None else min(capacity, rows + self.window - 1 + 127), 128)


class RetentionSpec:
    kind = RETENTION

    def __init__(self, heads, dim, vdim, decay, rot):
        if min(heads, dim, vdim) <= 0 or len(decay) != heads or rot.dims > dim:
            raise ValueError(f"retention: {heads} heads of {dim} x {vdim}, {len(decay)} decays, {rot.dims} rotated dimensions")
        self.heads, self.dim, self.vdim, self.decay, self.rot = heads, dim, vdim, decay, rot
        self.dim_p, self.vdim_p = up(dim, 16), up(vdim, 16)

    @classmethod
    def from_dict(cls, d):
        return cls(int(d["heads"]), int(d["dim"]), int(d["vdim"]), [float(x) for x in d["decay"]], Rotation.from_dict(d.get("rot")))

    def to_dict(self):
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay), "rot": self.rot.to_dict()}

    def tensor_shapes(self, w):
        k, v = self.heads * self.dim, self.heads * self.vdim
        return {"q": (k, w), "k": (k, w), "v": (v, w), "g": (v, w), "o": (w, v)}

    def in_columns(self):
        """Where q, k, v and the gate begin in the input product, and its columns."""
        k = up(self.heads * self.dim_p, 32)
        v = 2 * k
        g = v + up(self.heads * self.vdim_p, 32)
        return (0, k, v, g), up(g + self.heads * self.vdim_p, 8)


class DenseSpec:
    def __init__(self, ff):
        self.ff, self.ff_p = ff, up(ff, 8)

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff}

    def tensor_shapes(self, w):
        return {"up": (self.ff, w), "down": (w, self.ff)}


class RoutedSpec:
    def __init__(self, experts, top, ff):
        if not 0 < top <= experts:
            raise ValueError(f"routed feed-forward: {top} of {experts} experts")
        self.experts, self.top, self.ff, self.ff_p = experts, top, ff, up(ff, 8)

    def to_dict(self):
        return {"kind": "moe", "router": {"experts": self.experts, "top": self.top}, "expert": {"ff": self.ff}}

    def tensor_shapes(self, w):
        out = {"router": (self.experts, w), "router.b": (self.experts,)}
        for e in range(self.experts):
            out.update({f"e{e}.gate": (self.ff, w), f"e{e}.up": (self.ff, w), f"e{e}.down": (w, self.ff)})
        return out

    def tiles(self, rows):
        """(rows of a tile, most tiles) of the grouped products over `rows` tokens: up to 128 tokens share one tile per chosen
        expert, more are sorted by expert."""
        pairs = rows * self.top
        for n in (16, 64, 128):
            if rows <= n:
                return n, min(self.experts, pairs)
        return 128, min(pairs, self.experts + pairs // 128)


def _feed_forward(d, where):
    if d is None:
        return None
    if d["kind"] == "dense":
        return DenseSpec(int(d["ff"]))
    if d["kind"] == "moe":
        return RoutedSpec(int(d["router"]["experts"]), int(d["router"]["top"]), int(d["expert"]["ff"]))
    raise ValueError(f"{where}: feed-forward kind {d['kind']!r} is not part of this design")


class LayerSpec:
    def __init__(self, index, mixer, mlp):
        self.index, self.mixer, self.mlp = index, mixer, mlp


class ZisevikConfig:
    ARCHITECTURE = "Zisevik"

    def __init__(self, vocab, width, layers, eps, loop=None):
        self.vocab, self.width, self.layers, self.eps, self.loop = vocab, width, layers, eps, loop
        self.width_p = up(width, 8)
        if loop is not None and not (0 <= loop[0] < loop[1] <= len(layers) and loop[2] >= 1):
            raise ValueError(f"loop over layers {loop[0]} .. {loop[1]} of {len(layers)}, {loop[2]} times")

    @classmethod
    def from_dict(cls, d):
        if d.get("architecture") != cls.ARCHITECTURE:
            raise ValueError(f"config.json names architecture {d.get('architecture')!r}, not {cls.ARCHITECTURE!r}")
        layers = []
        for i, entry in enumerate(d["layers"]):
            kinds = {LATENT: LatentSpec, RETENTION: RetentionSpec}
            if entry["type"] not in kinds:
                raise ValueError(f"layer {i}: mixer type {entry['type']!r} is not part of this design")
            layers.append(LayerSpec(i, kinds[entry["type"]].from_dict(entry["mixer"]), _feed_forward(entry.get("mlp"), f"layer {i}")))
        loop = d.get("loop")
        return cls(int(d["vocab"]), int(d["width"]), layers, float(d["norm"]["eps"]),
                   None if not loop else (int(loop["start"]), int(loop["stop"]), int(loop["times"])))

    def to_dict(self):
        layers = [{"type": l.mixer.kind, "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()} for l in self.layers]
        out = {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width, "layers": layers, "norm": {"eps": self.eps}}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    def runs(self):
        """[(layer, is it the first of a pass over the loop)] in the order they run."""
        if self.loop is None:
            return [(l, False) for l in self.layers]
        start, stop, times = self.loop
        span = [(l, l.index == start) for l in self.layers[start:stop]]
        return [(l, False) for l in self.layers[:start]] + span * times + [(l, False) for l in self.layers[stop:]]

    def tensor_shapes(self):
        """Name -> shape of every tensor a checkpoint of this configuration holds."""
        w = self.width
        out = {"embed": (self.vocab, w)}
        if self.loop is not None:
            out["loop.in"] = (w, 2 * w)
        for l in self.layers:
            p = f"l{l.index}."
            out[p + "norm1"] = (w,)
            out.update({p + "mix." + n: s for n, s in l.mixer.tensor_shapes(w).items()})
            if l.mlp is not None:
                out[p + "norm2"] = (w,)
                out.update({p + "mlp." + n: s for n, s in l.mlp.tensor_shapes(w).items()})
        out["final.norm"], out["head"] = (w,), (self.vocab, w)
        return out


class _Step:
    """One step archive under construction."""

    def __init__(self, model, rows, capacity, portion):
        self.m, self.rows, self.capacity, self.portion = model, rows, capacity, portion
        self.w, self.sl, self.made = model._begin()
        self.work, self.tables = {}, {}
        step_in = self.sl.new(4 * (STEP_IN_IDS + rows))
        self.w.inputs.append(holo.Port("step_in", step_in, STEP_IN_IDS + rows, I32, [STEP_IN_IDS + rows]))
        self.pos, self.step = self.sl.ref(step_in, 0, 4), self.sl.ref(step_in, 0, 8)      # the position; (position, real rows)
        self.ids = self.sl.ref(step_in, 4 * STEP_IN_IDS)

    def const(self, name):
        return self.m._const(self.w, self.sl, self.made, name)

    def call(self, c):
        self.w.calls.append(c)

    def buffer(self, name, nbytes):
        """A work buffer, shared by every layer run that asks for the same name and size."""
        key = (name, nbytes)
        if key not in self.work:
            self.work[key] = self.sl.new(nbytes)
        return self.work[key]

    def state(self, name, dtype, shape):
        n = int(np.prod(shape))
        s = self.sl.new(n * (4 if dtype == F32 else 2))
        self.w.inputs.append(holo.Port(name, s, n, dtype, list(shape)))
        return s

    def table(self, rot):
        """The step's cosines and sines for a rotation, made where a layer first needs them."""
        if not rot.dims:
            return None
        if rot.key not in self.tables:
            half = rot.dims // 2
            t = self.sl.new(8 * self.rows * half)
            self.call(kc.KernelCall.RotaryTable(kc.RotaryTableCall(self.pos, self.const(self.m._rotary_name(rot)), self.sl.ref(t), self.rows, half)))
            self.tables[rot.key] = t
        return self.sl.ref(self.tables[rot.key])

    def norm(self, x, weight, out):
        c = self.m.config
        self.call(kc.KernelCall.RmsNormMulti(kc.RmsNormMultiCall(x, self.const(weight), kc.NONE, out, self.rows, c.width, c.width_p, kc.f32_bits(c.eps), self.m.dtype)))

    def linear(self, a, b, segs, k, n, m=None, **kw):
        self.call(kc.KernelCall.Linear(kc.LinearCall.make(a, self.const(b), segs, self.rows if m is None else m, k, n, self.m.dtype, **kw)))


class ZisevikModel(StepModel):
    """Configuration and device-layout weights of one model; builds its step archives."""

    CONFIG = ZisevikConfig

    # ---- weights ----
    @staticmethod
    def _rotary_name(rot):
        return f"rotary.{rot.dims}.{rot.base!r}"

    def _rows_to_columns(self, value, rows, rows_p, heads=1, order=None):
        """[heads * rows, w] -> [w8, heads * rows_p]: every head's rows (in `order`) become columns, padded with zeros."""
        w = value.shape[1]
        out = self._zeros((up(w, 8), heads, rows_p))
        v = value.reshape(heads, rows, w).transpose(2, 0, 1)
        out[:w, :, :rows] = v if order is None else v[:, :, order]
        return out.reshape(up(w, 8), heads * rows_p)

    def _side_by_side(self, parts, starts, cols):
        out = self._zeros((parts[0].shape[0], cols))
        for p, at in zip(parts, starts):
            out[:, at:at + p.shape[1]] = p
        return out

    def _out_matrix(self, value, heads, vdim, vdim_p):
        """W_o [w, heads * vdim] -> [heads * vdim_p, w8]."""
        w = value.shape[0]
        out = self._zeros((heads, vdim_p, up(w, 8)))
        out[:, :vdim, :w] = value.T.reshape(heads, vdim, w)
        return out.reshape(heads * vdim_p, up(w, 8))

    def _pack(self, t):
        c = self.config
        w, wp = c.width, c.width_p
        val = lambda name: self._value(t[name])
        self._add("embed", val("embed"))
        if c.loop is not None:
            b = self._zeros((2 * wp, wp))
            v = val("loop.in").T
            b[:w, :w], b[wp:wp + w, :w] = v[:w], v[w:]
            self._add("loop.in", b)
        for l in c.layers:
            p, a = f"l{l.index}.", l.mixer
            if a.rot.dims:
                self._add(self._rotary_name(a.rot), a.rot.frequencies())
            self._add(p + "norm1", t[p + "norm1"].as_f32())
            (self._pack_latent if a.kind == LATENT else self._pack_retention)(t, p + "mix.", a)
            self._add(p + "mix.o", self._out_matrix(val(p + "mix.o"), a.heads, a.vdim, a.vdim_p))
            if l.mlp is None:
                continue
            self._add(p + "norm2", t[p + "norm2"].as_f32())
            ff, ffp = l.mlp.ff, l.mlp.ff_p
            if isinstance(l.mlp, DenseSpec):
                self._add(p + "mlp.up", self._rows_to_columns(val(p + "mlp.up"), ff, ffp))
                self._add(p + "mlp.down", self._out_matrix(val(p + "mlp.down"), 1, ff, ffp))
                continue
            n = l.mlp.experts
            self._add(p + "mlp.router", self._rows_to_columns(val(p + "mlp.router"), n, up(n, 8)))
            self._add(p + "mlp.router.b", t[p + "mlp.router.b"].as_f32())
            pair, down = self._zeros((n, wp, ffp, 2)), self._zeros((n, ffp, wp))
            for e in range(n):
                pair[e, :w, :ff, 0], pair[e, :w, :ff, 1] = val(f"{p}mlp.e{e}.gate").T, val(f"{p}mlp.e{e}.up").T
                down[e, :ff, :w] = val(f"{p}mlp.e{e}.down").T
            self._add(p + "mlp.experts", pair.reshape(n * wp, 2 * ffp))
            self._add(p + "mlp.experts.down", down.reshape(n * ffp, wp))
        self._pack_head(t, t["final.norm"].as_f32())

    def _pack_latent(self, t, p, a):
        val = lambda name: self._value(t[p + name])
        dkv, order = val("dkv"), a.rot.order(a.rot_dim)
        (q, kv, rot), cols = a.in_columns()
        parts, starts = [self._rows_to_columns(val("dq"), a.q_rank, a.q_rank), self._rows_to_columns(dkv[:a.kv_rank], a.kv_rank, a.kv_rank)], [q, kv]
        if a.rot_dim:
            parts.append(self._rows_to_columns(dkv[a.kv_rank:], a.rot_dim, a.rot_p, order=order))
            starts.append(rot)
        self._add(p + "in", self._side_by_side(parts, starts, cols))
        self._add(p + "dq.norm", t[p + "dq.norm"].as_f32())
        self._add(p + "dkv.norm", t[p + "dkv.norm"].as_f32())
        self._add(p + "sink", t[p + "sink"].as_f32())
        uq = val("uq").reshape(a.heads, a.dim + a.rot_dim, a.q_rank)
        b = self._zeros((a.q_p, a.heads, a.head_p))
        b[:a.q_rank, :, :a.dim] = uq[:, :a.dim].transpose(2, 0, 1)
        b[:a.q_rank, :, a.dim_p:a.dim_p + a.rot_dim] = uq[:, a.dim:][:, order].transpose(2, 0, 1)
        self._add(p + "uq", b.reshape(a.q_p, a.heads * a.head_p))
        # keys and values of cached latents: one product for many rows; head by head for few (the keys transposed: they act on q)
        uk, uv = val("uk").reshape(a.heads, a.dim, a.kv_rank), val("uv").reshape(a.heads, a.vdim, a.kv_rank)
        v0, cols = a.expand_columns()
        b = self._zeros((a.kv_p, cols))
        b[:a.kv_rank, :a.heads * a.dim_p].reshape(a.kv_rank, a.heads, a.dim_p)[:, :, :a.dim] = uk.transpose(2, 0, 1)
        b[:a.kv_rank, v0:v0 + a.heads * a.vdim_p] = self._head_columns(uv, a.vdim_p)
        self._add(p + "expand", b)
        b = self._zeros((a.heads, a.dim_p, a.kv_p))
        b[:, :a.dim, :a.kv_rank] = uk
        self._add(p + "absorb", b)

    def _head_columns(self, value, width):
        """[heads, n, k] -> [k, heads * width]."""
        heads, n, k = value.shape
        out = self._zeros((k, heads, width))
        out[:, :, :n] = value.transpose(2, 0, 1)
        return out.reshape(k, heads * width)

    def _pack_retention(self, t, p, a):
        val = lambda name: self._value(t[p + name])
        order = a.rot.order(a.dim)
        parts = [self._rows_to_columns(val(n), a.dim, a.dim_p, a.heads, order) for n in "qk"] + [
            self._rows_to_columns(val(n), a.vdim, a.vdim_p, a.heads) for n in "vg"]
        starts, cols = a.in_columns()
        self._add(p + "in", self._side_by_side(parts, starts, cols))
        self._add(p + "decay", np.asarray(a.decay, dtype=np.float32))

    # ---- archives ----
    def step_writer(self, rows, capacity, hidden_rows, with_logits):
        """The archive of one step of `rows` tokens: ports `step_in`, `hidden`, and the caches (`l<r>.latent`) and states
        (`l<r>.state`) of every layer run; with `with_logits` also the output head over all rows (port `logits`)."""
        c, es = self.config, self.elem
        s = _Step(self, rows, capacity, hidden_rows)
        sl = s.sl
        hidden = self._hidden(s.w, sl, hidden_rows)
        x = sl.ref(hidden, 0, 4 * rows * c.width)
        self._embed(s.w, sl, s.made, s.ids, x, rows)
        h = s.buffer("h", rows * c.width_p * es)
        both = None
        if c.loop is not None:      # [x | embedding output]: the right half stays for every pass
            both = s.buffer("both", rows * 2 * c.width_p * es)
            self._copy(s, x, both, c.width_p)
        for run, (l, begins_pass) in enumerate(c.runs()):
            p = f"l{l.index}."
            if begins_pass:
                self._copy(s, x, both, 0)
                s.linear(sl.ref(both), "loop.in", [kc.LinearSeg.make(x, c.width, c.width, F32)], 2 * c.width_p, c.width_p)
            s.norm(x, p + "norm1", sl.ref(h))
            (self._latent if l.mixer.kind == LATENT else self._retention)(s, run, l.mixer, p + "mix.", h, x)
            if l.mlp is not None:
                s.norm(x, p + "norm2", sl.ref(h))
                (self._dense if isinstance(l.mlp, DenseSpec) else self._routed)(s, l.mlp, p + "mlp.", h, x)
        if with_logits:
            # this archive's session lends its weights to every other step shape: it holds all of them
            for name in self._constants:
                s.const(name)
            self._logits(s.w, sl, s.made, x, rows)
        return self._end(s.w, sl)

    def _copy(self, s, x, both, column):
        c = self.config
        part = kc.NormPart(kc.NONE, s.sl.ref(both, column * self.elem), 0, c.width, c.width_p, 2 * c.width_p, 0, 0)
        s.call(kc.KernelCall.RmsNormParts(kc.RmsNormPartsCall.make(x, [part], s.rows, c.width, c.eps, self.dtype)))

    def _add_to_residual(self, s, a, b, k, x):
        c = self.config
        s.linear(a, b, [kc.LinearSeg.make(x, c.width, c.width, F32)], k, c.width_p, residual=x)

    def _latent(self, s, run, a, p, h, x):
        c, es, dt, sl, rows = self.config, self.elem, self.dtype, s.sl, s.rows
        ring = a.cache_rows(s.capacity, s.portion)
        cache = s.state(f"l{run}.latent", dt, [ring, a.row_p])
        table = s.table(a.rot)
        rotated = lambda head, begin: (head, begin, a.rot.dims) if a.rot.dims else None
        # latents (f32, still to be normed) and the rotated key part
        kv0, ldd = a.down_columns()
        down = s.buffer("down", 4 * rows * ldd)
        (cq, ckv, crot), cols = a.in_columns()
        segs = [kc.LinearSeg.make(sl.ref(down), a.q_rank, ldd, F32, cq), kc.LinearSeg.make(sl.ref(down, 4 * kv0), a.kv_rank, ldd, F32, ckv)]
        if a.rot_dim:
            segs.append(kc.LinearSeg.make(sl.ref(cache, a.kv_p * es), a.rot_p, a.row_p, dt, crot, row_pos=s.step, ring=True, rotate=rotated(a.rot_p, 0)))
        s.linear(sl.ref(h), p + "in", segs, c.width_p, cols, rot=table)
        latent = s.buffer("latent", rows * a.q_p * es)
        parts = [kc.NormPart(s.const(p + "dq.norm"), sl.ref(latent), 0, a.q_rank, a.q_p, a.q_p, 1, 0),
                 kc.NormPart(s.const(p + "dkv.norm"), sl.ref(cache), kv0, a.kv_rank, a.kv_p, a.row_p, 1, 1)]
        s.call(kc.KernelCall.RmsNormParts(kc.RmsNormPartsCall.make(sl.ref(down), parts, rows, ldd, c.eps, dt, step=s.step)))
        ldq = a.heads * a.head_p
        q = s.buffer("q", rows * ldq * es)
        s.linear(sl.ref(latent), p + "uq", [kc.LinearSeg.make(sl.ref(q), ldq, ldq, dt, rotate=rotated(a.head_p, a.dim_p))], a.q_p, ldq, rot=table)
        # attention
        ldo = a.heads * a.vdim_p
        out = s.buffer("context", rows * ldo * es)
        v0, ecols = a.expand_columns()
        window, scale = a.window or 0, kc.f32_bits(a.scale)
        q2, k2 = (sl.ref(q, a.dim_p * es), sl.ref(cache, a.kv_p * es)) if a.rot_p else (kc.NONE, kc.NONE)
        if dt == F32 or rows <= ABSORB_ROWS:
            ldl = a.heads * a.kv_p
            ql, ol = s.buffer("query latents", rows * ldl * es), s.buffer("value latents", rows * ldl * es)
            s.call(kc.KernelCall.HeadLinear(kc.HeadLinearCall(sl.ref(q), s.const(p + "absorb"), sl.ref(ql), rows, a.heads, a.dim_p, a.kv_p, ldq, a.head_p,
                                                              a.kv_p, a.dim_p * a.kv_p, ldl, a.kv_p, dt)))
            s.call(kc.KernelCall.WindowAttention(kc.WindowAttentionCall(
                sl.ref(ql), sl.ref(cache), sl.ref(cache), q2, k2, s.pos, s.const(p + "sink"), sl.ref(ol), rows, a.heads, 1, a.kv_p, a.kv_p, a.rot_p,
                ldl, a.kv_p, a.row_p, a.row_p, ldq, a.head_p, a.row_p, ldl, ring, kc.WHOLE_CACHE, ring, window, scale, dt)))
            expand = s.const(p + "expand")
            values = kc.rb(expand.slot, v0 * es, expand.length - v0 * es)
            s.call(kc.KernelCall.HeadLinear(kc.HeadLinearCall(sl.ref(ol), values, sl.ref(out), rows, a.heads, a.kv_p, a.vdim_p, ldl, a.kv_p,
                                                              ecols, a.vdim_p, ldo, a.vdim_p, dt)))
        else:
            span, back = a.expand_rows(rows, s.capacity), kc.WHOLE_CACHE if a.window is None else a.window - 1
            ldk = a.heads * a.dim_p
            keys, values = s.buffer("keys", span * ldk * es), s.buffer("values", span * ldo * es)
            s.linear(sl.ref(cache), p + "expand", [kc.LinearSeg.make(sl.ref(keys), ldk, ldk, dt), kc.LinearSeg.make(sl.ref(values), ldo, ldo, dt, v0)],
                     a.kv_p, ecols, m=span, lda=a.row_p, a_pos=s.pos, a_back=back, a_rows=ring)
            s.call(kc.KernelCall.WindowAttention(kc.WindowAttentionCall(
                sl.ref(q), sl.ref(keys), sl.ref(values), q2, k2, s.pos, s.const(p + "sink"), sl.ref(out), rows, a.heads, a.heads, a.dim_p, a.vdim_p, a.rot_p,
                ldq, a.head_p, ldk, ldo, ldq, a.head_p, a.row_p, ldo, span, back, ring, window, scale, dt)))
        self._add_to_residual(s, sl.ref(out), p + "o", ldo, x)

    def _retention(self, s, run, a, p, h, x):
        c, es, dt, sl, rows = self.config, self.elem, self.dtype, s.sl, s.rows
        state = s.state(f"l{run}.state", F32, [a.heads, a.dim_p, a.vdim_p])
        table = s.table(a.rot)
        rotate = (a.dim_p, 0, a.rot.dims) if a.rot.dims else None
        ldk, ldv = a.heads * a.dim_p, a.heads * a.vdim_p
        q, k, v, g = (s.buffer("retention " + n, rows * ld * es) for n, ld in (("q", ldk), ("k", ldk), ("v", ldv), ("g", ldv)))
        (cq, ck, cv, cg), cols = a.in_columns()
        s.linear(sl.ref(h), p + "in", [
            kc.LinearSeg.make(sl.ref(q), ldk, ldk, dt, cq, rotate=rotate), kc.LinearSeg.make(sl.ref(k), ldk, ldk, dt, ck, rotate=rotate),
            kc.LinearSeg.make(sl.ref(v), ldv, ldv, dt, cv), kc.LinearSeg.make(sl.ref(g), ldv, ldv, dt, cg, act=kc.LINEAR_ACT_SILU)], c.width_p, cols, rot=table)
        out = s.buffer("context", rows * ldv * es)
        work = sl.ref(s.buffer("retention work", 4 * rows * ldv)) if dt == BF and rows > 1 else kc.NONE
        s.call(kc.KernelCall.Retention(kc.RetentionCall(
            sl.ref(q), sl.ref(k), sl.ref(v), sl.ref(g), s.const(p + "decay"), s.step, sl.ref(state), sl.ref(out), work, rows, a.heads, a.dim_p, a.vdim_p, a.vdim,
            ldk, ldk, ldv, ldv, ldv, kc.f32_bits(a.dim ** -0.5), kc.f32_bits(c.eps), dt)))
        self._add_to_residual(s, sl.ref(out), p + "o", ldv, x)

    def _dense(self, s, mlp, p, h, x):
        act = s.buffer("act", s.rows * mlp.ff_p * self.elem)
        s.linear(s.sl.ref(h), p + "up", [kc.LinearSeg.make(s.sl.ref(act), mlp.ff_p, mlp.ff_p, self.dtype, act=kc.LINEAR_ACT_GELU_TANH)], self.config.width_p, mlp.ff_p)
        self._add_to_residual(s, s.sl.ref(act), p + "down", mlp.ff_p, x)

    def _routed(self, s, mlp, p, h, x):
        c, es, dt, sl, rows = self.config, self.elem, self.dtype, s.sl, s.rows
        n, ffp, wp = mlp.experts, mlp.ff_p, c.width_p
        tile, most = mlp.tiles(rows)
        shared = rows <= tile           # every tile reads the step's rows as they are
        logits = s.buffer("router", 4 * rows * n)
        weight, place = s.buffer("weight", 4 * rows * mlp.top), s.buffer("place", 4 * rows * mlp.top)
        tiles, source = s.buffer("tiles", 4 * (1 + most)), s.buffer("source", 4 * most * tile)
        s.linear(sl.ref(h), p + "router", [kc.LinearSeg.make(sl.ref(logits), n, n, F32)], wp, up(n, 8))
        s.call(kc.KernelCall.MoePlan(kc.MoePlanCall(sl.ref(logits), s.const(p + "router.b"), s.step, sl.ref(weight), sl.ref(place), sl.ref(tiles), sl.ref(source),
                                                    rows, n, mlp.top, n, tile, most)))
        src = h
        if not shared:
            src = s.buffer("sorted", most * tile * wp * es)
            s.call(kc.KernelCall.Gather(kc.GatherCall(sl.ref(h), sl.ref(source), sl.ref(src), 1, rows, wp, most * tile, I32, dt)))
        act, y = s.buffer("expert act", most * tile * ffp * es), s.buffer("expert out", most * tile * wp * es)
        group = {"m": most * tile, "tiles": sl.ref(tiles), "tile_rows": tile, "experts": n}
        s.linear(sl.ref(src), p + "experts", [kc.LinearSeg.make(sl.ref(act), 2 * ffp, ffp, dt, act=kc.LINEAR_ACT_SILU_GATE)], wp, 2 * ffp,
                 a_shared=rows if shared else 0, **group)
        s.linear(sl.ref(act), p + "experts.down", [kc.LinearSeg.make(sl.ref(y), wp, wp, dt)], ffp, wp, **group)
        s.call(kc.KernelCall.MoeCombine(kc.MoeCombineCall(x, sl.ref(y), sl.ref(weight), sl.ref(place), s.step, rows, c.width, mlp.top, wp, most * tile, dt)))

    def launches(self, rows, with_logits):
        """Calls of one step's archive."""
        return len(self.step_writer(rows, rows, rows, with_logits).calls)
