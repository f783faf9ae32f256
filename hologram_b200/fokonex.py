"""Fokonex: a decoder-only design with parallel attention / feed-forward layers, as `.holo` step archives.

A layer adds `m * (mixer(norm1(x)) + ff(norm2(x)))` to an f32 residual stream x, both branches reading the same x
(RMS norms whose weights are stored around zero). The mixer is grouped-query attention without rotation, with its own
value width, a logarithmic query temperature, a score cap and one sink per query head in the softmax denominator; the
feed-forward is relu(W_up h)^2 through W_down. A layer may reuse another layer's tensors while keeping a cache of its own.

One archive is one step shape: `rows` new tokens of one sequence against a cache of `capacity` rows. Each layer is

    RmsNormMulti   x -> [h1 | h2]
    Linear         [h1 | h2] -> q, rows of the K cache, rows of the V cache (from h1), relu^2 of the up projection (from h2)
    CausalAttention over the cache -> the left part of the activation buffer (the up projection filled the right part)
    Linear         [attention | up] -> x += m * (...)   (W_o and W_down stacked along k)

Head widths are padded with zero columns to multiples of 16 and the model width to a multiple of 8, so that every row
pitch suits TMA whatever the configuration's sizes are; zero columns change no result.
"""
import numpy as np

from . import holo
from . import kernel_call as kc
from .step_model import BF, F32, I32, STEP_IN_IDS, StepModel, up as _up


class AttentionSpec:
    """Sizes and constants of one attention mixer."""

    def __init__(self, heads, kv_heads, dim, vdim, scale, softcap=0.0, temp_coef=0.0, temp_every=0.0):
        if heads <= 0 or kv_heads <= 0 or heads % kv_heads:
            raise ValueError(f"attention: {heads} query heads do not group over {kv_heads} key/value heads")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.softcap, self.temp_coef, self.temp_every = scale, softcap, temp_coef, temp_every
        self.dim_p, self.vdim_p = _up(dim, 16), _up(vdim, 16)

    @classmethod
    def from_dict(cls, d):
        temp = d.get("q_temp") or {}
        return cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]), float(d.get("softcap") or 0.0),
                   float(temp.get("coef", 0.0)), float(temp.get("every", 0.0)))


class LayerSpec:
    def __init__(self, index, mixer, ff, owner):
        self.index, self.mixer, self.ff, self.owner = index, mixer, ff, owner   # ff None = no feed-forward; owner = layer whose tensors it uses
        self.ff_p = _up(ff, 8) if ff is not None else 0


class FokonexConfig:
    ARCHITECTURE = "Fokonex"

    def __init__(self, vocab, width, layers, eps, residual_mult=1.0, logit_scale=1.0):
        self.vocab, self.width, self.layers, self.eps = vocab, width, layers, eps
        self.residual_mult, self.logit_scale = residual_mult, logit_scale
        self.width_p = _up(width, 8)

    @classmethod
    def from_dict(cls, d):
        if d.get("architecture") != cls.ARCHITECTURE:
            raise ValueError(f"config.json names architecture {d.get('architecture')!r}, not {cls.ARCHITECTURE!r}")
        layers = []
        for i, entry in enumerate(d["layers"]):
            if entry["type"] != "attention":
                raise ValueError(f"layer {i}: mixer type {entry['type']!r} is not part of this design")
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not part of this design")
            owner = i
            if entry.get("weights_of") is not None:
                j = int(entry["weights_of"])
                if not 0 <= j < len(d["layers"]) or j == i:
                    raise ValueError(f"layer {i}: weights_of {j}")
                owner, seen = j, {i}
                while d["layers"][owner].get("weights_of") is not None:
                    if owner in seen:
                        raise ValueError(f"layer {i}: weights_of goes in a circle")
                    seen.add(owner)
                    owner = int(d["layers"][owner]["weights_of"])
            layers.append(LayerSpec(i, AttentionSpec.from_dict(entry["mixer"]), int(mlp["ff"]) if mlp is not None else None, owner))
        return cls(int(d["vocab"]), int(d["width"]), layers, float(d["norm"]["eps"]), float(d.get("residual_mult", 1.0)),
                   float(d.get("logit_scale", 1.0)))

    def to_dict(self):
        out = []
        for l in self.layers:
            a = l.mixer
            mixer = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "softcap": a.softcap,
                     "q_temp": {"coef": a.temp_coef, "every": a.temp_every}}
            entry = {"type": "attention", "mixer": mixer, "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}}
            if l.owner != l.index:
                entry["weights_of"] = l.owner
            out.append(entry)
        return {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width, "layers": out, "norm": {"eps": self.eps},
                "residual_mult": self.residual_mult, "logit_scale": self.logit_scale}

    def tensor_shapes(self):
        """Name -> shape of every tensor a checkpoint of this configuration holds."""
        w = self.width
        out = {"embed": (self.vocab, w)}
        for l in self.layers:
            if l.owner != l.index:
                continue
            p, a = f"l{l.index}.", l.mixer
            out[p + "norm1"] = (w,)
            if l.ff is not None:
                out[p + "norm2"] = (w,)
            out[p + "mix.q"], out[p + "mix.k"] = (a.heads * a.dim, w), (a.kv_heads * a.dim, w)
            out[p + "mix.v"], out[p + "mix.sink"] = (a.kv_heads * a.vdim, w), (a.heads,)
            out[p + "mix.o"] = (w, a.heads * a.vdim)
            if l.ff is not None:
                out[p + "mlp.up"], out[p + "mlp.down"] = (l.ff, w), (w, l.ff)
        out["final.norm"], out["head"] = (w,), (self.vocab, w)
        return out


class FokonexModel(StepModel):
    """Configuration and device-layout weights of one model; builds its step archives."""

    CONFIG = FokonexConfig

    @staticmethod
    def _gain(tensor):
        return (np.float32(1.0) + tensor.as_f32()).astype(np.float32)

    def in_columns(self, layer):
        """Where q, k, v and the up projection begin in a layer's input product, and its column count."""
        a = layer.mixer
        q = 0
        k = _up(a.heads * a.dim_p, 32)
        v = k + _up(a.kv_heads * a.dim_p, 32)
        end = v + a.kv_heads * a.vdim_p
        if layer.ff is None:
            return (q, k, v, None), _up(end, 8)
        up = _up(end, 256)      # the up projection reads other columns of A: it starts a tile of its own
        return (q, k, v, up), _up(up + layer.ff, 8)

    def _pack(self, t):
        c = self.config
        w, wp = c.width, c.width_p
        self._add("embed", self._value(t["embed"]))

        def heads_in(src, heads, d, dp):        # [heads * d, w] -> [wp, heads * dp]
            out = self._zeros((wp, heads, dp))
            out[:w, :, :d] = self._value(src).reshape(heads, d, w).transpose(2, 0, 1)
            return out.reshape(wp, heads * dp)

        for l in c.layers:
            if l.owner != l.index:
                continue
            p, a = f"l{l.index}.", l.mixer
            self._add(p + "norm1", self._gain(t[p + "norm1"]))
            (q, k, v, up), cols = self.in_columns(l)
            b = self._zeros((wp, cols))
            for at, name, heads, d, dp in ((q, "q", a.heads, a.dim, a.dim_p), (k, "k", a.kv_heads, a.dim, a.dim_p), (v, "v", a.kv_heads, a.vdim, a.vdim_p)):
                b[:, at:at + heads * dp] = heads_in(t[p + "mix." + name], heads, d, dp)
            o = self._zeros((a.heads, a.vdim_p, wp))
            o[:, :a.vdim, :w] = self._value(t[p + "mix.o"]).T.reshape(a.heads, a.vdim, w)
            o = o.reshape(a.heads * a.vdim_p, wp)
            if l.ff is not None:
                self._add(p + "norm2", self._gain(t[p + "norm2"]))
                b[:w, up:up + l.ff] = self._value(t[p + "mlp.up"]).T
                down = self._zeros((l.ff_p, wp))
                down[:l.ff, :w] = self._value(t[p + "mlp.down"]).T
                o = np.concatenate([o, down])
            self._add(p + "in", b)
            self._add(p + "out", o)
            self._add(p + "sink", t[p + "mix.sink"].as_f32())
        self._pack_head(t, self._gain(t["final.norm"]), c.logit_scale)

    def step_writer(self, rows, capacity, hidden_rows, with_logits):
        """The archive of one step of `rows` tokens: ports `step_in` (i32: position, three unused words, the token ids),
        `hidden` (the residual stream, [hidden_rows, width]), `l<i>.k` / `l<i>.v` (the cache of layer run i); with
        `with_logits` also the output head over all rows (port `logits`)."""
        c, es, dt = self.config, self.elem, self.dtype
        w, sl, made = self._begin()
        step_in = sl.new(4 * (STEP_IN_IDS + rows))
        w.inputs.append(holo.Port("step_in", step_in, STEP_IN_IDS + rows, I32, [STEP_IN_IDS + rows]))
        pos, ids = sl.ref(step_in, 0, 4), sl.ref(step_in, 4 * STEP_IN_IDS)
        x = self._hidden(w, sl, hidden_rows)
        xr = sl.ref(x, 0, 4 * rows * c.width)
        self._embed(w, sl, made, ids, xr, rows)
        # activations: one set per distinct layer geometry, reused by every layer that has it
        work = {}
        for l in c.layers:
            a, p = l.mixer, f"l{l.owner}."
            ka = a.heads * a.vdim_p + l.ff_p
            key = (a.heads, a.dim_p, a.vdim_p, l.ff_p)
            nh = 1 if l.ff is None else 2
            if key not in work:
                work[key] = (sl.new(rows * nh * c.width_p * es), sl.new(rows * a.heads * a.dim_p * es), sl.new(rows * ka * es))
            h, q, act = work[key]
            lk, lv = a.kv_heads * a.dim_p, a.kv_heads * a.vdim_p
            kcache, vcache = sl.new(capacity * lk * es), sl.new(capacity * lv * es)
            w.inputs.append(holo.Port(f"l{l.index}.k", kcache, capacity * lk, dt, [capacity, a.kv_heads, a.dim_p]))
            w.inputs.append(holo.Port(f"l{l.index}.v", vcache, capacity * lv, dt, [capacity, a.kv_heads, a.vdim_p]))
            w.calls.append(kc.KernelCall.RmsNormMulti(kc.RmsNormMultiCall(
                xr, self._const(w, sl, made, p + "norm1"), kc.NONE if l.ff is None else self._const(w, sl, made, p + "norm2"), sl.ref(h),
                rows, c.width, c.width_p, kc.f32_bits(c.eps), dt)))
            (cq, ck, cv, cu), cols = self.in_columns(l)
            segs = [kc.LinearSeg.make(sl.ref(q), a.heads * a.dim_p, a.heads * a.dim_p, dt, cq),
                    kc.LinearSeg.make(sl.ref(kcache), lk, lk, dt, ck, row_pos=pos), kc.LinearSeg.make(sl.ref(vcache), lv, lv, dt, cv, row_pos=pos)]
            if l.ff is not None:
                segs.append(kc.LinearSeg.make(sl.ref(act, a.heads * a.vdim_p * es), l.ff, ka, dt, cu, c.width_p, kc.LINEAR_ACT_RELU2))
            w.calls.append(kc.KernelCall.Linear(kc.LinearCall.make(
                sl.ref(h), self._const(w, sl, made, p + "in"), segs, rows, c.width_p, cols, dt, lda=nh * c.width_p)))
            w.calls.append(kc.KernelCall.CausalAttention(kc.CausalAttentionCall(
                sl.ref(q), sl.ref(kcache), sl.ref(vcache), pos, self._const(w, sl, made, p + "sink"), sl.ref(act), rows, a.heads, a.kv_heads,
                a.dim_p, a.vdim_p, capacity, ka, kc.f32_bits(a.scale), kc.f32_bits(a.softcap), kc.f32_bits(a.temp_coef),
                kc.f32_bits(a.temp_every), dt)))
            seg = kc.LinearSeg.make(xr, c.width, c.width, F32)
            w.calls.append(kc.KernelCall.Linear(kc.LinearCall.make(
                sl.ref(act), self._const(w, sl, made, p + "out"), [seg], rows, ka, c.width_p, dt, residual=xr, alpha=c.residual_mult)))
        if with_logits:
            self._logits(w, sl, made, xr, rows)
        return self._end(w, sl)

    def launches(self, rows, with_logits):
        """Kernel launches of one step, by the archive's call count."""
        return (1 if self.dtype == F32 else 2) + 4 * len(self.config.layers) + (2 if with_logits else 0)
