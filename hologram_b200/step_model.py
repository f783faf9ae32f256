"""What decoder models served as `.holo` step archives have in common: a checkpoint packed into the kernels' layouts, the
slots of an archive under construction, the embedding at the start of a step and the output head at its end.

An archive is one step shape: `rows` new tokens of one sequence. Its ports are `step_in` (i32: the position of the first row,
the number of real rows, two unused words, the token ids), `hidden` (the f32 residual stream, [hidden_rows, width]) and the
model's caches and states; sessions of one model share the buffers of ports that have the same name.
"""
import json
import os

import numpy as np

from . import holo
from . import kernel_call as kc
from . import safetensors_io

BF, F32, I32 = kc.DTYPE_BF16, kc.DTYPE_F32, kc.DTYPE_I32
STEP_IN_IDS = 4            # the token ids follow four words: the position of the step's first row, the number of real rows, two unused


def up(n, multiple):
    return (n + multiple - 1) // multiple * multiple


class Slots:
    """Slot numbers and sizes of one archive under construction."""

    def __init__(self):
        self.nbytes = []

    def new(self, nbytes):
        self.nbytes.append(int(nbytes))
        return len(self.nbytes) - 1

    def ref(self, slot, offset=0, length=None):
        return kc.rb(slot, offset, self.nbytes[slot] - offset if length is None else length)


class StepModel:
    """Configuration and device-layout weights of one model. A subclass names its CONFIG class (ARCHITECTURE, from_dict,
    tensor_shapes, and the fields vocab, width, width_p, eps), packs its weights in `_pack` and writes a step's calls in `step_writer`."""

    CONFIG = None

    def __init__(self, config, tensors, dtype=BF):
        self.config, self.dtype = config, dtype
        self.elem = 2 if dtype == BF else 4
        missing = [n for n, s in config.tensor_shapes().items() if n not in tensors or tuple(tensors[n].shape) != tuple(s)]
        if missing:
            raise ValueError(f"checkpoint: missing or misshaped tensors: {', '.join(missing[:5])}")
        self._constants = {}       # name -> (array, fingerprint)
        self._pack(tensors)

    @classmethod
    def load(cls, path, dtype=BF):
        with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
            config = cls.CONFIG.from_dict(json.load(f))
        return cls(config, safetensors_io.read(os.path.join(path, "model.safetensors")), dtype)

    # ---- weights in the layout the kernels read: [in, out], columns of several products side by side ----
    def _value(self, tensor):
        return tensor.as_bf16() if self.dtype == BF else tensor.as_f32()

    def _zeros(self, shape):
        return np.zeros(shape, dtype=np.uint16 if self.dtype == BF else np.float32)

    def _add(self, name, array):
        array = np.ascontiguousarray(array)
        self._constants[name] = (array, holo.fingerprint(array.view(np.uint8).reshape(-1).data))

    def _pack(self, tensors):
        raise NotImplementedError

    def _pack_head(self, t, gain, logit_scale=1.0):
        c = self.config
        self.logit_scale = logit_scale
        self._add("final.norm", gain)
        head = self._zeros((c.width_p, up(c.vocab, 8)))
        head[:c.width, :c.vocab] = self._value(t["head"]).T
        self._add("head", head)

    # ---- archives ----
    def _begin(self):
        return holo.HoloWriter(), Slots(), {}

    def _end(self, w, sl):
        w.exec_plan = [[i] for i in range(len(w.calls))]
        w.slot_bytes = list(sl.nbytes)
        return w

    def _const(self, w, sl, made, name):
        if name not in made:
            array, fp = self._constants[name]
            made[name] = sl.new(array.nbytes)
            w.add_constant(made[name], F32 if array.dtype == np.float32 else BF, array.view(np.uint8).reshape(-1).data, known_fingerprint=fp)
        return sl.ref(made[name])

    def _hidden(self, w, sl, hidden_rows):
        n = hidden_rows * self.config.width
        s = sl.new(4 * n)
        w.inputs.append(holo.Port("hidden", s, n, F32, [hidden_rows, self.config.width]))
        return s

    def _embed(self, w, sl, made, ids, x, rows):
        """Embedding rows, widened to f32, into the residual stream."""
        c, dt = self.config, self.dtype
        emb = x if dt == F32 else sl.ref(sl.new(rows * c.width * 2))
        w.calls.append(kc.KernelCall.Gather(kc.GatherCall(self._const(w, sl, made, "embed"), ids, emb, 1, c.vocab, c.width, rows, I32, dt)))
        if dt != F32:
            w.calls.append(kc.KernelCall.Cast(kc.CastCall(emb, x, rows * c.width, BF, F32)))

    def _logits(self, w, sl, made, x, rows):
        """final norm and output head over `rows` rows of x; the f32 logits are port `logits`."""
        c, es = self.config, self.elem
        h, logits = sl.new(rows * c.width_p * es), sl.new(4 * rows * c.vocab)
        w.calls.append(kc.KernelCall.RmsNormMulti(kc.RmsNormMultiCall(
            x, self._const(w, sl, made, "final.norm"), kc.NONE, sl.ref(h), rows, c.width, c.width_p, kc.f32_bits(c.eps), self.dtype)))
        seg = kc.LinearSeg.make(sl.ref(logits), c.vocab, c.vocab, F32)
        w.calls.append(kc.KernelCall.Linear(kc.LinearCall.make(
            sl.ref(h), self._const(w, sl, made, "head"), [seg], rows, c.width_p, up(c.vocab, 8), self.dtype, alpha=self.logit_scale)))
        w.outputs.append(holo.Port("logits", logits, rows * c.vocab, F32, [rows, c.vocab]))

    def build_step(self, rows, capacity, hidden_rows, with_logits, weightless=False):
        return self.step_writer(rows, capacity, hidden_rows, with_logits).finish(weightless=weightless)

    def build_head(self, rows, hidden_rows, weightless=False):
        return self.head_writer(rows, hidden_rows).finish(weightless=weightless)

    def step_writer(self, rows, capacity, hidden_rows, with_logits):
        """The archive of one step of `rows` tokens; with `with_logits` also the output head over all rows (port `logits`)."""
        raise NotImplementedError

    def head_writer(self, rows, hidden_rows):
        """The archive that turns `rows` chosen rows of the residual stream (port `want`, i32) into logits."""
        c = self.config
        w, sl, made = self._begin()
        x = self._hidden(w, sl, hidden_rows)
        want = sl.new(4 * rows)
        w.inputs.append(holo.Port("want", want, rows, I32, [rows]))
        picked = sl.new(4 * rows * c.width)
        w.calls.append(kc.KernelCall.Gather(kc.GatherCall(sl.ref(x), sl.ref(want), sl.ref(picked), 1, hidden_rows, c.width, rows, I32, F32)))
        self._logits(w, sl, made, sl.ref(picked), rows)
        return self._end(w, sl)
