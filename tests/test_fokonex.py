"""Fokonex on the CPU: configuration, checkpoint reading, the step archives (interpreted call by call and compared with
the plain equations), the cache, the queue and sampling."""
import json

import numpy as np
import pytest

import fokonex_reference as ref
from hologram_b200 import decode as dc
from hologram_b200 import fokonex as fk
from hologram_b200 import kernel_call as kc
from hologram_b200 import models, safetensors_io
from oracle import interp


def make_model(name, dtype=kc.DTYPE_F32, seed=0):
    cfg = ref.CONFIGS[name]
    t = ref.random_tensors(cfg, seed)
    tensors = {n: safetensors_io.Tensor("BF16", ref.to_bf16_bits(v)) for n, v in t.items()}
    return fk.FokonexModel(fk.FokonexConfig.from_dict(cfg), tensors, dtype), ref.Reference(cfg, t)


class InterpretedSteps:
    """Runs a model's step archives on the CPU call interpreter, the caches kept between steps."""

    def __init__(self, model, capacity, hidden_rows):
        self.model, self.capacity, self.hidden_rows = model, capacity, hidden_rows
        self.ports, self.pos = {}, 0

    def _run(self, writer, feeds):
        slots = {s: np.frombuffer(bytes(body), dtype=np.uint8).copy() for s, _, body in writer.inline_constants + writer.weight_constants}
        for p in writer.inputs:
            size = p.element_count * {kc.DTYPE_F32: 4, kc.DTYPE_I32: 4, kc.DTYPE_BF16: 2}[p.dtype]
            if p.name in feeds:
                slots[p.slot] = np.ascontiguousarray(feeds[p.name]).view(np.uint8).reshape(-1).copy()
            else:
                slots[p.slot] = self.ports.get(p.name, np.zeros(size, dtype=np.uint8))
            assert slots[p.slot].size == size
        for s, n in enumerate(writer.slot_bytes):      # every other buffer starts as zeros, as the device workspace's do
            slots.setdefault(s, np.zeros(n, dtype=np.uint8))
        interp.run(writer.calls, slots)
        for p in writer.inputs:
            self.ports[p.name] = slots[p.slot]
        return {p.name: slots[p.slot] for p in writer.outputs}

    def step(self, tokens, pad_to=None):
        rows = pad_to or len(tokens)
        feed = np.zeros(4 + rows, dtype=np.int32)
        feed[0] = self.pos
        feed[4:4 + len(tokens)] = tokens
        vocab = self.model.config.vocab
        if rows == 1:
            out = self._run(self.model.step_writer(1, self.capacity, self.hidden_rows, True), {"step_in": feed})
        else:
            self._run(self.model.step_writer(rows, self.capacity, self.hidden_rows, False), {"step_in": feed})
            out = self._run(self.model.head_writer(len(tokens), self.hidden_rows), {"want": np.arange(len(tokens), dtype=np.int32)})
        self.pos += len(tokens)
        return out["logits"].view(np.float32).reshape(-1, vocab)


@pytest.mark.parametrize("name", sorted(ref.CONFIGS))
def test_archives_compute_the_equations(name):
    """Whole prompt, portions (padded, some past the cache's end) and single tokens, all against the plain model."""
    model, plain = make_model(name)
    rng = np.random.default_rng(1)
    tokens = rng.integers(0, model.config.vocab, size=19)
    want = plain.forward(tokens)
    whole = InterpretedSteps(model, 19, 32).step(tokens)
    assert ref.row_errors(whole, want).max() < 1e-5
    cut = InterpretedSteps(model, 19, 32)
    got = np.concatenate([cut.step(tokens[:2]), cut.step(tokens[2:5], pad_to=4), cut.step(tokens[5:6]), cut.step(tokens[6:16], pad_to=16), cut.step(tokens[16:], pad_to=8)])
    assert ref.row_errors(got, want).max() < 1e-5


def test_archive_in_bf16_stays_close():
    model, plain = make_model("odd", kc.DTYPE_BF16)
    tokens = np.random.default_rng(2).integers(0, model.config.vocab, size=12)
    got = InterpretedSteps(model, 16, 16).step(tokens, pad_to=16)
    assert ref.row_errors(got, plain.forward(tokens)).max() < 4e-2


def test_archive_image_parses_and_its_weights_can_be_left_out():
    from hologram_b200.session import archive_check
    model, _ = make_model("odd")
    full = model.build_step(8, 16, 16, False)
    calls, inputs, outputs, constants = archive_check(full)
    assert calls == model.launches(8, False)
    assert inputs == 2 + 2 * len(model.config.layers) and outputs == 0 and constants > 0
    assert len(model.build_step(8, 16, 16, False, weightless=True)) < len(full) // 2
    head = archive_check(model.build_head(4, 16))
    assert head[0] == 3 and head[2] == 1


def test_layers_that_share_tensors_share_constants_but_not_caches():
    model, _ = make_model("shared")
    w = model.step_writer(4, 8, 8, False)
    names = [p.name for p in w.inputs]
    assert {f"l{i}.{c}" for i in range(3) for c in "kv"} <= set(names)
    linears = [c.u.linear for c in w.calls if c.kind == kc.K_LINEAR]
    assert len({c.b.slot for c in linears[0::2]}) == 1 and len({c.b.slot for c in linears[1::2]}) == 1
    attn = [c.u.causal_attention for c in w.calls if c.kind == kc.K_CAUSAL_ATTENTION]
    assert len({c.k.slot for c in attn}) == 3 and len({c.v.slot for c in attn}) == 3


def test_config_reads_every_field_and_round_trips():
    cfg = ref.CONFIGS["odd"]
    c = fk.FokonexConfig.from_dict(cfg)
    assert (c.vocab, c.width, c.eps, c.residual_mult, c.logit_scale) == (61, 52, 1e-5, 0.7, 0.6)
    a = c.layers[2].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.softcap, a.temp_coef, a.temp_every) == (2, 2, 9, 33, 5.0, 0.3, 16.0)
    assert c.layers[1].ff is None and c.layers[2].ff == 70
    again = fk.FokonexConfig.from_dict(json.loads(json.dumps(c.to_dict())))
    assert again.to_dict() == c.to_dict()
    shared = fk.FokonexConfig.from_dict(ref.CONFIGS["shared"])
    assert [l.owner for l in shared.layers] == [1, 1, 1]
    assert not any(n.startswith(("l0.", "l2.")) for n in shared.tensor_shapes())


@pytest.mark.parametrize("change", [
    lambda d: d.update(architecture="Other"),
    lambda d: d["layers"][0].update(type="recurrent"),
    lambda d: d["layers"][0]["mlp"].update(kind="routed"),
    lambda d: d["layers"][0]["mixer"].update(kv_heads=4),
    lambda d: d["layers"][0].update(weights_of=0),
    lambda d: d["layers"][0].update(weights_of=9),
])
def test_config_refuses_what_the_design_does_not_have(change):
    d = json.loads(json.dumps(ref.CONFIGS["odd"]))
    change(d)
    with pytest.raises(ValueError):
        fk.FokonexConfig.from_dict(d)


def test_checkpoint_loading_and_registry(tmp_path):
    cfg = ref.CONFIGS["plain"]
    t = ref.random_tensors(cfg)
    path = ref.write_model(tmp_path / "m", cfg, t)
    read = safetensors_io.read(tmp_path / "m" / "model.safetensors")
    assert set(read) == set(t)
    assert all(np.array_equal(read[n].as_f32(), t[n]) for n in t)
    m = models.load_model(path, "float32")
    assert isinstance(m, fk.FokonexModel) and m.dtype == kc.DTYPE_F32
    missing = dict(t)
    del missing["l0.mix.sink"]
    ref.write_model(tmp_path / "n", cfg, missing)
    with pytest.raises(ValueError, match="mix.sink"):
        models.load_model(str(tmp_path / "n"))
    ref.write_model(tmp_path / "o", dict(cfg, architecture="Nobody"), t)
    with pytest.raises(ValueError, match="Nobody"):
        models.load_model(str(tmp_path / "o"))


def test_safetensors_reader_checks_bounds(tmp_path):
    p = tmp_path / "t.safetensors"
    h = json.dumps({"a": {"dtype": "F32", "shape": [4], "data_offsets": [0, 16]}}).encode()
    p.write_bytes(len(h).to_bytes(8, "little") + h + b"\0" * 8)
    with pytest.raises(ValueError):
        safetensors_io.read(p)
    p.write_bytes(len(h).to_bytes(8, "little") + h + np.arange(4, dtype=np.float32).tobytes())
    assert np.array_equal(safetensors_io.read(p)["a"].as_f32(), np.arange(4))


def test_input_product_columns_and_padding():
    """q, k, v and up sit where the call says, the up projection on a tile boundary, everything else is zero."""
    model, _ = make_model("odd")
    l = model.config.layers[0]
    (q, k, v, up), cols = model.in_columns(l)
    assert q == 0 and k % 32 == 0 and v % 32 == 0 and up % 256 == 0 and cols % 8 == 0
    b = model._constants["l0.in"][0]
    t = ref.random_tensors(ref.CONFIGS["odd"])
    assert b.shape == (model.config.width_p, cols) and not b[model.config.width:].any()
    heads = b[:52, :6 * 32].reshape(52, 6, 32)
    assert np.array_equal(heads[:, :, :20], t["l0.mix.q"].reshape(6, 20, 52).transpose(2, 0, 1)) and not heads[:, :, 20:].any()
    assert np.array_equal(b[:52, up:up + 37], t["l0.mlp.up"].T)
    used = np.zeros(cols, dtype=bool)
    for at, n in ((q, 6 * 32), (k, 2 * 32), (v, 2 * 32), (up, 37)):
        used[at:at + n] = True
    assert not b[:, ~used].any()


class FakeRunner:
    """Stands in for the step function: the next token is (last token + 1) mod vocab; records its calls."""

    def __init__(self, capacity=32, max_rows=8, vocab=10):
        self.cache = dc.SequenceCache(capacity)
        self.max_rows, self.vocab, self.calls = max_rows, vocab, []

    def step(self, seq, tokens, want=None):
        self.cache.acquire(seq)
        self.cache.check(len(tokens))
        self.cache.length += len(tokens)
        self.calls.append((seq, list(tokens)))
        want = [len(tokens) - 1] if want is None else want
        out = np.zeros((len(want), self.vocab), dtype=np.float32)
        for i, w in enumerate(want):
            out[i, (tokens[w] + 1) % self.vocab] = 1.0
        return out

    def end(self, seq):
        self.cache.release(seq)


def test_scheduler_runs_requests_one_after_another_in_portions():
    r = FakeRunner()
    s = dc.Scheduler(r, portion=3)
    a, b = dc.Request([1, 2, 3, 4, 5, 6, 7], 3), dc.Request([8], 4, stop={1})
    s.submit(a)
    s.submit(b)
    events = list(s.run())
    assert a.tokens == [8, 9, 0] and b.tokens == [9, 0, 1]
    assert events == [(0, 8), (0, 9), (0, 0), (1, 9), (1, 0), (1, 1)]
    assert [t for i, t in r.calls if i == 0] == [[1, 2, 3], [4, 5, 6], [7], [8], [9]]
    assert r.cache.owner is None


def test_scheduler_gives_the_cache_back_when_a_step_fails():
    r = FakeRunner(capacity=5)
    s = dc.Scheduler(r)
    with pytest.raises(dc.CacheFull):
        s.submit(dc.Request([1] * 4, 3))
    with pytest.raises(ValueError):
        s.submit(dc.Request([], 3))
    s.submit(dc.Request([1, 2], 3))
    r.cache.capacity = 2
    with pytest.raises(dc.CacheFull):
        list(s.run())
    assert r.cache.owner is None


def test_cache_is_held_by_one_sequence_until_released():
    c = dc.SequenceCache(4)
    c.acquire("a")
    c.length = 3
    with pytest.raises(dc.CacheFull):
        c.acquire("b")
    with pytest.raises(dc.CacheFull):
        c.check(2)
    c.release("b")
    assert c.owner == "a"
    c.release("a")
    c.acquire("b")
    assert c.length == 0


def test_sampler():
    logits = np.array([0.0, 3.0, 1.0, 2.9], dtype=np.float32)
    assert dc.Sampler()(logits) == 1
    draws = [dc.Sampler(temperature=1.0, top_k=2, seed=s)(logits) for s in range(40)]
    assert set(draws) == {1, 3}
    assert dc.Sampler(0.5, 0, 7)(logits) == dc.Sampler(0.5, 0, 7)(logits)
    hot = [dc.Sampler(100.0, 0, s)(logits) for s in range(60)]
    assert set(hot) == {0, 1, 2, 3}


def test_row_buckets():
    assert [dc.bucket(n) for n in (1, 2, 3, 4, 5, 37, 64, 65)] == [1, 2, 4, 4, 8, 64, 64, 128]


def test_command_line_lists_architectures(capsys):
    from hologram_b200.__main__ import main
    assert main(["models"]) == 0
    assert "Fokonex" in capsys.readouterr().out.split()
