"""Zisevik on the CPU: configuration, weight packing, and the step archives (interpreted call by call and compared with the
plain equations)."""
import json

import numpy as np
import pytest

import zisevik_reference as ref
from hologram_b200 import kernel_call as kc
from hologram_b200 import models, safetensors_io
from hologram_b200 import zisevik as zk
from test_fokonex import InterpretedSteps


def make_model(name, dtype=kc.DTYPE_F32, seed=0):
    cfg = ref.CONFIGS[name]
    t = ref.random_tensors(cfg, seed)
    tensors = {n: safetensors_io.Tensor("BF16", ref.to_bf16_bits(v)) for n, v in t.items()}
    return zk.ZisevikModel(zk.ZisevikConfig.from_dict(cfg), tensors, dtype), ref.Reference(cfg, t)


class Steps(InterpretedSteps):
    """The interpreter of step archives, with the count of real rows in every step."""

    def _run(self, writer, feeds):
        if "step_in" in feeds:
            feeds["step_in"][1] = self.real
        return super()._run(writer, feeds)

    def step(self, tokens, pad_to=None):
        self.real = len(tokens)
        return super().step(tokens, pad_to)


@pytest.mark.parametrize("name", ["odd", "looped", "plain"])
def test_archives_compute_the_equations(name):
    """Whole prompt, portions (padded) and single tokens, all against the plain model."""
    model, plain = make_model(name)
    tokens = np.random.default_rng(1).integers(0, model.config.vocab, size=23)
    want = plain.forward(tokens)
    assert ref.row_errors(Steps(model, 23, 32).step(tokens, pad_to=32), want).max() < 1e-5
    cut = Steps(model, 23, 32)
    got = np.concatenate([cut.step(tokens[:2]), cut.step(tokens[2:5], pad_to=4), cut.step(tokens[5:6]), cut.step(tokens[6:19], pad_to=16), cut.step(tokens[19:], pad_to=4)])
    assert ref.row_errors(got, want).max() < 1e-5


@pytest.mark.parametrize("name", ["odd", "looped"])
def test_archives_in_bf16_stay_close_on_both_attention_paths(name):
    model, plain = make_model(name, kc.DTYPE_BF16)
    tokens = np.random.default_rng(2).integers(0, model.config.vocab, size=30)
    want = plain.forward(tokens)
    steps = Steps(model, 32, 32)
    got = np.concatenate([steps.step(tokens[:9], pad_to=16), steps.step(tokens[9:], pad_to=32)])
    assert np.median(ref.row_errors(got, want)) < 5e-2


def test_caches_are_rings_and_padding_rows_leave_no_trace():
    """A window of 7 and portions of 8: 128 ring rows serve 300 positions, in f32 and through the expanded keys."""
    cfg = ref.config(40, 24, [ref.attention_layer(2, 6, 4, 5, 9, 8, 7, None)])
    t = ref.random_tensors(cfg, 3)
    tensors = {n: safetensors_io.Tensor("BF16", ref.to_bf16_bits(v)) for n, v in t.items()}
    tokens = np.random.default_rng(3).integers(0, 40, size=300)
    want = ref.Reference(cfg, t).forward(tokens)
    for dtype, rows, limit in ((kc.DTYPE_F32, 8, 1e-5), (kc.DTYPE_BF16, 32, 6e-2)):
        model = zk.ZisevikModel(zk.ZisevikConfig.from_dict(cfg), tensors, dtype)
        assert model.config.layers[0].mixer.cache_rows(1000, rows) == 128
        steps = Steps(model, 1000, rows)
        got = np.concatenate([steps.step(tokens[i:i + rows - 3], pad_to=rows) for i in range(0, 300, rows - 3)])
        assert ref.row_errors(got, want).max() < limit


def test_states_start_from_zero_with_every_sequence():
    model, plain = make_model("looped")
    steps = Steps(model, 32, 8)
    rng = np.random.default_rng(4)
    for _ in range(2):
        tokens = rng.integers(0, model.config.vocab, size=11)
        steps.pos = 0
        plain.reset()
        got = np.concatenate([steps.step(tokens[:7], pad_to=8), steps.step(tokens[7:])])
        assert ref.row_errors(got, plain.forward(tokens)).max() < 1e-5


def test_plain_model_does_not_depend_on_the_cut():
    _, plain = make_model("odd")
    tokens = np.random.default_rng(5).integers(0, 61, size=17)
    want = plain.forward(tokens)
    plain.reset()
    assert np.allclose(np.concatenate([plain.forward(tokens[:6]), plain.forward(tokens[6:])]), want, atol=1e-10)


def test_archive_images_parse_and_lend_their_weights():
    from hologram_b200.session import archive_check
    for name in ref.CONFIGS:
        model, _ = make_model(name, kc.DTYPE_BF16)
        root = model.step_writer(1, 64, 64, True)
        names = {p.name for p in root.inputs}
        kinds = [l.mixer.kind for l, _ in model.config.runs()]
        assert {f"l{r}.{'latent' if k == zk.LATENT else 'state'}" for r, k in enumerate(kinds)} <= names
        held = {bytes(b) for b in root.known_fingerprints.values()}
        for rows in (2, 32, 256):
            w = model.step_writer(rows, 64, 256, False)
            calls, inputs, outputs, _ = archive_check(w.finish())
            assert calls == len(w.calls) and inputs == len(names) and outputs == 0
            assert {bytes(b) for b in w.known_fingerprints.values()} <= held


def test_config_reads_every_field_and_round_trips():
    for cfg in ref.CONFIGS.values():
        c = zk.ZisevikConfig.from_dict(cfg)
        assert zk.ZisevikConfig.from_dict(json.loads(json.dumps(c.to_dict()))).to_dict() == c.to_dict()
        assert {n: tuple(s) for n, s in c.tensor_shapes().items()} == {n: v.shape for n, v in ref.random_tensors(cfg).items()}
        assert [(l.index, b) for l, b in c.runs()] == ref.layer_runs(cfg)
    a = zk.ZisevikConfig.from_dict(ref.CONFIGS["odd"]).layers[1].mixer
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank, a.window, a.rot.dims, a.rot.base) == (3, 20, 6, 11, 27, 23, 7, 6, 10000.0)


@pytest.mark.parametrize("change", [
    lambda d: d.update(architecture="Other"),
    lambda d: d["layers"][0].update(type="attention"),
    lambda d: d["layers"][0]["mlp"].update(kind="pooled"),
    lambda d: d["layers"][0]["mlp"]["router"].update(top=6),
    lambda d: d["layers"][0]["mixer"]["decay"].pop(),
    lambda d: d["layers"][1]["mixer"]["mask"].update(size=0),
    lambda d: d["layers"][1]["mixer"]["rot"].update(dims=8),
    lambda d: d["loop"].update(stop=9),
    lambda d: d["loop"].update(times=0),
])
def test_config_refuses_what_the_design_does_not_have(change):
    d = json.loads(json.dumps(ref.CONFIGS["odd"]))
    change(d)
    with pytest.raises(ValueError):
        zk.ZisevikConfig.from_dict(d)


def test_checkpoint_loading_and_registry(tmp_path):
    cfg = ref.CONFIGS["looped"]
    t = ref.random_tensors(cfg)
    m = models.load_model(ref.write_model(tmp_path / "m", cfg, t), "float32")
    assert isinstance(m, zk.ZisevikModel) and m.dtype == kc.DTYPE_F32
    assert set(models.ARCHITECTURES) == {"Fokonex", "Zisevik"}
    for name in ("loop.in", "l0.mlp.e6.down", "l1.mix.sink"):
        missing = {n: v for n, v in t.items() if n != name}
        with pytest.raises(ValueError, match=name.replace(".", r"\.")):
            models.load_model(ref.write_model(tmp_path / name, cfg, missing))


def test_rotated_pairs_are_stored_side_by_side():
    rot = zk.Rotation(6, 100.0)
    assert rot.order(8).tolist() == [0, 3, 1, 4, 2, 5, 6, 7]
    hi, lo = rot.frequencies()
    exact = 100.0 ** (-2.0 * np.arange(3) / 6) / (2.0 * np.pi)
    assert np.abs(hi.astype(np.float64) + lo - exact).max() < 1e-15 * 2
    model, _ = make_model("odd")
    t = ref.random_tensors(ref.CONFIGS["odd"])
    a = model.config.layers[0].mixer
    (q, k, v, g), cols = a.in_columns()
    b = model._constants["l0.mix.in"][0]
    assert b.shape == (56, cols) and k % 32 == 0 and v % 32 == 0 and g % 32 == 0
    got = b[:52, k:k + 3 * 16].reshape(52, 3, 16)
    want = t["l0.mix.k"].reshape(3, 10, 52)[:, a.rot.order(10)]
    assert np.array_equal(got[:, :, :10], want.transpose(2, 0, 1)) and not got[:, :, 10:].any()


def test_routed_tiles_always_suffice():
    rng = np.random.default_rng(6)
    for experts, top, rows in ((5, 3, 1), (16, 2, 16), (64, 6, 64), (7, 1, 200), (16, 4, 300), (3, 3, 129)):
        spec = zk.RoutedSpec(experts, top, 8)
        tile, most = spec.tiles(rows)
        for _ in range(20):
            bias = rng.standard_normal(experts) * rng.choice([0.0, 3.0])
            chosen = np.argsort(-(rng.standard_normal((rows, experts)) + bias), axis=1)[:, :top]
            counts = np.bincount(chosen.reshape(-1), minlength=experts)
            need = (counts > 0).sum() if rows <= tile else (-(-counts // tile)).sum()
            assert need <= most


def test_launches_counts_the_calls():
    model, _ = make_model("plain", kc.DTYPE_BF16)
    assert model.launches(1, True) == len(model.step_writer(1, 8, 8, True).calls)
