"""Fokonex on the GPU: every mechanism alone, then whole models through the step runner, the queue and the trace replay."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import fokonex_reference as ref
from hologram_b200 import kernel_call as kc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF = kc.DTYPE_F32, kc.DTYPE_BF16


def store(x, dtype):
    return ref.to_bf16_bits(x) if dtype == BF else np.ascontiguousarray(x, dtype=np.float32)


def load(raw, dtype):
    return ref.from_bf16_bits(raw.view(np.uint16)) if dtype == BF else raw.view(np.float32)


def rounded(x, dtype):
    return ref.bf16(x) if dtype == BF else np.asarray(x, dtype=np.float32)


def workspace(backend, arrays, outputs):
    """Slots 0.. hold `arrays`; then `outputs` buffers of the given byte counts."""
    import hologram_b200 as hb
    ws = hb.DeviceWorkspace(backend, len(arrays) + len(outputs))
    for i, a in enumerate(arrays):
        ws.put(i, a)
    for i, n in enumerate(outputs):
        ws.alloc(len(arrays) + i, n)
    return ws


# ---- norms ----
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rows,feature,step,two", [(1, 52, 56, True), (3, 64, 64, False), (70, 1030, 1032, True), (2, 5120, 5120, True), (1, 7, 8, False), (2, 17000, 17000, False)])
def test_rms_norm_multi(backend, dtype, rows, feature, step, two):
    rng = np.random.default_rng(0)
    x = rng.standard_normal((rows, feature)).astype(np.float32) * 3
    x[0] *= 1e-3                                          # eps matters there
    w = [(0.5 * rng.standard_normal(feature)).astype(np.float32) for _ in range(2 if two else 1)]
    gammas = [(1 + v).astype(np.float32) for v in w]
    n = len(gammas)
    ws = workspace(backend, [x] + gammas, [rows * n * step * (2 if dtype == BF else 4)])
    backend.dispatch(kc.KernelCall.RmsNormMulti(kc.RmsNormMultiCall(
        kc.rb(0), kc.rb(1), kc.rb(2) if two else kc.NONE, kc.rb(1 + n), rows, feature, step, kc.f32_bits(1e-5), dtype)), ws)
    got = load(ws.read(1 + n, rows * n * step * (2 if dtype == BF else 4)), dtype).reshape(rows, n, step)
    for i in range(n):
        want = ref.rms_norm(x, w[i], 1e-5)
        assert np.abs(got[:, i, :feature] - want).max() < (2e-2 if dtype == BF else 1e-5)
        assert np.abs(got[:, i, :feature] - want).max() / np.abs(want).max() < (4e-3 if dtype == BF else 1e-6)
        assert not got[:, i, feature:].any()


# ---- products ----
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("m,w,widths,up", [
    (1, 52, (40, 24, 33), 37), (1, 256, (384, 128, 128), 1000), (5, 104, (64, 32, 48), 40), (64, 512, (256, 64, 96), 512), (130, 192, (96, 33, 40), 300),
    (300, 320, (256, 64, 64), 640), (4096, 128, (1024, 256, 256), 2048), (2048, 256, (512, 128, 128), 2048)])
def test_linear_segments(backend, dtype, m, w, widths, up):
    """Three segments of the first half of A (two of them appended to a cache at a device-side row) and a squared-relu one
    of the second half."""
    if dtype == F32 and m * w * up > 1 << 27:
        pytest.skip("the per-cell kernel needs no large case")
    rng = np.random.default_rng(m + w)
    wp = (w + 7) // 8 * 8
    a = np.zeros((m, 2, wp), dtype=np.float32)
    a[:, :, :w] = rounded(rng.standard_normal((m, 2, w)), dtype)
    begins, col = [], 0
    for n in widths:
        begins.append(col)
        col = (col + n + 31) // 32 * 32
    cu = (col + 255) // 256 * 256
    cols = (cu + up + 7) // 8 * 8
    b = np.zeros((wp, cols), dtype=np.float32)
    parts = []
    for at, n in list(zip(begins, widths)) + [(cu, up)]:
        p = rounded(rng.standard_normal((w, n)) / np.sqrt(w), dtype)
        b[:w, at:at + n] = p
        parts.append(p)
    es = 2 if dtype == BF else 4
    first, room = 3, 3 + max(1, m - 2)                     # the last two rows fall off the end of the cache
    ld_up = up + 8
    pad = store(np.full((m, ld_up), 7.0), dtype)           # columns around the segment stay as they are
    cache = [store(np.full((room, n), -5.0), dtype) for n in widths[1:]]
    ws = workspace(backend, [store(a, dtype), store(b, dtype), np.array([first], np.int32), cache[0], cache[1], pad], [m * widths[0] * 4])
    seg = [kc.LinearSeg(kc.rb(6), kc.NONE, begins[0], widths[0], 0, widths[0], 0, F32),
           kc.LinearSeg(kc.rb(3, 0, room * widths[1] * es), kc.rb(2), begins[1], widths[1], 0, widths[1], 0, dtype),
           kc.LinearSeg(kc.rb(4, 0, room * widths[2] * es), kc.rb(2), begins[2], widths[2], 0, widths[2], 0, dtype),
           kc.LinearSeg(kc.rb(5, 8 * es), kc.NONE, cu, up, wp, ld_up, kc.LINEAR_ACT_RELU2, dtype)]
    backend.dispatch(kc.KernelCall.Linear(kc.LinearCall.make(kc.rb(0), kc.rb(1), seg, m, wp, cols, dtype, lda=2 * wp, alpha=0.75)), ws)
    tol = 6e-3 if dtype == BF else 2e-6
    close = lambda got, want: np.abs(got - want).max() <= tol * max(1.0, np.abs(want).max())
    h = a[:, :, :w].astype(np.float64)
    assert close(load(ws.read(6, m * widths[0] * 4), F32).reshape(m, -1), 0.75 * h[:, 0] @ parts[0])
    for s, n, p in ((3, widths[1], parts[1]), (4, widths[2], parts[2])):
        got = load(ws.read(s, room * n * es), dtype).reshape(room, n)
        assert (got[:first] == -5).all() and close(got[first:], (0.75 * h[:, 0] @ p)[:room - first])
    got = load(ws.read(5, m * ld_up * es), dtype).reshape(m, ld_up)
    assert (got[:, :8] == 7).all() and close(got[:, 8:], 0.75 * ref.relu_squared(h[:, 1] @ parts[3]))


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("m,k,n", [(1, 72, 52), (1, 2048, 1024), (17, 136, 96), (200, 264, 100), (2048, 512, 2048)])
def test_linear_adds_into_the_residual_stream(backend, dtype, m, k, n):
    if dtype == F32 and m * k * n > 1 << 27:
        pytest.skip("the per-cell kernel needs no large case")
    rng = np.random.default_rng(k)
    a, x = rounded(rng.standard_normal((m, k)), dtype), rng.standard_normal((m, n)).astype(np.float32)
    cols = (n + 7) // 8 * 8
    b = np.zeros((k, cols), dtype=np.float32)
    b[:, :n] = rounded(rng.standard_normal((k, n)) / np.sqrt(k), dtype)
    ws = workspace(backend, [store(a, dtype), store(b, dtype), x], [])
    c = kc.LinearCall.make(kc.rb(0), kc.rb(1), [kc.LinearSeg(kc.rb(2), kc.NONE, 0, n, 0, n, 0, F32)], m, k, cols, dtype, residual=kc.rb(2), alpha=0.3)
    backend.dispatch(kc.KernelCall.Linear(c), ws)
    want = x + 0.3 * (a.astype(np.float64) @ b[:, :n])
    assert np.abs(load(ws.read(2, m * n * 4), F32).reshape(m, n) - want).max() < 3e-5      # accumulation is f32 for both


def test_linear_refuses_what_it_cannot_do(backend):
    from hologram_b200 import BackendError
    ws = workspace(backend, [np.zeros(64 * 64, np.float32)] * 3, [])
    seg = lambda **k: kc.LinearSeg(kc.rb(2), kc.NONE, k.get("at", 0), k.get("n", 32), k.get("ko", 0), k.get("ld", 32), k.get("act", 0), F32)
    for segs in ([seg(at=8)], [seg(), seg(at=33)], [seg(n=80)], [seg(ko=40)], [seg(ld=16)], [seg(act=9)], [seg(), seg(at=32, ko=16)]):
        with pytest.raises(BackendError):
            backend.dispatch(kc.KernelCall.Linear(kc.LinearCall.make(kc.rb(0), kc.rb(1), segs, 4, 32, 64, F32, lda=64)), ws)


# ---- attention ----
def run_attention(backend, q, k, v, first, scale, softcap, coef, every, sinks, dtype, cache_rows=None, stale=None, ld_extra=0):
    """The CausalAttention call over a cache that may be longer than the keys (its other rows hold `stale`)."""
    rows, heads, dim = q.shape
    length, groups, vdim = k.shape[0], k.shape[1], v.shape[2]
    cache_rows = cache_rows or length
    kk, vv = np.zeros((cache_rows, groups, dim), np.float32), np.zeros((cache_rows, groups, vdim), np.float32)
    if stale is not None:
        kk[:], vv[:] = stale, stale
    kk[:length], vv[:length] = k, v
    ld = heads * vdim + ld_extra
    es = 2 if dtype == BF else 4
    ws = workspace(backend, [store(q, dtype), store(kk, dtype), store(vv, dtype), np.array([first], np.int32), np.zeros(heads, np.float32) if sinks is None else sinks.astype(np.float32)],
                   [rows * ld * es])
    backend.dispatch(kc.KernelCall.CausalAttention(kc.CausalAttentionCall(
        kc.rb(0), kc.rb(1), kc.rb(2), kc.rb(3), kc.NONE if sinks is None else kc.rb(4), kc.rb(5), rows, heads, groups, dim, vdim, cache_rows, ld,
        kc.f32_bits(scale), kc.f32_bits(softcap), kc.f32_bits(coef), kc.f32_bits(every), dtype)), ws)
    return load(ws.read(5, rows * ld * es), dtype).reshape(rows, ld)[:, :heads * vdim].reshape(rows, heads, vdim)


def random_attention(rows, heads, groups, dim, vdim, length, seed, amp=1.0):
    rng = np.random.default_rng(seed)
    return (ref.bf16(rng.standard_normal((rows, heads, dim)) * amp), ref.bf16(rng.standard_normal((length, groups, dim))),
            ref.bf16(rng.standard_normal((length, groups, vdim))), rng.standard_normal(heads) + 1.0)


ATTENTION_SHAPES = [   # rows, heads, kv heads, dim, vdim, first position, cache rows
    (1, 6, 2, 48, 80, 0, 64), (1, 6, 2, 48, 80, 15, 64), (1, 6, 2, 48, 80, 16, 64), (1, 16, 4, 128, 128, 1500, 1600), (3, 6, 2, 48, 80, 126, 200),
    (16, 4, 4, 32, 16, 40, 60), (2, 4, 1, 256, 256, 300, 310), (1, 2, 2, 16, 176, 33, 40), (9, 5, 1, 64, 96, 100, 128),
    (128, 6, 2, 48, 80, 0, 128), (129, 4, 4, 64, 64, 0, 129), (100, 12, 2, 96, 48, 28, 130), (77, 5, 1, 32, 112, 51, 128), (65, 2, 1, 128, 128, 700, 800),
    (140, 2, 2, 256, 256, 0, 150), (260, 4, 2, 80, 144, 255, 520), (70, 10, 1, 16, 32, 3, 73)]


@pytest.mark.parametrize("shape", ATTENTION_SHAPES, ids=lambda s: "-".join(map(str, s)))
def test_attention_bf16(backend, shape):
    rows, heads, groups, dim, vdim, first, cache_rows = shape
    q, k, v, sinks = random_attention(rows, heads, groups, dim, vdim, first + rows, seed=rows + dim)
    got = run_attention(backend, q, k, v, first, dim ** -0.5, 25.0, 0.3, 16, sinks, BF, cache_rows, stale=300.0, ld_extra=16)
    want = ref.attention(q, k, v, first, dim ** -0.5, 25.0, 0.3, 16, sinks)
    assert np.abs(got - want).max() / np.abs(want).max() < 1e-2


@pytest.mark.parametrize("shape", [s for s in ATTENTION_SHAPES[9:] if s[3] <= 128 and s[4] <= 128] + [(640, 4, 2, 64, 64, 700, 1400), (1000, 2, 1, 128, 128, 0, 1000)],
                         ids=lambda s: "-".join(map(str, s)))
@pytest.mark.parametrize("tiles", [1, 2])
def test_attention_query_tiles_per_cta(backend, shape, tiles, monkeypatch):
    """One and two query tiles per CTA (the choice by size needs more rows than these) give the same result."""
    monkeypatch.setenv("HOLO_CAUSAL_QUERY_TILES", str(tiles))
    rows, heads, groups, dim, vdim, first, cache_rows = shape
    q, k, v, sinks = random_attention(rows, heads, groups, dim, vdim, first + rows, seed=rows + dim)
    got = run_attention(backend, q, k, v, first, dim ** -0.5, 25.0, 0.3, 16, sinks, BF, cache_rows, stale=300.0)
    want = ref.attention(q, k, v, first, dim ** -0.5, 25.0, 0.3, 16, sinks)
    assert np.abs(got - want).max() / np.abs(want).max() < 1e-2


@pytest.mark.parametrize("shape", ATTENTION_SHAPES[:9:2] + [(20, 3, 1, 20, 33, 11, 40), (5, 2, 2, 7, 130, 60, 70)], ids=lambda s: "-".join(map(str, s)))
def test_attention_f32(backend, shape):
    rows, heads, groups, dim, vdim, first, cache_rows = shape
    q, k, v, sinks = random_attention(rows, heads, groups, dim, vdim, first + rows, seed=rows + dim)
    got = run_attention(backend, q, k, v, first, dim ** -0.5, 25.0, 0.3, 16, sinks, F32, cache_rows, stale=1e4)
    want = ref.attention(q, k, v, first, dim ** -0.5, 25.0, 0.3, 16, sinks)
    assert np.abs(got - want).max() / np.abs(want).max() < 3e-6


@pytest.mark.parametrize("rows", [1, 150])
@pytest.mark.parametrize("softcap,amp", [(0.0, 2.0), (90.0, 6.0), (4.0, 20.0), (64.0, 12.0), (0.5, 1.0), (30.0, 0.05)])
def test_attention_caps(backend, rows, softcap, amp):
    """No cap, a cap beyond the fixed range (general kernel), scores deep in the cap, at the range's end, far below the cap."""
    q, k, v, sinks = random_attention(rows, 6, 3, 64, 64, 40 + rows, seed=7, amp=amp)
    got = run_attention(backend, q, k, v, 40, 0.2, softcap, 0.1, 32, sinks, BF)
    want = ref.attention(q, k, v, 40, 0.2, softcap, 0.1, 32, sinks)
    assert np.abs(got - want).max() / np.abs(want).max() < 1.2e-2


@pytest.mark.parametrize("rows,dtype", [(1, BF), (4, BF), (140, BF), (1, F32), (6, F32)])
def test_attention_finds_one_far_key_and_respects_the_causal_edge(backend, rows, dtype):
    """One key takes nearly all weight. Planted at the last position a row sees it must dominate that row; one position
    later it must not show at all. Also at the sequence's start and around the key tiles' borders."""
    heads, groups, dim, vdim, first = 4, 2, 64, 32, 390
    q, k, v, sinks = random_attention(rows, heads, groups, dim, vdim, first + rows, seed=3, amp=0.02)
    q[:, :, 0] = 8.0
    k[:, :, 0] = 0.0
    for row in sorted({0, rows // 2, rows - 1}):
        for at in (0, 1, 15, 16, 127, 128, 255, 256, first - 1, first + row, first + row + 1):
            if at >= first + rows:
                continue
            planted, pv = k.copy(), v.copy()
            planted[at, :, 0] = 2.0
            pv[at] = 50.0
            got = run_attention(backend, q, planted, pv, first, 1.0, 30.0, 0.0, 0.0, sinks, dtype)
            seen = at <= first + row
            assert (np.abs(got[row] - 50.0).max() < 1.0) if seen else (np.abs(got[row]).max() < 2.0), (row, at)


@pytest.mark.parametrize("rows,dtype", [(1, BF), (140, BF), (3, F32)])
def test_attention_sink(backend, rows, dtype):
    """A sink of the scores' size takes its share per head; it is neither scaled nor capped; without it the weights sum to one."""
    heads, groups, dim, vdim = 4, 2, 32, 16
    q, k, v, _ = random_attention(rows, heads, groups, dim, vdim, 20 + rows, seed=5)
    v[:] = 1.0                                           # the output is then 1 - the sink's share
    sinks = np.array([-40.0, 3.0, 6.0, 12.0])
    args = (20, dim ** -0.5, 5.0, 0.2, 8)
    want = ref.attention(q, k, v, *args, sinks)
    got = run_attention(backend, q, k, v, *args, sinks, dtype)
    assert np.abs(got - want).max() < (5e-3 if dtype == BF else 1e-6)
    assert got[:, 0].min() > 0.99 and got[:, 3].max() < 0.3
    assert np.abs(run_attention(backend, q, k, v, *args, None, dtype) - 1.0).max() < (5e-3 if dtype == BF else 1e-6)


@pytest.mark.parametrize("rows,dtype", [(1, BF), (180, BF), (2, F32)])
def test_attention_query_factor_steps_at_its_period(backend, rows, dtype):
    """Two keys, one favoured by the factor: the output jumps exactly where floor((p + 1) / every) does."""
    every, dim = 48, 16
    for first in (0, every - 2, every - 1, every, 3 * every - 2, 3 * every - 1):
        q = np.zeros((rows, 1, dim), np.float32)
        q[:, :, 0] = 1.0
        length = first + rows
        k, v = np.zeros((length, 1, dim), np.float32), np.zeros((length, 1, dim), np.float32)
        k[0, 0, 0], v[0] = 2.0, 1.0
        args = (first, 1.0, 20.0, 2.0, every)
        want = ref.attention(q, k, v, *args, np.array([-3.0]))
        got = run_attention(backend, q, k, v, *args, np.array([-3.0]), dtype)
        assert np.abs(got - want).max() < (1e-2 if dtype == BF else 2e-6)


def test_attention_splits_give_the_same_bits_as_repeats(backend):
    """The partial buffers and counters are left clean: repeating a split call changes nothing."""
    q, k, v, sinks = random_attention(2, 8, 2, 64, 64, 3000, seed=11)
    first = run_attention(backend, q, k, v, 2998, 0.125, 20.0, 0.2, 64, sinks, BF)
    for _ in range(3):
        assert np.array_equal(run_attention(backend, q, k, v, 2998, 0.125, 20.0, 0.2, 64, sinks, BF), first)


# ---- whole models ----
TOL = {"float32": 2e-5, "bfloat16": 4e-2}


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    base = tmp_path_factory.mktemp("fokonex")
    out = {}
    for name, cfg in ref.CONFIGS.items():
        t = ref.random_tensors(cfg, seed=4)
        out[name] = (ref.write_model(base / name, cfg, t), cfg, t)
    return out


def make_runner(backend, path, dtype, capacity, **kw):
    from hologram_b200 import decode, models
    return decode.StepRunner(backend, models.load_model(path, dtype), capacity, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ref.CONFIGS))
def test_prompt_portions_and_single_tokens_agree_with_the_equations(backend, model_dirs, name, dtype):
    path, cfg, t = model_dirs[name]
    rng = np.random.default_rng(8)
    tokens = rng.integers(0, cfg["vocab"], size=150)
    want = ref.Reference(cfg, t).forward(tokens)
    runner = make_runner(backend, path, dtype, 150)
    everything = runner.step("whole", tokens, range(150))
    runner.end("whole")
    assert ref.row_errors(everything, want).max() < TOL[dtype]
    single = np.concatenate([runner.step("single", [tok]) for tok in tokens[:40]])
    runner.end("single")
    assert ref.row_errors(single, want[:40]).max() < TOL[dtype]
    for sizes in ((2,), (3, 2, 37), (100, 1, 1, 48), (64, 64), (5, 33)):
        at, i, got = 0, 0, []
        while at < 150:
            n = min(sizes[i % len(sizes)], 150 - at)
            got.append(runner.step("cut", tokens[at:at + n], range(n)))
            at, i = at + n, i + 1
        runner.end("cut")
        got = np.concatenate(got)
        assert ref.row_errors(got, want).max() < TOL[dtype], sizes
        assert ref.row_errors(got, everything).max() < TOL[dtype] / 2, sizes
    runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_cache_is_clean_for_the_next_sequence(backend, model_dirs, dtype):
    """A long sequence leaves its rows behind; shorter ones after it give the bits they give on a fresh runner."""
    path, cfg, _ = model_dirs["odd"]
    rng = np.random.default_rng(9)
    long, short = rng.integers(0, cfg["vocab"], size=90), rng.integers(0, cfg["vocab"], size=11)
    fresh = make_runner(backend, path, dtype, 100)
    want = [fresh.step("s", short[:7], range(7)), fresh.step("s", short[7:8]), fresh.step("s", short[8:], range(3))]
    fresh.close()
    used = make_runner(backend, path, dtype, 100)
    used.step("long", long, [])
    for tok in long[:10]:
        used.step("long", [tok])
    used.end("long")
    got = [used.step("s", short[:7], range(7)), used.step("s", short[7:8]), used.step("s", short[8:], range(3))]
    used.close()
    assert all(np.array_equal(a, b) for a, b in zip(got, want))


def test_cache_may_be_filled_to_its_last_row_and_no_further(backend, model_dirs):
    from hologram_b200 import decode
    path, cfg, t = model_dirs["plain"]
    tokens = np.random.default_rng(1).integers(0, cfg["vocab"], size=21)
    runner = make_runner(backend, path, "float32", 21)
    got = np.concatenate([runner.step("a", tokens[:18], range(18)), runner.step("a", tokens[18:], range(3))])   # padded past the end
    assert ref.row_errors(got, ref.Reference(cfg, t).forward(tokens)).max() < TOL["float32"]
    with pytest.raises(decode.CacheFull):
        runner.step("a", tokens[:1])
    with pytest.raises(decode.CacheFull):
        runner.step("b", tokens[:1])
    with pytest.raises(ValueError):
        runner.step("a", [cfg["vocab"]])
    runner.close()


def test_a_step_longer_than_the_largest_shape_runs_in_pieces(backend, model_dirs):
    path, cfg, t = model_dirs["shared"]
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], size=75)
    want = ref.Reference(cfg, t).forward(tokens)
    runner = make_runner(backend, path, "float32", 80, max_rows=16)
    assert runner.max_rows == 16
    got = runner.step("a", tokens, [74, 0, 31, 32, 15, 16])           # any order, across the pieces
    assert ref.row_errors(got, want[[74, 0, 31, 32, 15, 16]]).max() < TOL["float32"]
    runner.close()


def test_shapes_share_weights_cache_and_replay_graphs(backend, model_dirs):
    path, cfg, _ = model_dirs["plain"]
    runner = make_runner(backend, path, "bfloat16", 64)
    runner.step("a", list(range(10)), [9])
    runner.step("a", [1])
    root, big = runner._steps[1][0], runner._steps[16][0]
    assert root.device_ptr("l0.k")[0] == big.device_ptr("l0.k")[0] and root.device_ptr("hidden")[0] == big.device_ptr("hidden")[0]
    assert big.device_bytes < root.device_bytes
    assert runner._steps[1][1] and runner._steps[16][1]               # captured
    before = backend.launch_count
    runner.step("a", [2])
    assert backend.launch_count - before == runner.model.launches(1, True)
    plain = make_runner(backend, path, "bfloat16", 64, graphs=False)
    runner.end("a")
    a = [runner.step("x", [3, 4, 5], range(3)), runner.step("x", [6])]
    b = [plain.step("x", [3, 4, 5], range(3)), plain.step("x", [6])]
    assert all(np.array_equal(p, q) for p, q in zip(a, b))
    runner.close()
    plain.close()


def far_token_model():
    """Token 7 alone carries coordinate 0, every token carries coordinate 1. Keys read the former, queries the latter, so
    token 7's key scores high for every query; its values are large."""
    cfg = ref.config(40, 64, [ref.layer(4, 2, 32, 48, 64, softcap=12.0, every=24)], residual_mult=1.0)
    t = ref.random_tensors(cfg, seed=6, gain=0.1)
    t["l0.norm1"][:] = 0.0
    t["embed"][:, 0] = 0.0
    t["embed"][7, 0] = 8.0
    t["embed"][:, 1] = 4.0
    q, k, v = (t["l0.mix." + n].reshape(h, d, 64) for n, h, d in (("q", 4, 32), ("k", 2, 32), ("v", 2, 48)))
    q[:, 0, 1] = 4.0
    k[:, 0, 0] = 4.0
    v[:, :, 0] = np.where(np.arange(48) % 2 == 0, 2.0, -2.0)
    return cfg, t


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_token_is_still_read_after_long_decoding(backend, dtype):
    """Weights that make one early token stand out: its key matches every query, its value swings the logits. A model
    decoded token by token must agree with the equations to the end, and must react to that token."""
    cfg, t = far_token_model()
    from hologram_b200 import decode, fokonex as fk, safetensors_io as st
    tensors = {n: st.Tensor("BF16", ref.to_bf16_bits(v)) for n, v in t.items()}
    model = fk.FokonexModel(fk.FokonexConfig.from_dict(cfg), tensors, BF if dtype == "bfloat16" else F32)
    rng = np.random.default_rng(12)
    tokens = rng.integers(8, 40, size=420)
    other = tokens.copy()
    tokens[3] = 7
    want, without = ref.Reference(cfg, t).forward(tokens), ref.Reference(cfg, t).forward(other)
    runner = decode.StepRunner(backend, model, 420)
    got = [runner.step("a", tokens[:100], range(100))] + [runner.step("a", [tok]) for tok in tokens[100:]]
    got = np.concatenate(got)
    runner.close()
    assert ref.row_errors(got, want).max() < TOL[dtype]
    assert ref.row_errors(got[-50:], without[-50:]).min() > 3 * TOL[dtype]


@pytest.mark.parametrize("name,dtype", [("odd", "float32"), ("shared", "bfloat16")])
def test_greedy_generation_through_the_scheduler(backend, model_dirs, name, dtype):
    from hologram_b200 import decode
    path, cfg, t = model_dirs[name]
    rng = np.random.default_rng(13)
    prompts = [rng.integers(0, cfg["vocab"], size=n) for n in (9, 1, 30)]
    runner = make_runner(backend, path, dtype, 64)
    scheduler = decode.Scheduler(runner, portion=7)
    requests = [decode.Request(p, 12) for p in prompts]
    for r in requests:
        scheduler.submit(r)
    list(scheduler.run())
    for p, r in zip(prompts, requests):
        # teacher-forced: every token must be the plain model's best, or as good within the format's error
        logits = ref.Reference(cfg, t).forward(list(p) + r.tokens[:-1])[len(p) - 1:]
        spread = (logits - logits.mean(axis=1, keepdims=True)).std()
        assert len(r.tokens) == 12
        for row, tok in zip(logits, r.tokens):
            assert row.max() - row[tok] <= 2 * TOL[dtype] * spread
    assert decode.generate(runner, prompts[0], 12) == requests[0].tokens
    runner.close()


def test_command_line_generates(backend, model_dirs):
    path, cfg, _ = model_dirs["plain"]
    from hologram_b200 import decode
    runner = make_runner(backend, path, "float32", 40)
    want = decode.generate(runner, [5, 6, 7], 6)
    runner.close()
    out = subprocess.run([sys.executable, "-m", "hologram_b200", "generate", "--model", path, "--tokens", "5,6,7", "--tokens", "1", "--max-new", "6", "--dtype", "float32"],
                         cwd=ROOT, capture_output=True, text=True, timeout=120)
    assert out.returncode == 0, out.stderr
    lines = out.stdout.split()
    assert lines[0] == ",".join(map(str, want)) and len(lines) == 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(model_dirs, tmp_path, dtype):
    path, cfg, t = model_dirs["odd"]
    rng = np.random.default_rng(14)
    a, b = [int(x) for x in rng.integers(0, cfg["vocab"], size=20)], [int(x) for x in rng.integers(0, cfg["vocab"], size=6)]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:14], "want": [3, 13]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[14:16], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[16:], "want": [0, 3]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [5]}], "end": ["b"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "20"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "2.f32", "3.f32"]
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
    wa, wb = ref.Reference(cfg, t).forward(a), ref.Reference(cfg, t).forward(b)
    for got, want in ((read(0), wa[[3, 13]]), (read(2), wa[[16, 19]]), (read(3), wb[[5]])):
        assert got.shape == want.shape
        d = got - want
        assert np.abs(d - d.mean(axis=1, keepdims=True)).max() / wa.std() < 4 * TOL[dtype]
