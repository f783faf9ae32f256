"""Zisevik on the GPU: every mechanism alone against the plain equations, then whole models through the step runner, the queue
and the trace replay."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import zisevik_reference as ref
from hologram_b200 import kernel_call as kc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF, I32 = kc.DTYPE_F32, kc.DTYPE_BF16, kc.DTYPE_I32
rb = kc.rb


def store(x, dtype):
    return ref.to_bf16_bits(x) if dtype == BF else np.ascontiguousarray(x, dtype=np.float32)


def load(raw, dtype):
    return ref.from_bf16_bits(raw.view(np.uint16)) if dtype == BF else raw.view(np.float32)


def rounded(x, dtype):
    return ref.bf16(x) if dtype == BF else np.asarray(x, dtype=np.float32)


def words(*v):
    return np.array(v, dtype=np.int32)


def workspace(backend, arrays, outputs=()):
    """Slots 0.. hold `arrays`; then `outputs` buffers of the given byte counts."""
    import hologram_b200 as hb
    ws = hb.DeviceWorkspace(backend, len(arrays) + len(outputs))
    for i, a in enumerate(arrays):
        ws.put(i, a)
    for i, n in enumerate(outputs):
        ws.alloc(len(arrays) + i, n)
    return ws


def close(got, want, dtype, bf_tol=1e-2, f32_tol=1e-5):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err < (bf_tol if dtype == BF else f32_tol), err


# ---- rotary table, norms of parts ----
@pytest.mark.parametrize("first", [0, 5, 70000, 20000003])
def test_rotary_table(backend, first):
    rows, half, base = 9, 13, 1e6
    f = base ** (-2.0 * np.arange(half) / (2 * half)) / (2.0 * np.pi)
    hi = f.astype(np.float32)
    ws = workspace(backend, [words(first), np.stack([hi, (f - hi).astype(np.float32)])], [8 * rows * half])
    backend.dispatch(kc.KernelCall.RotaryTable(kc.RotaryTableCall(rb(0), rb(1), rb(2), rows, half)), ws)
    got = ws.read(rb(2), 8 * rows * half, np.float32).reshape(rows, half, 2)
    a = 2.0 * np.pi * np.remainder((first + np.arange(rows))[:, None] * f, 1.0)
    assert np.abs(got - np.stack([np.cos(a), np.sin(a)], axis=-1)).max() < 1e-6 + 5e-14 * first


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rows,count,first", [(1, 1, 37), (6, 4, 0), (40, 33, 127)])
def test_norm_parts_and_ring_rows(backend, dtype, rows, count, first):
    """Two normed parts (one into a ring that wraps, as columns of wider rows) and a copied one."""
    rng = np.random.default_rng(rows)
    widths, outs, ld_in, ring, ld = (23, 700, 31), (24, 704, 31), 780, 64, 720
    at = (0, 23, 740)
    x = (3 * rng.standard_normal((rows, ld_in))).astype(np.float32)
    x[0] *= 1e-3                                          # eps matters there
    w = [(1 + 0.3 * rng.standard_normal(n)).astype(np.float32) for n in widths[:2]]
    es = 2 if dtype == BF else 4
    ws = workspace(backend, [x, words(first, count), w[0], w[1], store(np.zeros((rows, 24)), dtype), store(np.full((ring, ld), 7.0), dtype), store(np.zeros((rows, 31)), dtype)])
    parts = [kc.NormPart(rb(2), rb(4), at[0], widths[0], outs[0], 24, 1, 0), kc.NormPart(rb(3), rb(5, 8 * es), at[1], widths[1], outs[1], ld, 1, 1),
             kc.NormPart(kc.NONE, rb(6), at[2], widths[2], outs[2], 31, 0, 0)]
    backend.dispatch(kc.KernelCall.RmsNormParts(kc.RmsNormPartsCall.make(rb(0), parts, rows, ld_in, 1e-4, dtype, step=rb(1))), ws)
    got = load(ws.read(rb(4), rows * 24 * es), dtype).reshape(rows, 24)
    close(got[:, :23], ref.rms_norm(x[:, :23], w[0], 1e-4), dtype)
    assert not got[:, 23:].any()
    close(load(ws.read(rb(6), rows * 31 * es), dtype).reshape(rows, 31), x[:, 740:771], dtype)
    got = load(ws.read(rb(5), ring * ld * es), dtype).reshape(ring, ld)
    want = np.full((ring, ld), 7.0)
    for i in range(count):
        want[(first + i) % ring, 8:8 + 704] = 0
        want[(first + i) % ring, 8:8 + 700] = ref.rms_norm(x[i, 23:723], w[1], 1e-4)
    close(got, want, dtype)


# ---- products ----
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rows", [1, 3, 70, 300])
def test_linear_rotates_appends_to_a_ring_and_activates(backend, dtype, rows):
    rng = np.random.default_rng(rows)
    k, ring, first, count = 72, 128 if rows < 128 else 384, 100, max(1, rows - 2)
    es = 2 if dtype == BF else 4
    a, b = rounded(rng.standard_normal((rows, k)), dtype), rounded(rng.standard_normal((k, 256)) / 8, dtype)
    angle = rng.uniform(-3, 3, (rows, 5))
    table = np.stack([np.cos(angle), np.sin(angle)], axis=-1).astype(np.float32)
    # segments: two heads of 16 whose columns 4 .. 13 turn, into a ring; silu; gelu; a gated pair
    ws = workspace(backend, [store(a, dtype), store(b, dtype), table, words(first, count), store(np.full((ring, 40), 3.0), dtype)],
                   [rows * 48 * es, rows * 32 * 4, rows * 30 * es])
    segs = [kc.LinearSeg.make(rb(4, 8 * es), 32, 40, dtype, 0, row_pos=rb(3), ring=True, rotate=(16, 4, 10)),
            kc.LinearSeg.make(rb(5), 47, 48, dtype, 32, act=kc.LINEAR_ACT_SILU), kc.LinearSeg.make(rb(6), 32, 32, F32, 96, act=kc.LINEAR_ACT_GELU_TANH),
            kc.LinearSeg.make(rb(7), 60, 30, dtype, 128, act=kc.LINEAR_ACT_SILU_GATE)]
    backend.dispatch(kc.KernelCall.Linear(kc.LinearCall.make(rb(0), rb(1), segs, rows, k, 256, dtype, alpha=0.5, rot=rb(2))), ws)
    v = a.astype(np.float64) @ b
    want = np.full((ring, 40), 3.0)
    turned = v[:, :32].reshape(rows, 2, 16).copy()
    u, w = turned[:, :, 4:14:2].copy(), turned[:, :, 5:14:2].copy()
    turned[:, :, 4:14:2] = u * np.cos(angle)[:, None] - w * np.sin(angle)[:, None]
    turned[:, :, 5:14:2] = w * np.cos(angle)[:, None] + u * np.sin(angle)[:, None]
    for i in range(count):
        want[(first + i) % ring, 8:] = 0.5 * turned[i].reshape(32)
    close(load(ws.read(rb(4), ring * 40 * es), dtype).reshape(ring, 40), want, dtype)
    close(load(ws.read(rb(5), rows * 48 * es), dtype).reshape(rows, 48)[:, :47], 0.5 * ref.silu(v[:, 32:79]), dtype)
    close(ws.read(rb(6), rows * 128, np.float32).reshape(rows, 32), 0.5 * ref.gelu_tanh(v[:, 96:128]), F32)
    close(load(ws.read(rb(7), rows * 30 * es), dtype).reshape(rows, 30), 0.5 * ref.silu(v[:, 128:188:2]) * v[:, 129:188:2], dtype)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("m,n,pos", [(128, 64, 0), (256, 64, 300), (384, 64, 1000), (384, 4096, 700), (640, 12288, 700)])
def test_linear_over_a_window_of_a_ring(backend, dtype, m, n, pos):
    """Rows of A come from a ring, starting a given distance before the position (all three tensor-core kernels)."""
    rng = np.random.default_rng(m)
    ring, lda, k, back = 512, 96, 80, 150
    es = 2 if dtype == BF else 4
    if dtype == F32 and n > 64:
        return
    a, b = rounded(rng.standard_normal((ring, lda)), dtype), rounded(rng.standard_normal((k, n)) / 9, dtype)
    ws = workspace(backend, [store(a, dtype), store(b, dtype), words(pos)], [m * n * es])
    backend.dispatch(kc.KernelCall.Linear(kc.LinearCall.make(rb(0), rb(1), [kc.LinearSeg.make(rb(3), n, n, dtype)], m, k, n, dtype, lda=lda, a_pos=rb(2), a_back=back, a_rows=ring)), ws)
    start = max(0, pos - back) // 128 * 128
    want = a[(start + np.arange(m)) % ring, :k].astype(np.float64) @ b
    close(load(ws.read(rb(3), m * n * es), dtype).reshape(m, n), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("tile_rows,shared,k,n,experts,tiles", [
    (16, 1, 72, 80, 5, [3, 0, 4]), (16, 13, 200, 48, 5, [0, 1, 2, 3, 4]), (64, 50, 64, 96, 3, [2]), (128, 128, 72, 64, 4, [1, 3]),
    (16, 0, 72, 80, 5, [3, 0, 4]), (64, 0, 520, 64, 3, [2, 0]), (128, 0, 104, 72, 4, [0, 0, 3]), (128, 0, 128, 4096, 4, [0, 0, 2, 3, 3, 3, 1, 1, 1, 2])])
def test_grouped_linear(backend, dtype, tile_rows, shared, k, n, experts, tiles):
    rng = np.random.default_rng(k + tile_rows)
    es, most = 2 if dtype == BF else 4, len(tiles) + 2
    m = most * tile_rows
    a = rounded(rng.standard_normal((shared or m, k)), dtype)
    b = rounded(rng.standard_normal((experts, k, n)) / np.sqrt(k), dtype)
    table = np.zeros(1 + most, dtype=np.int32)
    table[0], table[1:1 + len(tiles)] = len(tiles), tiles
    for act, width in ((kc.LINEAR_ACT_NONE, n), (kc.LINEAR_ACT_SILU_GATE, n // 2)):
        ws = workspace(backend, [store(a, dtype), store(b, dtype), table, store(np.full((m, width), 9.0), dtype)])
        backend.dispatch(kc.KernelCall.Linear(kc.LinearCall.make(rb(0), rb(1), [kc.LinearSeg.make(rb(3), n, width, dtype, act=act)], m, k, n, dtype, tiles=rb(2),
                                                                 tile_rows=tile_rows, experts=experts, a_shared=shared)), ws)
        got = load(ws.read(rb(3), m * width * es), dtype).reshape(most, tile_rows, width)
        for t, e in enumerate(tiles):
            rows = a if shared else a[t * tile_rows:(t + 1) * tile_rows]
            v = rows.astype(np.float64) @ b[e]
            close(got[t, :len(rows)], ref.silu(v[:, 0::2]) * v[:, 1::2] if act else v, dtype)
        assert (got[len(tiles):] == 9.0).all()


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rows,heads,k,n", [(1, 3, 48, 80), (5, 2, 130, 37), (16, 4, 512, 128), (1, 16, 128, 512)])
def test_head_linear(backend, dtype, rows, heads, k, n):
    rng = np.random.default_rng(n)
    es, lda, ld, bld = 2 if dtype == BF else 4, heads * (k + 8) + 8, heads * (n + 3), n + 8
    a, b = rounded(rng.standard_normal((rows, lda)), dtype), rounded(rng.standard_normal((heads, k, bld)) / np.sqrt(k), dtype)
    ws = workspace(backend, [store(a, dtype), store(b, dtype)], [rows * ld * es])
    backend.dispatch(kc.KernelCall.HeadLinear(kc.HeadLinearCall(rb(0), rb(1), rb(2), rows, heads, k, n, lda, k + 8, bld, k * bld, ld, n + 3, dtype)), ws)
    got = load(ws.read(rb(2), rows * ld * es), dtype).reshape(rows, heads, n + 3)
    for h in range(heads):
        close(got[:, h, :n], a[:, h * (k + 8):h * (k + 8) + k].astype(np.float64) @ b[h, :, :n], dtype)


# ---- attention ----
def attention_case(backend, dtype, rows, heads, kv_heads, dim, dim2, vdim, pos, window, shared_values=False, expanded=False, sink=True, seed=0, loud=None):
    """Runs WindowAttention over ring buffers and returns (got, want); `loud` = [(row, key)]: that score stands out."""
    rng = np.random.default_rng(seed)
    es = 2 if dtype == BF else 4
    length = pos + rows
    need = length if not window else min(length, rows + window - 1 + 127)
    ring = -(-need // 128) * 128
    q, q2 = rng.standard_normal((rows, heads, dim)), rng.standard_normal((rows, heads, max(dim2, 1)))
    k, v, k2 = rng.standard_normal((length, kv_heads, dim)), rng.standard_normal((length, kv_heads, vdim)), rng.standard_normal((length, max(dim2, 1)))
    for row, key in loud or ():
        if key < 0:
            continue
        direction = rng.standard_normal(dim)
        direction *= np.sqrt(dim) / np.linalg.norm(direction)
        q[row], k[key] = 1.5 * direction, 1.5 * direction
    q, q2, k, v, k2 = (rounded(t, dtype) for t in (q, q2, k, v, k2))
    if shared_values:
        v = k[..., :vdim]
    scale = (dim + dim2) ** -0.5 * 1.3
    sinks = rng.standard_normal(heads).astype(np.float32) * 2 if sink else None
    back = (window - 1) if window else kc.WHOLE_CACHE
    start = max(0, pos - back) // 128 * 128 if expanded and window else 0
    if not expanded:
        back = kc.WHOLE_CACHE
    lk, lv, l2 = kv_heads * dim + 16, kv_heads * vdim + 8, max(dim2, 8) + 24
    if dim2 % 8:
        l2 = dim2 + 3
    kb, vb, k2b = np.zeros((ring, lk)), np.zeros((ring, lv)), np.zeros((ring, l2))
    for j in range(max(0, length - ring), length):
        if j >= start:
            kb[(j - start) % ring, :kv_heads * dim], vb[(j - start) % ring, :kv_heads * vdim] = k[j].reshape(-1), v[j].reshape(-1)
        k2b[j % ring, :max(dim2, 1)] = k2[j]
    if shared_values:
        lv = lk
    qs, q2s, ld = dim + 8, dim2 + 8, heads * vdim + 8
    qb, q2b = np.zeros((rows, heads, qs)), np.zeros((rows, heads, q2s))
    qb[..., :dim] = q
    q2b[..., :dim2] = q2[..., :dim2]
    arrays = [store(t, dtype) for t in (qb, kb, kb if shared_values else vb, q2b, k2b)] + [words(pos), sinks if sink else np.zeros(heads, np.float32)]
    ws = workspace(backend, arrays, [rows * ld * es])
    none = kc.NONE
    backend.dispatch(kc.KernelCall.WindowAttention(kc.WindowAttentionCall(
        rb(0), rb(1), rb(1) if shared_values else rb(2), rb(3) if dim2 else none, rb(4) if dim2 else none, rb(5), rb(6) if sink else none, rb(7),
        rows, heads, kv_heads, dim, vdim, dim2, heads * qs, qs, lk, lv, heads * q2s, q2s, l2, ld, ring, back, ring, window, kc.f32_bits(scale), dtype)), ws)
    got = load(ws.read(rb(7), rows * ld * es), dtype).reshape(rows, ld)[:, :heads * vdim].reshape(rows, heads, vdim)
    kk, qq = k, q
    if dim2:
        kk = np.concatenate([k, np.broadcast_to(k2[:, None], (length, kv_heads, dim2))], axis=-1)
        qq = np.concatenate([q, q2], axis=-1)
    return got, ref.attend(qq, kk, v, pos, scale, window or None, sinks)


SHAPES = [(1, 4, 4, 24, 8, 20), (7, 6, 2, 33, 0, 40), (130, 3, 3, 64, 16, 64), (3, 2, 1, 300, 20, 200)]


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("pos,window", [(0, 0), (0, 5), (200, 1), (311, 96), (150, 4000)])
def test_window_attention_general(backend, monkeypatch, dtype, shape, pos, window):
    monkeypatch.setenv("HOLO_WINDOW_GENERAL", "1")
    got, want = attention_case(backend, dtype, *shape, pos, window)
    close(got, want, dtype)


@pytest.mark.parametrize("shape", [(1, 16, 1, 128, 16, 128), (1, 3, 1, 32, 16, 32), (5, 4, 1, 128, 16, 128), (16, 16, 1, 512, 64, 512), (2, 5, 1, 48, 0, 48),
                                   (1, 8, 1, 768, 64, 768), (3, 32, 1, 256, 32, 256)])
@pytest.mark.parametrize("pos,window", [(0, 0), (0, 96), (90, 96), (1500, 96), (1203, 1), (2000, 1000), (700, 0)])
def test_latent_attention_few_rows(backend, shape, pos, window):
    got, want = attention_case(backend, BF, *shape, pos, window, shared_values=True)
    close(got, want, BF)


@pytest.mark.parametrize("shape", [(128, 4, 4, 64, 16, 64), (17, 4, 4, 64, 16, 64), (300, 2, 2, 128, 64, 128), (511, 3, 3, 80, 32, 48), (200, 8, 2, 64, 0, 128),
                                   (260, 2, 2, 192, 64, 256), (140, 2, 2, 16, 16, 16), (700, 6, 2, 128, 0, 128)])
@pytest.mark.parametrize("pos,window,expanded", [(0, 0, False), (0, 96, True), (100, 96, True), (1111, 96, True), (515, 1, True), (3000, 1024, True), (400, 0, False), (900, 200, False)])
def test_window_attention_many_rows(backend, shape, pos, window, expanded):
    got, want = attention_case(backend, BF, *shape, pos, window, expanded=expanded)
    close(got, want, BF)


def test_window_attention_many_rows_one_query_tile_per_cta(backend, monkeypatch):
    monkeypatch.setenv("HOLO_WINDOW_QUERY_TILES", "1")
    for pos, window in ((0, 0), (777, 130)):
        got, want = attention_case(backend, BF, 300, 4, 4, 64, 32, 64, pos, window, expanded=bool(window))
        close(got, want, BF)


@pytest.mark.parametrize("kind", ["general f32", "general bf16", "few", "many"])
@pytest.mark.parametrize("window", [1, 2, 64, 96, 127, 128, 129, 256])
def test_window_edges(backend, monkeypatch, kind, window):
    """One loud key per probe row: just inside the window it dominates the row, one further back it must not count at all."""
    rows = 200 if kind == "many" else 12
    dtype = F32 if kind == "general f32" else BF
    if kind.startswith("general"):
        monkeypatch.setenv("HOLO_WINDOW_GENERAL", "1")
    shape = (rows, 4, 1, 64, 16, 64) if kind == "few" else (rows, 2, 2, 64, 16, 64)
    for probe in ({0, rows - 1, rows // 2} if kind != "many" else {0, 1, 63, 127, 128, 199}):
        for inside in (True, False):
            key = 300 + probe - window + (1 if inside else 0)
            got, want = attention_case(backend, dtype, *shape, 300, window, shared_values=kind == "few", expanded=kind == "many", loud=[(probe, key)], seed=probe)
            close(got, want, dtype)


@pytest.mark.parametrize("grow", [0.5, 3.0])
def test_running_maximum_rises_and_falls_over_many_key_tiles(backend, grow):
    """Keys that get louder from tile to tile make every row raise its reference again and again (and a sink that beats them)."""
    rows, pos = 160, 900
    loud = [(r, 130 * i + 7) for i in range(1, 8) for r in (5, 100, 159)]
    got, want = attention_case(backend, BF, rows, 2, 2, 64, 0, 64, pos, 0, loud=loud, seed=11)
    close(got, want, BF)
    rng = np.random.default_rng(5)
    length = pos + rows
    scale_up = grow ** (np.arange(length) / 128.0)
    q, k, v = ref.bf16(rng.standard_normal((rows, 2, 64))), ref.bf16(rng.standard_normal((length, 2, 64)) * scale_up[:, None, None]), ref.bf16(rng.standard_normal((length, 2, 64)))
    ring = -(-length // 128) * 128
    kb, vb = np.zeros((ring, 128)), np.zeros((ring, 128))
    kb[:length], vb[:length] = k.reshape(length, -1), v.reshape(length, -1)
    sinks = np.array([30.0, -50.0], np.float32)
    ws = workspace(backend, [store(q, BF), store(kb, BF), store(vb, BF), words(pos), sinks], [rows * 128 * 2])
    backend.dispatch(kc.KernelCall.WindowAttention(kc.WindowAttentionCall(
        rb(0), rb(1), rb(2), kc.NONE, kc.NONE, rb(3), rb(4), rb(5), rows, 2, 2, 64, 64, 0, 128, 64, 128, 128, 0, 0, 0, 128, ring, kc.WHOLE_CACHE, 0, 0, kc.f32_bits(0.125), BF)), ws)
    close(load(ws.read(rb(5), rows * 256), BF).reshape(rows, 2, 64), ref.attend(q, k, v, pos, 0.125, None, sinks), BF)


# ---- retention ----
def retention_case(backend, dtype, rows, count, heads, dim, vdim, vmean, first, state, seed=0, decay=None):
    rng = np.random.default_rng(seed)
    es = 2 if dtype == BF else 4
    q, k = (rounded(rng.standard_normal((rows, heads, dim)), dtype) for _ in range(2))
    v, gate = (rounded(rng.standard_normal((rows, heads, vdim)), dtype) for _ in range(2))
    v[:, :, vmean:] = 0
    decay = np.asarray(decay if decay is not None else [1 - 2.0 ** -(1 + 2 * h) for h in range(heads)], dtype=np.float32)
    scale, eps = dim ** -0.5, 1e-3
    ldq, ldv = heads * dim + 8, heads * vdim + 8

    def padded(x, ld):
        out = np.zeros((rows, ld))
        out[:, :x[0].size] = x.reshape(rows, -1)
        return store(out, dtype)
    ws = workspace(backend, [padded(q, ldq), padded(k, ldq), padded(v, ldv), padded(gate, ldv), decay, words(first, count), np.asarray(state, np.float32),
                             store(np.full((rows, ldv), 5.0), dtype)], [4 * rows * heads * vdim])
    backend.dispatch(kc.KernelCall.Retention(kc.RetentionCall(*[rb(i) for i in range(9)], rows, heads, dim, vdim, vmean, ldq, ldq, ldv, ldv, ldv,
                                                              kc.f32_bits(scale), kc.f32_bits(eps), dtype)), ws)
    got = load(ws.read(rb(7), rows * ldv * es), dtype).reshape(rows, ldv)[:, :heads * vdim].reshape(rows, heads, vdim)
    after = ws.read(rb(6), 4 * heads * dim * vdim, np.float32).reshape(heads, dim, vdim)
    want_state = np.array(state, dtype=np.float64) * (first != 0)
    o = ref.retain(q[:count].astype(np.float64), k[:count].astype(np.float64) * scale, v[:count].astype(np.float64), decay, want_state)
    # the call keeps S without k's factor
    return got, after, o, gate, eps, vmean


def check_retention(backend, dtype, rows, count, heads, dim, vdim, vmean, first, seed=0, decay=None):
    rng = np.random.default_rng(seed + 100)
    state = rng.standard_normal((heads, dim, vdim)) * 3
    state[:, :, vmean:] = 0
    scale = dim ** -0.5
    got, after, _, gate, eps, _ = retention_case(backend, dtype, rows, count, heads, dim, vdim, vmean, first, state, seed, decay)
    rng = np.random.default_rng(seed)
    q, k = (rounded(rng.standard_normal((rows, heads, dim)), dtype) for _ in range(2))
    v = rounded(rng.standard_normal((rows, heads, vdim)), dtype)
    v[:, :, vmean:] = 0
    d = np.asarray(decay if decay is not None else [1 - 2.0 ** -(1 + 2 * h) for h in range(heads)], dtype=np.float32)
    s = np.asarray(state, np.float32).astype(np.float64) * (first != 0)
    o = scale * ref.retain(q[:count].astype(np.float64), k[:count].astype(np.float64), v[:count].astype(np.float64), d, s)
    want = ref.rms(o[..., :vmean], eps) * gate[:count, :, :vmean]
    close(got[:count, :, :vmean], want, dtype)
    assert (got[count:] == 5.0).all()
    close(after, s, F32, f32_tol=2e-5)          # the state is f32 in either format


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("heads,dim,vdim,vmean", [(3, 16, 32, 22), (2, 64, 128, 128), (1, 32, 48, 33), (2, 128, 256, 256), (1, 256, 512, 512), (2, 48, 16, 7)])
@pytest.mark.parametrize("first", [0, 9])
def test_retention_one_row(backend, dtype, heads, dim, vdim, vmean, first):
    check_retention(backend, dtype, 1, 1, heads, dim, vdim, vmean, first)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("heads,dim,vdim,vmean", [(3, 16, 32, 22), (2, 64, 128, 128), (1, 32, 48, 33), (2, 128, 256, 256), (1, 256, 256, 250), (1, 256, 512, 512),
                                                  (2, 48, 16, 7), (1, 144, 144, 140), (1, 16, 384, 384), (2, 80, 64, 64)])
@pytest.mark.parametrize("rows,count,first", [(2, 2, 5), (16, 9, 0), (128, 127, 40), (256, 129, 0), (512, 400, 7)])
def test_retention_many_rows(backend, dtype, heads, dim, vdim, vmean, rows, count, first):
    check_retention(backend, dtype, rows, count, heads, dim, vdim, vmean, first)


@pytest.mark.parametrize("heads,dim,vdim,vmean", [(3, 128, 64, 64), (2, 128, 192, 180), (5, 256, 512, 500), (1, 256, 64, 64), (2, 128, 512, 512)])
@pytest.mark.parametrize("tile", [True, False])
def test_retention_long_prompts_in_both_chunked_forms(backend, monkeypatch, heads, dim, vdim, vmean, tile):
    if not tile:
        monkeypatch.setenv("HOLO_RETENTION_NO_TILE", "1")
    for rows, count, first in ((128, 128, 0), (1024, 1023, 3), (640, 1, 5)):
        check_retention(backend, BF, rows, count, heads, dim, vdim, vmean, first, seed=rows, decay=[1 - 2.0 ** -(h + 1) for h in range(heads)])


def test_retention_general_form_and_extreme_decays(backend, monkeypatch):
    for decay in ([1.0, 0.0, 0.5, 0.9999],):
        check_retention(backend, BF, 256, 200, 4, 32, 64, 64, 3, decay=decay)
        check_retention(backend, BF, 256, 200, 4, 128, 64, 64, 3, decay=decay)
        check_retention(backend, BF, 1, 1, 4, 32, 64, 64, 3, decay=decay)
        monkeypatch.setenv("HOLO_RETENTION_GENERAL", "1")
        check_retention(backend, BF, 64, 50, 4, 32, 64, 64, 3, decay=decay)
        check_retention(backend, F32, 64, 50, 1, 256, 512, 500, 0, decay=[0.97])   # the state does not fit shared memory


@pytest.mark.parametrize("dim", [64, 128, 256])
def test_retention_remembers_one_token_far_back(backend, dim):
    """A single loud key and value 300 tokens before a query that asks for it, everything between quiet."""
    rng = np.random.default_rng(8)
    rows, vdim = 512, 64
    q, k, v = (1e-3 * rng.standard_normal((rows, 1, n)) for n in (dim, dim, vdim))
    mark = rng.standard_normal(dim)
    k[77], v[77], q[377] = mark, rng.standard_normal(vdim), mark
    q, k, v = ref.bf16(q), ref.bf16(k), ref.bf16(v)
    ones = np.ones((rows, 1, vdim))
    ws = workspace(backend, [store(t, BF) for t in (q, k, v, ones)] + [np.array([0.995], np.float32), words(0, rows), np.zeros((dim, vdim), np.float32)], [rows * vdim * 2, rows * vdim * 4])
    backend.dispatch(kc.KernelCall.Retention(kc.RetentionCall(*[rb(i) for i in range(9)], rows, 1, dim, vdim, vdim, dim, dim, vdim, vdim, vdim, kc.f32_bits(1.0), kc.f32_bits(1e-6), BF)), ws)
    got = load(ws.read(rb(7), rows * vdim * 2), BF).reshape(rows, vdim)
    want = ref.rms(ref.retain(q.astype(np.float64), k.astype(np.float64), v.astype(np.float64), [0.995], np.zeros((1, dim, vdim)))[:, 0], 1e-6)
    close(got[377], want[377], BF)
    assert np.corrcoef(got[377], v[77, 0])[0, 1] > 0.999


# ---- routing ----
@pytest.mark.parametrize("rows,count,experts,top,tile", [(1, 1, 16, 2, 16), (16, 11, 5, 3, 16), (60, 60, 64, 6, 64), (128, 100, 300, 8, 128), (300, 290, 16, 4, 128),
                                                         (512, 512, 7, 1, 128), (2048, 2000, 64, 6, 128), (130, 129, 3, 3, 128), (200, 200, 1000, 32, 128)])
def test_moe_plan_and_combine(backend, rows, count, experts, top, tile):
    from hologram_b200.zisevik import RoutedSpec
    rng = np.random.default_rng(rows)
    want_tile, most = RoutedSpec(experts, top, 8).tiles(rows)
    assert want_tile == tile
    z = (3 * rng.standard_normal((rows, experts + 3))).astype(np.float32)
    bias = (2 * rng.standard_normal(experts)).astype(np.float32)
    width, slots = 52, most * tile
    y = rng.standard_normal((slots, 56)).astype(np.float32)
    x = rng.standard_normal((rows, width)).astype(np.float32)
    ws = workspace(backend, [z, bias, words(40, count), x, y], [4 * rows * top, 4 * rows * top, 4 * (1 + most), 4 * slots])
    backend.dispatch(kc.KernelCall.MoePlan(kc.MoePlanCall(rb(0), rb(1), rb(2), rb(5), rb(6), rb(7), rb(8), rows, experts, top, experts + 3, tile, most)), ws)
    weight = ws.read(rb(5), 4 * rows * top, np.float32).reshape(rows, top)[:count]
    place = ws.read(rb(6), 4 * rows * top, np.int32).reshape(rows, top)[:count]
    tiles = ws.read(rb(7), 4 * (1 + most), np.int32)
    source = ws.read(rb(8), 4 * slots, np.int32)
    chosen, want = ref.route((z[:count, :experts] + bias).astype(np.float64), top)
    close(weight, want, F32)
    used = tiles[0]
    assert 0 < used <= most
    assert np.array_equal(tiles[1 + place // tile], chosen)      # every pair lies in a tile of its expert
    if rows <= tile:
        assert np.array_equal(place % tile, np.broadcast_to(np.arange(count)[:, None], (count, top)))
        assert np.array_equal(tiles[1:1 + used], np.unique(chosen))
    else:
        assert len(np.unique(place)) == count * top
        assert np.array_equal(source[place], np.broadcast_to(np.arange(count)[:, None], (count, top)))
        assert used == sum(-(-n // tile) for n in np.bincount(chosen.reshape(-1)))
    for dtype in (F32, BF):
        ws.put(3, x)
        ws.put(4, store(y, dtype))
        backend.dispatch(kc.KernelCall.MoeCombine(kc.MoeCombineCall(rb(3), rb(4), rb(5), rb(6), rb(2), rows, width, top, 56, slots, dtype)), ws)
        got = ws.read(rb(3), 4 * rows * width, np.float32).reshape(rows, width)
        total = x[:count] + np.einsum("it,itc->ic", weight.astype(np.float64), rounded(y, dtype)[place][..., :width])
        close(got[:count], total, F32)
        assert np.array_equal(got[count:], x[count:])


def test_calls_refuse_wrong_geometry(backend):
    import hologram_b200 as hb
    ws = workspace(backend, [np.zeros(4096, np.float32) for _ in range(9)])
    plan = lambda **k: kc.KernelCall.MoePlan(kc.MoePlanCall(rb(0), rb(1), rb(2), rb(3), rb(4), rb(5), rb(6), 16, k.get("experts", 8), k.get("top", 2), 8, 16, k.get("most", 8)))
    for bad in ({"top": 9}, {"most": 3}, {"top": 0}):
        with pytest.raises(hb.BackendError):
            backend.dispatch(plan(**bad), ws)
    att = lambda heads, kv, **k: kc.KernelCall.WindowAttention(kc.WindowAttentionCall(
        rb(0), rb(1), rb(2), kc.NONE, kc.NONE, rb(3), kc.NONE, rb(4), 1, heads, kv, k.get("dim", 8), 8, 0, heads * 8, 8, kv * 8, kv * 8, 0, 0, 0, k.get("ld", heads * 8),
        k.get("kv_rows", 16), kc.WHOLE_CACHE, 0, 4, kc.f32_bits(1.0), F32))
    backend.dispatch(att(2, 2), ws)
    for call in (att(3, 2), att(2, 2, dim=2000), att(2, 2, ld=8), att(2, 2, kv_rows=100000)):
        with pytest.raises(hb.BackendError):
            backend.dispatch(call, ws)
    seg = lambda **k: kc.LinearSeg.make(rb(2), k.get("n", 32), 32, F32, act=k.get("act", 0), rotate=k.get("rot"), row_pos=None, ring=k.get("ring", False))
    lin = lambda s, **k: kc.KernelCall.Linear(kc.LinearCall.make(rb(0), rb(1), [s], 16, 8, 32, F32, **k))
    backend.dispatch(lin(seg()), ws)
    for call in (lin(seg(rot=(32, 0, 8))), lin(seg(rot=(32, 28, 8)), rot=rb(3)), lin(seg(ring=True)), lin(seg(act=kc.LINEAR_ACT_SILU_GATE, n=31)),
                 lin(seg(), tiles=rb(3), tile_rows=17, experts=2), lin(seg(), a_pos=rb(3))):
        with pytest.raises(hb.BackendError):
            backend.dispatch(call, ws)


# ---- whole models ----
def make_runner(backend, tmp_path, cfg, dtype, capacity, seed=0, tensors=None, **kw):
    from hologram_b200 import decode, models
    t = tensors or ref.random_tensors(cfg, seed)
    path = ref.write_model(tmp_path / f"m{seed}", cfg, t)
    return decode.StepRunner(backend, models.load_model(path, dtype), capacity, **kw), ref.Reference(cfg, t)


LIMIT = {"float32": 2e-5, "bfloat16": 8e-2}


def check_rows(got, want, dtype, cfg, what=None):
    """Every row close to the plain model's. With bf16 activations a token whose router logits nearly tie may go to another
    expert than in the plain model, in any of its layer runs: where experts are left out, most rows have to agree (in f32 all)."""
    err = ref.row_errors(got, want)
    picky = any(l["mlp"] and l["mlp"]["kind"] == "moe" and l["mlp"]["router"]["top"] < l["mlp"]["router"]["experts"] for l in cfg["layers"])
    if dtype == "bfloat16" and picky:
        assert np.quantile(err, 0.7) < LIMIT[dtype], (what, np.quantile(err, 0.7))
    else:
        assert err.max() < 2 * LIMIT[dtype], (what, err.max(), int(err.argmax()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ref.CONFIGS))
def test_prompt_portions_and_single_tokens_agree(backend, tmp_path, name, dtype):
    """A whole prompt, portions of several sizes down to two tokens, and token by token, each against the plain model."""
    cfg = ref.CONFIGS[name]
    runner, plain = make_runner(backend, tmp_path, cfg, dtype, 300, max_rows=256)
    tokens = np.random.default_rng(1).integers(0, cfg["vocab"], size=270)
    want = plain.forward(tokens)
    everywhere = lambda n: list(range(n))
    cuts = {"whole": [270], "portions": [2, 3, 17, 2, 64, 31, 130, 2, 19], "pairs": [2] * 20 + [100, 130], "tokens": [200] + [1] * 70, "alone": [1] * 40 + [230]}
    for name_, cut in cuts.items():
        assert sum(cut) == 270, name_
        got, at = [], 0
        for n in cut:
            got.append(runner.step(name_, tokens[at:at + n], everywhere(n)))
            at += n
        runner.end(name_)
        check_rows(np.concatenate(got), want, dtype, cfg, name_)
    runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_sequences_go_round_the_rings(backend, tmp_path, dtype):
    """More positions than the cache has rows, by portions and then one by one; afterwards another sequence in the same slots."""
    cfg = ref.config(64, 48, [ref.attention_layer(3, 20, 8, 16, 32, 24, 33, ref.dense(40)), ref.retention_layer(2, 16, 24, 16, ref.moe(6 if dtype == "float32" else 2, 2, 24)),
                              ref.attention_layer(2, 32, 16, 32, 48, 32, 100, None)], loop=(0, 2, 2))
    runner, plain = make_runner(backend, tmp_path, cfg, dtype, 1000, max_rows=32)
    assert [l.mixer.cache_rows(1000, 32) for l, _ in runner.model.config.runs() if l.mixer.kind == "latent_attention"] == [128, 128, 256]
    for seed in (2, 3):
        tokens = np.random.default_rng(seed).integers(0, 64, size=700)
        plain.reset()
        want = plain.forward(tokens)
        got, at = [], 0
        for n in [500, 29, 2] + [1] * 169:
            got.append(runner.step(seed, tokens[at:at + n], list(range(n))))
            at += n
        runner.end(seed)
        check_rows(np.concatenate(got), want, dtype, cfg, seed)
    runner.close()


def test_sequences_leave_nothing_behind(backend, tmp_path):
    """The same prompt after other sequences gives the same bits as in a fresh runner."""
    cfg = ref.CONFIGS["looped"]
    runner, _ = make_runner(backend, tmp_path, cfg, "bfloat16", 200, max_rows=64)
    rng = np.random.default_rng(9)
    a, b = rng.integers(0, 130, size=90), rng.integers(0, 130, size=150)
    fresh = [runner.step("a", a[:60], [0, 1, 59]), runner.step("a", a[60:], [29])]
    runner.end("a")
    runner.step("b", b, [])
    runner.end("b")
    again = [runner.step("c", a[:60], [0, 1, 59]), runner.step("c", a[60:], [29])]
    runner.end("c")
    assert all(np.array_equal(x, y) for x, y in zip(fresh, again))
    runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_window_edge_shows_in_the_logits(backend, tmp_path, dtype):
    """Changing the token just inside every window changes the last logits; the one just outside of all of them does not."""
    window = 40
    cfg = ref.config(90, 64, [ref.attention_layer(4, 32, 16, 32, 32, 32, window, ref.dense(64), scale=0.3)])
    runner, plain = make_runner(backend, tmp_path, cfg, dtype, 256, max_rows=256)
    tokens = np.random.default_rng(4).integers(0, 90, size=200)
    for cut in ([200], [199, 1]):
        def last(t):
            at = 0
            for n in cut:
                out = runner.step("s", t[at:at + n], [n - 1])
                at += n
            runner.end("s")
            return out[0]
        base = last(tokens)
        for back, seen in ((window - 1, True), (window, False), (window + 1, False)):
            changed = tokens.copy()
            changed[199 - back] = (changed[199 - back] + 7) % 90
            moved = np.abs(last(changed) - base).max()
            plain.reset()
            want = plain.forward(changed)[-1]
            assert (moved > 0) == seen, (cut, back, moved)
            assert ref.row_errors(last(changed)[None], want[None])[0] < LIMIT[dtype]
    runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sinks_and_gates_show_in_the_logits(backend, tmp_path, dtype):
    """Sinks far above and far below the scores, per head; a router bias that moves every token to other experts."""
    cfg = ref.config(70, 64, [ref.attention_layer(4, 16, 16, 16, 32, 32, 50, ref.moe(6, 2, 32))])
    t = ref.random_tensors(cfg, 5)
    outs = []
    for sinks, bias in (([-20, -20, -20, -20], 0), ([6, -20, 3, -20], 0), ([6, -20, 3, -20], 4)):
        t = dict(t)
        t["l0.mix.sink"] = ref.bf16(np.array(sinks, dtype=np.float32))
        t["l0.mlp.router.b"] = ref.bf16(np.array([bias, 0, 0, bias, 0, 0], dtype=np.float32))
        runner, plain = make_runner(backend, tmp_path, cfg, dtype, 128, seed=len(outs), tensors=t)
        tokens = np.random.default_rng(6).integers(0, 70, size=80)
        want = plain.forward(tokens)
        got = runner.step("s", tokens, list(range(80)))
        assert np.quantile(ref.row_errors(got, want), 0.95) < LIMIT[dtype]
        outs.append(want)
        runner.close()
    assert np.median(ref.row_errors(outs[0], outs[1])) > 0.1 and np.median(ref.row_errors(outs[1], outs[2])) > 0.1


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_queue(backend, tmp_path, dtype):
    """Unequal requests one after another, prompts in portions: every token is the plain model's choice (or as good as)."""
    from hologram_b200 import decode
    cfg = ref.CONFIGS["looped" if dtype == "float32" else "plain"]
    vocab = cfg["vocab"]
    runner, plain = make_runner(backend, tmp_path, cfg, dtype, 160, max_rows=32)
    rng = np.random.default_rng(7)
    requests = [decode.Request(rng.integers(0, vocab, size=n).tolist(), m) for n, m in ((1, 30), (70, 20), (9, 5), (33, 40))]
    scheduler = decode.Scheduler(runner, portion=24)
    for r in requests:
        scheduler.submit(r)
    assert len(list(scheduler.run())) == 95
    for r in requests:
        assert len(r.tokens) == r.max_new_tokens
        plain.reset()
        logits = plain.forward(r.prompt + r.tokens[:-1])[len(r.prompt) - 1:]
        spread = logits.std()
        for row, token in zip(logits, r.tokens):
            assert row[token] >= row.max() - (1e-3 if dtype == "float32" else 0.3) * spread
        if dtype == "float32":
            assert [int(i) for i in logits.argmax(axis=1)] == r.tokens
    assert decode.generate(runner, requests[1].prompt, 20, portion=7) == requests[1].tokens or dtype == "bfloat16"
    runner.close()


def test_command_line_and_trace_replay(backend, tmp_path):
    cfg = ref.CONFIGS["odd"]
    t = ref.random_tensors(cfg, 1)
    path = ref.write_model(tmp_path / "m", cfg, t)
    plain = ref.Reference(cfg, t)
    env = dict(os.environ, PYTHONPATH=ROOT)
    out = subprocess.run([sys.executable, "-m", "hologram_b200", "generate", "--model", path, "--tokens", "1,2,3", "--tokens", "9", "--max-new", "6", "--dtype", "float32"],
                         capture_output=True, text=True, env=env, cwd=ROOT, timeout=120, check=True).stdout.split()
    for prompt, line in zip(([1, 2, 3], [9]), out):
        new = [int(x) for x in line.split(",")]
        plain.reset()
        logits = plain.forward(prompt + new[:-1])[len(prompt) - 1:]
        assert [int(i) for i in logits.argmax(axis=1)] == new
    tokens = np.random.default_rng(3).integers(0, 61, size=40).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:25], "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[25:27], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[27:40], "want": [12]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": tokens[:1], "want": [0]}], "end": ["b"]}]
    plain.reset()
    want = plain.forward(tokens)
    for dtype in ("float32", "bfloat16"):
        folder = tmp_path / dtype
        folder.mkdir()
        run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(folder), "--max-tokens", "64"],
                             input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240, check=True)
        assert [l for l in run.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        got = {i: np.fromfile(folder / f"{i}.f32", dtype="<f4").reshape(-1, 61) for i in (0, 2, 3)}
        assert not (folder / "1.f32").exists()
        for rows, logits in ((got[0], want[[0, 24]]), (got[2], want[[39]]), (got[3], want[[0]])):
            assert ref.row_errors(rows, logits).max() < 3 * LIMIT[dtype]
