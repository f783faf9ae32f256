"""CPU interpreter of a KernelCall list over numpy byte slots, built on the oracle kernels.

TEST INFRASTRUCTURE ONLY (see oracle/hologram_oracle.c). It plays the role the reference's
CpuBackend + slot-vector TestWorkspace play in crates/hologram-compute/tests: each call reads
and writes `slots[slot]` (numpy uint8 arrays). `all_reduce(array_f32) -> array_f32` supplies
the tensor-parallel sum when the list contains AllReduce calls.
"""
import numpy as np

from hologram_b200 import kernel_call as kc
from . import oracle as orc

_NP = {kc.DTYPE_F32: np.float32, kc.DTYPE_BF16: np.uint16, kc.DTYPE_F16: np.uint16, kc.DTYPE_I8: np.int8,
       kc.DTYPE_I32: np.int32, kc.DTYPE_I64: np.int64, kc.DTYPE_U8: np.uint8}
_LUT = {kc.K_SIGMOID: kc.LUT_SIGMOID, kc.K_TANH: kc.LUT_TANH, kc.K_GELU: kc.LUT_GELU, kc.K_SILU: kc.LUT_SILU,
        kc.K_EXP: kc.LUT_EXP, kc.K_ERF: kc.LUT_ERF}

_REDUCE = {kc.K_REDUCE_SUM: (0, False), kc.K_REDUCE_MEAN: (0, True), kc.K_REDUCE_PROD: (1, False), kc.K_REDUCE_MIN: (2, False),
           kc.K_REDUCE_MAX: (3, False)}


def _get(slots, ref, nbytes, dtype):
    buf = slots[ref.slot]
    assert ref.offset + nbytes <= buf.size, f"slot {ref.slot} too short"
    return buf[ref.offset:ref.offset + nbytes].view(_NP[dtype])


def _put(slots, ref, arr):
    raw = np.ascontiguousarray(arr).view(np.uint8).reshape(-1)
    if ref.slot not in slots or slots[ref.slot].size < ref.offset + raw.size:
        new = np.zeros(ref.offset + raw.size, dtype=np.uint8)
        if ref.slot in slots:
            new[:slots[ref.slot].size] = slots[ref.slot]
        slots[ref.slot] = new
    slots[ref.slot][ref.offset:ref.offset + raw.size] = raw


def _f32(bits):
    return float(np.array([bits], dtype=np.uint32).view(np.float32)[0])


def _wide(a, dtype):
    """f64 values of a bf16 or f32 array."""
    return (orc.bf16_to_f32(a) if dtype == kc.DTYPE_BF16 else a).astype(np.float64)


def _narrow(a, dtype):
    return orc.f32_to_bf16_rne(np.ascontiguousarray(a).reshape(-1)) if dtype == kc.DTYPE_BF16 else np.asarray(a, dtype=np.float32)


def _word(slots, ref, index=0):
    return int(_get(slots, kc.rb(ref.slot, ref.offset + 4 * index), 4, kc.DTYPE_I32).view(np.uint32)[0])


def _extent(slots, ref):
    return ref.length or slots[ref.slot].size - ref.offset


def _matrix(slots, ref, rows, cols, ld, dtype):
    """f64 values of `rows` rows of `cols` columns at pitch `ld`."""
    size = np.dtype(_NP[dtype]).itemsize
    flat = _wide(_get(slots, ref, ((rows - 1) * ld + cols) * size, dtype), dtype)
    return np.lib.stride_tricks.as_strided(flat, (rows, cols), (8 * ld, 8)).copy()


def _put_matrix(slots, ref, values, ld, dtype):
    size = np.dtype(_NP[dtype]).itemsize
    for i, row in enumerate(values):
        _put(slots, kc.rb(ref.slot, ref.offset + i * ld * size), _narrow(row.astype(np.float32), dtype))


def _linear_act(v, act):
    if act == kc.LINEAR_ACT_RELU2:
        return np.maximum(v, 0.0) ** 2
    if act == kc.LINEAR_ACT_GELU_TANH:
        return 0.5 * v * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (v + 0.044715 * v ** 3)))
    if act == kc.LINEAR_ACT_SILU:
        return v / (1.0 + np.exp(-v))
    if act == kc.LINEAR_ACT_SILU_GATE:
        return v[:, 0::2] / (1.0 + np.exp(-v[:, 0::2])) * v[:, 1::2]
    return v


def _linear(slots, c, extended):
    size = np.dtype(_NP[c.dtype]).itemsize
    grouped, window = extended and c.tiles.slot != kc.NO_SLOT, extended and c.a_pos.slot != kc.NO_SLOT
    if window:
        start = max(0, _word(slots, c.a_pos) - c.a_back) // 128 * 128
        a = _matrix(slots, c.a, c.a_rows, c.lda, c.lda, c.dtype)[(start + np.arange(c.m)) % c.a_rows]
    elif grouped and c.a_shared:
        a = np.zeros((c.m, c.lda))
        shared = _matrix(slots, c.a, c.a_shared, c.lda, c.lda, c.dtype)
        for t in range(c.m // c.tile_rows):
            a[t * c.tile_rows:t * c.tile_rows + c.a_shared] = shared
    else:
        a = _matrix(slots, c.a, c.m, c.lda, c.lda, c.dtype)
    b = _wide(_get(slots, c.b, c.k * c.n * size * (c.experts if grouped else 1), c.dtype), c.dtype).reshape(-1, c.k, c.n)
    if grouped:
        tiles = _get(slots, c.tiles, 4 * (1 + c.m // c.tile_rows), kc.DTYPE_I32)
        tiles = tiles[1:1 + tiles[0]]
    for g in list(c.seg)[:c.nseg]:
        cols = slice(g.col_begin, g.col_begin + g.width)
        if grouped:
            part = [a[t * c.tile_rows:(t + 1) * c.tile_rows, g.k_offset:g.k_offset + c.k] @ b[e][:, cols] for t, e in enumerate(tiles)]
            v = np.concatenate(part) if part else np.zeros((0, g.width))
        else:
            v = a[:, g.k_offset:g.k_offset + c.k] @ b[0][:, cols]
        v = _linear_act(v, g.act)
        if extended and g.rot_head:
            table = _matrix(slots, c.rot, c.m, g.rot_dims, g.rot_dims, kc.DTYPE_F32).reshape(c.m, -1, 2)
            for head in range(0, g.width, g.rot_head):
                lo = head + g.rot_begin
                e, o = v[:, lo:lo + g.rot_dims:2].copy(), v[:, lo + 1:lo + g.rot_dims:2].copy()
                v[:, lo:lo + g.rot_dims:2] = e * table[..., 0] - o * table[..., 1]
                v[:, lo + 1:lo + g.rot_dims:2] = o * table[..., 0] + e * table[..., 1]
        v = _f32(c.alpha_bits) * v
        out_size = np.dtype(_NP[g.dtype]).itemsize
        appends, ring = g.row_pos.slot != kc.NO_SLOT, extended and g.ring
        first = _word(slots, g.row_pos) if appends else 0
        limit = _extent(slots, g.output) // (g.ld * out_size) if appends else c.m
        if ring:
            limit = (_extent(slots, g.output) - g.width * out_size) // (g.ld * out_size) + 1
        count = min(len(v), _word(slots, g.row_pos, 1)) if ring else min(len(v), limit - first)
        for i in range(count):
            row, cells = ((first + i) % limit if ring else first + i), v[i]
            if c.residual.slot != kc.NO_SLOT:
                cells = cells + _get(slots, kc.rb(c.residual.slot, c.residual.offset + i * g.ld * 4), g.width * 4, kc.DTYPE_F32)
            _put(slots, kc.rb(g.output.slot, g.output.offset + row * g.ld * out_size), _narrow(cells.astype(np.float32), g.dtype))


def run(calls, slots, all_reduce=None):
    es = lambda dt: np.dtype(_NP[dt]).itemsize
    for call in calls:
        k, u = call.kind, call.u
        if k in _LUT:
            c = u.unary
            _put(slots, c.output, orc.unary_lut(_LUT[k], c.dtype, _get(slots, c.input, c.element_count * 2, c.dtype)))
        elif k in (kc.K_ADD, kc.K_MUL):
            c = u.binary
            n = c.element_count * es(c.dtype)
            _put(slots, c.output, orc.binary(0 if k == kc.K_ADD else 1, _get(slots, c.a, n, c.dtype), _get(slots, c.b, n, c.dtype), c.dtype))
        elif k in (kc.K_MATMUL, kc.K_MATMUL_ACTIVATION, kc.K_MATMUL_ADD):
            mm = u.matmul
            a = _get(slots, mm.a, mm.m * mm.k * 2, mm.dtype)
            b = _get(slots, mm.b, mm.k * mm.n * 2, mm.dtype)
            act = u.matmul_activation.act if k == kc.K_MATMUL_ACTIVATION else 0
            res = _get(slots, u.matmul_add.residual, mm.m * mm.n * 2, mm.dtype) if k == kc.K_MATMUL_ADD else None
            _put(slots, mm.output, orc.matmul(a, b, mm.m, mm.k, mm.n, mm.dtype, act=act, residual=res))
        elif k == kc.K_RMS_NORM:
            c = u.norm
            x = _get(slots, c.x, c.batch * c.feature * es(c.dtype), c.dtype)
            g = _get(slots, c.gamma, c.feature * es(c.dtype), c.dtype) if c.gamma.slot != kc.NO_SLOT else None
            _put(slots, c.output, orc.rms_norm(x, g, c.batch, c.feature, c.epsilon_bits, c.dtype))
        elif k == kc.K_LAYER_NORM:
            c = u.norm
            row = c.feature * es(c.dtype)
            x = _get(slots, c.x, c.batch * row, c.dtype)
            g = _get(slots, c.gamma, row, c.dtype) if c.gamma.slot != kc.NO_SLOT else None
            b = _get(slots, c.beta, row, c.dtype) if c.beta.slot != kc.NO_SLOT else None
            _put(slots, c.output, orc.layer_norm(x, g, b, c.batch, c.feature, c.epsilon_bits, c.dtype))
        elif k == kc.K_SOFTMAX:
            c = u.softmax
            x = _get(slots, c.input, c.batch * c.feature * es(c.dtype), c.dtype)
            _put(slots, c.output, orc.softmax(x, c.batch, c.feature, c.dtype))
        elif k in _REDUCE:
            c = u.reduce
            dims = [c.dims[i] for i in range(c.rank)]
            kind, mean = _REDUCE[k]
            _put(slots, c.output, orc.reduce(_get(slots, c.input, c.element_count * es(c.dtype), c.dtype), dims, c.axes_mask, kind, mean, c.dtype))
        elif k in (kc.K_EXPAND, kc.K_BROADCAST_BINARY):
            c = u.expand if k == kc.K_EXPAND else u.broadcast_binary
            ind, outd = [c.in_dims[i] for i in range(c.rank)], [c.out_dims[i] for i in range(c.rank)]
            small = _get(slots, c.input if k == kc.K_EXPAND else c.small, int(np.prod(ind)) * es(c.dtype), c.dtype)
            if k == kc.K_EXPAND:
                _put(slots, c.output, orc.broadcast(small, None, ind, outd, es(c.dtype)))
            else:
                other = _get(slots, c.other, int(np.prod(outd)) * es(c.dtype), c.dtype)
                _put(slots, c.output, orc.broadcast(small, other, ind, outd, es(c.dtype), c.op, bool(c.small_is_lhs), c.dtype))
        elif k in kc.EXACT_UNARY:
            c = u.unary
            _put(slots, c.output, orc.elementwise(k, _get(slots, c.input, c.element_count * es(c.dtype), c.dtype), None, c.dtype))
        elif k in kc.EXACT_BINARY:
            c = u.binary
            n = c.element_count * es(c.dtype)
            _put(slots, c.output, orc.elementwise(k, _get(slots, c.a, n, c.dtype), _get(slots, c.b, n, c.dtype), c.dtype))
        elif k == kc.K_WHERE:
            c = u.where
            n = c.element_count * es(c.dtype)
            _put(slots, c.output, orc.where(_get(slots, c.cond, c.element_count, kc.DTYPE_U8), _get(slots, c.a, n, c.dtype), _get(slots, c.b, n, c.dtype), c.dtype))
        elif k == kc.K_ATTENTION:
            c = u.attention
            hkv = c.kv_heads or c.heads
            q = _get(slots, c.q, c.batch * c.heads * c.seq * c.head_dim * es(c.dtype), c.dtype)
            kk = _get(slots, c.k, c.batch * hkv * c.seq * c.head_dim * es(c.dtype), c.dtype)
            v = _get(slots, c.v, c.batch * hkv * c.seq * c.head_dim * es(c.dtype), c.dtype)
            _put(slots, c.output, orc.attention(q, kk, v, c.batch, c.heads, c.kv_heads, c.seq, c.head_dim, bool(c.causal), c.scale_bits, c.dtype))
        elif k == kc.K_CONCAT:
            c = u.binary
            a = slots[c.a.slot][c.a.offset:c.a.offset + c.a.length] if c.a.length else slots[c.a.slot][c.a.offset:]
            b = slots[c.b.slot][c.b.offset:c.b.offset + c.b.length] if c.b.length else slots[c.b.slot][c.b.offset:]
            _put(slots, c.output, np.concatenate([a, b]))
        elif k == kc.K_ADD_RMS_NORM:
            c = u.norm
            n = c.batch * c.feature * es(c.dtype)
            x = _get(slots, c.x, n, c.dtype)
            r = _get(slots, c.residual, n, c.dtype) if c.residual.slot != kc.NO_SLOT else None
            g = _get(slots, c.gamma, c.feature * es(c.dtype), c.dtype) if c.gamma.slot != kc.NO_SLOT else None
            _put(slots, c.output, orc.add_rms_norm(x, r, g, c.batch, c.feature, c.epsilon_bits, c.dtype))
        elif k == kc.K_TRANSPOSE:
            c = u.transpose
            dims = [c.dims[i] for i in range(c.rank)]
            total = int(np.prod(dims)) * es(c.dtype)
            _put(slots, c.output, orc.transpose(_get(slots, c.input, total, kc.DTYPE_U8), dims, [c.perm[i] for i in range(c.rank)], es(c.dtype)))
        elif k == kc.K_ROTARY:
            c = u.rope
            n = c.element_count * es(c.dtype)
            _put(slots, c.output, orc.rope(_get(slots, c.x, n, c.dtype), _get(slots, c.cos, n, c.dtype), _get(slots, c.sin, n, c.dtype), c.head_dim, c.dtype))
        elif k == kc.K_GATHER:
            c = u.gather
            data = _get(slots, c.data, c.outer * c.axis_dim * c.inner * es(c.dtype), c.dtype)
            idx = _get(slots, c.indices, c.num_indices * es(c.idx_dtype), c.idx_dtype)
            rc, out = orc.gather(data, idx, c.outer, c.axis_dim, c.inner, c.dtype)
            assert rc == 0
            _put(slots, c.output, out)
        elif k == kc.K_QUANTIZE_ROWS_I8:
            c = u.quantize_rows_i8
            x = _get(slots, c.input, c.rows * c.row_len * es(c.dtype), c.dtype)
            codes, scales = orc.quantize_rows_i8(x, c.dtype, c.rows, c.row_len)
            _put(slots, c.codes, codes)
            _put(slots, c.scales, scales)
        elif k == kc.K_DECODE_ATTENTION_VALID_Q8:
            c = u.decode_attention_valid_q8
            hkv = c.kv_heads or c.heads
            prow, nrow = c.batch * hkv * c.past_len, c.batch * hkv * c.new_len
            q = _get(slots, c.q, c.batch * c.heads * c.q_rows * c.head_dim * es(c.dtype), c.dtype)
            g8 = lambda r, n: _get(slots, r, n * c.head_dim, kc.DTYPE_I8)
            gs = lambda r, n: _get(slots, r, n * 4, kc.DTYPE_F32)
            vl = int(_get(slots, c.valid_len, 4, kc.DTYPE_I32).view(np.uint32)[0])
            rc, out = orc.decode_attention_valid_q8(q, c.dtype, g8(c.k_past, prow), gs(c.k_past_scales, prow), g8(c.v_past, prow),
                                                    gs(c.v_past_scales, prow), g8(c.k_new, nrow), gs(c.k_new_scales, nrow),
                                                    g8(c.v_new, nrow), gs(c.v_new_scales, nrow), vl, c.batch, c.heads, c.kv_heads,
                                                    c.q_rows, c.past_len, c.new_len, c.head_dim, c.scale_bits)
            assert rc == 0
            _put(slots, c.output, out)
        elif k == kc.K_KV_CACHE_WRITE:
            c = u.kv_cache_write
            total = c.planes * c.bucket_rows * c.row_bytes
            cache = _get(slots, c.cache, total, kc.DTYPE_U8)
            new = _get(slots, c.new, c.planes * c.new_rows * c.row_bytes, kc.DTYPE_U8)
            pos = int(_get(slots, c.pos, 4, kc.DTYPE_I32).view(np.uint32)[0])
            rc, out = orc.kv_cache_write(cache, new, pos, c.planes, c.bucket_rows, c.new_rows, c.row_bytes)
            assert rc == 0
            _put(slots, c.output, out)
        elif k == kc.K_CAST:
            c = u.cast
            _put(slots, c.output, orc.cast_float(_get(slots, c.input, c.element_count * es(c.src_dtype), c.src_dtype), c.src_dtype, c.dst_dtype))
        elif k == kc.K_RMS_NORM_MULTI:
            c = u.rms_norm_multi
            x = _get(slots, c.x, c.rows * c.feature * 4, kc.DTYPE_F32).reshape(c.rows, c.feature).astype(np.float64)
            gammas = [g for g in (c.gamma0, c.gamma1) if g.slot != kc.NO_SLOT]
            out = np.zeros((c.rows, len(gammas), c.step), dtype=np.float32)
            inv = 1.0 / np.sqrt((x * x).mean(axis=1, keepdims=True) + _f32(c.epsilon_bits))
            for i, g in enumerate(gammas):
                out[:, i, :c.feature] = x * inv * _get(slots, g, c.feature * 4, kc.DTYPE_F32)
            _put(slots, c.output, _narrow(out, c.dtype))
        elif k in (kc.K_LINEAR, kc.K_LINEAR_EX):
            _linear(slots, u.linear, k == kc.K_LINEAR_EX)
        elif k == kc.K_ROTARY_TABLE:
            c = u.rotary_table
            f = _get(slots, c.freq, 8 * c.half, kc.DTYPE_F32).astype(np.float64).reshape(2, c.half).sum(axis=0)
            a = 2.0 * np.pi * (_word(slots, c.pos) + np.arange(c.rows))[:, None] * f
            _put(slots, c.output, np.stack([np.cos(a), np.sin(a)], axis=-1).astype(np.float32))
        elif k == kc.K_RMS_NORM_PARTS:
            c = u.rms_norm_parts
            for p in list(c.part)[:c.nparts]:
                x = _matrix(slots, kc.rb(c.x.slot, c.x.offset + 4 * p.in_col), c.rows, p.width, c.ld_in, kc.DTYPE_F32)
                if p.norm:
                    x = x / np.sqrt((x * x).mean(axis=1, keepdims=True) + _f32(c.epsilon_bits))
                if p.weight.slot != kc.NO_SLOT:
                    x = x * _get(slots, p.weight, 4 * p.width, kc.DTYPE_F32)
                x = np.concatenate([x, np.zeros((c.rows, p.out_width - p.width))], axis=1)
                size = es(c.dtype)
                for i in range(min(c.rows, _word(slots, c.step, 1)) if p.ring else c.rows):
                    row = (_word(slots, c.step) + i) % ((_extent(slots, p.output) - p.out_width * size) // (p.ld * size) + 1) if p.ring else i
                    _put(slots, kc.rb(p.output.slot, p.output.offset + row * p.ld * size), _narrow(x[i].astype(np.float32), c.dtype))
        elif k == kc.K_HEAD_LINEAR:
            c = u.head_linear
            size = es(c.dtype)
            for h in range(c.heads):
                a = _matrix(slots, kc.rb(c.a.slot, c.a.offset + h * c.a_step * size), c.rows, c.k, c.lda, c.dtype)
                b = _matrix(slots, kc.rb(c.b.slot, c.b.offset + h * c.b_step * size), c.k, c.n, c.b_ld, c.dtype)
                _put_matrix(slots, kc.rb(c.output.slot, c.output.offset + h * c.out_step * size), a @ b, c.ld, c.dtype)
        elif k == kc.K_WINDOW_ATTENTION:
            c = u.window_attention
            size, first, scale = es(c.dtype), _word(slots, c.pos), _f32(c.scale_bits)
            start = 0 if c.kv_back == kc.WHOLE_CACHE else max(0, first - c.kv_back) // 128 * 128
            kk, vv = (_matrix(slots, r, c.kv_rows, c.kv_heads * d, ld, c.dtype) for r, d, ld in ((c.k, c.dim, c.k_ld), (c.v, c.vdim, c.v_ld)))
            k2 = _matrix(slots, c.k2, c.k2_rows, c.dim2, c.k2_ld, c.dtype) if c.dim2 else None
            for h in range(c.heads):
                g = h // (c.heads // c.kv_heads)
                q = _matrix(slots, kc.rb(c.q.slot, c.q.offset + h * c.q_step * size), c.rows, c.dim, c.q_ld, c.dtype)
                q2 = _matrix(slots, kc.rb(c.q2.slot, c.q2.offset + h * c.q2_step * size), c.rows, c.dim2, c.q2_ld, c.dtype) if c.dim2 else None
                sink = _get(slots, kc.rb(c.sink.slot, c.sink.offset + 4 * h), 4, kc.DTYPE_F32)[0] if c.sink.slot != kc.NO_SLOT else -np.inf
                out = np.zeros((c.rows, c.vdim))
                for i in range(c.rows):
                    p = first + i
                    j = np.arange(max(0, p + 1 - c.window) if c.window else 0, p + 1)
                    rows = (j - start) % c.kv_rows
                    s = kk[rows, g * c.dim:(g + 1) * c.dim] @ q[i]
                    if c.dim2:
                        s = s + k2[j % c.k2_rows] @ q2[i]
                    s = s * scale
                    top = max(s.max(), sink)
                    e = np.exp(s - top)
                    out[i] = e @ vv[rows, g * c.vdim:(g + 1) * c.vdim] / (e.sum() + np.exp(sink - top))
                _put_matrix(slots, kc.rb(c.output.slot, c.output.offset + h * c.vdim * size), out, c.ld, c.dtype)
        elif k == kc.K_RETENTION:
            c = u.retention
            q, kk = (_matrix(slots, r, c.rows, c.heads * c.dim, ld, c.dtype).reshape(c.rows, c.heads, c.dim) for r, ld in ((c.q, c.q_ld), (c.k, c.k_ld)))
            v, gate = (_matrix(slots, r, c.rows, c.heads * c.vdim, ld, c.dtype).reshape(c.rows, c.heads, c.vdim) for r, ld in ((c.v, c.v_ld), (c.gate, c.gate_ld)))
            decay = _get(slots, c.decay, 4 * c.heads, kc.DTYPE_F32).astype(np.float64)
            state = _get(slots, c.state, 4 * c.heads * c.dim * c.vdim, kc.DTYPE_F32).astype(np.float64).reshape(c.heads, c.dim, c.vdim)
            state = state * (_word(slots, c.step) != 0)
            size = es(c.dtype)
            for i in range(min(c.rows, _word(slots, c.step, 1))):
                state = decay[:, None, None] * state + kk[i][:, :, None] * v[i][:, None, :]
                o = _f32(c.scale_bits) * np.einsum("hde,hd->he", state, q[i])
                o = o / np.sqrt((o[:, :c.vmean] ** 2).mean(axis=1, keepdims=True) + _f32(c.epsilon_bits)) * gate[i]
                _put(slots, kc.rb(c.output.slot, c.output.offset + i * c.ld * size), _narrow(o.reshape(-1).astype(np.float32), c.dtype))
            _put(slots, c.state, state.astype(np.float32))
        elif k == kc.K_MOE_PLAN:
            c = u.moe_plan
            z = _matrix(slots, c.logits, c.rows, c.experts, c.ld_logits, kc.DTYPE_F32)
            if c.bias.slot != kc.NO_SLOT:
                z = z + _get(slots, c.bias, 4 * c.experts, kc.DTYPE_F32)
            n = min(c.rows, _word(slots, c.step, 1))
            chosen = np.argsort(-z[:n], axis=1, kind="stable")[:, :c.top]
            e = np.take_along_axis(z[:n], chosen, axis=1)
            e = np.exp(e - e[:, :1])
            weight, place = np.zeros((c.rows, c.top), dtype=np.float32), np.zeros((c.rows, c.top), dtype=np.int32)
            weight[:n] = e / e.sum(axis=1, keepdims=True)
            tiles, source = [], np.zeros(c.max_tiles * c.tile_rows, dtype=np.int32)
            for x in range(c.experts):
                pairs = np.argwhere(chosen == x)
                for at, (i, t) in enumerate(pairs):
                    place[i, t] = len(tiles) * c.tile_rows + (i if c.rows <= c.tile_rows else at)
                    source[place[i, t]] = i
                tiles += [x] * (min(1, len(pairs)) if c.rows <= c.tile_rows else -(-len(pairs) // c.tile_rows))
            assert len(tiles) <= c.max_tiles
            _put(slots, c.weight, weight)
            _put(slots, c.place, place)
            _put(slots, c.source, source)
            _put(slots, c.tiles, np.array([len(tiles)] + tiles, dtype=np.int32))
        elif k == kc.K_MOE_COMBINE:
            c = u.moe_combine
            x = _matrix(slots, c.x, c.rows, c.width, c.width, kc.DTYPE_F32)
            y = _matrix(slots, c.y, c.y_rows, c.width, c.ld, c.dtype)
            weight = _get(slots, c.weight, 4 * c.rows * c.top, kc.DTYPE_F32).reshape(c.rows, c.top)
            place = _get(slots, c.place, 4 * c.rows * c.top, kc.DTYPE_I32).reshape(c.rows, c.top)
            for i in range(min(c.rows, _word(slots, c.step, 1))):
                x[i] += weight[i].astype(np.float64) @ y[place[i]]
            _put(slots, c.x, x.astype(np.float32))
        elif k == kc.K_CAUSAL_ATTENTION:
            c = u.causal_attention
            size = es(c.dtype)
            load = lambda ref, *shape: _wide(_get(slots, ref, int(np.prod(shape)) * size, c.dtype), c.dtype).reshape(shape)
            q, kk = load(c.q, c.rows, c.heads, c.dim), load(c.k, c.cache_rows, c.kv_heads, c.dim)
            v = load(c.v, c.cache_rows, c.kv_heads, c.vdim)
            first = int(_get(slots, c.pos, 4, kc.DTYPE_I32)[0])
            every, cap = _f32(c.temp_every_bits), _f32(c.softcap_bits)
            scale = _f32(c.scale_bits) or c.dim ** -0.5
            for i in range(c.rows):
                n = min(first + i + 1, c.cache_rows)
                f = scale * (1.0 + _f32(c.temp_coef_bits) * np.log(np.floor((first + i + 1) / every) + 1.0) if every else 1.0)
                for h in range(c.heads):
                    kv = h // (c.heads // c.kv_heads)
                    s = kk[:n, kv] @ q[i, h] * f
                    s = cap * np.tanh(s / cap) if cap else s
                    sink = _get(slots, kc.rb(c.sink.slot, c.sink.offset + 4 * h), 4, kc.DTYPE_F32)[0] if c.sink.slot != kc.NO_SLOT else -np.inf
                    top = max(s.max(), sink)
                    e = np.exp(s - top)
                    o = e @ v[:n, kv] / (e.sum() + np.exp(sink - top))
                    _put(slots, kc.rb(c.output.slot, c.output.offset + (i * c.ld + h * c.vdim) * size), _narrow(o.astype(np.float32), c.dtype))
        elif k == kc.K_ALL_REDUCE:
            c = u.all_reduce
            assert c.dtype == kc.DTYPE_BF16
            part = orc.bf16_to_f32(_get(slots, c.buffer, c.element_count * 2, c.dtype))
            total = all_reduce(part) if all_reduce else part
            _put(slots, c.buffer, orc.f32_to_bf16_rne(total))
        else:
            raise NotImplementedError(f"oracle interpreter: KernelCall kind {k}")
    return slots
