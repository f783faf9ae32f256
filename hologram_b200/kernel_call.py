"""ctypes mirror of include/hologram_b200.h: the `KernelCall` tagged union and its payloads.

Names follow the reference (crates/hologram-compute/src/kernel_call.rs): BufferRef,
UnaryCall, MatMulCall, DecodeAttentionValidCall ... so tests read like the reference's own.
"""
import ctypes as C

# dtype tags (crates/hologram-types/src/dtype_id.rs:51-74)
DTYPE_BOOL, DTYPE_U8, DTYPE_I8, DTYPE_U64, DTYPE_I32, DTYPE_I64 = 0, 1, 2, 3, 4, 5
DTYPE_F16, DTYPE_BF16, DTYPE_F32, DTYPE_F64 = 6, 7, 8, 9
DTYPE_I4 = 10     # two signed nibbles per byte, low nibble first

# lut_act ids (kernel_call.rs:877-885)
LUT_SIGMOID, LUT_TANH, LUT_GELU, LUT_SILU, LUT_EXP, LUT_ERF = 0, 1, 2, 3, 4, 5
LUT_NAMES = {LUT_SIGMOID: "sigmoid", LUT_TANH: "tanh", LUT_GELU: "gelu", LUT_SILU: "silu", LUT_EXP: "exp", LUT_ERF: "erf"}

# fused_activation ids (kernel_call.rs:861-870)
FUSED_RELU, FUSED_GELU, FUSED_SILU, FUSED_SIGMOID, FUSED_TANH, FUSED_EXP = 1, 2, 3, 4, 5, 8

# variant tags = archive wire discriminants (crates/hologram-archive/src/kernel_codec.rs:19-128)
K_ADD, K_MUL = 5, 7
# exact elementwise variants (one IEEE operation per element)
K_NEG, K_RELU, K_SQRT, K_RECIPROCAL, K_CEIL, K_FLOOR, K_ROUND, K_IS_NAN, K_SIGN, K_ABS = 1, 11, 21, 22, 29, 30, 31, 33, 34, 35
K_SUB, K_DIV, K_MOD, K_MIN, K_MAX, K_EQUAL, K_LESS, K_LESS_OR_EQUAL, K_GREATER, K_GREATER_OR_EQUAL = 6, 36, 38, 39, 40, 41, 42, 43, 44, 45
EXACT_UNARY = (K_NEG, K_RELU, K_SQRT, K_RECIPROCAL, K_CEIL, K_FLOOR, K_ROUND, K_IS_NAN, K_SIGN, K_ABS)
EXACT_BINARY = (K_SUB, K_DIV, K_MOD, K_MIN, K_MAX, K_EQUAL, K_LESS, K_LESS_OR_EQUAL, K_GREATER, K_GREATER_OR_EQUAL)
K_SIGMOID, K_TANH, K_GELU, K_SILU, K_EXP, K_ERF = 12, 13, 14, 15, 18, 32
K_MATMUL, K_RMS_NORM, K_RESHAPE, K_ROTARY = 46, 51, 60, 75
K_LAYER_NORM, K_EXPAND, K_BROADCAST_BINARY, K_ATTENTION, K_DEQUANT_ACTIVATION, K_WHERE = 50, 72, 112, 69, 113, 78
BROADCAST_ADD, BROADCAST_SUB, BROADCAST_MUL = 0, 1, 2
K_REDUCE_SUM, K_REDUCE_MEAN, K_REDUCE_PROD, K_REDUCE_MIN, K_REDUCE_MAX = 55, 56, 57, 58, 59
K_ADD_RMS_NORM, K_TRANSPOSE, K_CONCAT, K_SLICE, K_SOFTMAX = 54, 61, 62, 63, 64
K_DECODE_ATTENTION = 119
K_MATMUL_DEQUANT = 116
K_MATMUL_DEQUANT_PLAIN = 111      # the all-default wire form ([k,n] weight, f32 activations)
K_MATMUL_ADD_ACTIVATION = 108
K_MATMUL_DEQUANT_CODEBOOK = 117   # the same call with a codebook operand bound (E8 codebook weights)
DTYPE_E8CB = 11
K_DEQUANTIZE, K_MATMUL_ACTIVATION, K_MATMUL_ADD = 105, 106, 107
K_GATHER, K_CAST, K_KV_CACHE_WRITE, K_DECODE_ATTENTION_VALID = 114, 115, 120, 121
K_QUANTIZE_ROWS_I8, K_DECODE_ATTENTION_VALID_Q8, K_ALL_REDUCE = 0x8001, 0x8002, 0x8003
K_ROPE_QUANTIZE_ROWS_I8 = 0x8004
K_RMS_NORM_MULTI, K_LINEAR, K_CAUSAL_ATTENTION = 0x8005, 0x8006, 0x8007
K_LINEAR_EX, K_ROTARY_TABLE, K_RMS_NORM_PARTS, K_HEAD_LINEAR = 0x8008, 0x8009, 0x800a, 0x800b
K_WINDOW_ATTENTION, K_RETENTION, K_MOE_PLAN, K_MOE_COMBINE = 0x800c, 0x800d, 0x800e, 0x800f
LUT_KIND = {LUT_SIGMOID: K_SIGMOID, LUT_TANH: K_TANH, LUT_GELU: K_GELU, LUT_SILU: K_SILU, LUT_EXP: K_EXP, LUT_ERF: K_ERF}

NO_SLOT = 0xFFFFFFFF

# status codes (crates/hologram-compute/src/error.rs:6-20)
OK, ERR_SLOT_OUT_OF_RANGE, ERR_SHAPE_MISMATCH, ERR_UNSUPPORTED_OP, ERR_INIT, ERR_DISPATCH = 0, -1, -2, -3, -4, -5


class BufferRef(C.Structure):
    _fields_ = [("slot", C.c_uint32), ("offset", C.c_uint64), ("length", C.c_uint64)]


def rb(slot, offset=0, length=0):
    """BufferRef over a whole slot (the reference tests' `rb` helper, tests/lut.rs:51-57)."""
    return BufferRef(slot, offset, length)


NONE = BufferRef(NO_SLOT, 0, 0)


def f32_bits(x):
    """The bit pattern of an f32 scalar, as the calls carry their constants."""
    return C.c_uint32.from_buffer(C.c_float(x)).value


class UnaryCall(C.Structure):
    _fields_ = [("input", BufferRef), ("output", BufferRef), ("element_count", C.c_uint64),
                ("witt_bits", C.c_uint16), ("dtype", C.c_uint8)]


class BinaryCall(C.Structure):
    _fields_ = [("a", BufferRef), ("b", BufferRef), ("output", BufferRef), ("element_count", C.c_uint64),
                ("witt_bits", C.c_uint16), ("dtype", C.c_uint8)]


class MatMulCall(C.Structure):
    _fields_ = [("a", BufferRef), ("b", BufferRef), ("output", BufferRef), ("m", C.c_uint32), ("k", C.c_uint32),
                ("n", C.c_uint32), ("dtype", C.c_uint8), ("b_packed", C.c_uint8)]


class MatMulActivationCall(C.Structure):
    _fields_ = [("mm", MatMulCall), ("act", C.c_uint8)]


class MatMulAddCall(C.Structure):
    _fields_ = [("mm", MatMulCall), ("residual", BufferRef)]


class MatMulAddActivationCall(C.Structure):
    """kernel_call.rs:913-929: out = act(A . B + residual)."""
    _fields_ = [("mm", MatMulCall), ("residual", BufferRef), ("act", C.c_uint8)]


class MatMulDequantCall(C.Structure):
    """kernel_call.rs:152-213 (wire forms 111 / 116 / 117). Served: output-major W8A8 (bq_omajor=1, act_quant=1) over
    i8 / i4 / e8cb weights, and the [k,n] form with f32 activations (bq_omajor=0, act_quant=0) over i8 / u8 / i4."""
    _fields_ = [("a", BufferRef), ("bq", BufferRef), ("scales", BufferRef), ("zero_points", BufferRef), ("output", BufferRef),
                ("m", C.c_uint32), ("k", C.c_uint32), ("n", C.c_uint32), ("channels", C.c_uint32), ("inner", C.c_uint32),
                ("quant_dtype", C.c_uint8), ("dtype", C.c_uint8), ("scale_bits", C.c_uint32), ("zero_point", C.c_int32),
                ("bq_omajor", C.c_uint8), ("act_quant", C.c_uint8), ("act", C.c_uint8), ("residual", BufferRef), ("codebook", BufferRef)]

    def __init__(self, *args, **kw):
        super().__init__(*args, **kw)
        if len(args) < 19 and "codebook" not in kw:
            self.codebook = NONE


class NormCall(C.Structure):
    _fields_ = [("x", BufferRef), ("gamma", BufferRef), ("beta", BufferRef), ("residual", BufferRef),
                ("output", BufferRef), ("batch", C.c_uint32), ("feature", C.c_uint32), ("channels", C.c_uint32),
                ("num_groups", C.c_uint32), ("epsilon_bits", C.c_uint64), ("dtype", C.c_uint8)]


class RoPECall(C.Structure):
    _fields_ = [("x", BufferRef), ("cos", BufferRef), ("sin", BufferRef), ("output", BufferRef),
                ("head_dim", C.c_uint32), ("element_count", C.c_uint64), ("dtype", C.c_uint8)]


class GatherCall(C.Structure):
    _fields_ = [("data", BufferRef), ("indices", BufferRef), ("output", BufferRef), ("outer", C.c_uint64),
                ("axis_dim", C.c_uint64), ("inner", C.c_uint64), ("num_indices", C.c_uint64),
                ("idx_dtype", C.c_uint8), ("dtype", C.c_uint8)]


class CastCall(C.Structure):
    _fields_ = [("input", BufferRef), ("output", BufferRef), ("element_count", C.c_uint64),
                ("src_dtype", C.c_uint8), ("dst_dtype", C.c_uint8)]


class LayoutCall(C.Structure):
    _fields_ = [("input", BufferRef), ("output", BufferRef), ("element_count", C.c_uint64), ("dtype", C.c_uint8)]


class SoftmaxCall(C.Structure):
    _fields_ = [("input", BufferRef), ("output", BufferRef), ("batch", C.c_uint32), ("feature", C.c_uint32), ("dtype", C.c_uint8)]


class WhereCall(C.Structure):
    """kernel_call.rs:761-769: out[i] = cond[i] != 0 ? a[i] : b[i]; one condition byte per element."""
    _fields_ = [("cond", BufferRef), ("a", BufferRef), ("b", BufferRef), ("output", BufferRef), ("element_count", C.c_uint64),
                ("dtype", C.c_uint8)]


class DequantActivationCall(C.Structure):
    """kernel_call.rs:265-290: out = act((q - zero_point) * scale), i8 / u8 / i4 in, f32 out; act is a LUT_* id."""
    _fields_ = [("input", BufferRef), ("output", BufferRef), ("element_count", C.c_uint64), ("quant_dtype", C.c_uint8),
                ("act", C.c_uint8), ("dtype", C.c_uint8), ("scale_bits", C.c_uint32), ("zero_point", C.c_int32)]


class AttentionCall(C.Structure):
    """kernel_call.rs:575-594: q [b, heads, seq, d], k / v [b, kv_heads, seq, d]; causal: row i sees keys j <= i."""
    _fields_ = [("q", BufferRef), ("k", BufferRef), ("v", BufferRef), ("output", BufferRef), ("batch", C.c_uint32),
                ("heads", C.c_uint32), ("seq", C.c_uint32), ("head_dim", C.c_uint32), ("kv_heads", C.c_uint32),
                ("causal", C.c_uint8), ("scale_bits", C.c_uint32), ("dtype", C.c_uint8)]


class ReduceCall(C.Structure):
    """kernel_call.rs:461-477: fold the axes set in axes_mask (0 = all); keepdims layout."""
    _fields_ = [("input", BufferRef), ("output", BufferRef), ("element_count", C.c_uint64), ("rank", C.c_uint8),
                ("dims", C.c_uint32 * 8), ("axes_mask", C.c_uint32), ("keepdims", C.c_uint8), ("dtype", C.c_uint8)]

    @classmethod
    def make(cls, inp, out, dims, axes_mask, dtype, keepdims=True):
        c = cls()
        c.input, c.output, c.rank, c.axes_mask, c.keepdims, c.dtype = inp, out, len(dims), axes_mask, int(keepdims), dtype
        n = 1
        for i, d in enumerate(dims):
            c.dims[i] = d
            n *= d
        c.element_count = n
        return c


class ExpandCall(C.Structure):
    """kernel_call.rs:539-547: an axis with in_dims[i] == 1 reads index 0, the others map 1:1."""
    _fields_ = [("input", BufferRef), ("output", BufferRef), ("rank", C.c_uint8), ("in_dims", C.c_uint32 * 8),
                ("out_dims", C.c_uint32 * 8), ("dtype", C.c_uint8)]

    @classmethod
    def make(cls, inp, out, in_dims, out_dims, dtype):
        c = cls()
        c.input, c.output, c.rank, c.dtype = inp, out, len(out_dims), dtype
        for i, (a, b) in enumerate(zip(in_dims, out_dims)):
            c.in_dims[i], c.out_dims[i] = a, b
        return c


class BroadcastBinaryCall(C.Structure):
    """kernel_call.rs:292-317: out[o] = op(small[bcast(o)], other[o]) (swapped when small_is_lhs is 0)."""
    _fields_ = [("small", BufferRef), ("other", BufferRef), ("output", BufferRef), ("rank", C.c_uint8),
                ("in_dims", C.c_uint32 * 8), ("out_dims", C.c_uint32 * 8), ("op", C.c_uint8), ("small_is_lhs", C.c_uint8),
                ("dtype", C.c_uint8)]

    @classmethod
    def make(cls, small, other, out, in_dims, out_dims, op, small_is_lhs, dtype):
        c = cls()
        c.small, c.other, c.output, c.rank = small, other, out, len(out_dims)
        c.op, c.small_is_lhs, c.dtype = op, int(small_is_lhs), dtype
        for i, (a, b) in enumerate(zip(in_dims, out_dims)):
            c.in_dims[i], c.out_dims[i] = a, b
        return c


class TransposeCall(C.Structure):
    """kernel_call.rs:491-499: output axis i is input axis perm[i]."""
    _fields_ = [("input", BufferRef), ("output", BufferRef), ("rank", C.c_uint8), ("dims", C.c_uint32 * 8),
                ("perm", C.c_uint8 * 8), ("dtype", C.c_uint8)]

    @classmethod
    def make(cls, inp, out, dims, perm, dtype):
        c = cls()
        c.input, c.output, c.rank, c.dtype = inp, out, len(dims), dtype
        for i, (d, p) in enumerate(zip(dims, perm)):
            c.dims[i], c.perm[i] = d, p
        return c


class DequantizeCall(C.Structure):
    _fields_ = [("input", BufferRef), ("scales", BufferRef), ("zero_points", BufferRef), ("output", BufferRef),
                ("element_count", C.c_uint64), ("channels", C.c_uint32), ("inner", C.c_uint32),
                ("quant_dtype", C.c_uint8), ("dtype", C.c_uint8), ("scale_bits", C.c_uint32),
                ("zero_point", C.c_int32)]


class KvCacheWriteCall(C.Structure):
    _fields_ = [("cache", BufferRef), ("new", BufferRef), ("pos", BufferRef), ("output", BufferRef),
                ("planes", C.c_uint32), ("bucket_rows", C.c_uint32), ("new_rows", C.c_uint32),
                ("row_bytes", C.c_uint32)]


class DecodeAttentionValidCall(C.Structure):
    _fields_ = [("q", BufferRef), ("k_past", BufferRef), ("v_past", BufferRef), ("k_new", BufferRef),
                ("v_new", BufferRef), ("valid_len", BufferRef), ("output", BufferRef), ("batch", C.c_uint32),
                ("heads", C.c_uint32), ("kv_heads", C.c_uint32), ("q_rows", C.c_uint32), ("past_len", C.c_uint32),
                ("new_len", C.c_uint32), ("head_dim", C.c_uint32), ("scale_bits", C.c_uint32), ("dtype", C.c_uint8)]


class DecodeAttentionCall(C.Structure):
    """The additive-mask form (kernel_call.rs:632-655): mask is f32 [q_rows, past_len + new_len]."""
    _fields_ = [("q", BufferRef), ("k_past", BufferRef), ("v_past", BufferRef), ("k_new", BufferRef),
                ("v_new", BufferRef), ("mask", BufferRef), ("output", BufferRef), ("batch", C.c_uint32),
                ("heads", C.c_uint32), ("kv_heads", C.c_uint32), ("q_rows", C.c_uint32), ("past_len", C.c_uint32),
                ("new_len", C.c_uint32), ("head_dim", C.c_uint32), ("scale_bits", C.c_uint32), ("dtype", C.c_uint8)]


class QuantizeRowsI8Call(C.Structure):
    _fields_ = [("input", BufferRef), ("codes", BufferRef), ("scales", BufferRef), ("rows", C.c_uint64),
                ("row_len", C.c_uint32), ("dtype", C.c_uint8)]


class DecodeAttentionValidQ8Call(C.Structure):
    _fields_ = [("q", BufferRef), ("k_past", BufferRef), ("k_past_scales", BufferRef), ("v_past", BufferRef),
                ("v_past_scales", BufferRef), ("k_new", BufferRef), ("k_new_scales", BufferRef), ("v_new", BufferRef),
                ("v_new_scales", BufferRef), ("valid_len", BufferRef), ("output", BufferRef), ("batch", C.c_uint32),
                ("heads", C.c_uint32), ("kv_heads", C.c_uint32), ("q_rows", C.c_uint32), ("past_len", C.c_uint32),
                ("new_len", C.c_uint32), ("head_dim", C.c_uint32), ("scale_bits", C.c_uint32), ("dtype", C.c_uint8)]


class RopeQuantizeCall(C.Structure):
    """Extension: RotaryEmbedding then QuantizeRowsI8 of its result, one row = one head."""
    _fields_ = [("x", BufferRef), ("cos", BufferRef), ("sin", BufferRef), ("rope_output", BufferRef), ("codes", BufferRef),
                ("scales", BufferRef), ("rows", C.c_uint64), ("row_len", C.c_uint32), ("dtype", C.c_uint8)]


class AllReduceCall(C.Structure):
    _fields_ = [("buffer", BufferRef), ("element_count", C.c_uint64), ("dtype", C.c_uint8)]


class RmsNormMultiCall(C.Structure):
    """Extension: f32 rows normalised under one or two f32 weights, side by side in the output (`step` columns each)."""
    _fields_ = [("x", BufferRef), ("gamma0", BufferRef), ("gamma1", BufferRef), ("output", BufferRef), ("rows", C.c_uint32),
                ("feature", C.c_uint32), ("step", C.c_uint32), ("epsilon_bits", C.c_uint32), ("dtype", C.c_uint8)]


LINEAR_MAX_SEGS = 4
LINEAR_ACT_NONE, LINEAR_ACT_RELU2, LINEAR_ACT_GELU_TANH, LINEAR_ACT_SILU, LINEAR_ACT_SILU_GATE = range(5)


class LinearSeg(C.Structure):
    _fields_ = [("output", BufferRef), ("row_pos", BufferRef), ("col_begin", C.c_uint32), ("width", C.c_uint32),
                ("k_offset", C.c_uint32), ("ld", C.c_uint32), ("act", C.c_uint8), ("dtype", C.c_uint8), ("ring", C.c_uint8),
                ("rot_head", C.c_uint32), ("rot_begin", C.c_uint32), ("rot_dims", C.c_uint32)]

    @classmethod
    def make(cls, output, width, ld, dtype, col_begin=0, k_offset=0, act=LINEAR_ACT_NONE, row_pos=None, ring=False, rotate=None):
        """`rotate` = (columns per head, first rotated column, rotated columns)."""
        head, begin, dims = rotate or (0, 0, 0)
        return cls(output, NONE if row_pos is None else row_pos, col_begin, width, k_offset, ld, act, dtype, int(ring), head, begin, dims)


class LinearCall(C.Structure):
    """Extension: out_s[i, j] = residual + alpha * act_s(A[i, k_offset:k_offset + k] . B[:, col_begin + j]) for up to four segments;
    the extended fields add rotation, ring rows, a row window of A and groups."""
    _fields_ = [("a", BufferRef), ("b", BufferRef), ("residual", BufferRef), ("rot", BufferRef), ("a_pos", BufferRef), ("tiles", BufferRef),
                ("seg", LinearSeg * LINEAR_MAX_SEGS), ("m", C.c_uint32), ("k", C.c_uint32), ("n", C.c_uint32), ("lda", C.c_uint32),
                ("nseg", C.c_uint32), ("alpha_bits", C.c_uint32), ("a_back", C.c_uint32), ("a_rows", C.c_uint32), ("tile_rows", C.c_uint32),
                ("experts", C.c_uint32), ("a_shared", C.c_uint32), ("dtype", C.c_uint8)]

    @classmethod
    def make(cls, a, b, segs, m, k, n, dtype, lda=None, residual=None, alpha=1.0, rot=None, a_pos=None, a_back=0, a_rows=0, tiles=None,
             tile_rows=0, experts=0, a_shared=0):
        c = cls()
        c.a, c.b, c.residual = a, b, NONE if residual is None else residual
        c.rot, c.a_pos, c.tiles = (NONE if r is None else r for r in (rot, a_pos, tiles))
        c.m, c.k, c.n, c.lda, c.nseg, c.dtype = m, k, n, k if lda is None else lda, len(segs), dtype
        c.a_back, c.a_rows, c.tile_rows, c.experts, c.a_shared = a_back, a_rows, tile_rows, experts, a_shared
        c.alpha_bits = f32_bits(alpha)
        for i, g in enumerate(segs):
            c.seg[i] = g
        return c

    @property
    def extended(self):
        refs = (self.rot, self.a_pos, self.tiles)
        return any(r.slot != NO_SLOT for r in refs) or any(g.ring or g.rot_head for g in list(self.seg)[:self.nseg])


class CausalAttentionCall(C.Structure):
    """Extension: new rows of one sequence over the cache that already holds them (score cap, sink, query temperature)."""
    _fields_ = [("q", BufferRef), ("k", BufferRef), ("v", BufferRef), ("pos", BufferRef), ("sink", BufferRef), ("output", BufferRef),
                ("rows", C.c_uint32), ("heads", C.c_uint32), ("kv_heads", C.c_uint32), ("dim", C.c_uint32), ("vdim", C.c_uint32),
                ("cache_rows", C.c_uint32), ("ld", C.c_uint32), ("scale_bits", C.c_uint32), ("softcap_bits", C.c_uint32),
                ("temp_coef_bits", C.c_uint32), ("temp_every_bits", C.c_uint32), ("dtype", C.c_uint8)]


class RotaryTableCall(C.Structure):
    """Extension: (cos, sin) of every row's angles."""
    _fields_ = [("pos", BufferRef), ("freq", BufferRef), ("output", BufferRef), ("rows", C.c_uint32), ("half", C.c_uint32)]


NORM_MAX_PARTS = 3


class NormPart(C.Structure):
    _fields_ = [("weight", BufferRef), ("output", BufferRef), ("in_col", C.c_uint32), ("width", C.c_uint32), ("out_width", C.c_uint32),
                ("ld", C.c_uint32), ("norm", C.c_uint8), ("ring", C.c_uint8)]


class RmsNormPartsCall(C.Structure):
    """Extension: column ranges of f32 rows, each normalised (or copied) into a buffer of its own."""
    _fields_ = [("x", BufferRef), ("step", BufferRef), ("part", NormPart * NORM_MAX_PARTS), ("rows", C.c_uint32), ("ld_in", C.c_uint32),
                ("nparts", C.c_uint32), ("epsilon_bits", C.c_uint32), ("dtype", C.c_uint8)]

    @classmethod
    def make(cls, x, parts, rows, ld_in, eps, dtype, step=None):
        c = cls()
        c.x, c.step, c.rows, c.ld_in, c.nparts, c.epsilon_bits, c.dtype = x, NONE if step is None else step, rows, ld_in, len(parts), f32_bits(eps), dtype
        for i, p in enumerate(parts):
            c.part[i] = p
        return c


class HeadLinearCall(C.Structure):
    """Extension: every head's columns times a matrix of its own."""
    _fields_ = [("a", BufferRef), ("b", BufferRef), ("output", BufferRef)] + [(n, C.c_uint32) for n in (
        "rows", "heads", "k", "n", "lda", "a_step", "b_ld", "b_step", "ld", "out_step")] + [("dtype", C.c_uint8)]


WHOLE_CACHE = 0xFFFFFFFF     # kv_back of keys whose row 0 is position 0


class WindowAttentionCall(C.Structure):
    """Extension: sliding-window attention with a sink and an optional key part all heads share."""
    _fields_ = [(n, BufferRef) for n in ("q", "k", "v", "q2", "k2", "pos", "sink", "output")] + [(n, C.c_uint32) for n in (
        "rows", "heads", "kv_heads", "dim", "vdim", "dim2", "q_ld", "q_step", "k_ld", "v_ld", "q2_ld", "q2_step", "k2_ld", "ld",
        "kv_rows", "kv_back", "k2_rows", "window", "scale_bits")] + [("dtype", C.c_uint8)]


class RetentionCall(C.Structure):
    """Extension: linear attention with one decay per head, an f32 state, and a normed, gated output."""
    _fields_ = [(n, BufferRef) for n in ("q", "k", "v", "gate", "decay", "step", "state", "output", "work")] + [(n, C.c_uint32) for n in (
        "rows", "heads", "dim", "vdim", "vmean", "q_ld", "k_ld", "v_ld", "gate_ld", "ld", "scale_bits", "epsilon_bits")] + [("dtype", C.c_uint8)]


class MoePlanCall(C.Structure):
    """Extension: router logits -> chosen experts, weights and the row tiles of the grouped products."""
    _fields_ = [(n, BufferRef) for n in ("logits", "bias", "step", "weight", "place", "tiles", "source")] + [(n, C.c_uint32) for n in (
        "rows", "experts", "top", "ld_logits", "tile_rows", "max_tiles")]


class MoeCombineCall(C.Structure):
    """Extension: x += the weighted sum of the chosen experts' outputs."""
    _fields_ = [(n, BufferRef) for n in ("x", "y", "weight", "place", "step")] + [(n, C.c_uint32) for n in (
        "rows", "width", "top", "ld", "y_rows")] + [("dtype", C.c_uint8)]


class _Payload(C.Union):
    _fields_ = [("unary", UnaryCall), ("binary", BinaryCall), ("matmul", MatMulCall),
                ("matmul_activation", MatMulActivationCall), ("matmul_add", MatMulAddCall), ("matmul_add_activation", MatMulAddActivationCall), ("matmul_dequant", MatMulDequantCall), ("norm", NormCall),
                ("rope", RoPECall), ("gather", GatherCall), ("cast", CastCall), ("layout", LayoutCall),
                ("transpose", TransposeCall), ("softmax", SoftmaxCall), ("expand", ExpandCall), ("reduce", ReduceCall), ("attention", AttentionCall), ("dequant_activation", DequantActivationCall), ("where", WhereCall), ("broadcast_binary", BroadcastBinaryCall), ("dequantize", DequantizeCall), ("kv_cache_write", KvCacheWriteCall),
                ("decode_attention", DecodeAttentionCall),
                ("decode_attention_valid", DecodeAttentionValidCall), ("quantize_rows_i8", QuantizeRowsI8Call),
                ("decode_attention_valid_q8", DecodeAttentionValidQ8Call), ("all_reduce", AllReduceCall),
                ("rope_quantize", RopeQuantizeCall), ("rms_norm_multi", RmsNormMultiCall), ("linear", LinearCall),
                ("causal_attention", CausalAttentionCall), ("rotary_table", RotaryTableCall), ("rms_norm_parts", RmsNormPartsCall),
                ("head_linear", HeadLinearCall), ("window_attention", WindowAttentionCall), ("retention", RetentionCall),
                ("moe_plan", MoePlanCall), ("moe_combine", MoeCombineCall)]


class KernelCall(C.Structure):
    """`enum KernelCall` (kernel_call.rs:1146-1276) as tag + union."""
    _fields_ = [("kind", C.c_uint16), ("u", _Payload)]

    _FIELD = {}

    @classmethod
    def of(cls, kind, payload):
        kc = cls()
        kc.kind = kind
        setattr(kc.u, cls._FIELD[type(payload)], payload)
        return kc

    @classmethod
    def Elementwise(cls, kind, c):
        """Any of EXACT_UNARY (UnaryCall) or EXACT_BINARY (BinaryCall), by wire discriminant."""
        assert kind in EXACT_UNARY + EXACT_BINARY
        return cls.of(kind, c)

    # constructors named after the reference variants
    @classmethod
    def Sigmoid(cls, c): return cls.of(K_SIGMOID, c)
    @classmethod
    def Tanh(cls, c): return cls.of(K_TANH, c)
    @classmethod
    def Gelu(cls, c): return cls.of(K_GELU, c)
    @classmethod
    def Silu(cls, c): return cls.of(K_SILU, c)
    @classmethod
    def Exp(cls, c): return cls.of(K_EXP, c)
    @classmethod
    def Erf(cls, c): return cls.of(K_ERF, c)
    @classmethod
    def Add(cls, c): return cls.of(K_ADD, c)
    @classmethod
    def Mul(cls, c): return cls.of(K_MUL, c)
    @classmethod
    def MatMul(cls, c): return cls.of(K_MATMUL, c)
    @classmethod
    def MatMulActivation(cls, c): return cls.of(K_MATMUL_ACTIVATION, c)
    @classmethod
    def MatMulAdd(cls, c): return cls.of(K_MATMUL_ADD, c)
    @classmethod
    def MatMulAddActivation(cls, c): return cls.of(K_MATMUL_ADD_ACTIVATION, c)
    @classmethod
    def MatMulDequant(cls, c):
        # the wire form follows the call (kernel_codec.rs:525-544): a codebook takes 117, any extended field 116, else 111
        if c.codebook.slot != NO_SLOT:
            return cls.of(K_MATMUL_DEQUANT_CODEBOOK, c)
        extended = c.bq_omajor or c.act_quant or c.act or c.residual.slot != NO_SLOT
        return cls.of(K_MATMUL_DEQUANT if extended else K_MATMUL_DEQUANT_PLAIN, c)
    @classmethod
    def RmsNorm(cls, c): return cls.of(K_RMS_NORM, c)
    @classmethod
    def LayerNorm(cls, c): return cls.of(K_LAYER_NORM, c)
    @classmethod
    def AddRmsNorm(cls, c): return cls.of(K_ADD_RMS_NORM, c)
    @classmethod
    def Softmax(cls, c): return cls.of(K_SOFTMAX, c)
    @classmethod
    def Expand(cls, c): return cls.of(K_EXPAND, c)
    @classmethod
    def Attention(cls, c): return cls.of(K_ATTENTION, c)
    @classmethod
    def DequantActivation(cls, c): return cls.of(K_DEQUANT_ACTIVATION, c)
    @classmethod
    def Where(cls, c): return cls.of(K_WHERE, c)
    @classmethod
    def ReduceSum(cls, c): return cls.of(K_REDUCE_SUM, c)
    @classmethod
    def ReduceMean(cls, c): return cls.of(K_REDUCE_MEAN, c)
    @classmethod
    def ReduceProd(cls, c): return cls.of(K_REDUCE_PROD, c)
    @classmethod
    def ReduceMin(cls, c): return cls.of(K_REDUCE_MIN, c)
    @classmethod
    def ReduceMax(cls, c): return cls.of(K_REDUCE_MAX, c)
    @classmethod
    def BroadcastBinary(cls, c): return cls.of(K_BROADCAST_BINARY, c)
    @classmethod
    def Transpose(cls, c): return cls.of(K_TRANSPOSE, c)
    @classmethod
    def Concat(cls, c): return cls.of(K_CONCAT, c)
    @classmethod
    def Slice(cls, c): return cls.of(K_SLICE, c)
    @classmethod
    def RotaryEmbedding(cls, c): return cls.of(K_ROTARY, c)
    @classmethod
    def Gather(cls, c): return cls.of(K_GATHER, c)
    @classmethod
    def Cast(cls, c): return cls.of(K_CAST, c)
    @classmethod
    def Reshape(cls, c): return cls.of(K_RESHAPE, c)
    @classmethod
    def Dequantize(cls, c): return cls.of(K_DEQUANTIZE, c)
    @classmethod
    def KvCacheWrite(cls, c): return cls.of(K_KV_CACHE_WRITE, c)
    @classmethod
    def DecodeAttention(cls, c): return cls.of(K_DECODE_ATTENTION, c)
    @classmethod
    def DecodeAttentionValid(cls, c): return cls.of(K_DECODE_ATTENTION_VALID, c)
    @classmethod
    def QuantizeRowsI8(cls, c): return cls.of(K_QUANTIZE_ROWS_I8, c)
    @classmethod
    def DecodeAttentionValidQ8(cls, c): return cls.of(K_DECODE_ATTENTION_VALID_Q8, c)
    @classmethod
    def AllReduce(cls, c): return cls.of(K_ALL_REDUCE, c)
    @classmethod
    def RopeQuantizeRowsI8(cls, c): return cls.of(K_ROPE_QUANTIZE_ROWS_I8, c)
    @classmethod
    def RmsNormMulti(cls, c): return cls.of(K_RMS_NORM_MULTI, c)
    @classmethod
    def Linear(cls, c): return cls.of(K_LINEAR_EX if c.extended else K_LINEAR, c)    # the wire form follows the call
    @classmethod
    def CausalAttention(cls, c): return cls.of(K_CAUSAL_ATTENTION, c)
    @classmethod
    def RotaryTable(cls, c): return cls.of(K_ROTARY_TABLE, c)
    @classmethod
    def RmsNormParts(cls, c): return cls.of(K_RMS_NORM_PARTS, c)
    @classmethod
    def HeadLinear(cls, c): return cls.of(K_HEAD_LINEAR, c)
    @classmethod
    def WindowAttention(cls, c): return cls.of(K_WINDOW_ATTENTION, c)
    @classmethod
    def Retention(cls, c): return cls.of(K_RETENTION, c)
    @classmethod
    def MoePlan(cls, c): return cls.of(K_MOE_PLAN, c)
    @classmethod
    def MoeCombine(cls, c): return cls.of(K_MOE_COMBINE, c)


KernelCall._FIELD = {
    UnaryCall: "unary", BinaryCall: "binary", MatMulCall: "matmul", MatMulActivationCall: "matmul_activation",
    MatMulAddCall: "matmul_add", MatMulAddActivationCall: "matmul_add_activation", MatMulDequantCall: "matmul_dequant", NormCall: "norm", RoPECall: "rope", GatherCall: "gather", CastCall: "cast",
    LayoutCall: "layout", TransposeCall: "transpose", SoftmaxCall: "softmax", ExpandCall: "expand", ReduceCall: "reduce", AttentionCall: "attention", DequantActivationCall: "dequant_activation", WhereCall: "where", BroadcastBinaryCall: "broadcast_binary", DequantizeCall: "dequantize", KvCacheWriteCall: "kv_cache_write",
    DecodeAttentionCall: "decode_attention", DecodeAttentionValidCall: "decode_attention_valid", QuantizeRowsI8Call: "quantize_rows_i8",
    DecodeAttentionValidQ8Call: "decode_attention_valid_q8", AllReduceCall: "all_reduce", RopeQuantizeCall: "rope_quantize",
    RmsNormMultiCall: "rms_norm_multi", LinearCall: "linear", CausalAttentionCall: "causal_attention",
    RotaryTableCall: "rotary_table", RmsNormPartsCall: "rms_norm_parts", HeadLinearCall: "head_linear", WindowAttentionCall: "window_attention",
    RetentionCall: "retention", MoePlanCall: "moe_plan", MoeCombineCall: "moe_combine",
}


class HostSlot(C.Structure):
    _fields_ = [("ptr", C.c_void_p), ("bytes", C.c_uint64)]


def lut_call(act, c):
    """KernelCall for LUT activation id `act` over UnaryCall `c`."""
    return KernelCall.of(LUT_KIND[act], c)
