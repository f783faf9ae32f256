// bf16 / f16 matmul with the reference's epilogues: the per-cell kernel and the launchers. The tensor-core kernels
// are in gemm_kernels.cuh.
#include "gemm_kernels.cuh"

namespace {

// Shapes the tensor-core path cannot take (row pitches that are not 16-byte multiples,
// unaligned bases), tiny problems and every f32 product: one thread per output cell running the
// reference's own per-cell recurrence, an ascending-k fused multiply-add chain (mul-then-add in
// the n % 8 column tail, cpu/simd.rs:746-799) -- bit-identical to the CPU kernel. For f32 the
// fused activation is the scalar function itself (no table exists for 32-bit patterns).
// `add_first` (MatMulAddActivation, cpu/float_kernels.rs:899-938): the residual is added before the activation and
// nothing is narrowed between the two; for 16-bit dtypes the product itself is narrowed once, as the matmul stores it.
__global__ void matmul_cell_kernel(const void* __restrict__ a, const void* __restrict__ b, void* __restrict__ out,
                                   const uint16_t* __restrict__ table, int act, const void* __restrict__ residual, uint32_t m,
                                   uint32_t k, uint32_t n, int dtype, int add_first) {
    holo_pdl_trigger();
    holo_pdl_wait();
    const uint32_t j = blockIdx.x * blockDim.x + threadIdx.x, i = blockIdx.y;
    if (j >= n || i >= m) return;
    const bool fused = j < n - (n % 8);
    float acc = 0.0f;
    for (uint32_t kk = 0; kk < k; ++kk) {
        float av = holo::load_float(a, (uint64_t)i * k + kk, dtype), bv = holo::load_float(b, (uint64_t)kk * n + j, dtype);
        acc = fused ? __fmaf_rn(av, bv, acc) : __fadd_rn(acc, __fmul_rn(av, bv));
    }
    const uint64_t idx = (uint64_t)i * n + j;
    if (add_first) {
        if (dtype == HOLO_DTYPE_F32) {
            acc = __fadd_rn(acc, reinterpret_cast<const float*>(residual)[idx]);
            reinterpret_cast<float*>(out)[idx] = holo::lut_act_ref(act, acc);
        } else {
            const float v = __fadd_rn(holo::widen16(holo::narrow16(acc, dtype), dtype), holo::widen16(reinterpret_cast<const uint16_t*>(residual)[idx], dtype));
            reinterpret_cast<uint16_t*>(out)[idx] = holo::narrow16(holo::lut_act_ref(act, v), dtype);
        }
        return;
    }
    if (dtype == HOLO_DTYPE_F32) {
        if (act >= 0) acc = holo::lut_act_ref(act, acc);
        if (residual) acc = __fadd_rn(acc, reinterpret_cast<const float*>(residual)[idx]);
        reinterpret_cast<float*>(out)[idx] = acc;
    } else {
        const uint16_t* res16 = reinterpret_cast<const uint16_t*>(residual);
        reinterpret_cast<uint16_t*>(out)[idx] = dtype == HOLO_DTYPE_F16 ? epilogue_elem<true>(acc, table, res16, idx) : epilogue_elem<false>(acc, table, res16, idx);
    }
}

}  // namespace

static int lut_id_of_fused(uint8_t fused_act) {
    return fused_act == HOLO_FUSED_GELU ? HOLO_LUT_GELU : fused_act == HOLO_FUSED_SILU ? HOLO_LUT_SILU
         : fused_act == HOLO_FUSED_SIGMOID ? HOLO_LUT_SIGMOID : fused_act == HOLO_FUSED_TANH ? HOLO_LUT_TANH : HOLO_LUT_EXP;
}

static int32_t act_table(holo_b200_ctx* ctx, uint8_t fused_act, uint8_t dtype, const uint16_t** table) {
    *table = nullptr;
    if (fused_act) {
        int act = fused_act == HOLO_FUSED_GELU ? HOLO_LUT_GELU : fused_act == HOLO_FUSED_SILU ? HOLO_LUT_SILU
                : fused_act == HOLO_FUSED_SIGMOID ? HOLO_LUT_SIGMOID : fused_act == HOLO_FUSED_TANH ? HOLO_LUT_TANH : HOLO_LUT_EXP;
        HOLO_TRY(holo_lut_table(ctx, (uint8_t)act, dtype, table));
    }
    return HOLO_OK;
}

int32_t holo_launch_matmul(holo_b200_ctx* ctx, const void* a, const void* b, void* out, uint32_t m, uint32_t k, uint32_t n,
                           uint8_t dtype, uint8_t fused_act, const void* residual, bool b_constant) {
    HoloMatmulSeg sg = {out, residual, n, fused_act};
    sg.b_constant = b_constant ? 1 : 0;
    return holo_launch_matmul_multi(ctx, a, b, m, k, n, dtype, &sg, 1);
}

int32_t holo_launch_matmul_add_activation(holo_b200_ctx* ctx, const void* a, const void* b, void* out, uint32_t m, uint32_t k, uint32_t n,
                                          uint8_t dtype, uint8_t fused_act, const void* residual) {
    if (m > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: matmul m %u on the per-cell path", m);
    HOLO_CUDA(holo_launch_kernel(ctx, matmul_cell_kernel, dim3((n + 127) / 128, m), dim3(128), 0, 1, a, b, out, (const uint16_t*)nullptr,
                                 lut_id_of_fused(fused_act), residual, m, k, n, (int)dtype, 1));
    ctx->launches++;
    return HOLO_OK;
}

// C[:, segment i] = epilogue_i(A . B[:, segment i]) for 1..3 column segments of one [k, n] B.
// Whether the segments' head_op requests can ride this product: the tensor-core path with one row tile, K
// split at least two ways inside a cluster, every segment a whole number of 128-column heads, no gate, no
// tensor-parallel sum. The session asks before it folds a RotaryEmbedding / QuantizeRowsI8 into a product.
bool holo_matmul_head_ops_ok(uint32_t m, uint32_t k, uint32_t n, uint8_t dtype, const HoloMatmulSeg* segs, uint32_t nseg) {
    if (dtype != HOLO_DTYPE_BF16 && dtype != HOLO_DTYPE_F16) return false;
    if (m == 0 || m > (uint32_t)BM || k < 2 * BK || (k % 8) != 0 || (n % 128) != 0 || nseg < 1 || nseg > MAX_SEGS) return false;
    if ((uint64_t)m * n * k < (1ull << 18) || encode_tiled_fn() == nullptr) return false;
    // the compute-bound kernels have no head epilogue (they need two row tiles, excluded above)
    for (uint32_t i = 0; i < nseg; ++i) {
        if ((segs[i].width % 128) != 0 || segs[i].gated || segs[i].all_reduce) return false;
        if (segs[i].head_op > 3) return false;
        if (segs[i].head_op == 1 || segs[i].head_op == 2)
            if (!segs[i].cos || !segs[i].sin || !segs[i].rope_out || (((uintptr_t)segs[i].cos | (uintptr_t)segs[i].sin | (uintptr_t)segs[i].rope_out) & 7u)) return false;
        if (segs[i].head_op >= 2)
            if (!segs[i].codes || !segs[i].scales || ((uintptr_t)segs[i].codes & 3u) || ((uintptr_t)segs[i].scales & 3u)) return false;
        if (segs[i].head_op && ((uintptr_t)segs[i].out & 7u)) return false;
    }
    return true;
}

int32_t holo_launch_matmul_multi(holo_b200_ctx* ctx, const void* a, const void* b, uint32_t m, uint32_t k, uint32_t n,
                                 uint8_t dtype, const HoloMatmulSeg* segs, uint32_t nseg) {
    if (nseg < 1 || nseg > MAX_SEGS) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: matmul segment count %u", nseg);
    GemmSeg gs[MAX_SEGS] = {};
    uint32_t col = 0;
    bool head_ops = false;
    for (uint32_t i = 0; i < nseg; ++i) {
        if (dtype != HOLO_DTYPE_F32) HOLO_TRY(act_table(ctx, segs[i].fused_act, dtype, &gs[i].table));
        gs[i].out = (uint16_t*)segs[i].out;
        gs[i].residual = (const uint16_t*)segs[i].residual;
        gs[i].col_begin = col;
        col += segs[i].width;
        gs[i].col_end = col;
        if (i + 1 < nseg && (col % 32) != 0) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: matmul segment boundary %u is not a multiple of 32", col);
        gs[i].head_op = segs[i].head_op;
        gs[i].cos = (const uint16_t*)segs[i].cos;
        gs[i].sin = (const uint16_t*)segs[i].sin;
        gs[i].rope_out = (uint16_t*)segs[i].rope_out;
        gs[i].codes = segs[i].codes;
        gs[i].scales = segs[i].scales;
        head_ops |= segs[i].head_op != 0;
    }
    if (head_ops && !holo_matmul_head_ops_ok(m, k, n, dtype, segs, nseg))
        return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: matmul head epilogue needs m <= 128, k >= 128 and 128-column segments");
    const bool gated = segs[0].gated != 0;
    if (gated) {
        if (nseg != 1 || (segs[0].width % 64) != 0 || dtype == HOLO_DTYPE_F32)
            return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: gated matmul takes one 16-bit segment whose width is a multiple of 64");
        col *= 2;
        gs[0].col_end = col;
    }
    if (col != n) return holo_fail(HOLO_ERR_SHAPE_MISMATCH, "shape mismatch: matmul segments cover %u of %u columns", col, n);
    const uint16_t* table = gs[0].table;
    const void* residual = gs[0].residual;
    void* out = gs[0].out;
    const bool tma_ok = dtype != HOLO_DTYPE_F32 && (k % 8) == 0 && (n % 8) == 0 && (((uintptr_t)a | (uintptr_t)b) & 15u) == 0 && encode_tiled_fn() != nullptr;
    const bool tiny = (uint64_t)m * n * k < (1ull << 18);
    if ((nseg > 1 || gated) && (!tma_ok || tiny))
        return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: merged matmul needs the tensor-core path");
    const bool cell_path = !tma_ok || tiny || getenv("HOLO_GEMM_FORCE_CELL");
    if (cell_path && segs[0].all_reduce && ctx->tp_world > 1) {
        // the per-cell kernel has no exchange of its own: product first, then the all-reduce launch
        HoloMatmulSeg plain = segs[0];
        plain.all_reduce = 0;
        plain.residual = nullptr;
        HOLO_TRY(holo_launch_matmul_multi(ctx, a, b, m, k, n, dtype, &plain, 1));
        return holo_all_reduce_add(ctx, segs[0].out, segs[0].residual, segs[0].out, (uint64_t)m * n, dtype);
    }
    if (cell_path) {
        dim3 grid((n + 127) / 128, m);
        if (m > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: matmul m %u on the per-cell path", m);
        HOLO_CUDA(holo_launch_kernel(ctx, matmul_cell_kernel, dim3(grid), dim3(128), 0, 1, a, b, out, table,
                                     segs[0].fused_act ? lut_id_of_fused(segs[0].fused_act) : -1, residual, m, k, n, (int)dtype, 0));
        HOLO_CUDA(cudaGetLastError());
        ctx->launches++;
        return HOLO_OK;
    }
    const uint32_t kblocks = (k + BK - 1) / BK, mtiles = (m + BM - 1) / BM;
    // Compute-bound shapes (at least one 128 x 256 tile per SM): the persistent kernel.
    {
        bool persistent, paired;
        persistent_choice(ctx, m, n, &persistent, &paired);
        if (gated || (segs[0].all_reduce && ctx->tp_world > 1)) persistent = paired = false;
        if (persistent) {
            GemmParams p;
            memset(&p, 0, sizeof p);
            for (uint32_t i = 0; i < MAX_SEGS; ++i) p.seg[i] = gs[i];
            p.nseg = nseg;
            p.status = ctx->dev_status;
            p.m = m; p.n = n; p.k = k; p.kblocks = kblocks; p.splits = 1;
            p.box_m = BM;
            p.dtype = dtype;
            CUtensorMap ma, mb;
            HOLO_TRY(make_map_2d(&ma, a, k, m, BK, BM));
            HOLO_TRY(make_map_2d(&mb, b, n, k, 64, BK));
            if (dtype == HOLO_DTYPE_F16) return paired ? launch_pair<true, false>(ctx, ma, mb, p) : launch_persistent<true, false>(ctx, ma, mb, p);
            return paired ? launch_pair<false, false>(ctx, ma, mb, p) : launch_persistent<false, false>(ctx, ma, mb, p);
        }
    }
    int bn;
    uint32_t splits;
    tile_choice(ctx, m, n, kblocks, &bn, &splits);
    const uint32_t tiles128 = mtiles * ((n + 127) / 128);
    if (const char* e = getenv("HOLO_GEMM_BN")) bn = atoi(e) == 64 ? 64 : atoi(e) == 256 ? 256 : 128;
    if (gated && bn != 128) {   // the gate / up pairing is per 128-wide tile
        bn = 128;
        splits = tiles128 >= 148 ? 1 : (192 + tiles128 - 1) / tiles128;
        if (splits > 8) splits = 8;
        if (splits > kblocks / 8) splits = kblocks / 8 ? kblocks / 8 : 1;
    }
    if (const char* e = getenv("HOLO_GEMM_SPLITS")) splits = (uint32_t)atoi(e) > 0 ? (uint32_t)atoi(e) : 1;
    if (head_ops) {
        // the per-head epilogue lives in the cluster reduction of 128-wide tiles (one head per tile)
        if (bn != 128) {
            bn = 128;
            splits = (240 + tiles128 - 1) / tiles128;
            if (splits > kblocks / 8) splits = kblocks / 8 ? kblocks / 8 : 1;
        }
        if (splits < 2) splits = 2;
    }
    if (splits > kblocks) splits = kblocks;
    if (splits > 8) splits = 8;  // one cluster (portable size) per output tile
    if (mtiles > 65535 || splits > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: matmul grid too large");

    // Tensor-parallel sum in the epilogue: needs the peer-memory transport, a single plain 16-bit
    // segment, a message that fits the one-shot mailbox regions, and every CTA of the launch resident
    // at once (a CTA waits for the same tile's CTAs on the other GPUs; with more CTAs than fit, a
    // waiting first wave here could face a second wave there). Otherwise the matmul stores its
    // narrowed partial and the all-reduce kernel follows.
    const bool want_ar = segs[0].all_reduce != 0 && ctx->tp_world > 1;
    // Opt-in (HOLO_TP_FUSED_GEMM; two ranks, or any group size with HOLO_TP_FUSED_GEMM_ANY_WORLD): measured on two
    // GPUs the product followed by the all-reduce kernel is faster (1.376 against 1.456 ms per decoder step), because
    // the fused launch must trim its K split to keep every CTA resident and its tiles wait on the peer's tiles.
    bool fused_ar = want_ar && ctx->tp_p2p && nseg == 1 && !gated && !segs[0].fused_act && (n % 4) == 0 &&
                    4ull * (uint64_t)ctx->tp_world * m * n <= P2P_ONESHOT_BYTES &&
                    ((ctx->tp_world == 2 && getenv("HOLO_TP_FUSED_GEMM")) || getenv("HOLO_TP_FUSED_GEMM_ANY_WORLD"));
    if (fused_ar) {
        // one CTA per SM is always resident, clusters included: trim the K split to stay within that
        const uint32_t tiles = ((n + bn - 1) / bn) * mtiles;
        if (tiles > (uint32_t)ctx->sm_count) fused_ar = false;
        else if (tiles * splits > (uint32_t)ctx->sm_count) splits = (uint32_t)ctx->sm_count / tiles;
    }
    if (want_ar && !fused_ar) {
        HoloMatmulSeg plain = segs[0];
        plain.all_reduce = 0;
        plain.residual = nullptr;
        HOLO_TRY(holo_launch_matmul_multi(ctx, a, b, m, k, n, dtype, &plain, 1));
        return holo_all_reduce_add(ctx, segs[0].out, segs[0].residual, segs[0].out, (uint64_t)m * n, dtype);
    }
    GemmParams p;
    p.ar_world = 0;
    p.ar_rank = 0;
    p.ar_state = nullptr;
    for (int r = 0; r < 8; ++r) p.ar_mailbox[r] = nullptr;
    if (fused_ar) {
        p.ar_world = (uint32_t)ctx->tp_world;
        p.ar_rank = (uint32_t)ctx->tp_rank;
        p.ar_state = ctx->tp_epochs;
        for (int r = 0; r < 8; ++r) p.ar_mailbox[r] = ctx->tp_mailbox[r];
    }
    for (uint32_t i = 0; i < MAX_SEGS; ++i) p.seg[i] = gs[i];
    p.nseg = nseg;
    p.status = ctx->dev_status;
    p.m = m; p.n = n; p.k = k; p.kblocks = kblocks; p.splits = splits;
    p.box_m = m < (uint32_t)BM ? m : (uint32_t)BM;
    p.dtype = dtype;
    p.gated = gated ? 1u : 0u;
    p.head_ops = head_ops ? 1u : 0u;
    p.b_constant = segs[0].b_constant && !getenv("HOLO_GEMM_NO_EARLY_B") ? 1u : 0u;
    CUtensorMap ma, mb;
    HOLO_TRY(make_map_2d(&ma, a, k, m, BK, p.box_m));
    HOLO_TRY(make_map_2d(&mb, b, n, k, 64, BK));
    dim3 grid((n + bn - 1) / bn, mtiles, splits);
    if (bn == 256) {
        if (m <= 16) HOLO_TRY((launch_umma<256, 6, 16>(ctx, ma, mb, p, grid)));
        else if (m <= 64) HOLO_TRY((launch_umma<256, 5, 64>(ctx, ma, mb, p, grid)));
        else HOLO_TRY((launch_umma<256, 4, 128>(ctx, ma, mb, p, grid)));
    } else if (bn == 128) {
        if (m <= 16) HOLO_TRY((launch_umma<128, 5, 16>(ctx, ma, mb, p, grid)));
        else if (m <= 64) HOLO_TRY((launch_umma<128, 4, 64>(ctx, ma, mb, p, grid)));
        else HOLO_TRY((launch_umma<128, 3, 128>(ctx, ma, mb, p, grid)));
    } else {
        if (m <= 16) HOLO_TRY((launch_umma<64, 9, 16>(ctx, ma, mb, p, grid)));
        else if (m <= 64) HOLO_TRY((launch_umma<64, 6, 64>(ctx, ma, mb, p, grid)));
        else HOLO_TRY((launch_umma<64, 4, 128>(ctx, ma, mb, p, grid)));
    }
    return HOLO_OK;
}
