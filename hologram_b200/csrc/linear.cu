// Products and norms of decoder steps whose residual stream is f32 (the Linear and RmsNormMulti calls).
//
// Linear: out_s = residual + alpha * act_s(A[:, k_offset_s ..] . B[:, columns of s]) for up to four column segments of
// one B, stored as f32 or as bf16 rounded to nearest, with a row pitch and an optional device-side row offset per
// segment. bf16 operands run on the tensor-core kernels of gemm_kernels.cuh (LIN instantiations: same tiles, rings and
// K splits as the matmul, other epilogue). f32 operands and shapes TMA cannot take run one thread per cell with an
// ascending-k fused multiply-add chain in f32 (no reduced-precision mode anywhere).
#include "gemm_kernels.cuh"

namespace {

constexpr int CELL_ROWS = 4, CELL_THREADS = 128;

// One thread: one column, up to CELL_ROWS rows (B is read once for them).
template <typename T>
__global__ void __launch_bounds__(CELL_THREADS)
linear_cell_kernel(const T* __restrict__ a, const T* __restrict__ b, const GemmParams p, uint32_t lda) {
    holo_pdl_trigger();
    holo_pdl_wait();
    const uint32_t col = blockIdx.x * CELL_THREADS + threadIdx.x, row0 = blockIdx.y * CELL_ROWS;
    if (col >= p.n) return;
    const GemmLin& g = p.lin[lin_segment(p, col)];
    const uint32_t c = col - g.col_begin;
    if (c >= g.width) return;
    float acc[CELL_ROWS] = {};
    const uint32_t rows = min((uint32_t)CELL_ROWS, p.m - row0);
    for (uint32_t kk = 0; kk < p.k; ++kk) {
        const float bv = (float)b[(uint64_t)kk * p.n + col];
#pragma unroll
        for (int r = 0; r < CELL_ROWS; ++r)
            if ((uint32_t)r < rows) acc[r] = __fmaf_rn((float)a[(uint64_t)(row0 + r) * lda + g.k_offset + kk], bv, acc[r]);
    }
    const uint64_t base = g.row_pos ? *g.row_pos : 0u;
#pragma unroll
    for (int r = 0; r < CELL_ROWS; ++r) {
        const uint64_t orow = base + row0 + r;
        if ((uint32_t)r >= rows || orow >= g.row_limit) continue;
        const uint64_t idx = orow * g.ld + c;
        const float v = p.alpha * lin_act(acc[r], g.act);
        if (g.f32) reinterpret_cast<float*>(g.out)[idx] = v + (g.residual ? g.residual[idx] : 0.0f);
        else reinterpret_cast<__nv_bfloat16*>(g.out)[idx] = __float2bfloat16_rn(v);
    }
}

__device__ __forceinline__ void store_norm(float* out, uint64_t i, float v) { out[i] = v; }
__device__ __forceinline__ void store_norm(__nv_bfloat16* out, uint64_t i, float v) { out[i] = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store_norm4(float* out, uint64_t i, float4 v) { *reinterpret_cast<float4*>(out + i) = v; }
__device__ __forceinline__ void store_norm4(__nv_bfloat16* out, uint64_t i, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(out + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// One CTA per row. VEC: feature and step are multiples of 4 and the row fits NORM_VECS float4 per thread, held in
// registers between the reduction and the scaling; the scalar form re-reads the row.
constexpr int NORM_VECS = 4, NORM_THREADS = 1024;
template <typename T, bool VEC>
__global__ void __launch_bounds__(NORM_THREADS)
rms_norm_multi_kernel(const float* __restrict__ x, const float* __restrict__ gamma0, const float* __restrict__ gamma1, T* __restrict__ out,
                      uint32_t feature, uint32_t step, float eps) {
    holo_pdl_trigger();
    __shared__ float s_part[32];
    const uint32_t tid = threadIdx.x, nt = blockDim.x;
    const uint32_t nvec = feature >> 2;
    holo_pdl_wait();
    const float* row = x + (uint64_t)blockIdx.x * feature;
    float4 v[NORM_VECS];
    float acc = 0.0f;
    if (VEC) {
#pragma unroll
        for (int i = 0; i < NORM_VECS; ++i) {
            const uint32_t j = tid + i * nt;
            v[i] = j < nvec ? reinterpret_cast<const float4*>(row)[j] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < NORM_VECS; ++i) acc = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, acc))));
    } else {
        for (uint32_t j = tid; j < feature; j += nt) acc = fmaf(row[j], row[j], acc);
    }
    for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if ((tid & 31) == 0) s_part[tid >> 5] = acc;
    __syncthreads();
    float t = (tid & 31) < (nt >> 5) ? s_part[tid & 31] : 0.0f;
    for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
    const float inv = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(t, (float)feature), eps)));
    const uint32_t nout = gamma1 ? 2 : 1;
    const uint64_t base = (uint64_t)blockIdx.x * step * nout;
    for (uint32_t w = 0; w < nout; ++w) {
        const float* gm = w ? gamma1 : gamma0;
        const uint64_t off = base + (uint64_t)w * step;
        if (VEC) {
#pragma unroll
            for (int i = 0; i < NORM_VECS; ++i) {
                const uint32_t j = tid + i * nt;
                if (j < nvec) {
                    const float4 g = reinterpret_cast<const float4*>(gm)[j];
                    store_norm4(out, off + 4 * j, make_float4(v[i].x * inv * g.x, v[i].y * inv * g.y, v[i].z * inv * g.z, v[i].w * inv * g.w));
                }
            }
        } else {
            for (uint32_t j = tid; j < feature; j += nt) store_norm(out, off + j, row[j] * inv * gm[j]);
        }
        for (uint32_t j = feature + tid; j < step; j += nt) store_norm(out, off + j, 0.0f);
    }
}

template <typename T>
int32_t launch_norm(holo_b200_ctx* ctx, const float* x, const float* g0, const float* g1, T* out, uint32_t rows, uint32_t feature, uint32_t step, float eps) {
    const bool vec = feature % 4 == 0 && step % 4 == 0 && feature <= 4u * NORM_VECS * NORM_THREADS &&
                     (((uintptr_t)x | (uintptr_t)g0 | (uintptr_t)g1 | (uintptr_t)out) & 15u) == 0;
    // one float4 per thread where that gives whole warps; many rows keep smaller CTAs so that several share an SM
    uint32_t threads = ((feature / 4 + 31) / 32) * 32;
    if (rows > 64 && threads > 256 && feature <= 4u * NORM_VECS * 256) threads = 256;
    threads = threads < 32 ? 32 : threads > (uint32_t)NORM_THREADS ? (uint32_t)NORM_THREADS : threads;
    if (vec) HOLO_CUDA(holo_launch_kernel(ctx, rms_norm_multi_kernel<T, true>, dim3(rows), dim3(threads), 0, 1, x, g0, g1, out, feature, step, eps));
    else HOLO_CUDA(holo_launch_kernel(ctx, rms_norm_multi_kernel<T, false>, dim3(rows), dim3(256), 0, 1, x, g0, g1, out, feature, step, eps));
    ctx->launches++;
    return HOLO_OK;
}

template <int BN, int STAGES, int A_ROWS>
int32_t launch_lin(holo_b200_ctx* ctx, const CUtensorMap& ma, const CUtensorMap& mb, const GemmParams& p, dim3 grid) {
    return launch_umma_ar<BN, STAGES, A_ROWS, false, false, true>(ctx, ma, mb, p, grid);
}

}  // namespace

int32_t holo_launch_rms_norm_multi(holo_b200_ctx* ctx, const float* x, const float* gamma0, const float* gamma1, void* out, uint32_t rows,
                                   uint32_t feature, uint32_t step, float eps, uint8_t dtype) {
    if (dtype == HOLO_DTYPE_F32) return launch_norm(ctx, x, gamma0, gamma1, (float*)out, rows, feature, step, eps);
    return launch_norm(ctx, x, gamma0, gamma1, (__nv_bfloat16*)out, rows, feature, step, eps);
}

int32_t holo_launch_linear(holo_b200_ctx* ctx, const HoloLinearArgs& a) {
    GemmParams p;
    memset(&p, 0, sizeof p);
    p.m = a.m; p.n = a.n; p.k = a.k;
    p.nlin = a.nseg;
    p.alpha = a.alpha;
    p.status = ctx->dev_status;
    p.dtype = a.dtype;
    bool k_offsets_ok = true;   // a TMA load starts on a 16-byte boundary
    for (uint32_t i = 0; i < a.nseg; ++i) {
        const HoloLinearSegArgs& s = a.seg[i];
        GemmLin& g = p.lin[i];
        g.out = s.out;
        g.residual = a.residual;
        g.row_pos = s.row_pos;
        g.row_limit = s.row_limit;
        g.col_begin = s.col_begin; g.width = s.width; g.k_offset = s.k_offset; g.ld = s.ld;
        g.act = s.act;
        g.f32 = s.dtype == HOLO_DTYPE_F32;
        k_offsets_ok = k_offsets_ok && s.k_offset % 8 == 0;
    }
    const bool tma_ok = a.dtype == HOLO_DTYPE_BF16 && a.lda % 8 == 0 && a.n % 8 == 0 && k_offsets_ok && (((uintptr_t)a.a | (uintptr_t)a.b) & 15u) == 0 &&
                        encode_tiled_fn() != nullptr && !getenv("HOLO_GEMM_FORCE_CELL");
    if (!tma_ok) {
        const uint32_t rows = (a.m + CELL_ROWS - 1) / CELL_ROWS;
        if (rows > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: linear m %u on the per-cell path", a.m);
        const dim3 grid((a.n + CELL_THREADS - 1) / CELL_THREADS, rows);
        if (a.dtype == HOLO_DTYPE_F32)
            HOLO_CUDA(holo_launch_kernel(ctx, linear_cell_kernel<float>, grid, dim3(CELL_THREADS), 0, 1, (const float*)a.a, (const float*)a.b, p, a.lda));
        else
            HOLO_CUDA(holo_launch_kernel(ctx, linear_cell_kernel<__nv_bfloat16>, grid, dim3(CELL_THREADS), 0, 1, (const __nv_bfloat16*)a.a, (const __nv_bfloat16*)a.b, p, a.lda));
        ctx->launches++;
        return HOLO_OK;
    }
    const uint32_t kblocks = (a.k + BK - 1) / BK, mtiles = (a.m + BM - 1) / BM;
    p.kblocks = kblocks;
    p.splits = 1;
    p.b_constant = a.b_constant && !getenv("HOLO_GEMM_NO_EARLY_B") ? 1u : 0u;
    CUtensorMap ma, mb;
    HOLO_TRY(make_map_2d(&mb, a.b, a.n, a.k, 64, BK));
    bool persistent, paired;
    persistent_choice(ctx, a.m, a.n, &persistent, &paired);
    if (persistent) {
        p.box_m = BM;
        HOLO_TRY(make_map_2d(&ma, a.a, a.lda, a.m, BK, BM));
        return paired ? launch_pair<false, true>(ctx, ma, mb, p) : launch_persistent<false, true>(ctx, ma, mb, p);
    }
    int bn;
    uint32_t splits;
    tile_choice(ctx, a.m, a.n, kblocks, &bn, &splits);
    if (const char* e = getenv("HOLO_GEMM_BN")) bn = atoi(e) == 64 ? 64 : 128;
    if (const char* e = getenv("HOLO_GEMM_SPLITS")) splits = (uint32_t)atoi(e) > 0 ? (uint32_t)atoi(e) : 1;
    if (splits > kblocks) splits = kblocks;
    if (splits > 8) splits = 8;
    if (mtiles > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: matmul grid too large");
    p.splits = splits;
    p.box_m = a.m < (uint32_t)BM ? a.m : (uint32_t)BM;
    HOLO_TRY(make_map_2d(&ma, a.a, a.lda, a.m, BK, p.box_m));
    const dim3 grid((a.n + bn - 1) / bn, mtiles, splits);
    if (bn == 128) {
        if (a.m <= 16) return launch_lin<128, 5, 16>(ctx, ma, mb, p, grid);
        if (a.m <= 64) return launch_lin<128, 4, 64>(ctx, ma, mb, p, grid);
        return launch_lin<128, 3, 128>(ctx, ma, mb, p, grid);
    }
    if (a.m <= 16) return launch_lin<64, 9, 16>(ctx, ma, mb, p, grid);
    if (a.m <= 64) return launch_lin<64, 6, 64>(ctx, ma, mb, p, grid);
    return launch_lin<64, 4, 128>(ctx, ma, mb, p, grid);
}
