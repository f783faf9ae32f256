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

// One thread: one column, up to CELL_ROWS rows (B is read once for them). Column pairs (rotation, gate) lie in neighbouring lanes.
template <typename T>
__global__ void __launch_bounds__(CELL_THREADS)
linear_cell_kernel(const T* __restrict__ a, const T* __restrict__ b, const GemmParams p, uint32_t lda) {
    holo_pdl_trigger();
    holo_pdl_wait();
    const uint32_t col = blockIdx.x * CELL_THREADS + threadIdx.x, row0 = blockIdx.y * CELL_ROWS;
    const GemmLin& g = p.lin[lin_segment(p, col)];
    const uint32_t c = col - g.col_begin;
    const bool valid = col < p.n && c < g.width;
    uint32_t rows = min((uint32_t)CELL_ROWS, p.m - row0);
    const T* arow[CELL_ROWS];
    if (p.tiles) {
        const uint32_t tile = row0 / p.tile_rows, in_tile = row0 % p.tile_rows;
        if (tile >= (uint32_t)p.tiles[0]) return;
        b += (uint64_t)p.tiles[1 + tile] * p.k * p.n;
        if (p.a_shared) {
            if (in_tile >= p.a_shared) return;
            rows = min(rows, p.a_shared - in_tile);
        }
    }
#pragma unroll
    for (int r = 0; r < CELL_ROWS; ++r) {
        uint32_t ar = row0 + min((uint32_t)r, rows - 1);
        if (p.tiles && p.a_shared) ar %= p.tile_rows;
        else if (p.a_pos) ar = lin_a_row(p, lin_a_start(p), ar);
        arow[r] = a + (uint64_t)ar * lda + g.k_offset;
    }
    float acc[CELL_ROWS] = {};
    if (valid)
        for (uint32_t kk = 0; kk < p.k; ++kk) {
            const float bv = (float)b[(uint64_t)kk * p.n + col];
#pragma unroll
            for (int r = 0; r < CELL_ROWS; ++r) acc[r] = __fmaf_rn((float)arow[r][kk], bv, acc[r]);
        }
#pragma unroll
    for (int r = 0; r < CELL_ROWS; ++r) {
        const float v0 = lin_act<false>(acc[r], g.act == HOLO_LINEAR_ACT_SILU_GATE ? HOLO_LINEAR_ACT_NONE : g.act);
        const float v1 = __shfl_xor_sync(0xffffffffu, v0, 1);
        uint64_t orow;
        if (!valid || (uint32_t)r >= rows || !lin_out_row(g, row0 + r, &orow)) continue;
        float v = v0;
        uint32_t oc = c;
        if (g.act == HOLO_LINEAR_ACT_SILU_GATE) {
            if (c & 1u) continue;
            v = sigmoid_times<false>(v0, v0) * v1;
            oc = c >> 1;
        } else if (g.rot_head) {
            const uint32_t cc = c % g.rot_head;
            if (cc >= g.rot_begin && cc < g.rot_begin + g.rot_dims) {
                const float2 t = p.rot[(uint64_t)(row0 + r) * (g.rot_dims >> 1) + ((cc - g.rot_begin) >> 1)];
                v = (c & 1u) ? v0 * t.x + v1 * t.y : v0 * t.x - v1 * t.y;
            }
        }
        v *= p.alpha;
        const uint64_t idx = orow * g.ld + oc;
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
    p.rot = (const float2*)a.rot;
    p.a_pos = a.a_pos; p.a_back = a.a_back; p.a_rows = a.a_rows;
    p.tiles = a.tiles; p.tile_rows = a.tile_rows; p.a_shared = a.a_shared;
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
        g.ring = s.ring;
        g.rot_head = s.rot_head; g.rot_begin = s.rot_begin; g.rot_dims = s.rot_dims;
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
    p.b_constant = a.b_constant && !a.tiles && !getenv("HOLO_GEMM_NO_EARLY_B") ? 1u : 0u;
    CUtensorMap ma, mb;
    HOLO_TRY(make_map_2d(&mb, a.b, a.n, (uint64_t)a.k * (a.tiles ? a.experts : 1), 64, BK));
    // rows A has: the matrix's own, a ring's, or the ones all tiles of a group share
    const uint64_t a_rows = a.a_pos ? a.a_rows : a.a_shared ? a.a_shared : a.m;
    bool persistent, paired;
    persistent_choice(ctx, a.m, a.n, &persistent, &paired);
    if (a.tiles) {
        persistent = persistent && a.tile_rows == (uint32_t)BM && !a.a_shared;
        paired = false;      // neighbouring row tiles may belong to different experts
    }
    if (persistent) {
        p.box_m = BM;
        HOLO_TRY(make_map_2d(&ma, a.a, a.lda, a_rows, BK, BM));
        return paired ? launch_pair<false, true>(ctx, ma, mb, p) : launch_persistent<false, true>(ctx, ma, mb, p);
    }
    int bn;
    uint32_t splits;
    const uint32_t gtiles = a.tiles ? a.m / a.tile_rows : 0;
    // a group is weight streaming like one product as wide as all its tiles together
    if (a.tiles) tile_choice(ctx, a.tile_rows, a.n * gtiles, kblocks, &bn, &splits);
    else tile_choice(ctx, a.m, a.n, kblocks, &bn, &splits);
    if (!a.tiles && mtiles > 1 && splits == 1) {      // many rows, few columns (a router): K slices fill the chip
        const uint32_t tiles = mtiles * ((a.n + bn - 1) / bn);
        splits = (uint32_t)ctx->sm_count / tiles;
        if (splits > kblocks / 4) splits = kblocks / 4;
        if (splits < 1) splits = 1;
    }
    if (const char* e = getenv("HOLO_GEMM_BN")) bn = atoi(e) == 64 ? 64 : 128;
    if (const char* e = getenv("HOLO_GEMM_SPLITS")) splits = (uint32_t)atoi(e) > 0 ? (uint32_t)atoi(e) : 1;
    if (splits > kblocks) splits = kblocks;
    if (splits > 8) splits = 8;
    if ((a.tiles ? gtiles : mtiles) > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: matmul grid too large");
    p.splits = splits;
    const uint32_t rows = a.tiles ? (a.a_shared ? a.a_shared : a.tile_rows) : a.m;     // of one row tile, or all
    p.box_m = rows < (uint32_t)BM ? rows : (uint32_t)BM;
    HOLO_TRY(make_map_2d(&ma, a.a, a.lda, a_rows, BK, p.box_m));
    const dim3 grid((a.n + bn - 1) / bn, a.tiles ? gtiles : mtiles, splits);
    if (bn == 128) {
        if (rows <= 16) return launch_lin<128, 5, 16>(ctx, ma, mb, p, grid);
        if (rows <= 64) return launch_lin<128, 4, 64>(ctx, ma, mb, p, grid);
        return launch_lin<128, 3, 128>(ctx, ma, mb, p, grid);
    }
    if (rows <= 16) return launch_lin<64, 9, 16>(ctx, ma, mb, p, grid);
    if (rows <= 64) return launch_lin<64, 6, 64>(ctx, ma, mb, p, grid);
    return launch_lin<64, 4, 128>(ctx, ma, mb, p, grid);
}

// ---- further row operations of decoder steps ----------------------------------------------------------------------
namespace {

// (cos, sin) of (*pos + row) times frequency j. The frequency is in turns, as a rounded value and its remainder; the product is
// split the same way and its whole turns dropped, which is exact: the angle's error is one f32 rounding below half a turn
// at any position.
__device__ __forceinline__ float turns(float x, float hi, float lo) {
    const float t = x * hi;
    return (t - rintf(t)) + fmaf(x, lo, fmaf(x, hi, -t));
}
__global__ void rotary_table_kernel(const uint32_t* __restrict__ pos, const float* __restrict__ freq, float2* __restrict__ out, uint32_t rows, uint32_t half) {
    holo_pdl_trigger();
    holo_pdl_wait();
    const uint32_t i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= rows * half) return;
    const uint32_t row = i / half, j = i % half, at = *pos + row, low = at & 0xfffffu;      // both parts are exact in f32
    float r = turns((float)low, freq[j], freq[half + j]);
    if (at != low) {
        r += turns((float)(at - low), freq[j], freq[half + j]);
        r -= rintf(r);
    }
    float s, c;
    sincospif(2.0f * r, &s, &c);
    out[i] = make_float2(c, s);
}

// One CTA per (row, part). VEC: everything is a multiple of four wide and aligned; up to PARTS_HELD vectors per thread stay in
// registers between the reduction and the scaling.
constexpr int PARTS_THREADS = 128, PARTS_HELD = 4;
template <typename T, bool VEC>
__global__ void __launch_bounds__(PARTS_THREADS)
rms_norm_parts_kernel(const HoloNormPartsArgs a) {
    __shared__ float s_part[PARTS_THREADS / 32];
    holo_pdl_trigger();
    const uint32_t row = blockIdx.x, tid = threadIdx.x;
    const HoloNormPartArgs& p = a.part[blockIdx.y];
    constexpr int V = VEC ? 4 : 1;
    const uint32_t nvec = p.width / V;
    holo_pdl_wait();
    const float* x = a.x + (uint64_t)row * a.ld_in + p.in_col;
    auto fetch = [&](uint32_t j) {
        if constexpr (VEC) return reinterpret_cast<const float4*>(x)[j];
        else return make_float4(x[j], 0.f, 0.f, 0.f);
    };
    auto square = [](const float4& v, float acc) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, acc)))); };
    float4 held[PARTS_HELD];
#pragma unroll
    for (int i = 0; i < PARTS_HELD; ++i) {
        const uint32_t j = tid + PARTS_THREADS * i;
        held[i] = j < nvec ? fetch(j) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    uint64_t orow = row;
    if (p.ring) {
        if (row >= a.step[1]) return;
        orow = (a.step[0] + row) % (uint32_t)p.row_limit;
    }
    float inv = 1.0f;
    if (p.norm) {
        float acc = 0.0f;
#pragma unroll
        for (int i = 0; i < PARTS_HELD; ++i) acc = square(held[i], acc);
        for (uint32_t j = tid + PARTS_THREADS * PARTS_HELD; j < nvec; j += PARTS_THREADS) acc = square(fetch(j), acc);
        for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if ((tid & 31u) == 0) s_part[tid >> 5] = acc;
        __syncthreads();
        acc = 0.0f;
#pragma unroll
        for (int w = 0; w < PARTS_THREADS / 32; ++w) acc += s_part[w];
        inv = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(acc, (float)p.width), a.eps)));
    }
    T* out = (T*)p.out + orow * p.ld;
    auto put = [&](uint32_t j, const float4& v) {
        if constexpr (VEC) {
            const float4 w = p.weight ? reinterpret_cast<const float4*>(p.weight)[j] : make_float4(1.f, 1.f, 1.f, 1.f);
            store_norm4(out, 4 * j, make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w));
        } else {
            store_norm(out, j, v.x * inv * (p.weight ? p.weight[j] : 1.0f));
        }
    };
#pragma unroll
    for (int i = 0; i < PARTS_HELD; ++i) {
        const uint32_t j = tid + PARTS_THREADS * i;
        if (j < nvec) put(j, held[i]);
    }
    for (uint32_t j = tid + PARTS_THREADS * PARTS_HELD; j < nvec; j += PARTS_THREADS) put(j, fetch(j));
    for (uint32_t j = p.width + tid; j < p.out_width; j += PARTS_THREADS) store_norm(out, j, 0.0f);
}

// A CTA takes HEAD_COLS columns of one head for up to R rows; its threads split k and add up through shared memory.
constexpr int HEAD_THREADS = 256;
template <typename T> struct HeadVec;
template <> struct HeadVec<float> { static constexpr int N = 4; };
template <> struct HeadVec<__nv_bfloat16> { static constexpr int N = 8; };
template <typename T>
__device__ __forceinline__ void load_vec(const T* src, bool vec, uint32_t left, float (&v)[HeadVec<T>::N]) {
    constexpr int N = HeadVec<T>::N;
    if (vec) {
        const uint4 raw = *reinterpret_cast<const uint4*>(src);
        const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = (float)e[i];
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = (uint32_t)i < left ? (float)src[i] : 0.0f;
    }
}
template <typename T, int R>
__global__ void __launch_bounds__(HEAD_THREADS)
head_linear_kernel(const HoloHeadLinearArgs a, uint32_t vec) {
    constexpr int N = HeadVec<T>::N, COLS = 4 * N, KG = HEAD_THREADS / 4;     // four column vectors, 64 slices of k
    __shared__ float part[HEAD_THREADS / 32][R][COLS];
    holo_pdl_trigger();
    const uint32_t cv = threadIdx.x & 3u, kg = threadIdx.x >> 2, h = blockIdx.y, r0 = blockIdx.z * R;
    const uint32_t col = blockIdx.x * COLS + cv * N;
    const T* b = (const T*)a.b + (uint64_t)h * a.b_step + col;
    const T* x = (const T*)a.a + (uint64_t)r0 * a.lda + (uint64_t)h * a.a_step;
    const uint32_t rows = min((uint32_t)R, a.rows - r0), left = col < a.n ? a.n - col : 0u;
    float acc[R][N] = {};
    holo_pdl_wait();
    if (left) {
        const bool whole = vec && left >= (uint32_t)N;
#pragma unroll 8
        for (uint32_t k = kg; k < a.k; k += KG) {
            float v[N];
            load_vec<T>(b + (uint64_t)k * a.b_ld, whole, left, v);
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float xv = (uint32_t)r < rows ? (float)x[(uint64_t)r * a.lda + k] : 0.0f;
#pragma unroll
                for (int i = 0; i < N; ++i) acc[r][i] = fmaf(xv, v[i], acc[r][i]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
        for (int i = 0; i < N; ++i) {
            for (int o = 4; o < 32; o <<= 1) acc[r][i] += __shfl_xor_sync(0xffffffffu, acc[r][i], o);
            if ((threadIdx.x & 31u) < 4) part[threadIdx.x >> 5][r][cv * N + i] = acc[r][i];
        }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < rows * COLS; i += HEAD_THREADS) {
        const uint32_t r = i / COLS, c = i % COLS, oc = blockIdx.x * COLS + c;
        if (oc >= a.n) continue;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < HEAD_THREADS / 32; ++w) v += part[w][r][c];
        store_norm((T*)a.out, (uint64_t)(r0 + r) * a.ld + (uint64_t)h * a.out_step + oc, v);
    }
}

template <typename T>
int32_t launch_head(holo_b200_ctx* ctx, const HoloHeadLinearArgs& a) {
    constexpr int N = HeadVec<T>::N;
    const uint32_t vec = a.b_ld % N == 0 && a.b_step % N == 0 && ((uintptr_t)a.b & 15u) == 0 ? 1u : 0u;
    const uint32_t cols = (a.n + 4 * N - 1) / (4 * N);
    const uint32_t per = a.rows == 1 ? 1 : 4, blocks = (a.rows + per - 1) / per;
    if (blocks > 65535 || a.heads > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: head_linear rows %u", a.rows);
    if (per == 1) HOLO_CUDA(holo_launch_kernel(ctx, head_linear_kernel<T, 1>, dim3(cols, a.heads, blocks), dim3(HEAD_THREADS), 0, 1, a, vec));
    else HOLO_CUDA(holo_launch_kernel(ctx, head_linear_kernel<T, 4>, dim3(cols, a.heads, blocks), dim3(HEAD_THREADS), 0, 1, a, vec));
    ctx->launches++;
    return HOLO_OK;
}

}  // namespace

int32_t holo_launch_rotary_table(holo_b200_ctx* ctx, const uint32_t* pos, const float* freq, float* out, uint32_t rows, uint32_t half) {
    const uint64_t n = (uint64_t)rows * half;
    if (n > 0x7fffffffull) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: rotary table of %u rows", rows);
    HOLO_CUDA(holo_launch_kernel(ctx, rotary_table_kernel, dim3((uint32_t)((n + 127) / 128)), dim3(128), 0, 1, pos, freq, (float2*)out, rows, half));
    ctx->launches++;
    return HOLO_OK;
}

template <typename T>
static int32_t launch_norm_parts(holo_b200_ctx* ctx, const HoloNormPartsArgs& a) {
    bool vec = a.ld_in % 4 == 0 && ((uintptr_t)a.x & 15u) == 0;
    for (uint32_t i = 0; i < a.nparts; ++i) {
        const HoloNormPartArgs& p = a.part[i];
        vec = vec && p.width % 4 == 0 && p.in_col % 4 == 0 && p.ld % 4 == 0 && (((uintptr_t)p.weight & 15u) | ((uintptr_t)p.out & (4 * sizeof(T) - 1))) == 0;
    }
    const dim3 grid(a.rows, a.nparts);
    if (vec) HOLO_CUDA(holo_launch_kernel(ctx, rms_norm_parts_kernel<T, true>, grid, dim3(PARTS_THREADS), 0, 1, a));
    else HOLO_CUDA(holo_launch_kernel(ctx, rms_norm_parts_kernel<T, false>, grid, dim3(PARTS_THREADS), 0, 1, a));
    ctx->launches++;
    return HOLO_OK;
}
int32_t holo_launch_rms_norm_parts(holo_b200_ctx* ctx, const HoloNormPartsArgs& a) {
    return a.dtype == HOLO_DTYPE_F32 ? launch_norm_parts<float>(ctx, a) : launch_norm_parts<__nv_bfloat16>(ctx, a);
}

int32_t holo_launch_head_linear(holo_b200_ctx* ctx, const HoloHeadLinearArgs& a) {
    return a.dtype == HOLO_DTYPE_F32 ? launch_head<float>(ctx, a) : launch_head<__nv_bfloat16>(ctx, a);
}
