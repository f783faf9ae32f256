// Sliding-window attention of new rows over keys that already hold them (the WindowAttention call): row i of the step is at
// p = *pos + i and sees the last `window` positions up to p. A learned sink per head joins the softmax denominator; a second
// part of every score (q2 . k2) may come from a key part that all heads share.
//
//   latent_attention_kernel   bf16, one key head whose values are the first columns of its keys (latent attention with the
//                             up projections absorbed into query and output): key tiles in shared memory serve 16 (row, head)
//                             pairs for both products (mma.sync), the window split over the chip
//   window_attention_kernel   everything else, f32 included: one CTA per (row, head)
#include "gemm_kernels.cuh"

#include <algorithm>

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void store_out(float* out, uint64_t i, float v) { out[i] = v; }
__device__ __forceinline__ void store_out(__nv_bfloat16* out, uint64_t i, float v) { out[i] = __float2bfloat16_rn(v); }

// The position row 0 of k and v holds, and the first position a row at p sees.
__device__ __forceinline__ uint32_t kv_start(const HoloWindowArgs& a, uint32_t pos) {
    return a.kv_back == 0xffffffffu || pos <= a.kv_back ? 0u : (pos - a.kv_back) & ~127u;
}
__device__ __forceinline__ uint32_t first_seen(const HoloWindowArgs& a, uint32_t p) { return a.window == 0 || p + 1 <= a.window ? 0u : p + 1 - a.window; }

// ---- general form --------------------------------------------------------------------------------------------------
constexpr int GEN_WARPS = 8;
template <typename T, int PL>   // vdim <= 32 PL
__global__ void __launch_bounds__(GEN_WARPS * 32)
window_attention_kernel(const HoloWindowArgs a) {
    holo_pdl_trigger();
    extern __shared__ float s_mem[];   // q [dim], q2 [dim2], then [GEN_WARPS][vdim + 2]
    const uint32_t h = blockIdx.x, i = blockIdx.y, g = h / (a.heads / a.kv_heads);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* s_q2 = s_mem + a.dim;
    float* s_merge = s_q2 + a.dim2;
    holo_pdl_wait();
    const uint32_t pos = *a.pos, p = pos + i;
    for (uint32_t c = threadIdx.x; c < a.dim; c += blockDim.x) s_mem[c] = (float)((const T*)a.q)[(uint64_t)i * a.q_ld + (uint64_t)h * a.q_step + c];
    for (uint32_t c = threadIdx.x; c < a.dim2; c += blockDim.x) s_q2[c] = (float)((const T*)a.q2)[(uint64_t)i * a.q2_ld + (uint64_t)h * a.q2_step + c];
    __syncthreads();
    float o[PL], mx = -INFINITY, sum = 0.0f;
#pragma unroll
    for (int e = 0; e < PL; ++e) o[e] = 0.0f;
    const uint32_t start = kv_start(a, pos);
    for (uint32_t j = first_seen(a, p) + warp; j <= p; j += GEN_WARPS) {
        const uint64_t row = (j - start) % a.kv_rows;
        const T* k = (const T*)a.k + row * a.k_ld + (uint64_t)g * a.dim;
        const T* v = (const T*)a.v + row * a.v_ld + (uint64_t)g * a.vdim;
        float s = 0.0f;
        for (uint32_t c = lane; c < a.dim; c += 32) s = fmaf(s_mem[c], (float)k[c], s);
        if (a.dim2) {
            const T* k2 = (const T*)a.k2 + (uint64_t)(j % a.k2_rows) * a.k2_ld;
            for (uint32_t c = lane; c < a.dim2; c += 32) s = fmaf(s_q2[c], (float)k2[c], s);
        }
        for (int off = 16; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
        s *= a.scale;
        const float nm = fmaxf(mx, s), corr = expf(mx - nm), w = expf(s - nm);   // exp(-inf) = 0 on the first key
        sum = sum * corr + w;
#pragma unroll
        for (int e = 0; e < PL; ++e) {
            const uint32_t c = lane + 32 * e;
            if (c < a.vdim) o[e] = fmaf(w, (float)v[c], o[e] * corr);
        }
        mx = nm;
    }
    float* mine = s_merge + (size_t)warp * (a.vdim + 2);
#pragma unroll
    for (int e = 0; e < PL; ++e) {
        const uint32_t c = lane + 32 * e;
        if (c < a.vdim) mine[c] = o[e];
    }
    if (lane == 0) {
        mine[a.vdim] = mx;
        mine[a.vdim + 1] = sum;
    }
    __syncthreads();
    const float sink = a.sink ? a.sink[h] : -INFINITY;
    float gm = sink;
    for (int w = 0; w < GEN_WARPS; ++w) gm = fmaxf(gm, s_merge[(size_t)w * (a.vdim + 2) + a.vdim]);
    float factor[GEN_WARPS], denom = expf(sink - gm);
#pragma unroll
    for (int w = 0; w < GEN_WARPS; ++w) {
        factor[w] = expf(s_merge[(size_t)w * (a.vdim + 2) + a.vdim] - gm);
        denom += s_merge[(size_t)w * (a.vdim + 2) + a.vdim + 1] * factor[w];
    }
    T* out = (T*)a.out + (uint64_t)i * a.ld + (uint64_t)h * a.vdim;
    for (uint32_t c = threadIdx.x; c < a.vdim; c += blockDim.x) {
        float acc = 0.0f;
#pragma unroll
        for (int w = 0; w < GEN_WARPS; ++w) acc += s_merge[(size_t)w * (a.vdim + 2) + c] * factor[w];
        store_out(out, c, acc / denom);
    }
}

template <typename T, int PL>
int32_t launch_general_as(holo_b200_ctx* ctx, const HoloWindowArgs& a) {
    if (a.rows > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: window_attention rows %u on the general path", a.rows);
    const size_t smem = (a.dim + a.dim2 + GEN_WARPS * (a.vdim + 2)) * sizeof(float);     // at most 41 KiB
    HOLO_CUDA(holo_launch_kernel(ctx, window_attention_kernel<T, PL>, dim3(a.heads, a.rows), dim3(GEN_WARPS * 32), smem, 1, a));
    ctx->launches++;
    return HOLO_OK;
}
template <typename T>
int32_t launch_general(holo_b200_ctx* ctx, const HoloWindowArgs& a) {
    if (a.vdim <= 128) return launch_general_as<T, 4>(ctx, a);
    if (a.vdim <= 512) return launch_general_as<T, 16>(ctx, a);
    return launch_general_as<T, 32>(ctx, a);
}

// ---- one key head, values inside the keys -----------------------------------------------------------------------------
// A CTA (8 warps) takes 16 (row, head) pairs and a contiguous share of the key tiles the pairs see. Per tile of KT keys:
//   scores   warp w: keys 8 w .. 8 w + 7 against all pairs, over the whole key width
//   weights  warp w: pairs 2 w, 2 w + 1: running maximum, exponentials, the factor the accumulators shrink by
//   values   warp w: value columns [16 u, 16 u + 16), u = w, w + 8, ...
// Shares of one pair tile meet in a second launch (latent_merge_kernel) through a partial buffer.
constexpr int LAT_WARPS = 8;
constexpr uint32_t LAT_PARTIAL_FLOATS = 6u << 20;

struct LatentParams {
    HoloWindowArgs a;
    float* partials;     // [pair tile][split][16][vdim + 2]
    uint32_t splits;
};

__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool take) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(take ? 16u : 0u) : "memory");
}

// The keys a pair tile sees: positions [lo, hi].
struct LatentRange {
    uint32_t lo, hi;
};
__device__ __forceinline__ LatentRange latent_range(const HoloWindowArgs& a, uint32_t tile, uint32_t pos) {
    const uint32_t first = tile * 16 / a.heads, last = min((tile * 16 + 15) / a.heads, a.rows - 1);
    return {first_seen(a, pos + first), pos + last};
}

template <int KT>
struct LatentSmem {
    uint32_t pitch, q, ring, scores, weights, stats, total;
    __host__ __device__ explicit LatentSmem(uint32_t width) {
        pitch = width * 2 + 16;                      // an odd number of 16-byte units: rows start in different banks
        q = 0;
        ring = q + 16 * pitch;
        scores = ring + 2 * KT * pitch;
        weights = scores + 16 * (KT + 4) * 4;        // bf16 rows of KT + 8
        stats = weights + 16 * (KT + 8) * 2;         // maximum, sum, factor
        total = stats + 3 * 16 * 4;
    }
};

template <int KT, int UW>   // vdim <= 128 UW
__global__ void __launch_bounds__(LAT_WARPS * 32)
latent_attention_kernel(const LatentParams p) {
    extern __shared__ __align__(16) uint8_t sm[];
    const HoloWindowArgs& a = p.a;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t split = blockIdx.x, tile = blockIdx.y, width = a.dim + a.dim2;
    const LatentSmem<KT> s(width);
    float* s_scores = reinterpret_cast<float*>(sm + s.scores);
    __nv_bfloat16* s_weights = reinterpret_cast<__nv_bfloat16*>(sm + s.weights);
    float* s_max = reinterpret_cast<float*>(sm + s.stats);
    float *s_sum = s_max + 16, *s_factor = s_max + 32;
    const uint32_t base = smem_u32(sm);
    holo_pdl_trigger();
    holo_pdl_wait();
    const uint32_t pos = *a.pos;
    const LatentRange range = latent_range(a, tile, pos);
    const uint32_t tiles = (range.hi - range.lo + KT) / KT, used = min(p.splits, tiles);
    if (split >= used) return;
    const uint32_t t_begin = (uint32_t)((uint64_t)tiles * split / used), t_end = (uint32_t)((uint64_t)tiles * (split + 1) / used);
    const uint32_t start = kv_start(a, pos), vec1 = a.dim / 8, vecs = width / 8;

    auto load_tile = [&](uint32_t t, uint32_t stage) {
        for (uint32_t r = warp; r < KT; r += LAT_WARPS) {
            const uint32_t key = range.lo + t * KT + r;
            const bool take = key <= range.hi;
            const __nv_bfloat16* k = (const __nv_bfloat16*)a.k + (uint64_t)((min(key, range.hi) - start) % a.kv_rows) * a.k_ld;
            const __nv_bfloat16* k2 = a.dim2 ? (const __nv_bfloat16*)a.k2 + (uint64_t)(min(key, range.hi) % a.k2_rows) * a.k2_ld : nullptr;
            const uint32_t dst = base + s.ring + (stage * KT + r) * s.pitch;
            for (uint32_t c = lane; c < vecs; c += 32) cp_async16(dst + c * 16, c < vec1 ? k + c * 8 : k2 + (c - vec1) * 8, take);
        }
    };
    load_tile(t_begin, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (uint32_t i = threadIdx.x; i < 16 * vecs; i += blockDim.x) {
        const uint32_t r = i / vecs, c = i % vecs, pair = tile * 16 + r, row = pair / a.heads, head = pair % a.heads;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (row < a.rows)
            v = *reinterpret_cast<const uint4*>(c < vec1 ? (const __nv_bfloat16*)a.q + (uint64_t)row * a.q_ld + (uint64_t)head * a.q_step + c * 8
                                                         : (const __nv_bfloat16*)a.q2 + (uint64_t)row * a.q2_ld + (uint64_t)head * a.q2_step + (c - vec1) * 8);
        *reinterpret_cast<uint4*>(sm + s.q + r * s.pitch + c * 16) = v;
    }
    if (threadIdx.x < 16) {
        s_max[threadIdx.x] = -INFINITY;
        s_sum[threadIdx.x] = 0.0f;
    }
    float o[UW][2][4];
#pragma unroll
    for (int u = 0; u < UW; ++u)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[u][0][e] = o[u][1][e] = 0.0f;
    const uint32_t q_addr = base + s.q + (lane & 15) * s.pitch + (lane >> 4) * 16;
    const uint32_t p_addr = base + s.weights + (lane & 15) * (KT + 8) * 2 + (lane >> 4) * 16;
    const uint32_t k_off = (warp * 8 + (lane & 7)) * s.pitch + (lane >> 3) * 16;
    const uint32_t v_off = ((lane & 7) + (((lane >> 3) & 1) << 3)) * s.pitch + (lane >> 4) * 16;
    const uint32_t ksteps = width / 16, units = a.vdim / 16, r0 = lane >> 2;
    const float scale = a.scale * LOG2E;
    uint32_t stage = 0;
    for (uint32_t t = t_begin; t < t_end; ++t) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                               // tile t is here, and nobody reads the other stage any more
        if (t + 1 < t_end) load_tile(t + 1, stage ^ 1u);
        asm volatile("cp.async.commit_group;" ::: "memory");
        const uint32_t keys = base + s.ring + stage * KT * s.pitch;
        if (warp * 8 < KT) {
            float c0[4] = {}, c1[4] = {};
#pragma unroll 4
            for (uint32_t k = 0; k < ksteps; k += 2) {
                uint32_t kb[4], qa[4];
                ldsm4(keys + k_off + k * 32, kb);      // 8 keys, two steps (past the last step: bytes nobody uses)
                ldsm4(q_addr + k * 32, qa);
                mma16816(c0, qa, kb[0], kb[1]);
                if (k + 1 < ksteps) {
                    ldsm4(q_addr + k * 32 + 32, qa);
                    mma16816(c1, qa, kb[2], kb[3]);
                }
            }
            float* dst = s_scores + r0 * (KT + 4) + warp * 8 + (lane & 3) * 2;
            *reinterpret_cast<float2*>(dst) = make_float2(c0[0] + c1[0], c0[1] + c1[1]);
            *reinterpret_cast<float2*>(dst + 8 * (KT + 4)) = make_float2(c0[2] + c1[2], c0[3] + c1[3]);
        }
        __syncthreads();
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const uint32_t r = warp * 2 + x, at = pos + (tile * 16 + r) / a.heads, seen = first_seen(a, at);
            float v[KT / 32], top = -INFINITY;
#pragma unroll
            for (int i = 0; i < KT / 32; ++i) {
                const uint32_t key = range.lo + t * KT + lane + 32 * i;
                v[i] = key <= at && key >= seen && key <= range.hi ? s_scores[r * (KT + 4) + lane + 32 * i] * scale : -INFINITY;
                top = fmaxf(top, v[i]);
            }
            for (int off = 16; off > 0; off >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, off));
            const float old = s_max[r], now = fmaxf(old, top), ref = now == -INFINITY ? 0.0f : now;
            float part = 0.0f;
#pragma unroll
            for (int i = 0; i < KT / 32; ++i) {
                const float w = exp2f(v[i] - ref);
                part += w;
                s_weights[r * (KT + 8) + lane + 32 * i] = __float2bfloat16_rn(w);
            }
            for (int off = 16; off > 0; off >>= 1) part += __shfl_xor_sync(0xffffffffu, part, off);
            __syncwarp();
            if (lane == 0) {
                const float f = exp2f(old - ref);
                s_max[r] = now;
                s_factor[r] = f;
                s_sum[r] = s_sum[r] * f + part;
            }
            __syncwarp();
        }
        __syncthreads();
        const float f0 = s_factor[r0], f1 = s_factor[r0 + 8];
#pragma unroll
        for (int u = 0; u < UW; ++u)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                o[u][n][0] *= f0; o[u][n][1] *= f0;
                o[u][n][2] *= f1; o[u][n][3] *= f1;
            }
#pragma unroll
        for (int ks = 0; ks < KT / 16; ++ks) {
            uint32_t pa[4];
            ldsm4(p_addr + ks * 32, pa);
#pragma unroll
            for (int u = 0; u < UW; ++u) {
                const uint32_t unit = warp + LAT_WARPS * u;
                if (unit < units) {
                    uint32_t vb[4];
                    ldsm4t(keys + ks * 16 * s.pitch + v_off + unit * 32, vb);
                    mma16816(o[u][0], pa, vb[0], vb[1]);
                    mma16816(o[u][1], pa, vb[2], vb[3]);
                }
            }
        }
        stage ^= 1u;
    }
    // (maximum in log2 units, sum, unscaled context) of this share
    const uint32_t ml = a.vdim + 2;
    if (used > 1) {
        float* part = p.partials + ((uint64_t)tile * p.splits + split) * 16 * ml;
#pragma unroll
        for (int u = 0; u < UW; ++u) {
            const uint32_t unit = warp + LAT_WARPS * u;
            if (unit < units)
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        *reinterpret_cast<float2*>(part + (r0 + 8 * e) * ml + unit * 16 + n * 8 + (lane & 3) * 2) = make_float2(o[u][n][2 * e], o[u][n][2 * e + 1]);
        }
        if (threadIdx.x < 16) *reinterpret_cast<float2*>(part + threadIdx.x * ml + a.vdim) = make_float2(s_max[threadIdx.x], s_sum[threadIdx.x]);
        return;
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const uint32_t r = r0 + 8 * e, pair = tile * 16 + r, row = pair / a.heads, head = pair % a.heads;
        if (row >= a.rows) continue;
        const float sink = a.sink ? a.sink[head] * LOG2E : -INFINITY, top = fmaxf(s_max[r], sink);
        const float f = exp2f(s_max[r] - top), inv = f / (s_sum[r] * f + exp2f(sink - top));
        __nv_bfloat16* out = (__nv_bfloat16*)a.out + (uint64_t)row * a.ld + (uint64_t)head * a.vdim;
#pragma unroll
        for (int u = 0; u < UW; ++u) {
            const uint32_t unit = warp + LAT_WARPS * u;
            if (unit < units)
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const __nv_bfloat162 v = __floats2bfloat162_rn(o[u][n][2 * e] * inv, o[u][n][2 * e + 1] * inv);
                    *reinterpret_cast<__nv_bfloat162*>(out + unit * 16 + n * 8 + (lane & 3) * 2) = v;
                }
        }
    }
}

// One CTA per (pair, 128 value columns).
template <int KT>
__global__ void __launch_bounds__(128)
latent_merge_kernel(const LatentParams p) {
    const HoloWindowArgs& a = p.a;
    const uint32_t pair = blockIdx.x, tile = pair >> 4, row = pair / a.heads, head = pair % a.heads, c = blockIdx.y * 128 + threadIdx.x;
    holo_pdl_trigger();
    holo_pdl_wait();
    const LatentRange range = latent_range(a, tile, *a.pos);
    const uint32_t used = min(p.splits, (range.hi - range.lo + KT) / KT), ml = a.vdim + 2;
    if (used < 2 || c >= a.vdim) return;
    const float* part = p.partials + (uint64_t)tile * p.splits * 16 * ml + (pair & 15u) * ml;
    const float sink = a.sink ? a.sink[head] * LOG2E : -INFINITY;
    float top = sink;
    for (uint32_t i = 0; i < used; ++i) top = fmaxf(top, part[(uint64_t)i * 16 * ml + a.vdim]);
    float denom = exp2f(sink - top), acc = 0.0f;
#pragma unroll 8
    for (uint32_t i = 0; i < used; ++i) {
        const float* share = part + (uint64_t)i * 16 * ml;
        const float f = exp2f(share[a.vdim] - top);
        denom = fmaf(share[a.vdim + 1], f, denom);
        acc = fmaf(share[c], f, acc);
    }
    ((__nv_bfloat16*)a.out)[(uint64_t)row * a.ld + (uint64_t)head * a.vdim + c] = __float2bfloat16_rn(acc / denom);
}

template <int KT, int UW>
int32_t launch_latent(holo_b200_ctx* ctx, LatentParams p, uint32_t pair_tiles) {
    static thread_local int configured_device = -1;
    if (configured_device != ctx->device) {
        HOLO_CUDA(cudaFuncSetAttribute(latent_attention_kernel<KT, UW>, cudaFuncAttributeMaxDynamicSharedMemorySize, ctx->smem_optin - 1024));
        configured_device = ctx->device;
    }
    const HoloWindowArgs& a = p.a;
    const uint32_t rows_in_tile = 15 / a.heads + 2;
    const uint64_t keys = a.window ? std::min<uint64_t>((uint64_t)a.window + rows_in_tile, a.kv_rows) : a.kv_rows;
    uint64_t splits = std::max<uint64_t>(1, (uint64_t)ctx->sm_count / pair_tiles);
    splits = std::min<uint64_t>(splits, (keys + KT - 1) / KT);
    splits = std::min<uint64_t>(splits, LAT_PARTIAL_FLOATS / ((uint64_t)pair_tiles * 16 * (a.vdim + 2)));
    p.splits = (uint32_t)std::max<uint64_t>(splits, 1);
    HOLO_CUDA(holo_launch_kernel(ctx, latent_attention_kernel<KT, UW>, dim3(p.splits, pair_tiles), dim3(LAT_WARPS * 32), LatentSmem<KT>(a.dim + a.dim2).total, 1, p));
    ctx->launches++;
    if (p.splits > 1) {
        HOLO_CUDA(holo_launch_kernel(ctx, latent_merge_kernel<KT>, dim3(a.rows * a.heads, (a.vdim + 127) / 128), dim3(128), 0, 1, p));
        ctx->launches++;
    }
    return HOLO_OK;
}
template <int KT>
int32_t launch_latent_kt(holo_b200_ctx* ctx, const LatentParams& p, uint32_t pair_tiles) {
    if (p.a.vdim <= 128) return launch_latent<KT, 1>(ctx, p, pair_tiles);
    if (p.a.vdim <= 256) return launch_latent<KT, 2>(ctx, p, pair_tiles);
    if (p.a.vdim <= 512) return launch_latent<KT, 4>(ctx, p, pair_tiles);
    return launch_latent<KT, 8>(ctx, p, pair_tiles);
}

// Launches the latent kernel, or returns with *taken false when the shape does not suit it.
int32_t try_latent(holo_b200_ctx* ctx, const HoloWindowArgs& a, bool* taken) {
    *taken = false;
    const uint64_t pair_tiles = ((uint64_t)a.rows * a.heads + 15) / 16;
    const uint32_t width = a.dim + a.dim2, limit = (uint32_t)ctx->smem_optin - 1024;
    if (a.dtype != HOLO_DTYPE_BF16 || a.kv_heads != 1 || a.k != a.v || a.k_ld != a.v_ld || a.vdim > a.dim || a.dim % 16 || a.dim2 % 16 || a.vdim % 16 ||
        (a.k_ld | a.k2_ld | a.q_ld | a.q_step | a.q2_ld | a.q2_step) % 8 || a.ld % 2 || pair_tiles > 65535 ||
        (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.q2 | (uintptr_t)a.k2) & 15u) || ((uintptr_t)a.out & 3u))
        return HOLO_OK;
    const bool wide = LatentSmem<64>(width).total <= limit;
    if (!wide && LatentSmem<32>(width).total > limit) return HOLO_OK;
    LatentParams p;
    p.a = a;
    if (!ctx->latent_partials) HOLO_CUDA(cudaMalloc(&ctx->latent_partials, (size_t)LAT_PARTIAL_FLOATS * 4));
    p.partials = ctx->latent_partials;
    *taken = true;
    return wide ? launch_latent_kt<64>(ctx, p, (uint32_t)pair_tiles) : launch_latent_kt<32>(ctx, p, (uint32_t)pair_tiles);
}

}  // namespace

int32_t holo_launch_window_attention(holo_b200_ctx* ctx, const HoloWindowArgs& a) {
    if (!getenv("HOLO_WINDOW_GENERAL")) {
        bool taken = false;
        HOLO_TRY(try_latent(ctx, a, &taken));
        if (taken) return HOLO_OK;
    }
    return a.dtype == HOLO_DTYPE_F32 ? launch_general<float>(ctx, a) : launch_general<__nv_bfloat16>(ctx, a);
}
