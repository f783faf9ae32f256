// Sliding-window attention of new rows over keys that already hold them (the WindowAttention call): row i of the step is at
// p = *pos + i and sees the last `window` positions up to p. A learned sink per head joins the softmax denominator; a second
// part of every score (q2 . k2) may come from a key part that all heads share.
//
//   latent_attention_kernel   bf16, one key head whose values are the first columns of its keys (latent attention with the
//                             up projections absorbed into query and output): key tiles in shared memory serve 16 (row, head)
//                             pairs for both products (mma.sync), the window split over the chip
//   window_tile_kernel        bf16, many rows: 128-row query tiles on tcgen05 with scores, weights and output in TMEM, a running
//                             maximum per row and an accumulator that is rescaled only when the maximum has grown by a lot
//   window_attention_kernel   everything else, f32 included: one CTA per (row, head)
#include "attention_tile.cuh"

#include <algorithm>

namespace {

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

// One CTA per (pair, 128 value columns). At most MERGE_SPLITS shares.
constexpr uint32_t MERGE_SPLITS = 256;
template <int KT>
__global__ void __launch_bounds__(128)
latent_merge_kernel(const LatentParams p) {
    __shared__ float s_factor[MERGE_SPLITS], s_red[8];
    const HoloWindowArgs& a = p.a;
    const uint32_t pair = blockIdx.x, tile = pair >> 4, row = pair / a.heads, head = pair % a.heads, tid = threadIdx.x, c = blockIdx.y * 128 + tid;
    holo_pdl_trigger();
    holo_pdl_wait();
    const LatentRange range = latent_range(a, tile, *a.pos);
    const uint32_t used = min(p.splits, (range.hi - range.lo + KT) / KT), ml = a.vdim + 2;
    if (used < 2) return;
    const float* part = p.partials + (uint64_t)tile * p.splits * 16 * ml + (pair & 15u) * ml;
    const float sink = a.sink ? a.sink[head] * LOG2E : -INFINITY;
    float2 mine[MERGE_SPLITS / 128];
    float top = sink;
#pragma unroll
    for (uint32_t i = 0; i < MERGE_SPLITS / 128; ++i) {
        const uint32_t share = tid + 128 * i;
        mine[i] = share < used ? *reinterpret_cast<const float2*>(part + (uint64_t)share * 16 * ml + a.vdim) : make_float2(-INFINITY, 0.0f);
        top = fmaxf(top, mine[i].x);
    }
    for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
    if ((tid & 31u) == 0) s_red[tid >> 5] = top;
    __syncthreads();
    top = fmaxf(fmaxf(s_red[0], s_red[1]), fmaxf(s_red[2], s_red[3]));
    float denom = 0.0f;
#pragma unroll
    for (uint32_t i = 0; i < MERGE_SPLITS / 128; ++i) {
        const uint32_t share = tid + 128 * i;
        const float f = exp2f(mine[i].x - top);
        if (share < used) s_factor[share] = f;
        denom = fmaf(mine[i].y, f, denom);
    }
    for (int o = 16; o > 0; o >>= 1) denom += __shfl_xor_sync(0xffffffffu, denom, o);
    if ((tid & 31u) == 0) s_red[4 + (tid >> 5)] = denom;
    __syncthreads();
    if (c >= a.vdim) return;
    denom = (s_red[4] + s_red[5]) + (s_red[6] + s_red[7]) + exp2f(sink - top);
    float acc = 0.0f;
#pragma unroll 16
    for (uint32_t i = 0; i < used; ++i) acc = fmaf(part[(uint64_t)i * 16 * ml + c], s_factor[i], acc);
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
    splits = std::min<uint64_t>(splits, MERGE_SPLITS);
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
    // tiles of 32 keys where those of 64 would not reach every SM
    const uint64_t keys = a.window ? std::min<uint64_t>(a.window, a.kv_rows) : a.kv_rows;
    return wide && pair_tiles * ((keys + 63) / 64) > (uint64_t)ctx->sm_count / 2 ? launch_latent_kt<64>(ctx, p, (uint32_t)pair_tiles)
                                                                                : launch_latent_kt<32>(ctx, p, (uint32_t)pair_tiles);
}

// ---- many rows: 128-row tiles on tcgen05 ------------------------------------------------------------------------------
// A tile of 128 rows packs `rpt` rows times the heads of a group. One CTA works on NQ tiles of a key head, the keys in tiles
// of 128; while the weight warps of one query tile exponentiate, the tensor core works for the other.
//   warp 0      TMA producer: the query tiles once; key chunks (128 keys x 64 columns; the shared key part follows the head's
//               own) and value tiles through rings
//   warp 1      tcgen05.mma issuer. Per key tile and query tile q: O_q += P_q V as soon as the weights are stored, then
//               S_q = Q_q K^T of the next key tile into the same columns (one thread's products execute in order)
//   warps 2-9   weights and output, four warps per query tile, one thread per row
// The weights are exp2(s - m) with m a reference that follows the row's maximum only when it has grown by more than RAISE
// (log2 units): weights stay below 2^RAISE, and O is rarely rescaled. TMEM: S_q (P_q over its first half) at 128 q, O_q at
// 256 + 128 q (NQ 2) or 256 (NQ 1, up to 256 columns). Allocated after the dependency wait, dependents released after that.
constexpr int WT_THREADS = 320;
constexpr float RAISE = 8.0f;

struct WindowTileParams {
    HoloWindowArgs a;
    uint32_t* status;
    uint32_t group, rpt, chunks1, chunks2, vchunks, kslots, vslots;
};

template <int NQ>
__global__ void __launch_bounds__(WT_THREADS, 1)
window_tile_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_q2, const __grid_constant__ CUtensorMap map_k,
                   const __grid_constant__ CUtensorMap map_k2, const __grid_constant__ CUtensorMap map_v, const WindowTileParams p) {
    extern __shared__ uint8_t smem_raw[];
    const HoloWindowArgs& a = p.a;
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    uint8_t* sm = smem_raw + (base - raw);
    const uint32_t kchunks = p.chunks1 + p.chunks2, qbytes = kchunks * TILE_CHUNK, vbytes = p.vchunks * TILE_CHUNK;
    const uint32_t s_q = base, s_k = s_q + NQ * qbytes, s_v = s_k + p.kslots * TILE_CHUNK;
    const uint32_t off_bars = NQ * qbytes + p.kslots * TILE_CHUNK + p.vslots * vbytes;
    // at most 16 key slots and 2 value slots
    const uint32_t bar_q = base + off_bars, bar_k_full = bar_q + 8, bar_k_empty = bar_k_full + 128, bar_v_full = bar_k_empty + 128, bar_v_empty = bar_v_full + 16,
                   bar_s = bar_v_empty + 16, bar_p = bar_s + 16, bar_pv = bar_p + 16;
    uint32_t* s_tmem = reinterpret_cast<uint32_t*>(sm + off_bars + 384);
    volatile uint32_t* s_abort = reinterpret_cast<volatile uint32_t*>(sm + off_bars + 388);

    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t g = blockIdx.x, row0 = (gridDim.y - 1 - blockIdx.y) * NQ * p.rpt;   // the tiles with the most keys first
    if (threadIdx.x == 0) {
        mbar_init(bar_q, 1);
        for (uint32_t i = 0; i < p.kslots; ++i) {
            mbar_init(bar_k_full + 8 * i, 1);
            mbar_init(bar_k_empty + 8 * i, 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(bar_v_full + 8 * i, 1);
            mbar_init(bar_v_empty + 8 * i, 1);
            mbar_init(bar_s + 8 * i, 1);
            mbar_init(bar_p + 8 * i, 4);     // one arrival per weight warp
            mbar_init(bar_pv + 8 * i, 1);
        }
        *s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    holo_pdl_wait();
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(s_tmem)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    holo_pdl_trigger();
    const uint32_t tmem_base = *s_tmem;
    const uint32_t pos = *a.pos, start = kv_start(a, pos);
    const uint32_t t_lo = first_seen(a, pos + row0) / 128, t_hi = (pos + min(row0 + NQ * p.rpt, a.rows) - 1) / 128, ntiles = t_hi - t_lo + 1;

    if (warp == 0) {
        // ---------------- TMA producer ----------------
        if (lane == 0) {
            mbar_arrive_expect_tx(bar_q, NQ * kchunks * p.rpt * p.group * 128);
            for (uint32_t i = 0; i < NQ; ++i) {
                const int row = (int)(row0 + i * p.rpt), head = (int)(g * p.group);
                for (uint32_t c = 0; c < p.chunks1; ++c) tma_load_3d(s_q + i * qbytes + c * TILE_CHUNK, &map_q, (int)(64 * c), head, row, bar_q);
                for (uint32_t c = 0; c < p.chunks2; ++c) tma_load_3d(s_q + i * qbytes + (p.chunks1 + c) * TILE_CHUNK, &map_q2, (int)(64 * c), head, row, bar_q);
            }
            uint32_t ks = 0, kuse = 0, vs = 0, vuse = 0;      // slot, and how often the ring has gone round
            bool ok = true;
            for (uint32_t t = t_lo; t <= t_hi && ok; ++t) {
                const int krow = (int)((t * 128 - start) % a.kv_rows), k2row = a.dim2 ? (int)(t * 128 % a.k2_rows) : 0;
                for (uint32_t c = 0; c < kchunks && ok; ++c) {
                    ok = kuse == 0 || mbar_wait(bar_k_empty + 8 * ks, (kuse - 1) & 1, s_abort, p.status);
                    if (!ok) break;
                    mbar_arrive_expect_tx(bar_k_full + 8 * ks, TILE_CHUNK);
                    if (c < p.chunks1) tma_load_2d(s_k + ks * TILE_CHUNK, &map_k, (int)(g * a.dim + 64 * c), krow, bar_k_full + 8 * ks);
                    else tma_load_2d(s_k + ks * TILE_CHUNK, &map_k2, (int)(64 * (c - p.chunks1)), k2row, bar_k_full + 8 * ks);
                    if (++ks == p.kslots) ks = 0, ++kuse;
                }
                ok = ok && (vuse == 0 || mbar_wait(bar_v_empty + 8 * vs, (vuse - 1) & 1, s_abort, p.status));
                if (!ok) break;
                mbar_arrive_expect_tx(bar_v_full + 8 * vs, vbytes);
                for (uint32_t c = 0; c < p.vchunks; ++c) tma_load_2d(s_v + vs * vbytes + c * TILE_CHUNK, &map_v, (int)(g * a.vdim + 64 * c), krow, bar_v_full + 8 * vs);
                if (++vs == p.vslots) vs = 0, ++vuse;
            }
            if (!ok) {
                // nothing may still be on its way into this CTA's shared memory when it ends: the last load of every slot
                for (uint32_t it = 0; it < WAIT_LIMIT && !mbar_try_wait(bar_q, 0); ++it) __nanosleep(64);
                for (uint32_t i = 0; i < p.kslots; ++i) {
                    const uint32_t loads = kuse + (i < ks ? 1u : 0u);
                    for (uint32_t it = 0; loads && it < WAIT_LIMIT && !mbar_try_wait(bar_k_full + 8 * i, (loads - 1) & 1); ++it) __nanosleep(64);
                }
                for (uint32_t i = 0; i < p.vslots; ++i) {
                    const uint32_t loads = vuse + (i < vs ? 1u : 0u);
                    for (uint32_t it = 0; loads && it < WAIT_LIMIT && !mbar_try_wait(bar_v_full + 8 * i, (loads - 1) & 1); ++it) __nanosleep(64);
                }
            }
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer ----------------
        if (lane == 0) {
            // D = f32, A = B = bf16, M = 128; S: both operands K-major, N = 128; O: V is N-major, N = vdim
            const uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 3) << 17) | ((128u >> 4) << 24);
            const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((a.vdim >> 3) << 17) | ((128u >> 4) << 24);
            const uint64_t desc_q = smem_desc(s_q, 16, 1024), desc_k = smem_desc(s_k, 16, 1024), desc_v = smem_desc(s_v, TILE_CHUNK, 1024);
            uint32_t ks = 0, kphase = 0, vs = 0, vphase = 0;
            // S_q of the key tile whose chunks begin at slot ks; the last query tile gives every chunk back
            auto scores = [&](uint32_t q) {
                uint32_t slot = ks, phase = kphase;
                for (uint32_t c = 0; c < kchunks; ++c) {
                    if (q == 0 && !mbar_wait(bar_k_full + 8 * slot, phase, s_abort, p.status)) return false;
                    if (q == 0) asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint32_t width = c < p.chunks1 ? a.dim - 64 * c : a.dim2 - 64 * (c - p.chunks1);
                    const uint64_t dq = desc_q + ((q * qbytes + c * TILE_CHUNK) >> 4), dk = desc_k + ((slot * TILE_CHUNK) >> 4);
#pragma unroll
                    for (uint32_t k = 0; k < 4; ++k)
                        if (16 * k < width) umma_bf16(tmem_base + q * 128, dq + 2 * k, dk + 2 * k, idesc_s, (c | k) != 0);
                    if (q == NQ - 1) umma_commit(bar_k_empty + 8 * slot);
                    if (++slot == p.kslots) slot = 0, phase ^= 1;
                }
                umma_commit(bar_s + 8 * q);
                if (q == NQ - 1) ks = slot, kphase = phase;
                return true;
            };
            bool ok = mbar_wait(bar_q, 0, s_abort, p.status);
            for (uint32_t q = 0; q < NQ && ok; ++q) ok = scores(q);
            for (uint32_t i = 0; i < ntiles && ok; ++i) {
                for (uint32_t q = 0; q < NQ && ok; ++q) {
                    if (q == 0) ok = mbar_wait(bar_v_full + 8 * vs, vphase, s_abort, p.status);
                    ok = ok && mbar_wait(bar_p + 8 * q, i & 1, s_abort, p.status);
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint64_t dv = desc_v + ((vs * vbytes) >> 4);
#pragma unroll
                    for (uint32_t k = 0; k < 8; ++k)
                        umma_bf16_ts(tmem_base + 256 + q * 128, tmem_base + q * 128 + k * 8, dv + 128 * k, idesc_o, k != 0 || i != 0);
                    umma_commit(bar_pv + 8 * q);
                    if (q == NQ - 1) {
                        umma_commit(bar_v_empty + 8 * vs);
                        if (++vs == p.vslots) vs = 0, vphase ^= 1;
                    }
                    if (i + 1 < ntiles) ok = scores(q);
                }
            }
        }
    } else if ((warp - 2) >> 2 < NQ) {
        // ---------------- weights (TMEM lane quarter = warp % 4), then the output ----------------
        const uint32_t q = (warp - 2) >> 2, quarter = warp & 3u, tr = quarter * 32 + lane;
        const uint32_t first = row0 + q * p.rpt, row = first + tr / p.group, head = g * p.group + tr % p.group;
        const bool valid = tr < p.rpt * p.group && row < a.rows;
        const uint32_t at = pos + min(row, a.rows - 1), seen = first_seen(a, at);
        const uint32_t last_seen = first_seen(a, pos + min(first + p.rpt, a.rows) - 1);   // the first key the tile's last row sees
        const uint32_t lanes = (quarter * 32u) << 16, tmem_s = tmem_base + q * 128 + lanes, tmem_o = tmem_base + 256 + q * 128 + lanes;
        const float c = a.scale * LOG2E;
        const uint64_t c2 = pair(c, c);
        float ref = -1e30f, sum = 0.0f;
        bool ok = true;
        for (uint32_t i = 0; i < ntiles; ++i) {
            ok = mbar_wait(bar_s + 8 * q, i & 1, s_abort, p.status) && !*s_abort;
            // the product before these scores (it has finished: they were issued after it)
            if (ok && i > 0) ok = mbar_wait(bar_pv + 8 * q, (i - 1) & 1, s_abort, p.status);
            ok = __all_sync(0xffffffffu, ok);   // the TMEM accesses below are whole-warp instructions
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t key0 = (t_lo + i) * 128;
            uint32_t v[4][32];
#pragma unroll
            for (int x = 0; x < 4; ++x) tmem_ld32_request(tmem_s + 32 * x, v[x]);
            tmem_ld32_wait(v[0]);
#pragma unroll
            for (int x = 1; x < 4; ++x) tmem_ld32_pass(v[x]);
            if (key0 + 127 > pos + first || key0 < last_seen) {      // some row does not see some key
#pragma unroll
                for (int x = 0; x < 4; ++x)
#pragma unroll
                    for (int e = 0; e < 32; ++e) {
                        const uint32_t key = key0 + 32 * x + e;
                        if (key > at || key < seen) v[x][e] = 0xff800000u;   // -infinity
                    }
            }
            float top[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int x = 0; x < 4; ++x)
#pragma unroll
                for (int e = 0; e < 32; ++e) top[e & 3] = fmaxf(top[e & 3], __uint_as_float(v[x][e]));
            const float most = fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])) * c;
            const bool raise = most > ref + RAISE;
            if (__any_sync(0xffffffffu, raise)) {
                const float f = raise ? ex2(ref - most) : 1.0f;
                if (raise) ref = most;
                sum *= f;
                if (i > 0) {     // the products so far are in O, the next one waits for this warp's weights
                    for (uint32_t x = 0; x < a.vdim / 16; ++x) {
                        uint32_t o[16];
                        tmem_ld16(tmem_o + 16 * x, o);
#pragma unroll
                        for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * f);
                        tmem_st16(tmem_o + 16 * x, o);
                    }
                }
            }
            const uint64_t minus = pair(-ref, -ref);
            uint64_t part[2] = {0, 0};
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                uint32_t w[16];
#pragma unroll
                for (int e = 0; e < 16; ++e) {
                    const float2 s = unpair(fma2(pair(__uint_as_float(v[x][2 * e]), __uint_as_float(v[x][2 * e + 1])), c2, minus));
                    const float lo = ex2(s.x), hi = ex2(s.y);
                    part[e & 1] = add2(part[e & 1], pair(lo, hi));
                    w[e] = pack_bf16(lo, hi);
                }
                tmem_st16(tmem_s + 16 * x, w);      // over scores this warp has already read
            }
            const float2 a0 = unpair(part[0]), a1 = unpair(part[1]);
            sum += (a0.x + a0.y) + (a1.x + a1.y);
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar_p + 8 * q) : "memory");
        }
        ok = ok && mbar_wait(bar_pv + 8 * q, (ntiles - 1) & 1, s_abort, p.status) && !*s_abort && !(*reinterpret_cast<volatile uint32_t*>(p.status) & 4u);
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const float denom = sum + (a.sink && valid ? ex2(fmaf(a.sink[head], LOG2E, -ref)) : 0.0f);
            const float inv = __fdiv_rn(1.0f, denom);
            __nv_bfloat16* out = (__nv_bfloat16*)a.out + (uint64_t)row * a.ld + (uint64_t)head * a.vdim;
            for (uint32_t x = 0; x < a.vdim / 16; ++x) {
                uint32_t v[16], w[8];
                tmem_ld16(tmem_o + 16 * x, v);
#pragma unroll
                for (int e = 0; e < 8; ++e) w[e] = pack_bf16(__uint_as_float(v[2 * e]) * inv, __uint_as_float(v[2 * e + 1]) * inv);
                if (valid) {
                    reinterpret_cast<uint4*>(out + 16 * x)[0] = make_uint4(w[0], w[1], w[2], w[3]);
                    reinterpret_cast<uint4*>(out + 16 * x)[1] = make_uint4(w[4], w[5], w[6], w[7]);
                }
            }
        }
    }
    // everyone meets here, whatever happened above, so that TMEM is always released
    __syncwarp();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(512u) : "memory");
    }
}

// `cols` columns of every head over all rows, a box of 64 columns of a group's heads over the tile's rows.
int32_t make_map_heads(CUtensorMap* map, const void* ptr, uint32_t cols, uint32_t heads, uint32_t rows, uint64_t step, uint64_t ld, uint32_t group, uint32_t rpt) {
    cuuint64_t dims[3] = {cols, heads, rows};
    cuuint64_t strides[2] = {step * 2, ld * 2};
    cuuint32_t box[3] = {64, group, rpt};
    cuuint32_t es[3] = {1, 1, 1};
    const CUresult r = encode_tiled_fn()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? HOLO_OK : holo_fail(HOLO_ERR_DISPATCH, "dispatch failed: cuTensorMapEncodeTiled (attention) returned %d", (int)r);
}
// `cols` columns of rows of pitch ld, boxes of 64 columns and 128 rows.
int32_t make_map_keys(CUtensorMap* map, const void* ptr, uint64_t cols, uint64_t rows, uint64_t ld) {
    cuuint64_t dims[2] = {cols, rows};
    cuuint64_t strides[1] = {ld * 2};
    cuuint32_t box[2] = {64, 128};
    cuuint32_t es[2] = {1, 1};
    const CUresult r = encode_tiled_fn()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? HOLO_OK : holo_fail(HOLO_ERR_DISPATCH, "dispatch failed: cuTensorMapEncodeTiled (attention) returned %d", (int)r);
}

template <int NQ>
int32_t launch_window_tile(holo_b200_ctx* ctx, const CUtensorMap (&m)[5], const WindowTileParams& p, uint32_t ctas, uint32_t smem) {
    static thread_local int configured_device = -1;
    if (configured_device != ctx->device) {
        HOLO_CUDA(cudaFuncSetAttribute(window_tile_kernel<NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, ctx->smem_optin));
        configured_device = ctx->device;
    }
    HOLO_CUDA(holo_launch_kernel(ctx, window_tile_kernel<NQ>, dim3(p.a.kv_heads, ctas), dim3(WT_THREADS), smem, 1, m[0], m[1], m[2], m[3], m[4], p));
    ctx->launches++;
    return HOLO_OK;
}

// Launches the tile kernel, or returns with *taken false when the shape does not suit it.
int32_t try_window_tile(holo_b200_ctx* ctx, const HoloWindowArgs& a, bool* taken) {
    *taken = false;
    WindowTileParams p;
    p.a = a;
    p.status = ctx->dev_status;
    p.group = a.heads / a.kv_heads;
    if (a.dtype != HOLO_DTYPE_BF16 || !(a.scale > 0.0f) || a.dim % 16 || a.dim2 % 16 || a.vdim % 16 || a.dim > 512 || a.dim2 > 512 || a.vdim > 256 || p.group > 128 ||
        a.kv_rows % 128 || a.k2_rows % 128 || (a.q_ld | a.q_step | a.k_ld | a.v_ld | a.q2_ld | a.q2_step | a.k2_ld | a.ld) % 8 ||
        (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.q2 | (uintptr_t)a.k2 | (uintptr_t)a.out) & 15u) || encode_tiled_fn() == nullptr)
        return HOLO_OK;
    p.rpt = 128 / p.group;
    p.chunks1 = (a.dim + 63) / 64;
    p.chunks2 = (a.dim2 + 63) / 64;
    p.vchunks = (a.vdim + 63) / 64;
    const uint32_t kchunks = p.chunks1 + p.chunks2, extra = 512 + 1024, slots = ((uint32_t)ctx->smem_optin - extra) / TILE_CHUNK;
    const uint32_t qtiles = (a.rows + p.rpt - 1) / p.rpt;
    if (qtiles > 65535) return HOLO_OK;
    // two query tiles per CTA where they fit beside a whole key tile and a value tile; two value slots where one more key chunk fits as well
    uint32_t nq = a.vdim <= 128 && qtiles > 1 && 3 * kchunks + p.vchunks <= slots ? 2 : 1;
    if (const char* e = getenv("HOLO_WINDOW_QUERY_TILES")) nq = atoi(e) == 1 ? 1 : nq;
    if ((nq + 1) * kchunks + p.vchunks > slots) return HOLO_OK;
    p.vslots = (nq + 1) * kchunks + 1 + 2 * p.vchunks <= slots ? 2 : 1;
    p.kslots = std::min<uint32_t>(slots - nq * kchunks - p.vslots * p.vchunks, 2 * kchunks);
    p.kslots = std::min<uint32_t>(p.kslots, 16);
    if (p.kslots < kchunks) return HOLO_OK;
    const uint32_t smem = (nq * kchunks + p.kslots + p.vslots * p.vchunks) * TILE_CHUNK + extra;
    CUtensorMap m[5];
    HOLO_TRY(make_map_heads(&m[0], a.q, a.dim, a.heads, a.rows, a.q_step, a.q_ld, p.group, p.rpt));
    HOLO_TRY(make_map_keys(&m[2], a.k, (uint64_t)a.kv_heads * a.dim, a.kv_rows, a.k_ld));
    HOLO_TRY(make_map_keys(&m[4], a.v, (uint64_t)a.kv_heads * a.vdim, a.kv_rows, a.v_ld));
    m[1] = m[0];
    m[3] = m[2];
    if (a.dim2) {
        HOLO_TRY(make_map_heads(&m[1], a.q2, a.dim2, a.heads, a.rows, a.q2_step, a.q2_ld, p.group, p.rpt));
        HOLO_TRY(make_map_keys(&m[3], a.k2, a.dim2, a.k2_rows, a.k2_ld));
    }
    *taken = true;
    return nq == 2 ? launch_window_tile<2>(ctx, m, p, (qtiles + 1) / 2, smem) : launch_window_tile<1>(ctx, m, p, qtiles, smem);
}

}  // namespace

int32_t holo_launch_window_attention(holo_b200_ctx* ctx, const HoloWindowArgs& a) {
    if (!getenv("HOLO_WINDOW_GENERAL")) {
        bool taken = false;
        HOLO_TRY(try_latent(ctx, a, &taken));
        if (!taken) HOLO_TRY(try_window_tile(ctx, a, &taken));
        if (taken) return HOLO_OK;
    }
    return a.dtype == HOLO_DTYPE_F32 ? launch_general<float>(ctx, a) : launch_general<__nv_bfloat16>(ctx, a);
}
