// Causal attention of new rows over a cache that already holds them (the CausalAttention call): row i of the step is
// at position p = *pos + i and sees cache rows 0 .. p. Optional score cap (softcap * tanh(s / softcap)), one learned
// sink per head in the softmax denominator, and a query factor that grows with the logarithm of the position.
//
// bf16 with a cap of at most CAP_LIMIT needs no running maximum: every capped score lies in [-cap, cap], so exp(s) of any
// row fits f32 (and bf16, which has f32's exponent range) as it is, partial sums over disjoint keys simply add, and the
// accumulator is never rescaled. Two kernels use that:
//   causal_attention_split_kernel  few rows (decode): warps stream 16-key tiles through their own cp.async rings, both
//                                  products on mma.sync (HBM- or latency-bound), the keys split over the chip
//   causal_attention_tile_kernel   many rows (prefill): 128-row tiles on tcgen05 with scores, weights and output in TMEM
// Everything else (f32, no cap, larger caps, sizes TMA cannot take) runs the general kernel.
#include "attention_tile.cuh"

#include <algorithm>

namespace {

constexpr float CAP_LIMIT = 64.0f;

// The factor of a query at position p: 1 + coef * ln(floor((p + 1) / every) + 1). IEEE division: an exact quotient
// stays exact, so the floor steps exactly at multiples of `every`.
__device__ __forceinline__ float query_factor(uint32_t p, float coef, float every) {
    if (every == 0.0f) return 1.0f;
    return 1.0f + coef * logf(floorf(__fdiv_rn((float)(p + 1), every)) + 1.0f);
}

__device__ __forceinline__ void store_out(float* out, uint64_t i, float v) { out[i] = v; }
__device__ __forceinline__ void store_out(__nv_bfloat16* out, uint64_t i, float v) { out[i] = __float2bfloat16_rn(v); }

// ---- general form: any dim / vdim up to 512, any group, f32 or bf16, with or without cap -------------------------
// One CTA per (row, head); its warps take interleaved keys with a running (max, sum, context) triple each and merge
// through shared memory at the end.
constexpr int GEN_WARPS = 8, GEN_PER_LANE = 16;
template <typename T>
__global__ void __launch_bounds__(GEN_WARPS * 32)
causal_attention_generic_kernel(const HoloCausalArgs a) {
    holo_pdl_trigger();
    extern __shared__ float s_mem[];   // [GEN_WARPS][vdim + 2]
    const uint32_t h = blockIdx.x, i = blockIdx.y, g = h / (a.heads / a.kv_heads);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    holo_pdl_wait();
    const uint32_t p = *a.pos + i, visible = min(p + 1, a.cache_rows);
    const T* q = (const T*)a.q + ((uint64_t)i * a.heads + h) * a.dim;
    const float factor = a.scale * query_factor(p, a.temp_coef, a.temp_every);
    float qv[GEN_PER_LANE], o[GEN_PER_LANE];
#pragma unroll
    for (int e = 0; e < GEN_PER_LANE; ++e) {
        const uint32_t c = lane + 32 * e;
        qv[e] = c < a.dim ? (float)q[c] : 0.0f;
        o[e] = 0.0f;
    }
    float mx = -INFINITY, sum = 0.0f;
    for (uint32_t j = warp; j < visible; j += GEN_WARPS) {
        const T* k = (const T*)a.k + ((uint64_t)j * a.kv_heads + g) * a.dim;
        const T* v = (const T*)a.v + ((uint64_t)j * a.kv_heads + g) * a.vdim;
        float s = 0.0f;
#pragma unroll
        for (int e = 0; e < GEN_PER_LANE; ++e) {
            const uint32_t c = lane + 32 * e;
            if (c < a.dim) s = fmaf(qv[e], (float)k[c], s);
        }
        for (int off = 16; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
        s *= factor;
        if (a.softcap > 0.0f) s = a.softcap * tanhf(s / a.softcap);
        const float nm = fmaxf(mx, s), corr = expf(mx - nm), w = expf(s - nm);   // exp(-inf) = 0 on the first key
        sum = sum * corr + w;
#pragma unroll
        for (int e = 0; e < GEN_PER_LANE; ++e) {
            const uint32_t c = lane + 32 * e;
            if (c < a.vdim) o[e] = fmaf(w, (float)v[c], o[e] * corr);
        }
        mx = nm;
    }
    float* mine = s_mem + (size_t)warp * (a.vdim + 2);
#pragma unroll
    for (int e = 0; e < GEN_PER_LANE; ++e) {
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
    for (int w = 0; w < GEN_WARPS; ++w) gm = fmaxf(gm, s_mem[(size_t)w * (a.vdim + 2) + a.vdim]);
    float denom = expf(sink - gm);
    for (int w = 0; w < GEN_WARPS; ++w) denom += s_mem[(size_t)w * (a.vdim + 2) + a.vdim + 1] * expf(s_mem[(size_t)w * (a.vdim + 2) + a.vdim] - gm);
    T* out = (T*)a.out + (uint64_t)i * a.ld + (uint64_t)h * a.vdim;
    for (uint32_t c = threadIdx.x; c < a.vdim; c += blockDim.x) {
        float acc = 0.0f;
        for (int w = 0; w < GEN_WARPS; ++w) acc += s_mem[(size_t)w * (a.vdim + 2) + c] * expf(s_mem[(size_t)w * (a.vdim + 2) + a.vdim] - gm);
        store_out(out, c, acc / denom);
    }
}

int32_t launch_generic(holo_b200_ctx* ctx, const HoloCausalArgs& a) {
    if (a.rows > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: causal_attention rows %u on the general path", a.rows);
    const size_t smem = GEN_WARPS * (a.vdim + 2) * sizeof(float);
    if (a.dtype == HOLO_DTYPE_F32) HOLO_CUDA(holo_launch_kernel(ctx, causal_attention_generic_kernel<float>, dim3(a.heads, a.rows), dim3(GEN_WARPS * 32), smem, 1, a));
    else HOLO_CUDA(holo_launch_kernel(ctx, causal_attention_generic_kernel<__nv_bfloat16>, dim3(a.heads, a.rows), dim3(GEN_WARPS * 32), smem, 1, a));
    ctx->launches++;
    return HOLO_OK;
}


// ---- capped scores without a maximum -----------------------------------------------------------------------------
// exp(cap * tanh(s * factor / cap)), with c1 = 2 factor log2(e) / cap and c2 = cap log2(e):
// tanh(y) = 1 - 2 / (exp(2y) + 1), so the exponent in log2 units is c2 - 2 c2 / (2^(s c1) + 1).
__device__ __forceinline__ float capped_exp(float s, float c1, float c2) { return ex2(fmaf(-2.0f * c2, rcp(ex2(s * c1) + 1.0f), c2)); }

// The same for scores well inside the cap, |y| = |s factor / cap| <= TANH_SMALL, two at a time on the packed f32 pipe: tanh(y) / y as
// a degree-5 polynomial in y^2 (a Chebyshev fit over the interval; |error| of tanh below 1e-7, f32 rounding included). One
// special-function operation per score instead of three, which is what bounds the many-row kernel.
constexpr float TANH_SMALL = 0.75f;
// c0 = factor / cap, c2 = cap log2(e), each twice
__device__ __forceinline__ float2 capped_exp_small(uint64_t s, uint64_t c0, uint64_t c2) {
    const uint64_t y = mul2(s, c0), z = mul2(y, y);
    uint64_t t = fma2(z, pair(-0.0047239522f, -0.0047239522f), pair(0.0195937865f, 0.0195937865f));
    t = fma2(t, z, pair(-0.0533498190f, -0.0533498190f));
    t = fma2(t, z, pair(0.1332551539f, 0.1332551539f));
    t = fma2(t, z, pair(-0.3333296776f, -0.3333296776f));
    t = fma2(t, z, pair(1.0f, 1.0f));
    const float2 e = unpair(mul2(mul2(t, y), c2));
    return make_float2(ex2(e.x), ex2(e.y));
}

// ---- few rows: keys split over CTAs and warps ----------------------------------------------------------------------
// A tile of 16 query rows packs (row, head of the group) pairs of one kv head, so every K/V row is read once for all of
// them. Warp w of split c takes 16-key tiles w, w + W, ... of the split's range through a private ring of STAGES tiles
// (no block-wide synchronisation in the loop). Warps merge through shared memory, splits through a partial buffer: the
// last CTA of a (kv head, row tile) to count in adds the partials in split order; nobody waits.
constexpr uint32_t SPLIT_SLOTS = 1024, SPLIT_SLOT_FLOATS = 16 * 257;

struct SplitParams {
    HoloCausalArgs a;
    float* partials;
    uint32_t* arrivals;
    uint32_t group, splits;
};

template <int VT, int STAGES>   // vdim <= 16 VT
__global__ void __launch_bounds__(256)
causal_attention_split_kernel(const SplitParams p) {
    extern __shared__ __align__(16) uint8_t sm[];
    const HoloCausalArgs& a = p.a;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    const uint32_t split = blockIdx.x, g = blockIdx.y, z = blockIdx.z;
    const uint32_t kp = a.dim * 2 + 16, vp = a.vdim * 2 + 16;      // shared-memory row pitches: an odd number of 16-byte units
    const uint32_t tile_bytes = 16 * (kp + vp);
    const uint32_t s_q = smem_u32(sm), s_ring = s_q + 16 * kp + warp * STAGES * tile_bytes;
    const uint32_t kv_ld = a.kv_heads * a.dim, vv_ld = a.kv_heads * a.vdim;
    holo_pdl_trigger();
    holo_pdl_wait();
    const uint32_t pos = *a.pos;
    // the last position any row of this tile sees
    const uint32_t last_row = min((z * 16 + 15) / p.group, a.rows - 1);
    const uint32_t visible = min(pos + last_row + 1, a.cache_rows);
    const uint32_t tiles = (visible + 15) / 16;
    const uint32_t used = min(p.splits, (tiles + nwarps - 1) / nwarps);
    if (split >= used) return;
    const uint32_t t_begin = (uint32_t)((uint64_t)tiles * split / used), t_end = (uint32_t)((uint64_t)tiles * (split + 1) / used);
    const __nv_bfloat16* kbase = (const __nv_bfloat16*)a.k + g * a.dim;
    const __nv_bfloat16* vbase = (const __nv_bfloat16*)a.v + g * a.vdim;
    const uint32_t kvec = a.dim / 8, vvec = a.vdim / 8;

    auto load_tile = [&](uint32_t tile, uint32_t stage) {
        const uint32_t dst = s_ring + stage * tile_bytes;
        for (uint32_t i = lane; i < 16 * kvec; i += 32) {
            const uint32_t r = i / kvec, c = i % kvec, key = tile * 16 + r;
            cp_async16(dst + r * kp + c * 16, kbase + (uint64_t)min(key, a.cache_rows - 1) * kv_ld + c * 8, key < visible);
        }
        for (uint32_t i = lane; i < 16 * vvec; i += 32) {
            const uint32_t r = i / vvec, c = i % vvec, key = tile * 16 + r;
            cp_async16(dst + 16 * kp + r * vp + c * 16, vbase + (uint64_t)min(key, a.cache_rows - 1) * vv_ld + c * 8, key < visible);
        }
    };
    const uint32_t first = t_begin + warp;
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) {
        const uint32_t t = first + s * nwarps;
        if (t < t_end) load_tile(t, s);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    // the query tile (rows past the step's last one are zero)
    for (uint32_t i = threadIdx.x; i < 16 * kvec; i += blockDim.x) {
        const uint32_t r = i / kvec, c = i % kvec, qr = z * 16 + r, row = qr / p.group;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (row < a.rows) v = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)a.q + ((uint64_t)row * a.heads + g * p.group + qr % p.group) * a.dim + c * 8);
        *reinterpret_cast<uint4*>(sm + r * kp + c * 16) = v;
    }
    __syncthreads();

    const uint32_t r0 = lane >> 2;                        // this thread's rows of the tile: r0 and r0 + 8
    const float c2 = a.softcap * LOG2E;
    float c1[2];
    uint32_t limit[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const uint32_t row = min((z * 16 + r0 + 8 * e) / p.group, a.rows - 1);
        c1[e] = 2.0f * LOG2E * a.scale * query_factor(pos + row, a.temp_coef, a.temp_every) / a.softcap;
        limit[e] = pos + row;
    }
    // with at most eight rows the upper half of the tile is all padding
    const bool upper = a.rows * p.group > z * 16 + 8;
    float o[VT][2][4];
    float sum[2] = {0.0f, 0.0f};
#pragma unroll
    for (int n = 0; n < VT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][0][e] = o[n][1][e] = 0.0f;
    const uint32_t q_addr = s_q + (lane & 15) * kp + (lane >> 4) * 16;
    const uint32_t k_off = ((lane & 7) + ((lane >> 4) << 3)) * kp + ((lane >> 3) & 1) * 16;
    const uint32_t v_off = 16 * kp + ((lane & 7) + (((lane >> 3) & 1) << 3)) * vp + (lane >> 4) * 16;
    const uint32_t ksteps = a.dim / 16, vsteps = a.vdim / 16;
    uint32_t stage = 0;
    for (uint32_t t = first; t < t_end; t += nwarps) {
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
        __syncwarp();
        {   // refill the stage the previous iteration has emptied
            const uint32_t nt = t + (STAGES - 1) * nwarps;
            if (nt < t_end) load_tile(nt, stage == 0 ? STAGES - 1 : stage - 1);
            asm volatile("cp.async.commit_group;" ::: "memory");
        }
        const uint32_t tile = s_ring + stage * tile_bytes;
        float s[2][4] = {};
#pragma unroll 4
        for (uint32_t k = 0; k < ksteps; ++k) {
            uint32_t qa[4], kb[4];
            ldsm4(q_addr + k * 32, qa);
            ldsm4(tile + k_off + k * 32, kb);
            mma16816(s[0], qa, kb[0], kb[1]);
            mma16816(s[1], qa, kb[2], kb[3]);
        }
        float w[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int half = e >> 1;
                const uint32_t key = t * 16 + n * 8 + (lane & 3) * 2 + (e & 1);
                w[n][e] = 0.0f;
                if ((half == 0 || upper) && key <= limit[half]) w[n][e] = capped_exp(s[n][e], c1[half], c2);
                sum[half] += w[n][e];
            }
        const uint32_t pa[4] = {pack_bf16(w[0][0], w[0][1]), pack_bf16(w[0][2], w[0][3]), pack_bf16(w[1][0], w[1][1]), pack_bf16(w[1][2], w[1][3])};
#pragma unroll
        for (int n = 0; n < VT; ++n) {
            if ((uint32_t)n < vsteps) {
                uint32_t vb[4];
                ldsm4t(tile + v_off + n * 32, vb);
                mma16816(o[n][0], pa, vb[0], vb[1]);
                mma16816(o[n][1], pa, vb[2], vb[3]);
            }
        }
        stage = stage + 1 == STAGES ? 0 : stage + 1;
        __syncwarp();
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 1);
        sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 2);
    }
    __syncthreads();   // every warp is through with its ring: it becomes the merge buffer [warp][16][vdim + 1]
    float* merge = reinterpret_cast<float*>(sm);
    const uint32_t ml = a.vdim + 1;
    float* mine = merge + (size_t)warp * 16 * ml;
#pragma unroll
    for (int n = 0; n < VT; ++n)
        if ((uint32_t)n < vsteps)
#pragma unroll
            for (int h = 0; h < 2; ++h)
#pragma unroll
                for (int e = 0; e < 4; ++e) mine[(r0 + 8 * (e >> 1)) * ml + n * 16 + h * 8 + (lane & 3) * 2 + (e & 1)] = o[n][h][e];
    if ((lane & 3) == 0) {
        mine[r0 * ml + a.vdim] = sum[0];
        mine[(r0 + 8) * ml + a.vdim] = sum[1];
    }
    __syncthreads();
    const uint32_t nrows = min(16u, a.rows * p.group - z * 16), cells = nrows * ml;
    const uint32_t tile_id = z * a.kv_heads + g;
    float* part = p.partials + ((uint64_t)tile_id * p.splits + split) * SPLIT_SLOT_FLOATS;
    for (uint32_t i = threadIdx.x; i < cells; i += blockDim.x) {
        float v = 0.0f;
        for (uint32_t w = 0; w < nwarps; ++w) v += merge[(size_t)w * 16 * ml + i];
        if (used == 1) merge[i] = v;     // only this thread touches cell i of every warp's part
        else __stcg(part + i, v);
    }
    if (used > 1) {
        __shared__ uint32_t s_last;
        __threadfence();
        __syncthreads();
        if (threadIdx.x == 0) s_last = atomicAdd(p.arrivals + tile_id, 1u) == used - 1 ? 1u : 0u;
        __syncthreads();
        if (!s_last) return;
        __threadfence();
        if (threadIdx.x == 0) p.arrivals[tile_id] = 0;
        const float* all = p.partials + (uint64_t)tile_id * p.splits * SPLIT_SLOT_FLOATS;
        for (uint32_t i = threadIdx.x; i < cells; i += blockDim.x) {
            float v = 0.0f;
#pragma unroll 16
            for (uint32_t c = 0; c < used; ++c) v += __ldcg(all + (uint64_t)c * SPLIT_SLOT_FLOATS + i);
            merge[i] = v;
        }
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < nrows * (a.vdim / 2); i += blockDim.x) {
        const uint32_t r = i / (a.vdim / 2), c = 2 * (i % (a.vdim / 2)), qr = z * 16 + r, head = g * p.group + qr % p.group;
        const float denom = merge[r * ml + a.vdim] + (a.sink ? ex2(a.sink[head] * LOG2E) : 0.0f);
        const float inv = __fdiv_rn(1.0f, denom);
        *reinterpret_cast<uint32_t*>((__nv_bfloat16*)a.out + (uint64_t)(qr / p.group) * a.ld + head * a.vdim + c) =
            pack_bf16(merge[r * ml + c] * inv, merge[r * ml + c + 1] * inv);
    }
}

template <int VT, int STAGES>
int32_t launch_split(holo_b200_ctx* ctx, const SplitParams& p, uint32_t qtiles, uint32_t warps, size_t smem) {
    static thread_local int configured_device = -1;
    if (configured_device != ctx->device) {
        HOLO_CUDA(cudaFuncSetAttribute(causal_attention_split_kernel<VT, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, ctx->smem_optin - 1024));
        configured_device = ctx->device;
    }
    HOLO_CUDA(holo_launch_kernel(ctx, causal_attention_split_kernel<VT, STAGES>, dim3(p.splits, p.a.kv_heads, qtiles), dim3(warps * 32), smem, 1, p));
    ctx->launches++;
    return HOLO_OK;
}

// Launches the split kernel, or returns with *taken false when the shape does not suit it.
int32_t try_split(holo_b200_ctx* ctx, const HoloCausalArgs& a, bool* taken) {
    *taken = false;
    const uint32_t group = a.heads / a.kv_heads, qtiles = (a.rows * group + 15) / 16;
    const uint32_t pairs = qtiles * a.kv_heads;
    if (a.vdim > 256 || a.dim > 256 || pairs > SPLIT_SLOTS || qtiles > 65535) return HOLO_OK;
    const int stages = a.vdim <= 64 ? 4 : a.vdim <= 128 ? 3 : 2;
    const size_t kp = a.dim * 2 + 16, vp = a.vdim * 2 + 16, limit = (size_t)ctx->smem_optin - 1024;
    uint32_t warps = 8;
    auto bytes = [&](uint32_t w) { return std::max(16 * kp + w * stages * 16 * (kp + vp), (size_t)w * 16 * (a.vdim + 1) * 4); };
    while (warps > 1 && bytes(warps) > limit) warps /= 2;
    if (bytes(warps) > limit) return HOLO_OK;
    if (!ctx->causal_partials) HOLO_CUDA(cudaMalloc(&ctx->causal_partials, (size_t)SPLIT_SLOTS * SPLIT_SLOT_FLOATS * 4));
    SplitParams p;
    p.a = a;
    p.partials = ctx->causal_partials;
    p.arrivals = ctx->attn_arrivals;
    p.group = group;
    p.splits = (uint32_t)ctx->sm_count / pairs;
    const uint32_t most = (a.cache_rows + 16 * warps - 1) / (16 * warps);
    if (p.splits > most) p.splits = most;
    if (p.splits < 1) p.splits = 1;
    *taken = true;
    if (a.vdim <= 64) return launch_split<4, 4>(ctx, p, qtiles, warps, bytes(warps));
    if (a.vdim <= 128) return launch_split<8, 3>(ctx, p, qtiles, warps, bytes(warps));
    return launch_split<16, 2>(ctx, p, qtiles, warps, bytes(warps));
}

// ---- many rows: 128-row tiles on tcgen05 ------------------------------------------------------------------------------
// A tile of 128 rows packs `rpt` rows times the group's heads, so the keys are read once for the whole group. One CTA works
// on NQ such tiles of a kv head: two where there are enough rows to fill the chip and both fit (every K/V tile from L2 then
// serves 256 rows; with one, the loop waits for L2), else one. Keys come in tiles of 128; an item is one key tile against one
// query tile, and two items are in flight, one per S buffer.
//   warp 0     TMA producer: the query tiles once, K and V tiles through rings
//   warp 1     tcgen05.mma issuer: S = Q K^T, O += P V with P read from TMEM; as soon as an item's weights are stored its
//              product is issued, and the scores of the item after next into its buffer
//   warps 2-17 weights, four groups of four warps (one per TMEM lane quarter): group j takes key half j / 2 of the items of
//              buffer j % 2: tcgen05.ld half a row of S, cap, exponentiate, sum, tcgen05.st the bf16 weights
// Without a running maximum O needs no correction: it stays in TMEM from the first tile to the last.
// TMEM (all 512 columns): S at 0 and 128, O from 256; P at 384 and 448 where vdim leaves room, else over the S it came from,
// each key half's weights over the first half of its scores (the next scores then wait for the item's product). It is allocated after the dependency wait, and dependents are
// released only after the allocation, so no neighbouring launch can hold columns this kernel or its predecessor waits for.
constexpr int TILE_THREADS = 576;

struct TileParams {
    HoloCausalArgs a;
    uint32_t* status;
    uint32_t group, rpt, qchunks, vchunks, kstages, vstages;
    uint32_t alias;     // P lies over S
    uint32_t ostride;   // TMEM columns between the accumulators of two query tiles
};

template <int NQ>
__global__ void __launch_bounds__(TILE_THREADS, 1)
causal_attention_tile_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                             const __grid_constant__ CUtensorMap map_v, const TileParams p) {
    extern __shared__ uint8_t smem_raw[];
    const HoloCausalArgs& a = p.a;
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    uint8_t* sm = smem_raw + (base - raw);
    const uint32_t kbytes = p.qchunks * TILE_CHUNK, vbytes = p.vchunks * TILE_CHUNK;
    const uint32_t s_q = base, s_k = s_q + NQ * kbytes, s_v = s_k + p.kstages * kbytes;
    const uint32_t off_bars = (NQ + p.kstages) * kbytes + p.vstages * vbytes;
    const uint32_t bar_q = base + off_bars, bar_k_full = bar_q + 8, bar_k_empty = bar_k_full + 16, bar_v_full = bar_k_empty + 16,
                   bar_v_empty = bar_v_full + 16, bar_s = bar_v_empty + 16, bar_p = bar_s + 16, bar_pv = bar_p + 16, bar_o = bar_pv + 16;
    uint32_t* s_tmem = reinterpret_cast<uint32_t*>(sm + off_bars + 128);
    volatile uint32_t* s_abort = reinterpret_cast<volatile uint32_t*>(sm + off_bars + 132);
    float* s_sum = reinterpret_cast<float*>(sm + off_bars + 256);   // [4][128]

    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t g = blockIdx.x, qtile = gridDim.y - 1 - blockIdx.y;   // the tiles with the most keys first
    const uint32_t row0 = qtile * NQ * p.rpt;
    if (threadIdx.x == 0) {
        mbar_init(bar_q, 1);
        for (int s = 0; s < 2; ++s) {
            mbar_init(bar_k_full + 8 * s, 1);
            mbar_init(bar_k_empty + 8 * s, 1);
            mbar_init(bar_v_full + 8 * s, 1);
            mbar_init(bar_v_empty + 8 * s, 1);
            mbar_init(bar_s + 8 * s, 1);
            mbar_init(bar_p + 8 * s, 8);     // one arrival per weight warp
            mbar_init(bar_pv + 8 * s, 1);
        }
        mbar_init(bar_o, 1);
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
    const uint32_t tmem_base = *s_tmem, tmem_o = tmem_base + 256;
    const uint32_t pos = *a.pos;
    const uint32_t visible = min(pos + min(row0 + NQ * p.rpt, a.rows), a.cache_rows);
    const uint32_t ntiles = (visible + 127) / 128, items = ntiles * NQ;

    if (warp == 0) {
        // ---------------- TMA producer ----------------
        if (lane == 0) {
            mbar_arrive_expect_tx(bar_q, NQ * p.qchunks * p.rpt * p.group * 128);
            for (uint32_t i = 0; i < NQ; ++i)
                for (uint32_t c = 0; c < p.qchunks; ++c)
                    tma_load_3d(s_q + i * kbytes + c * TILE_CHUNK, &map_q, (int)(64 * c), (int)(g * p.group), (int)(row0 + i * p.rpt), bar_q);
            uint32_t kt = 0, vt = 0;
            bool ok = true;
            for (uint32_t t = 0; t < ntiles && ok; ++t) {
                const uint32_t ks = t % p.kstages, vs = t % p.vstages;
                ok = t < p.kstages || mbar_wait(bar_k_empty + 8 * ks, (t / p.kstages - 1) & 1, s_abort, p.status);
                if (!ok) break;
                mbar_arrive_expect_tx(bar_k_full + 8 * ks, kbytes);
                for (uint32_t c = 0; c < p.qchunks; ++c)
                    tma_load_2d(s_k + ks * kbytes + c * TILE_CHUNK, &map_k, (int)(g * a.dim + 64 * c), (int)(t * 128), bar_k_full + 8 * ks);
                ++kt;
                ok = t < p.vstages || mbar_wait(bar_v_empty + 8 * vs, (t / p.vstages - 1) & 1, s_abort, p.status);
                if (!ok) break;
                mbar_arrive_expect_tx(bar_v_full + 8 * vs, vbytes);
                for (uint32_t c = 0; c < p.vchunks; ++c)
                    tma_load_2d(s_v + vs * vbytes + c * TILE_CHUNK, &map_v, (int)(g * a.vdim + 64 * c), (int)(t * 128), bar_v_full + 8 * vs);
                ++vt;
            }
            if (!ok) {
                // nothing may still be on its way into this CTA's shared memory when it ends
                for (uint32_t it = 0; it < WAIT_LIMIT && !mbar_try_wait(bar_q, 0); ++it) __nanosleep(64);
                for (uint32_t t = kt > p.kstages ? kt - p.kstages : 0; t < kt; ++t)
                    for (uint32_t it = 0; it < WAIT_LIMIT && !mbar_try_wait(bar_k_full + 8 * (t % p.kstages), (t / p.kstages) & 1); ++it) __nanosleep(64);
                for (uint32_t t = vt > p.vstages ? vt - p.vstages : 0; t < vt; ++t)
                    for (uint32_t it = 0; it < WAIT_LIMIT && !mbar_try_wait(bar_v_full + 8 * (t % p.vstages), (t / p.vstages) & 1); ++it) __nanosleep(64);
            }
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer ----------------
        if (lane == 0) {
            // D = f32, A = B = bf16, M = 128; S: both operands K-major, N = 128; O: V is N-major, N = vdim
            const uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 3) << 17) | ((128u >> 4) << 24);
            const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((a.vdim >> 3) << 17) | ((128u >> 4) << 24);
            const uint32_t ksteps = a.dim / 16;
            // Item i is key tile i / NQ against query tile i % NQ, its scores in buffer i & 1. Between an item's weights and its
            // buffer's next scores lies what this one thread does, so it works on ready-made descriptors (a step of 16 k-elements
            // adds 32 bytes, four of them a chunk; a step of 16 keys adds 2048 bytes) and running stage numbers.
            const uint64_t desc_q = smem_desc(s_q, 16, 1024), desc_k = smem_desc(s_k, 16, 1024), desc_v = smem_desc(s_v, TILE_CHUNK, 1024);
            const uint32_t kstep = kbytes >> 4, vstep = vbytes >> 4;
            const bool alias = p.alias != 0;
            uint32_t ks = 0, kphase = 0, vs = 0, vphase = 0;
            auto scores = [&](uint32_t i) {
                const uint32_t qi = NQ == 2 ? i & 1u : 0u, buf = i & 1u;
                if (qi == 0 && !mbar_wait(bar_k_full + 8 * ks, kphase, s_abort, p.status)) return false;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint64_t dq = desc_q + qi * kstep, dk = desc_k + ks * kstep;
                const uint32_t d = tmem_base + buf * 128;
                for (uint32_t k0 = 0, off = 0; k0 < ksteps; k0 += 4, off += TILE_CHUNK >> 4) {
#pragma unroll
                    for (uint32_t k = 0; k < 4; ++k)
                        if (k0 + k < ksteps) umma_bf16(d, dq + off + 2 * k, dk + off + 2 * k, idesc_s, (k0 | k) != 0);
                }
                umma_commit(bar_s + 8 * buf);
                if (qi == NQ - 1) {
                    umma_commit(bar_k_empty + 8 * ks);
                    if (++ks == p.kstages) ks = 0, kphase ^= 1;
                }
                return true;
            };
            bool ok = mbar_wait(bar_q, 0, s_abort, p.status) && scores(0) && (items < 2 || scores(1));
            for (uint32_t i = 0; i < items && ok; ++i) {
                const uint32_t qi = NQ == 2 ? i & 1u : 0u, buf = i & 1u, phase = (i >> 1) & 1;
                if (qi == 0) ok = mbar_wait(bar_v_full + 8 * vs, vphase, s_abort, p.status);
                ok = ok && mbar_wait(bar_p + 8 * buf, phase, s_abort, p.status);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (!alias && i + 2 < items) ok = scores(i + 2);
                if (!ok) break;
                const uint32_t tmem_p = tmem_base + (alias ? buf * 128 : 384 + buf * 64), d = tmem_o + qi * p.ostride, gap = alias ? 32 : 0;
                const uint64_t dv = desc_v + vs * vstep;
#pragma unroll
                for (uint32_t k = 0; k < 8; ++k) umma_bf16_ts(d, tmem_p + k * 8 + (k >= 4 ? gap : 0), dv + 128 * k, idesc_o, k != 0 || i >= NQ);
                umma_commit(bar_pv + 8 * buf);
                if (qi == NQ - 1) {
                    umma_commit(bar_v_empty + 8 * vs);
                    if (++vs == p.vstages) vs = 0, vphase ^= 1;
                }
                if (alias && i + 2 < items) ok = mbar_wait(bar_pv + 8 * buf, phase, s_abort, p.status) && scores(i + 2);
            }
            if (ok) umma_commit(bar_o);
        }
    } else {
        // ---------------- weights (TMEM lane quarter = warp % 4), then the output ----------------
        const uint32_t quarter = warp & 3u, wg = (warp - 2) >> 2, buf = wg & 1u, half = wg >> 1, tr = quarter * 32 + lane;
        const uint32_t first = row0 + (NQ == 2 ? buf * p.rpt : 0), row = first + tr / p.group, head = g * p.group + tr % p.group;
        const bool valid = tr < p.rpt * p.group && row < a.rows;
        const uint32_t at = pos + min(row, a.rows - 1);
        const uint32_t lanes = (quarter * 32u) << 16;
        const float c2 = a.softcap * LOG2E;
        const float c0 = a.scale * query_factor(at, a.temp_coef, a.temp_every) / a.softcap, c1 = 2.0f * LOG2E * c0;
        const float small = TANH_SMALL / fabsf(c0);      // scores up to here take the short form
        const uint64_t c0_2 = pair(c0, c0), c2_2 = pair(c2, c2);
        float sum = 0.0f;
        bool ok = true;
        for (uint32_t i = buf; i < items; i += 2) {
            const uint32_t t = i / NQ;
            ok = mbar_wait(bar_s + 8 * buf, (i >> 1) & 1, s_abort, p.status) && !*s_abort;
            ok = __all_sync(0xffffffffu, ok);   // the TMEM accesses below are whole-warp instructions
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t tmem_s = tmem_base + buf * 128 + half * 64 + lanes;
            const uint32_t tmem_p = (p.alias ? tmem_s : tmem_base + 384 + buf * 64 + half * 32 + lanes);
            const uint32_t key0 = t * 128 + half * 64;
            // every key of the tile is at or before the first row's position: no mask
            const bool whole = t * 128 + 127 <= pos + first;
            uint32_t v[2][32];
            tmem_ld32_request(tmem_s, v[0]);
            tmem_ld32_request(tmem_s + 32, v[1]);
            tmem_ld32_wait(v[0]);
            tmem_ld32_pass(v[1]);
            float most[4] = {};
#pragma unroll
            for (int x = 0; x < 32; ++x) most[x & 3] = fmaxf(most[x & 3], fmaxf(fabsf(__uint_as_float(v[0][x])), fabsf(__uint_as_float(v[1][x]))));
            const bool short_form = __all_sync(0xffffffffu, fmaxf(fmaxf(most[0], most[1]), fmaxf(most[2], most[3])) <= small);
            if (!p.alias && i >= 2) {   // the product of item i - 2 reads this P buffer
                ok = mbar_wait(bar_pv + 8 * buf, ((i >> 1) - 1) & 1, s_abort, p.status);
                ok = __all_sync(0xffffffffu, ok);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            }
            if (short_form) {
                uint64_t s2[2] = {0, 0};
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    uint32_t w[16];
#pragma unroll
                    for (int x = 0; x < 16; ++x) {
                        float2 e = capped_exp_small(pair(__uint_as_float(v[c][2 * x]), __uint_as_float(v[c][2 * x + 1])), c0_2, c2_2);
                        if (!whole) {
                            e.x = key0 + c * 32 + 2 * x <= at ? e.x : 0.0f;
                            e.y = key0 + c * 32 + 2 * x + 1 <= at ? e.y : 0.0f;
                        }
                        s2[x & 1] = fma2(pair(e.x, e.y), pair(1.0f, 1.0f), s2[x & 1]);
                        w[x] = pack_bf16(e.x, e.y);
                    }
                    tmem_st16(tmem_p + c * 16, w);   // aliased: over scores this warp has already read
                }
                const float2 s1 = unpair(s2[0]), s3 = unpair(s2[1]);
                sum += (s1.x + s1.y) + (s3.x + s3.y);
            } else {
#pragma unroll 1
                for (uint32_t c = 0; c < 4; ++c) {   // compact: the scores are fetched again, sixteen at a time
                    uint32_t u[16], w[8];
                    tmem_ld16(tmem_s + c * 16, u);
                    float part = 0.0f;
#pragma unroll
                    for (int x = 0; x < 8; ++x) {
                        const uint32_t key = key0 + c * 16 + 2 * x;
                        const float lo = key <= at ? capped_exp(__uint_as_float(u[2 * x]), c1, c2) : 0.0f;
                        const float hi = key + 1 <= at ? capped_exp(__uint_as_float(u[2 * x + 1]), c1, c2) : 0.0f;
                        part += lo + hi;
                        w[x] = pack_bf16(lo, hi);
                    }
                    sum += part;
                    tmem_st8(tmem_p + c * 8, w);
                }
            }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar_p + 8 * buf) : "memory");
        }
        s_sum[wg * 128 + tr] = sum;
        asm volatile("bar.sync 1, 512;" ::: "memory");
        ok = mbar_wait(bar_o, 0, s_abort, p.status) && !*s_abort && !(*reinterpret_cast<volatile uint32_t*>(p.status) & 4u);
        // the loads below are whole-warp instructions: the warp takes one decision
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const float total = NQ == 2 ? s_sum[buf * 128 + tr] + s_sum[(buf + 2) * 128 + tr] : (s_sum[tr] + s_sum[128 + tr]) + (s_sum[256 + tr] + s_sum[384 + tr]);
            const float denom = total + (a.sink && valid ? ex2(a.sink[head] * LOG2E) : 0.0f);
            const float inv = __fdiv_rn(1.0f, denom);
            __nv_bfloat16* out = (__nv_bfloat16*)a.out + (uint64_t)row * a.ld + head * a.vdim;
            for (uint32_t c = NQ == 2 ? half : wg; c < a.vdim / 16; c += NQ == 2 ? 2 : 4) {
                uint32_t v[16], w[8];
                tmem_ld16(tmem_o + (NQ == 2 ? buf * p.ostride : 0) + lanes + c * 16, v);
#pragma unroll
                for (int x = 0; x < 8; ++x) w[x] = pack_bf16(__uint_as_float(v[2 * x]) * inv, __uint_as_float(v[2 * x + 1]) * inv);
                if (valid) {
                    reinterpret_cast<uint4*>(out + c * 16)[0] = make_uint4(w[0], w[1], w[2], w[3]);
                    reinterpret_cast<uint4*>(out + c * 16)[1] = make_uint4(w[4], w[5], w[6], w[7]);
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

template <int NQ>
int32_t launch_tile(holo_b200_ctx* ctx, const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const TileParams& p, uint32_t ctas, uint32_t smem) {
    static thread_local int configured_device = -1;
    if (configured_device != ctx->device) {
        HOLO_CUDA(cudaFuncSetAttribute(causal_attention_tile_kernel<NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, ctx->smem_optin));
        configured_device = ctx->device;
    }
    HOLO_CUDA(holo_launch_kernel(ctx, causal_attention_tile_kernel<NQ>, dim3(p.a.kv_heads, ctas), dim3(TILE_THREADS), smem, 1, mq, mk, mv, p));
    ctx->launches++;
    return HOLO_OK;
}

// Launches the tile kernel, or returns with *taken false when the shape does not suit it.
int32_t try_tile(holo_b200_ctx* ctx, const HoloCausalArgs& a, bool* taken) {
    *taken = false;
    TileParams p;
    p.a = a;
    p.status = ctx->dev_status;
    p.group = a.heads / a.kv_heads;
    if (a.dim > 256 || a.vdim > 256 || p.group > 128 || a.ld % 8 != 0 || encode_tiled_fn() == nullptr) return HOLO_OK;
    p.rpt = 128 / p.group;
    p.qchunks = (a.dim + 63) / 64;
    p.vchunks = (a.vdim + 63) / 64;
    const uint32_t extra = 256 + 2048 + 1024, limit = (uint32_t)ctx->smem_optin;   // barriers, row sums, alignment slack
    auto bytes = [&](uint32_t nq, uint32_t ks, uint32_t vs) { return ((nq + ks) * p.qchunks + vs * p.vchunks) * TILE_CHUNK + extra; };
    const uint32_t qtiles = (a.rows + p.rpt - 1) / p.rpt;
    if (qtiles > 65535) return HOLO_OK;
    p.kstages = p.vstages = 2;
    bool two = a.vdim <= 128 && bytes(2, 2, 2) <= limit && ((qtiles + 1) / 2) * a.kv_heads >= (uint32_t)ctx->sm_count;
    if (const char* e = getenv("HOLO_CAUSAL_QUERY_TILES")) two = atoi(e) == 2 && a.vdim <= 128 && bytes(2, 2, 2) <= limit;
    if (two) {
        p.ostride = a.vdim <= 64 ? 64 : 128;
        p.alias = a.vdim > 64 ? 1 : 0;
    } else {
        p.ostride = 0;
        p.alias = a.vdim > 128 ? 1 : 0;
        if (bytes(1, 2, 2) > limit) p.kstages = 1;
        if (bytes(1, p.kstages, 2) > limit) {
            p.vstages = 1;
            p.alias = 1;   // K(t + 2) is loaded after V(t + 1): with one V stage tile t's product must come before S(t + 2)
        }
    }
    const uint32_t smem = bytes(two ? 2 : 1, p.kstages, p.vstages);
    if (smem > limit) return HOLO_OK;
    CUtensorMap mq, mk, mv;
    {   // q as [rows][heads][dim]: a box is 64 columns of the group's heads over rpt rows
        cuuint64_t dims[3] = {a.dim, a.heads, a.rows};
        cuuint64_t strides[2] = {(cuuint64_t)a.dim * 2, (cuuint64_t)a.heads * a.dim * 2};
        cuuint32_t box[3] = {64, p.group, p.rpt};
        cuuint32_t es[3] = {1, 1, 1};
        const CUresult r = encode_tiled_fn()(&mq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(a.q), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
        if (r != CUDA_SUCCESS) return holo_fail(HOLO_ERR_DISPATCH, "dispatch failed: cuTensorMapEncodeTiled (attention) returned %d", (int)r);
    }
    HOLO_TRY(make_map_2d(&mk, a.k, (uint64_t)a.kv_heads * a.dim, a.cache_rows, 64, 128));
    HOLO_TRY(make_map_2d(&mv, a.v, (uint64_t)a.kv_heads * a.vdim, a.cache_rows, 64, 128));
    *taken = true;
    return two ? launch_tile<2>(ctx, mq, mk, mv, p, (qtiles + 1) / 2, smem) : launch_tile<1>(ctx, mq, mk, mv, p, qtiles, smem);
}

}  // namespace

int32_t holo_launch_causal_attention(holo_b200_ctx* ctx, const HoloCausalArgs& a) {
    const bool capped16 = a.dtype == HOLO_DTYPE_BF16 && a.softcap > 0.0f && a.softcap <= CAP_LIMIT && a.dim % 16 == 0 && a.vdim % 16 == 0 &&
                          a.ld % 2 == 0 && (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.out) & 15u) == 0 &&
                          !getenv("HOLO_CAUSAL_GENERIC");
    if (capped16) {
        bool taken = false;
        if (a.rows * (a.heads / a.kv_heads) <= 64) HOLO_TRY(try_split(ctx, a, &taken));
        if (!taken) HOLO_TRY(try_tile(ctx, a, &taken));
        if (taken) return HOLO_OK;
    }
    return launch_generic(ctx, a);
}
