// Causal attention of new rows over a cache that already holds them (the CausalAttention call): row i of the step is
// at position p = *pos + i and sees cache rows 0 .. p. Optional score cap (softcap * tanh(s / softcap)), one learned
// sink per head in the softmax denominator, and a query factor that grows with the logarithm of the position.
#include "common.h"

#include <cuda_bf16.h>
#include <stdlib.h>

namespace {

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

}  // namespace

int32_t holo_launch_causal_attention(holo_b200_ctx* ctx, const HoloCausalArgs& a) {
    return launch_generic(ctx, a);
}
