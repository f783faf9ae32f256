// Routed experts (the MoePlan and MoeCombine calls): from router logits to the row tiles the grouped Linear products work on,
// and from the experts' outputs back to the residual stream.
#include "common.h"

#include <cuda_bf16.h>

namespace {

constexpr int PLAN_THREADS = 1024, ROUTE_WARPS = 8, MAX_EXPERTS = 1024;

// One warp, one row: the `top` largest logits (ties to the lower expert) and the softmax over them. The experts' numbers go to
// `chosen`, in descending order of their logits.
template <int PL>
__device__ __forceinline__ void route_row(const HoloMoePlanArgs& a, uint32_t row, uint32_t lane, int32_t* chosen, float* weight) {
    float v[PL];
#pragma unroll
    for (int i = 0; i < PL; ++i) {
        const uint32_t e = lane + 32 * i;
        v[i] = e < a.experts ? a.logits[(uint64_t)row * a.ld_logits + e] + (a.bias ? a.bias[e] : 0.0f) : -INFINITY;
    }
    float first = 0.0f, sum = 0.0f, mine = 0.0f;
    for (uint32_t t = 0; t < a.top; ++t) {
        float best = -INFINITY;
        uint32_t at = 0xffffffffu;
#pragma unroll
        for (int i = 0; i < PL; ++i)
            if (v[i] > best || (at == 0xffffffffu && lane + 32 * i < a.experts && v[i] == best)) {
                best = v[i];
                at = lane + 32 * i;
            }
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const uint32_t oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (ob > best || (ob == best && oa < at)) {
                best = ob;
                at = oa;
            }
        }
        if (at >= a.experts) at = 0;       // only when logits are not numbers: stay within the tables
        if (t == 0) first = best;
        const float e = expf(best - first);
        sum += e;
        if (lane == t) {
            mine = e;
            chosen[(uint64_t)row * a.top + t] = (int32_t)at;
        }
#pragma unroll
        for (int i = 0; i < PL; ++i)
            if (at == lane + 32 * i) v[i] = -INFINITY;
    }
    if (lane < a.top) weight[(uint64_t)row * a.top + lane] = mine / sum;
}

template <int PL>
__global__ void __launch_bounds__(ROUTE_WARPS * 32)
moe_route_kernel(const HoloMoePlanArgs a) {
    holo_pdl_trigger();
    holo_pdl_wait();
    const uint32_t row = blockIdx.x * ROUTE_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row < min(a.rows, a.step[1])) route_row<PL>(a, row, lane, a.place, a.weight);
}

// Inclusive sums of n <= PLAN_THREADS values in shared memory.
__device__ __forceinline__ void scan(uint32_t* s, uint32_t n) {
    for (uint32_t d = 1; d < n; d <<= 1) {
        const uint32_t v = threadIdx.x < n && threadIdx.x >= d ? s[threadIdx.x - d] : 0u;
        __syncthreads();
        if (threadIdx.x < n) s[threadIdx.x] += v;
        __syncthreads();
    }
}

// One CTA. Few rows (at most one tile's worth): routes them, then one tile per expert in use. PL = 0: many rows, already
// routed (`place` holds the experts): counts, tiles, and a place for every pair.
template <int PL>
__global__ void __launch_bounds__(PLAN_THREADS)
moe_plan_kernel(const HoloMoePlanArgs a) {
    __shared__ uint32_t s_count[MAX_EXPERTS], s_end[MAX_EXPERTS];
    holo_pdl_trigger();
    const uint32_t tid = threadIdx.x;
    for (uint32_t e = tid; e < a.experts; e += PLAN_THREADS) s_count[e] = 0;
    holo_pdl_wait();
    const uint32_t rows = min(a.rows, a.step[1]), pairs = rows * a.top;
    if (PL > 0)
        for (uint32_t row = tid >> 5; row < rows; row += PLAN_THREADS / 32) route_row<PL == 0 ? 1 : PL>(a, row, tid & 31, a.place, a.weight);
    __syncthreads();
    for (uint32_t i = tid; i < pairs; i += PLAN_THREADS) atomicAdd(&s_count[a.place[i]], 1u);
    __syncthreads();
    uint32_t mine = 0;
    if (tid < a.experts) {
        mine = PL > 0 ? (s_count[tid] ? 1u : 0u) : (s_count[tid] + a.tile_rows - 1) / a.tile_rows;
        s_end[tid] = mine;
    }
    __syncthreads();
    scan(s_end, a.experts);
    if (tid < a.experts) {
        const uint32_t begin = s_end[tid] - mine;
        for (uint32_t t = 0; t < mine && begin + t < a.max_tiles; ++t) a.tiles[1 + begin + t] = (int32_t)tid;
        s_count[tid] = begin * a.tile_rows;      // where the expert's next pair goes
        if (tid == a.experts - 1) a.tiles[0] = (int32_t)min(s_end[tid], a.max_tiles);
    }
    if (PL == 0)
        for (uint32_t i = tid; i < a.max_tiles * a.tile_rows; i += PLAN_THREADS) a.source[i] = 0;
    __syncthreads();
    for (uint32_t i = tid; i < pairs; i += PLAN_THREADS) {
        const uint32_t e = (uint32_t)a.place[i], row = i / a.top;
        const uint32_t at = PL > 0 ? s_count[e] + row : atomicAdd(&s_count[e], 1u);
        a.place[i] = (int32_t)at;
        if (PL == 0) a.source[at] = (int32_t)row;
    }
}

// One thread: V columns of one row.
template <typename T, int V>
__global__ void __launch_bounds__(128)
moe_combine_kernel(float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ weight, const int32_t* __restrict__ place,
                   const uint32_t* __restrict__ step, uint32_t width, uint32_t top, uint32_t ld) {
    holo_pdl_trigger();
    holo_pdl_wait();
    const uint32_t row = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * V;
    if (row >= step[1] || c >= width) return;
    float acc[V];
    float* dst = x + (uint64_t)row * width + c;
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] = dst[i];
    for (uint32_t t = 0; t < top; ++t) {
        const float w = weight[(uint64_t)row * top + t];
        const T* src = y + (uint64_t)place[(uint64_t)row * top + t] * ld + c;
        T v[V];
        if constexpr (V * sizeof(T) == 16) *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(src);
        else if constexpr (V * sizeof(T) == 8) *reinterpret_cast<uint2*>(v) = *reinterpret_cast<const uint2*>(src);
        else
#pragma unroll
            for (int i = 0; i < V; ++i) v[i] = src[i];
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(w, (float)v[i], acc[i]);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) dst[i] = acc[i];
}

template <int PL>
int32_t launch_plan(holo_b200_ctx* ctx, const HoloMoePlanArgs& a) {
    if (a.rows <= a.tile_rows) {
        HOLO_CUDA(holo_launch_kernel(ctx, moe_plan_kernel<PL>, dim3(1), dim3(PLAN_THREADS), 0, 1, a));
        ctx->launches++;
        return HOLO_OK;
    }
    HOLO_CUDA(holo_launch_kernel(ctx, moe_route_kernel<PL>, dim3((a.rows + ROUTE_WARPS - 1) / ROUTE_WARPS), dim3(ROUTE_WARPS * 32), 0, 1, a));
    HOLO_CUDA(holo_launch_kernel(ctx, moe_plan_kernel<0>, dim3(1), dim3(PLAN_THREADS), 0, 1, a));
    ctx->launches += 2;
    return HOLO_OK;
}

template <typename T>
int32_t launch_combine(holo_b200_ctx* ctx, float* x, const void* y, const float* weight, const int32_t* place, const uint32_t* step, uint32_t rows,
                       uint32_t width, uint32_t top, uint32_t ld) {
    if (rows > 65535) return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: moe_combine rows %u", rows);
    const bool vec = width % 4 == 0 && ld % 4 == 0 && (((uintptr_t)x | (uintptr_t)y) & 15u) == 0;
    const uint32_t per = 128 * (vec ? 4 : 1);
    const dim3 grid((width + per - 1) / per, rows);
    if (vec) HOLO_CUDA(holo_launch_kernel(ctx, moe_combine_kernel<T, 4>, grid, dim3(128), 0, 1, x, (const T*)y, weight, place, step, width, top, ld));
    else HOLO_CUDA(holo_launch_kernel(ctx, moe_combine_kernel<T, 1>, grid, dim3(128), 0, 1, x, (const T*)y, weight, place, step, width, top, ld));
    ctx->launches++;
    return HOLO_OK;
}

}  // namespace

int32_t holo_launch_moe_plan(holo_b200_ctx* ctx, const HoloMoePlanArgs& a) {
    if (a.experts <= 64) return launch_plan<2>(ctx, a);
    if (a.experts <= 256) return launch_plan<8>(ctx, a);
    return launch_plan<32>(ctx, a);
}

int32_t holo_launch_moe_combine(holo_b200_ctx* ctx, float* x, const void* y, const float* weight, const int32_t* place, const uint32_t* step, uint32_t rows,
                                uint32_t width, uint32_t top, uint32_t ld, uint32_t, uint8_t dtype) {
    return dtype == HOLO_DTYPE_F32 ? launch_combine<float>(ctx, x, y, weight, place, step, rows, width, top, ld)
                                   : launch_combine<__nv_bfloat16>(ctx, x, y, weight, place, step, rows, width, top, ld);
}
