// Retention (linear attention with one fixed decay per head): S = decay S + k v^T, o = scale S^T q, every head's o divided by its
// root mean square and multiplied by the gate. The state is f32 and stays in place between steps.
#include "common.h"

#include <cuda_bf16.h>
#include <stdlib.h>

#include <algorithm>

namespace {

__device__ __forceinline__ void store_out(float* out, uint64_t i, float v) { out[i] = v; }
__device__ __forceinline__ void store_out(__nv_bfloat16* out, uint64_t i, float v) { out[i] = __float2bfloat16_rn(v); }

// ---- general form: one CTA per head, token by token ---------------------------------------------------------------------
// 64 value columns at a time, four threads per column over the key dimensions. The state sits in shared memory where it fits.
constexpr int SEQ_THREADS = 256, SEQ_COLS = 64, SEQ_GROUPS = SEQ_THREADS / SEQ_COLS;
template <typename T, bool HELD>
__global__ void __launch_bounds__(SEQ_THREADS)
retention_sequence_kernel(const HoloRetentionArgs a) {
    extern __shared__ float s_mem[];   // q [dim], k [dim], o [vdim], parts [4][64], sums [8], state [dim][vdim] when HELD
    const uint32_t h = blockIdx.x, tid = threadIdx.x, col = tid % SEQ_COLS, group = tid / SEQ_COLS;
    float *s_q = s_mem, *s_k = s_q + a.dim, *s_o = s_k + a.dim, *s_part = s_o + a.vdim, *s_sum = s_part + SEQ_THREADS;
    holo_pdl_trigger();
    holo_pdl_wait();
    const uint32_t count = min(a.rows, a.step[1]);
    const bool fresh = a.step[0] == 0;
    float* home = a.state + (uint64_t)h * a.dim * a.vdim;
    float* state = HELD ? s_sum + 8 : home;
    const uint32_t cells = a.dim * a.vdim;
    if (HELD || fresh)
        for (uint32_t i = tid; i < cells; i += SEQ_THREADS) state[i] = fresh ? 0.0f : home[i];
    const float decay = a.decay[h];
    for (uint32_t row = 0; row < count; ++row) {
        __syncthreads();
        for (uint32_t i = tid; i < a.dim; i += SEQ_THREADS) {
            s_q[i] = (float)((const T*)a.q)[(uint64_t)row * a.q_ld + (uint64_t)h * a.dim + i];
            s_k[i] = (float)((const T*)a.k)[(uint64_t)row * a.k_ld + (uint64_t)h * a.dim + i];
        }
        __syncthreads();
        for (uint32_t c0 = 0; c0 < a.vdim; c0 += SEQ_COLS) {
            const uint32_t c = c0 + col;
            float acc = 0.0f;
            if (c < a.vdim) {
                const float v = (float)((const T*)a.v)[(uint64_t)row * a.v_ld + (uint64_t)h * a.vdim + c];
                for (uint32_t d = group; d < a.dim; d += SEQ_GROUPS) {
                    const float s = fmaf(decay, state[d * a.vdim + c], s_k[d] * v);
                    state[d * a.vdim + c] = s;
                    acc = fmaf(s, s_q[d], acc);
                }
            }
            s_part[tid] = acc;
            __syncthreads();
            if (group == 0 && c < a.vdim) s_o[c] = a.scale * ((s_part[col] + s_part[SEQ_COLS + col]) + (s_part[2 * SEQ_COLS + col] + s_part[3 * SEQ_COLS + col]));
            __syncthreads();
        }
        float sq = 0.0f;
        for (uint32_t c = tid; c < a.vmean; c += SEQ_THREADS) sq = fmaf(s_o[c], s_o[c], sq);
        for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
        if ((tid & 31u) == 0) s_sum[tid >> 5] = sq;
        __syncthreads();
        float total = 0.0f;
#pragma unroll
        for (int w = 0; w < SEQ_THREADS / 32; ++w) total += s_sum[w];
        const float inv = 1.0f / sqrtf(total / (float)a.vmean + a.eps);
        for (uint32_t c = tid; c < a.vdim; c += SEQ_THREADS)
            store_out((T*)a.out, (uint64_t)row * a.ld + (uint64_t)h * a.vdim + c,
                      s_o[c] * inv * (float)((const T*)a.gate)[(uint64_t)row * a.gate_ld + (uint64_t)h * a.vdim + c]);
    }
    if (HELD) {
        __syncthreads();
        for (uint32_t i = tid; i < cells; i += SEQ_THREADS) home[i] = state[i];
    }
}

template <typename T, bool HELD>
int32_t launch_sequence_as(holo_b200_ctx* ctx, const HoloRetentionArgs& a, size_t smem) {
    static thread_local int configured_device = -1;
    if (configured_device != ctx->device) {
        HOLO_CUDA(cudaFuncSetAttribute(retention_sequence_kernel<T, HELD>, cudaFuncAttributeMaxDynamicSharedMemorySize, ctx->smem_optin - 1024));
        configured_device = ctx->device;
    }
    HOLO_CUDA(holo_launch_kernel(ctx, retention_sequence_kernel<T, HELD>, dim3(a.heads), dim3(SEQ_THREADS), smem, 1, a));
    ctx->launches++;
    return HOLO_OK;
}
template <typename T>
int32_t launch_sequence(holo_b200_ctx* ctx, const HoloRetentionArgs& a) {
    const size_t small = (2 * a.dim + a.vdim + SEQ_THREADS + 8) * sizeof(float), state = (size_t)a.dim * a.vdim * sizeof(float);
    return small + state <= (size_t)ctx->smem_optin - 1024 ? launch_sequence_as<T, true>(ctx, a, small + state) : launch_sequence_as<T, false>(ctx, a, small);
}

}  // namespace

int32_t holo_launch_retention(holo_b200_ctx* ctx, const HoloRetentionArgs& a) {
    return a.dtype == HOLO_DTYPE_F32 ? launch_sequence<float>(ctx, a) : launch_sequence<__nv_bfloat16>(ctx, a);
}
