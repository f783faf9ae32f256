// Retention (linear attention with one fixed decay per head): S = decay S + k v^T, o = scale S^T q, every head's o divided by its
// root mean square and multiplied by the gate. The state is f32 and stays in place between steps.
//
//   retention_tile_kernel       bf16, many rows, heads of 128 or 256 key dimensions: chunks of 128 tokens on tcgen05, the state
//                               in tensor memory from the first chunk to the last
//   retention_chunk_kernel      bf16, several rows, other heads: the same chunks on mma.sync, the state in registers
//   retention_token_kernel      one row
//   retention_sequence_kernel   everything else: token by token, one CTA per head
//
// In all but the last the CTAs of a head have a slice of the value columns each; for one row and for other heads they are a
// cluster and exchange the sums of squares.
#include "attention_tile.cuh"

#include <algorithm>

namespace {

__device__ __forceinline__ void store_out(float* out, uint64_t i, float v) { out[i] = v; }
__device__ __forceinline__ void store_out(__nv_bfloat16* out, uint64_t i, float v) { out[i] = __float2bfloat16_rn(v); }

// ---- value slices of a head in a cluster ----------------------------------------------------------------------------------
constexpr uint32_t MAX_SLICES = 8;
__device__ __forceinline__ void store_remote(uint32_t addr, uint32_t rank, float v) {
    uint32_t r;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(r), "f"(v) : "memory");
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

// ---- one row --------------------------------------------------------------------------------------------------------------
// Grid (slices, heads). A thread owns four columns of the slice and every GROUPS-th key dimension; the state is read, advanced
// and written once.
constexpr int TOK_THREADS = 256;
template <typename T, int HELD>   // a thread's share of the key dimensions, requested at once
__global__ void __launch_bounds__(TOK_THREADS)
retention_token_kernel(const HoloRetentionArgs a, uint32_t width) {
    extern __shared__ __align__(16) float t_mem[];      // parts [groups][width], o [width]
    __shared__ float s_sq[MAX_SLICES], s_part[TOK_THREADS / 32];
    const uint32_t slice = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, vecs = width / 4, groups = TOK_THREADS / vecs;
    float *s_parts = t_mem, *s_o = s_parts + groups * width;
    const uint32_t cv = tid % vecs, group = tid / vecs, e0 = slice * width + cv * 4;
    float* state = a.state + (uint64_t)h * a.dim * a.vdim + e0;
    const T *q = (const T*)a.q + (uint64_t)h * a.dim, *k = (const T*)a.k + (uint64_t)h * a.dim;
    holo_pdl_trigger();
    cluster_arrive();       // everyone has started: their shared memory may be written
    holo_pdl_wait();
    cluster_wait();
    float4 s[HELD];
    float qk[HELD][2], v[4] = {};
#pragma unroll
    for (int i = 0; i < HELD; ++i) {
        const uint32_t d = group + groups * i;
        const bool mine = group < groups && d < a.dim;
        s[i] = mine ? *reinterpret_cast<const float4*>(state + (uint64_t)d * a.vdim) : make_float4(0.f, 0.f, 0.f, 0.f);
        qk[i][0] = mine ? (float)q[d] : 0.0f;
        qk[i][1] = mine ? (float)k[d] : 0.0f;
    }
    if (group < groups)
#pragma unroll
        for (int i = 0; i < 4; ++i) v[i] = (float)((const T*)a.v)[(uint64_t)h * a.vdim + e0 + i];
    float gate = 0.0f;      // of the column this thread finishes (width is at most the CTA's threads)
    if (tid < width) gate = (float)((const T*)a.gate)[(uint64_t)h * a.vdim + slice * width + tid];
    const bool run = a.step[1] != 0;     // the same for every thread of the cluster
    const float decay = a.step[0] == 0 ? 0.0f : a.decay[h];
    const bool fresh = a.step[0] == 0;
    if (run) {
        float acc[4] = {};
#pragma unroll
        for (int i = 0; i < HELD; ++i) {
            const uint32_t d = group + groups * i;
            if (fresh) s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            s[i].x = fmaf(decay, s[i].x, qk[i][1] * v[0]); s[i].y = fmaf(decay, s[i].y, qk[i][1] * v[1]);
            s[i].z = fmaf(decay, s[i].z, qk[i][1] * v[2]); s[i].w = fmaf(decay, s[i].w, qk[i][1] * v[3]);
            if (group < groups && d < a.dim) *reinterpret_cast<float4*>(state + (uint64_t)d * a.vdim) = s[i];
            acc[0] = fmaf(s[i].x, qk[i][0], acc[0]); acc[1] = fmaf(s[i].y, qk[i][0], acc[1]);
            acc[2] = fmaf(s[i].z, qk[i][0], acc[2]); acc[3] = fmaf(s[i].w, qk[i][0], acc[3]);
        }
        if (group < groups) *reinterpret_cast<float4*>(s_parts + group * width + cv * 4) = make_float4(acc[0], acc[1], acc[2], acc[3]);
        __syncthreads();
        float sq = 0.0f;
        if (tid < width) {
            float o = 0.0f;
            for (uint32_t g = 0; g < groups; ++g) o += s_parts[g * width + tid];
            o *= a.scale;
            s_o[tid] = o;
            if (slice * width + tid < a.vmean) sq = o * o;
        }
        for (int o = 16; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
        if ((tid & 31u) == 0) s_part[tid >> 5] = sq;
        __syncthreads();
        if (tid < gridDim.x) {
            float total = 0.0f;
#pragma unroll
            for (int w = 0; w < TOK_THREADS / 32; ++w) total += s_part[w];
            store_remote(smem_u32(&s_sq[slice]), tid, total);
        }
    }
    __syncwarp();
    cluster_arrive();
    cluster_wait();
    if (!run || tid >= width) return;
    float total = 0.0f;
    for (uint32_t i = 0; i < gridDim.x; ++i) total += s_sq[i];
    const float inv = 1.0f / sqrtf(total / (float)a.vmean + a.eps);
    store_out((T*)a.out, (uint64_t)h * a.vdim + slice * width + tid, s_o[tid] * inv * gate);
}

template <typename T, int HELD>
int32_t launch_token_as(holo_b200_ctx* ctx, const HoloRetentionArgs& a, uint32_t slices, uint32_t width) {
    const size_t smem = ((TOK_THREADS / (width / 4)) * width + width) * sizeof(float);    // at most 5 KiB
    HOLO_CUDA(holo_launch_kernel_cluster(ctx, retention_token_kernel<T, HELD>, dim3(slices, a.heads), dim3(TOK_THREADS), smem, slices, 1u, a, width));
    ctx->launches++;
    return HOLO_OK;
}
// Launches the one-row kernel, or returns with *taken false when the shape does not suit it.
template <typename T>
int32_t try_token(holo_b200_ctx* ctx, const HoloRetentionArgs& a, bool* taken) {
    *taken = false;
    uint32_t slices = MAX_SLICES;
    while (slices > 1 && (a.vdim % (4 * slices) != 0 || a.vdim / slices < 16)) slices /= 2;
    const uint32_t width = a.vdim / slices;
    if (a.vdim % 4 || width > TOK_THREADS) return HOLO_OK;
    const uint32_t groups = TOK_THREADS / (width / 4), share = (a.dim + groups - 1) / groups;
    if (share > 32) return HOLO_OK;
    *taken = true;
    if (share <= 4) return launch_token_as<T, 4>(ctx, a, slices, width);
    if (share <= 8) return launch_token_as<T, 8>(ctx, a, slices, width);
    if (share <= 16) return launch_token_as<T, 16>(ctx, a, slices, width);
    return launch_token_as<T, 32>(ctx, a, slices, width);
}

// ---- several rows -----------------------------------------------------------------------------------------------------------
// Grid (slices, heads), a slice has W value columns. Per chunk of up to 128 tokens (64 where those do not fit), with p(n) = decay^n, L tokens in the chunk:
//   o_i  = p(i + 1) S^T q_i + sum_{j <= i} p(i - j) (q_i . k_j) v_j          warp w: tokens 16 w .. 16 w + 15
//   S    = p(L) S + sum_j p(L - 1 - j) k_j v_j^T                             warp w: key dimensions 8 (w + 8 n) .. + 7
// S is held transposed in the accumulator registers of the second product. What enters a product besides q, k and v (S, the
// decayed scores, the decayed values) is f32 and goes in as the sum of two bf16 values, so that it keeps 16 significant bits;
// everything is added up in f32.
constexpr int CHUNK_WARPS = 8;

__device__ __forceinline__ void split_bf16(float lo, float hi, uint32_t& big, uint32_t& small) {
    big = pack_bf16(lo, hi);
    const __nv_bfloat162 b = *reinterpret_cast<const __nv_bfloat162*>(&big);
    small = pack_bf16(lo - __low2float(b), hi - __high2float(b));
}

template <int W, int CHUNK>
struct ChunkSmem {
    static constexpr uint32_t VP = W * 2 + 16;      // row pitches: an odd number of 16-byte units
    uint32_t qk, stage, stages, sbig, vbig, power, sums, total;
    __host__ __device__ ChunkSmem(uint32_t dim, uint32_t nstages) {
        qk = dim * 2 + 16;
        stages = nstages;
        stage = CHUNK * (2 * qk + VP);               // q, k, v rows
        sbig = nstages * stage;                      // S^T as [W][dim], twice
        vbig = sbig + 2 * W * qk;                    // decayed values [CHUNK][W], twice
        power = vbig + 2 * CHUNK * VP;               // p(0) .. p(CHUNK)
        sums = power + (CHUNK + 4) * 4;              // sums of squares [2][MAX_SLICES][CHUNK]
        total = sums + 2 * MAX_SLICES * CHUNK * 4;
    }
};

template <int W, int NT, int CHUNK>   // dim <= 64 NT, CHUNK at most 16 tokens per warp
__global__ void __launch_bounds__(CHUNK_WARPS * 32)
retention_chunk_kernel(const HoloRetentionArgs a, uint32_t nstages) {
    extern __shared__ __align__(16) uint8_t sm[];
    constexpr int MT = W / 16, OT = W / 8;
    const ChunkSmem<W, CHUNK> s(a.dim, nstages);
    constexpr uint32_t VP = ChunkSmem<W, CHUNK>::VP;
    const uint32_t slice = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r0 = lane >> 2, c0 = (lane & 3) * 2;
    const uint32_t base = smem_u32(sm), ntiles = a.dim / 8, ksteps = a.dim / 16;
    float* s_power = reinterpret_cast<float*>(sm + s.power);
    float* s_sums = reinterpret_cast<float*>(sm + s.sums);
    holo_pdl_trigger();
    cluster_arrive();       // everyone has started: their shared memory may be written
    holo_pdl_wait();
    cluster_wait();
    const uint32_t count = min(a.rows, a.step[1]), chunks = (count + CHUNK - 1) / CHUNK;
    const bool fresh = a.step[0] == 0;
    if (chunks == 0) return;                         // the same for the whole cluster
    const float decay = a.decay[h];
    for (uint32_t i = tid; i <= CHUNK; i += blockDim.x) s_power[i] = i == 0 ? 1.0f : powf(decay, (float)i);
    const __nv_bfloat16* q = (const __nv_bfloat16*)a.q + (uint64_t)h * a.dim;
    const __nv_bfloat16* k = (const __nv_bfloat16*)a.k + (uint64_t)h * a.dim;
    const uint64_t col = (uint64_t)h * a.vdim + slice * W;
    const __nv_bfloat16* v = (const __nv_bfloat16*)a.v + col;

    auto load_chunk = [&](uint32_t chunk, uint32_t stage) {
        const uint32_t dst = base + stage * s.stage, vecs = a.dim / 8;
        for (uint32_t i = tid; i < CHUNK * vecs; i += blockDim.x) {
            const uint32_t r = i / vecs, c = i % vecs, row = chunk * CHUNK + r;
            const uint64_t from = min(row, count - 1);
            cp_async16(dst + r * s.qk + c * 16, q + from * a.q_ld + c * 8, row < count);
            cp_async16(dst + (CHUNK + r) * s.qk + c * 16, k + from * a.k_ld + c * 8, row < count);
        }
        for (uint32_t i = tid; i < CHUNK * (W / 8); i += blockDim.x) {
            const uint32_t r = i / (W / 8), c = i % (W / 8), row = chunk * CHUNK + r;
            cp_async16(dst + 2 * CHUNK * s.qk + r * VP + c * 16, v + (uint64_t)min(row, count - 1) * a.v_ld + c * 8, row < count);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_chunk(0, 0);
    // S^T: rows = value columns 16 m + r0 (+ 8), columns = key dimensions 8 (warp + 8 n) + c0 (+ 1)
    float st[NT][MT][4];
    float* home = a.state + (uint64_t)h * a.dim * a.vdim + slice * W;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t d = (warp + 8 * n) * 8 + c0 + (e & 1), x = 16 * m + r0 + 8 * (e >> 1);
                st[n][m][e] = !fresh && d < a.dim ? home[(uint64_t)d * a.vdim + x] : 0.0f;
            }
    for (uint32_t chunk = 0; chunk < chunks; ++chunk) {
        const uint32_t stage = s.stages == 2 ? chunk & 1u : 0u, tokens = min((uint32_t)CHUNK, count - chunk * CHUNK);
        const uint32_t s_q = base + stage * s.stage, s_k = s_q + CHUNK * s.qk, s_v = s_k + CHUNK * s.qk;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                             // the chunk is here; everyone is through with the one before
        if (s.stages == 2 && chunk + 1 < chunks) load_chunk(chunk + 1, stage ^ 1u);
        // S and the decayed values as pairs of bf16
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            if ((warp + 8 * n) < ntiles)
#pragma unroll
                for (int m = 0; m < MT; ++m)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        uint32_t big, small;
                        split_bf16(st[n][m][2 * e], st[n][m][2 * e + 1], big, small);
                        uint8_t* at = sm + s.sbig + (16 * m + r0 + 8 * e) * s.qk + ((warp + 8 * n) * 8 + c0) * 2;
                        *reinterpret_cast<uint32_t*>(at) = big;
                        *reinterpret_cast<uint32_t*>(at + W * s.qk) = small;
                    }
        }
        for (uint32_t i = tid; i < CHUNK * (W / 2); i += blockDim.x) {
            const uint32_t r = i / (W / 2), c = i % (W / 2);
            const float f = r < tokens ? s_power[tokens - 1 - r] : 0.0f;
            const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(sm + (s_v - base) + r * VP + c * 4);
            uint32_t big, small;
            split_bf16(__low2float(x) * f, __high2float(x) * f, big, small);
            uint8_t* at = sm + s.vbig + r * VP + c * 4;
            *reinterpret_cast<uint32_t*>(at) = big;
            *reinterpret_cast<uint32_t*>(at + CHUNK * VP) = small;
        }
        __syncthreads();
        // outputs of this warp's 16 tokens
        const uint32_t row = warp * 16;
        float o[OT][4];
#pragma unroll
        for (int n = 0; n < OT; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[n][e] = 0.0f;
        const bool active = row < tokens;
        if (active) {
            const uint32_t q_addr = s_q + (row + (lane & 15)) * s.qk + (lane >> 4) * 16;
            // operands whose rows are the output's columns: 16 rows, one step of 16
            const uint32_t n_off = ((lane & 7) + ((lane >> 4) << 3)) * s.qk + ((lane >> 3) & 1) * 16;
            for (uint32_t x = 0; x < ksteps; ++x) {
                uint32_t qa[4], sb[4];
                ldsm4(q_addr + x * 32, qa);
#pragma unroll
                for (int n = 0; n < OT; n += 2) {
                    const uint32_t at = base + s.sbig + n * 8 * s.qk + n_off + x * 32;
                    ldsm4(at, sb);
                    mma16816(o[n], qa, sb[0], sb[1]);
                    mma16816(o[n + 1], qa, sb[2], sb[3]);
                    ldsm4(at + W * s.qk, sb);
                    mma16816(o[n], qa, sb[0], sb[1]);
                    mma16816(o[n + 1], qa, sb[2], sb[3]);
                }
            }
            const float f0 = s_power[row + r0 + 1], f1 = s_power[row + r0 + 9];
#pragma unroll
            for (int n = 0; n < OT; ++n) {
                o[n][0] *= f0; o[n][1] *= f0;
                o[n][2] *= f1; o[n][3] *= f1;
            }
            const uint32_t v_off = ((lane & 7) + (((lane >> 3) & 1) << 3)) * VP + (lane >> 4) * 16;
            for (uint32_t j = 0; j <= warp; ++j) {
                float sc[2][4] = {};
                const uint32_t k_addr = s_k + j * 16 * s.qk + n_off;
#pragma unroll 4
                for (uint32_t x = 0; x < ksteps; ++x) {
                    uint32_t qa[4], kb[4];
                    ldsm4(q_addr + x * 32, qa);
                    ldsm4(k_addr + x * 32, kb);
                    mma16816(sc[0], qa, kb[0], kb[1]);
                    mma16816(sc[1], qa, kb[2], kb[3]);
                }
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int back = (int)(row + r0 + 8 * (e >> 1)) - (int)(j * 16 + n * 8 + c0 + (e & 1));
                        sc[n][e] = back >= 0 ? sc[n][e] * s_power[back] : 0.0f;
                    }
                uint32_t big[4], small[4];
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    split_bf16(sc[n][0], sc[n][1], big[2 * n], small[2 * n]);
                    split_bf16(sc[n][2], sc[n][3], big[2 * n + 1], small[2 * n + 1]);
                }
#pragma unroll
                for (int n = 0; n < OT; n += 2) {
                    uint32_t vb[4];
                    ldsm4t(s_v + j * 16 * VP + v_off + n * 16, vb);
                    mma16816(o[n], big, vb[0], vb[1]);
                    mma16816(o[n + 1], big, vb[2], vb[3]);
                    mma16816(o[n], small, vb[0], vb[1]);
                    mma16816(o[n + 1], small, vb[2], vb[3]);
                }
            }
        }
        // sums of squares of this slice, to every CTA of the head
        float sq[2] = {};
#pragma unroll
        for (int n = 0; n < OT; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                o[n][e] *= a.scale;
                if (slice * W + n * 8 + c0 + (e & 1) < a.vmean) sq[e >> 1] = fmaf(o[n][e], o[n][e], sq[e >> 1]);
            }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            sq[e] += __shfl_xor_sync(0xffffffffu, sq[e], 1);
            sq[e] += __shfl_xor_sync(0xffffffffu, sq[e], 2);
        }
        const uint32_t sums = (chunk & 1u) * MAX_SLICES * CHUNK;
        if (row < CHUNK)
            for (uint32_t to = lane & 3; to < gridDim.x; to += 4)
#pragma unroll
                for (int e = 0; e < 2; ++e) store_remote(base + s.sums + (sums + slice * CHUNK + row + r0 + 8 * e) * 4, to, sq[e]);
        __syncwarp();
        cluster_arrive();
        // while the sums travel: the gates of this warp's tokens, and the state
        __nv_bfloat162 gate[2][OT];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const uint32_t i = chunk * CHUNK + row + r0 + 8 * e;
#pragma unroll
            for (int n = 0; n < OT; ++n)
                if (row < CHUNK && i < count) gate[e][n] = *reinterpret_cast<const __nv_bfloat162*>((const __nv_bfloat16*)a.gate + (uint64_t)i * a.gate_ld + col + n * 8 + c0);
        }
        const float keep = s_power[tokens];
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int e = 0; e < 4; ++e) st[n][m][e] *= keep;
        {
            // A: rows = value columns (the stored rows are tokens: transposed), B: rows = tokens, columns = key dimensions
            const uint32_t a_off = ((lane & 7) + ((lane >> 4) << 3)) * VP + ((lane >> 3) & 1) * 16;
            const uint32_t b_off = ((lane & 7) + (((lane >> 3) & 1) << 3)) * s.qk;
            const uint32_t steps = (tokens + 15) / 16;
            for (uint32_t x = 0; x < steps; ++x) {
                uint32_t big[MT][4], small[MT][4];
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    const uint32_t at = base + s.vbig + x * 16 * VP + a_off + m * 32;
                    ldsm4t(at, big[m]);
                    ldsm4t(at + CHUNK * VP, small[m]);
                }
#pragma unroll
                for (int n = 0; n < NT; n += 2) {
                    // two tiles of eight key dimensions at once: lanes 16 .. 31 address the second one
                    const uint32_t t0 = warp + 8 * n, t1 = t0 + 8;
                    if (t0 < ntiles) {
                        uint32_t kb[4];
                        ldsm4t(s_k + x * 16 * s.qk + b_off + ((lane >> 4) && t1 < ntiles ? t1 : t0) * 16, kb);
#pragma unroll
                        for (int m = 0; m < MT; ++m) {
                            mma16816(st[n][m], big[m], kb[0], kb[1]);
                            mma16816(st[n][m], small[m], kb[0], kb[1]);
                            if (n + 1 < NT && t1 < ntiles) {
                                mma16816(st[n + 1 < NT ? n + 1 : n][m], big[m], kb[2], kb[3]);
                                mma16816(st[n + 1 < NT ? n + 1 : n][m], small[m], kb[2], kb[3]);
                            }
                        }
                    }
                }
            }
        }
        __syncwarp();
        cluster_wait();
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const uint32_t i = chunk * CHUNK + row + r0 + 8 * e;
            if (row >= CHUNK || i >= count) continue;
            float total = 0.0f;
            for (uint32_t x = 0; x < gridDim.x; ++x) total += s_sums[sums + x * CHUNK + row + r0 + 8 * e];
            const float inv = 1.0f / sqrtf(total / (float)a.vmean + a.eps);
            __nv_bfloat16* out = (__nv_bfloat16*)a.out + (uint64_t)i * a.ld + col;
#pragma unroll
            for (int n = 0; n < OT; ++n)
                *reinterpret_cast<__nv_bfloat162*>(out + n * 8 + c0) =
                    __floats2bfloat162_rn(o[n][2 * e] * inv * __low2float(gate[e][n]), o[n][2 * e + 1] * inv * __high2float(gate[e][n]));
        }
        if (s.stages == 1 && chunk + 1 < chunks) {
            __syncthreads();
            load_chunk(chunk + 1, 0);
        }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t d = (warp + 8 * n) * 8 + c0 + (e & 1), x = 16 * m + r0 + 8 * (e >> 1);
                if (d < a.dim) home[(uint64_t)d * a.vdim + x] = st[n][m][e];
            }
}

template <int W, int NT, int CHUNK>
int32_t launch_chunk_as(holo_b200_ctx* ctx, const HoloRetentionArgs& a, bool* taken) {
    const uint32_t limit = (uint32_t)ctx->smem_optin - 1024;
    uint32_t stages = a.rows > (uint32_t)CHUNK ? 2 : 1;
    if (ChunkSmem<W, CHUNK>(a.dim, stages).total > limit) stages = 1;
    const uint32_t smem = ChunkSmem<W, CHUNK>(a.dim, stages).total;
    if (smem > limit) return HOLO_OK;
    static thread_local int configured_device = -1;
    if (configured_device != ctx->device) {
        HOLO_CUDA(cudaFuncSetAttribute(retention_chunk_kernel<W, NT, CHUNK>, cudaFuncAttributeMaxDynamicSharedMemorySize, limit));
        configured_device = ctx->device;
    }
    const uint32_t slices = a.vdim / W;
    HOLO_CUDA(holo_launch_kernel_cluster(ctx, retention_chunk_kernel<W, NT, CHUNK>, dim3(slices, a.heads), dim3(CHUNK_WARPS * 32), smem, slices, 1u, a, stages));
    ctx->launches++;
    *taken = true;
    return HOLO_OK;
}
template <int W>
int32_t launch_chunk(holo_b200_ctx* ctx, const HoloRetentionArgs& a, bool* taken) {
    if (a.dim <= 128) return launch_chunk_as<W, 2, 128>(ctx, a, taken);
    HOLO_TRY((launch_chunk_as<W, 4, 128>(ctx, a, taken)));
    return *taken ? HOLO_OK : launch_chunk_as<W, 4, 64>(ctx, a, taken);      // wide keys and values: shorter chunks
}
// Launches the chunk kernel, or returns with *taken false when the shape does not suit it.
int32_t try_chunk(holo_b200_ctx* ctx, const HoloRetentionArgs& a, bool* taken) {
    *taken = false;
    if (a.dtype != HOLO_DTYPE_BF16 || a.dim % 16 || a.vdim % 16 || a.dim > 256 || (a.q_ld | a.k_ld | a.v_ld) % 8 || (a.gate_ld | a.ld) % 2 ||
        (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v) & 15u) || (((uintptr_t)a.gate | (uintptr_t)a.out) & 3u))
        return HOLO_OK;
    const auto fits = [&](uint32_t w) { return a.vdim % w == 0 && a.vdim / w <= MAX_SLICES; };
    if (fits(32)) return launch_chunk<32>(ctx, a, taken);
    if (fits(16)) return launch_chunk<16>(ctx, a, taken);
    if (fits(48)) return launch_chunk<48>(ctx, a, taken);
    if (fits(64)) return launch_chunk<64>(ctx, a, taken);
    return HOLO_OK;
}

// ---- many rows, heads of 128 or 256 key dimensions: tcgen05 ------------------------------------------------------------------
// The same chunks of 128 tokens and the same sums, a slice of 64 value columns per CTA; all four products run on tcgen05 with
// their f32 results in TMEM, where the state stays from the first chunk to the last. S and the decayed values enter their
// products as two bf16 parts; the decayed scores P, which touch nothing but their own token's output, as one, like the softmax
// weights of the attention kernels.
//   warp 0      TMA producer: q and k tiles (a ring of one or two chunks), v tiles
//   warp 1      MMA issuer. Per chunk: scores = Q K^T; O2 = P V; S += K^T V'; O1 = Q S (128 key dimensions at a time). Where two
//               chunks of q and k fit, P V and the next chunk's scores come first (the weights are ready by then, and v can be
//               replaced early), else last (the scores wait for their chunk)
//   warps 2-5   one thread per token: scores -> P over them, V -> V'
//   warps 6-9   one thread per key dimension: S -> shared memory and p(L) S -> TMEM
//   warps 10-13 one thread per token: o = scale (p(i + 1) O1 + O2), f32, through shared memory to the call's work buffer (TMA)
// A second launch divides every head's o by its root mean square and applies the gate. (A cluster per head that exchanged its
// sums of squares needed no second launch, but eight CTAs of this size rarely find room in one GPC: half the chip stood idle.)
// TMEM columns: O1 0 and 64, O2 128 and 192 (by turns), S 256 (+ 64 for the upper 128 key dimensions), scores 384. It is
// allocated after the dependency wait, dependents are released after that. Every wait is bounded.
constexpr int RT_THREADS = 448, RT_W = 64;

struct RetentionTileParams {
    HoloRetentionArgs a;
    uint32_t* status;
};

__device__ __forceinline__ void tma_prefetch_2d(const CUtensorMap* map, int x, int y) {
    asm volatile("cp.async.bulk.prefetch.tensor.2d.L2.global.tile [%0, {%1, %2}];" ::"l"(map), "r"(x), "r"(y) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint32_t bar) { asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory"); }
__device__ __forceinline__ void fence_async_smem() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

template <int DT>   // dim = 128 DT
__global__ void __launch_bounds__(RT_THREADS, 1)
retention_tile_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                      const __grid_constant__ CUtensorMap map_work, const RetentionTileParams p) {
    constexpr uint32_t NS = DT == 1 ? 2 : 1, QK = 2 * DT * TILE_CHUNK, STAGE = 2 * QK;      // q and k tiles of a chunk
    constexpr uint32_t OFF_V = NS * STAGE, OFF_VBIG = OFF_V + TILE_CHUNK, OFF_VSMALL = OFF_VBIG + TILE_CHUNK, OFF_SBIG = OFF_VSMALL + TILE_CHUNK,
                       OFF_SSMALL = OFF_SBIG + TILE_CHUNK, OFF_OUT = OFF_SSMALL + TILE_CHUNK, OFF_POWER = OFF_OUT + TILE_CHUNK, OFF_BARS = OFF_POWER + 1024;
    extern __shared__ uint8_t smem_raw[];
    const HoloRetentionArgs& a = p.a;
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    uint8_t* sm = smem_raw + (base - raw);
    const uint32_t bars = base + OFF_BARS, bar_q_full = bars, bar_q_empty = bars + 16, bar_sc = bars + 32, bar_o = bars + 48, bar_sbuf = bars + 64, bar_m2 = bars + 80,
                   bar_v_full = bars + 96, bar_v_empty = bars + 104, bar_ready = bars + 112, bar_vready = bars + 120, bar_oread = bars + 128, bar_s4 = bars + 144,
                   bar_k_full = bars + 168, bar_k_empty = bars + 184, bar_p = bars + 200;
    uint32_t* s_tmem = reinterpret_cast<uint32_t*>(sm + OFF_BARS + 160);
    volatile uint32_t* s_abort = reinterpret_cast<volatile uint32_t*>(sm + OFF_BARS + 164);
    float* s_power = reinterpret_cast<float*>(sm + OFF_POWER);      // [127 + n] = decay^n, 0 for n < 0
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, slice = blockIdx.x, slices = gridDim.x, h = blockIdx.y;
    if (tid == 0) {
        for (int i = 0; i < 2; ++i) {
            mbar_init(bar_q_full + 8 * i, 1);
            mbar_init(bar_q_empty + 8 * i, 1);
            mbar_init(bar_k_full + 8 * i, 1);
            mbar_init(bar_k_empty + 8 * i, 1);
            mbar_init(bar_sc + 8 * i, 1);
            mbar_init(bar_p + 8 * i, 4);
            mbar_init(bar_o + 8 * i, 1);
            mbar_init(bar_oread + 8 * i, 4);
            mbar_init(bar_sbuf + 8 * i, 4);
            mbar_init(bar_m2 + 8 * i, 1);
        }
        mbar_init(bar_v_full, 1);
        mbar_init(bar_v_empty, 5);                     // the product that read v, and the four warps that decayed it
        mbar_init(bar_ready, 4);
        mbar_init(bar_vready, 4);
        mbar_init(bar_s4, 1);
        *s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    holo_pdl_wait();
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(s_tmem)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    const float decay = a.decay[h];
    if (tid < 256) s_power[tid] = tid < 127 ? 0.0f : tid == 127 ? 1.0f : powf(decay, (float)(tid - 127));
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    holo_pdl_trigger();
    const uint32_t tmem = *s_tmem, tmem_o1 = tmem, tmem_o2 = tmem + 128, tmem_s = tmem + 256, tmem_sc = tmem + 384;
    const uint32_t count = min(a.rows, a.step[1]), chunks = (count + 127) / 128;

    if (warp == 0) {
        // ---------------- TMA producer ----------------
        if (lane == 0) {
            uint32_t nk = 0, nq = 0, nv = 0;       // loads requested
            for (uint32_t c = 0; c < chunks; ++c) {
                const uint32_t s = c % NS, st = base + s * STAGE;
                // two chunks ahead, into L2 (every slice of the head asks for its share of q and k)
                for (uint32_t f = c == 0 ? 1 : c + 2; f <= c + 2 && f < chunks; ++f) {
                    tma_prefetch_2d(&map_v, (int)(h * a.vdim + slice * RT_W), (int)(f * 128));
                    for (uint32_t x = slice; x < 2 * DT; x += slices) {
                        tma_prefetch_2d(&map_k, (int)(h * a.dim + 64 * x), (int)(f * 128));
                        tma_prefetch_2d(&map_q, (int)(h * a.dim + 64 * x), (int)(f * 128));
                    }
                }
                if (c >= NS && !mbar_wait(bar_k_empty + 8 * s, (c / NS - 1) & 1, s_abort, p.status)) break;
                mbar_arrive_expect_tx(bar_k_full + 8 * s, QK);
                for (uint32_t x = 0; x < 2 * DT; ++x) tma_load_2d(st + QK + x * TILE_CHUNK, &map_k, (int)(h * a.dim + 64 * x), (int)(c * 128), bar_k_full + 8 * s);
                ++nk;
                // (the values last: their buffer is free only after the product that follows the next chunk's scores)
                if (c >= NS && !mbar_wait(bar_q_empty + 8 * s, (c / NS - 1) & 1, s_abort, p.status)) break;
                mbar_arrive_expect_tx(bar_q_full + 8 * s, QK);
                for (uint32_t x = 0; x < 2 * DT; ++x) tma_load_2d(st + x * TILE_CHUNK, &map_q, (int)(h * a.dim + 64 * x), (int)(c * 128), bar_q_full + 8 * s);
                ++nq;
                if (c > 0 && !mbar_wait(bar_v_empty, (c - 1) & 1, s_abort, p.status)) break;
                mbar_arrive_expect_tx(bar_v_full, TILE_CHUNK);
                tma_load_2d(base + OFF_V, &map_v, (int)(h * a.vdim + slice * RT_W), (int)(c * 128), bar_v_full);
                ++nv;
            }
            // nothing may still be on its way into this CTA's shared memory when it ends
            for (uint32_t c = nk > NS ? nk - NS : 0; c < nk; ++c)
                for (uint32_t it = 0; it < WAIT_LIMIT && !mbar_try_wait(bar_k_full + 8 * (c % NS), (c / NS) & 1); ++it) __nanosleep(64);
            for (uint32_t c = nq > NS ? nq - NS : 0; c < nq; ++c)
                for (uint32_t it = 0; it < WAIT_LIMIT && !mbar_try_wait(bar_q_full + 8 * (c % NS), (c / NS) & 1); ++it) __nanosleep(64);
            for (uint32_t it = 0; nv && it < WAIT_LIMIT && !mbar_try_wait(bar_v_full, (nv - 1) & 1); ++it) __nanosleep(64);
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer ----------------
        if (lane == 0) {
            // D = f32, A = B = bf16, M = 128; scores: both operands K-major, N = 128; the others: B N-major, N = 64; the state's A is K^T (M-major)
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 4) << 24);
            constexpr uint32_t idesc_sc = idesc | ((128u >> 3) << 17), idesc_n = idesc | (1u << 16) | ((64u >> 3) << 17), idesc_st = idesc_n | (1u << 15);
            const uint64_t d_v = smem_desc(base + OFF_V, TILE_CHUNK, 1024), d_vb = smem_desc(base + OFF_VBIG, TILE_CHUNK, 1024), d_sb = smem_desc(base + OFF_SBIG, TILE_CHUNK, 1024);
            constexpr uint64_t PART = TILE_CHUNK >> 4;       // from a big part to its small one
            // the scores of a chunk, over weights that the product before has read
            auto scores = [&](uint32_t c) {
                const uint32_t s = c % NS, st = base + s * STAGE;
                if (!mbar_wait(bar_k_full + 8 * s, (c / NS) & 1, s_abort, p.status) || !mbar_wait(bar_q_full + 8 * s, (c / NS) & 1, s_abort, p.status)) return false;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint64_t d_q = smem_desc(st, 16, 1024), d_k = smem_desc(st + QK, 16, 1024);
#pragma unroll
                for (uint32_t k = 0; k < 8 * DT; ++k) umma_bf16(tmem_sc, d_q + (k >> 2) * PART + 2 * (k & 3), d_k + (k >> 2) * PART + 2 * (k & 3), idesc_sc, k != 0);
                umma_commit(bar_sc + 8 * (c & 1u));
                return true;
            };
            bool ok = chunks == 0 || scores(0);
            for (uint32_t c = 0; c < chunks && ok; ++c) {
                const uint32_t s = c % NS, st = base + s * STAGE, o = (c & 1u) * 64;
                const uint64_t d_q = smem_desc(st, 16, 1024), d_kt = smem_desc(st + QK, TILE_CHUNK, 1024);
                // O1 of 128 key dimensions
                auto inter = [&](uint32_t half) {
#pragma unroll
                    for (uint32_t part = 0; part < 2; ++part)
#pragma unroll
                        for (uint32_t k = 0; k < 8; ++k)
                            umma_bf16(tmem_o1 + o, d_q + (2 * half + (k >> 2)) * PART + 2 * (k & 3), d_sb + part * PART + 128 * k, idesc_n, (half | part | k) != 0);
                    umma_commit(bar_m2 + 8 * half);
                };
                // O2 = P V
                auto near = [&]() {
                    if (!mbar_wait(bar_v_full, c & 1, s_abort, p.status) || !mbar_wait(bar_p + 8 * (c & 1u), (c >> 1) & 1, s_abort, p.status)) return false;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
                    for (uint32_t k = 0; k < 8; ++k) umma_bf16_ts(tmem_o2 + o, tmem_sc + 8 * k, d_v + 128 * k, idesc_n, k != 0);
                    umma_commit(bar_v_empty);
                    return true;
                };
                ok = (c < 2 || mbar_wait(bar_oread + 8 * (c & 1u), ((c >> 1) - 1) & 1, s_abort, p.status)) &&
                     (NS == 1 || (near() && (c + 1 == chunks || scores(c + 1)))) && mbar_wait(bar_ready, c & 1, s_abort, p.status) && mbar_wait(bar_vready, c & 1, s_abort, p.status);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
                for (uint32_t half = 0; half < DT; ++half)
#pragma unroll
                    for (uint32_t part = 0; part < 2; ++part)
#pragma unroll
                        for (uint32_t k = 0; k < 8; ++k) umma_bf16(tmem_s + 64 * half, d_kt + 2 * half * PART + 128 * k, d_vb + part * PART + 128 * k, idesc_st, 1u);
                umma_commit(bar_s4);
                umma_commit(bar_k_empty + 8 * s);
                inter(0);
                if (DT == 2) {
                    if (!(ok = mbar_wait(bar_sbuf + 8, c & 1, s_abort, p.status))) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    inter(1);
                }
                umma_commit(bar_q_empty + 8 * s);
                if (NS == 1 && !(ok = near())) break;
                umma_commit(bar_o + 8 * (c & 1u));
                if (NS == 1 && c + 1 < chunks) ok = scores(c + 1);
            }
        }
    } else if (warp < 6) {
        // ---------------- weights and decayed values (TMEM lane quarter = warp % 4) ----------------
        const uint32_t quarter = warp & 3u, i = quarter * 32 + lane, lanes = (quarter * 32u) << 16;
        const float* power = s_power + 127;
        float diagonal[32];      // the decays among this warp's own 32 tokens
#pragma unroll
        for (int e = 0; e < 32; ++e) diagonal[e] = power[(int)lane - e];
        // scores -> weights, 32 tokens at a time: token 32 b + e is p(i - 32 b - 31) p(31 - e) away from the tokens of later blocks
        auto weights = [&](uint32_t c) {
            const uint32_t sc = tmem_sc + lanes;
            bool ok = mbar_wait(bar_sc + 8 * (c & 1u), (c >> 1) & 1, s_abort, p.status) && !*s_abort;
            if (!__all_sync(0xffffffffu, ok)) return false;   // the TMEM accesses below are whole-warp instructions
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
            for (uint32_t b2 = 0; b2 < 2; ++b2) {
                uint32_t v[2][32];
                if (2 * b2 <= quarter) {
                    tmem_ld32_request(sc + 64 * b2, v[0]);
                    tmem_ld32_request(sc + 64 * b2 + 32, v[1]);
                    tmem_ld32_wait(v[0]);
                    tmem_ld32_pass(v[1]);
                }
#pragma unroll
                for (uint32_t x = 0; x < 2; ++x) {
                    const uint32_t b = 2 * b2 + x;
                    uint32_t w[16];
                    if (b < quarter) {
                        const float far = power[(int)i - (int)(32 * b) - 31];
#pragma unroll
                        for (int e = 0; e < 16; ++e)
                            w[e] = pack_bf16(__uint_as_float(v[x][2 * e]) * (power[31 - 2 * e] * far), __uint_as_float(v[x][2 * e + 1]) * (power[30 - 2 * e] * far));
                    } else if (b == quarter) {
#pragma unroll
                        for (int e = 0; e < 16; ++e) w[e] = pack_bf16(__uint_as_float(v[x][2 * e]) * diagonal[2 * e], __uint_as_float(v[x][2 * e + 1]) * diagonal[2 * e + 1]);
                    } else {
#pragma unroll
                        for (int e = 0; e < 16; ++e) w[e] = 0;
                    }
                    tmem_st16(sc + 16 * b, w);          // over scores this warp has already read
                }
            }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_p + 8 * (c & 1u));
            return true;
        };
        // one token's values, the same places in both parts (units taken in another order by every lane: no bank is asked twice)
        auto values = [&](uint32_t c) {
            bool ok = (c == 0 || mbar_wait(bar_s4, (c - 1) & 1, s_abort, p.status)) && mbar_wait(bar_v_full, c & 1, s_abort, p.status);   // the last product has read V'
            if (!__all_sync(0xffffffffu, ok)) return false;
            const uint32_t tokens = min(128u, count - c * 128);
            const float f = i < tokens ? power[tokens - 1 - i] : 0.0f;
            uint4 x[8];
#pragma unroll
            for (uint32_t u0 = 0; u0 < 8; ++u0) x[u0] = *reinterpret_cast<const uint4*>(sm + OFF_V + i * 128 + (((u0 + lane) & 7u) << 4));
#pragma unroll
            for (uint32_t u0 = 0; u0 < 8; ++u0) {
                const uint32_t at = i * 128 + (((u0 + lane) & 7u) << 4);
                const uint32_t in[4] = {x[u0].x, x[u0].y, x[u0].z, x[u0].w};
                uint32_t big[4], small[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const __nv_bfloat162 y = *reinterpret_cast<const __nv_bfloat162*>(&in[e]);
                    split_bf16(__low2float(y) * f, __high2float(y) * f, big[e], small[e]);
                }
                *reinterpret_cast<uint4*>(sm + OFF_VBIG + at) = make_uint4(big[0], big[1], big[2], big[3]);
                *reinterpret_cast<uint4*>(sm + OFF_VSMALL + at) = make_uint4(small[0], small[1], small[2], small[3]);
            }
            fence_async_smem();
            __syncwarp();
            if (lane == 0) {
                mbar_arrive(bar_v_empty);
                mbar_arrive(bar_vready);
            }
            return true;
        };
        // with two chunks of q and k in flight a chunk's scores are there before the state's last product is through, else after
        for (uint32_t c = 0; c < chunks; ++c)
            if (NS == 2 ? !(weights(c) && values(c)) : !(values(c) && weights(c))) break;
    } else if (warp < 10) {
        // ---------------- state and values (TMEM lane quarter = warp % 4) ----------------
        const uint32_t quarter = warp & 3u, r = quarter * 32 + lane, lanes = (quarter * 32u) << 16;
        const float* power = s_power + 127;
        const bool fresh = a.step[0] == 0;
        float* home = a.state + ((uint64_t)h * a.dim + r) * a.vdim + slice * RT_W;      // key dimension r; the upper 128 follow 128 rows later
        if (chunks != 0) {
#pragma unroll
            for (int half = 0; half < DT; ++half)
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    uint32_t v[16];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const float4 f = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : reinterpret_cast<const float4*>(home + (uint64_t)half * 128 * a.vdim)[4 * x + e];
                        v[4 * e] = __float_as_uint(f.x); v[4 * e + 1] = __float_as_uint(f.y); v[4 * e + 2] = __float_as_uint(f.z); v[4 * e + 3] = __float_as_uint(f.w);
                    }
                    tmem_st16(tmem_s + 64 * half + lanes + 16 * x, v);
                }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
        // a row of S as two bf16 parts, 16-byte units swizzled as the matrix descriptor says
        auto stage_state = [&](const uint32_t (&v)[2][32]) {
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                uint32_t big[4], small[4];
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    split_bf16(__uint_as_float(v[u >> 2][8 * (u & 3) + 2 * e]), __uint_as_float(v[u >> 2][8 * (u & 3) + 2 * e + 1]), big[e], small[e]);
                const uint32_t at = r * 128 + (((uint32_t)u ^ (r & 7u)) << 4);
                *reinterpret_cast<uint4*>(sm + OFF_SBIG + at) = make_uint4(big[0], big[1], big[2], big[3]);
                *reinterpret_cast<uint4*>(sm + OFF_SSMALL + at) = make_uint4(small[0], small[1], small[2], small[3]);
            }
        };
        auto load_state = [&](int half, uint32_t (&v)[2][32]) {
            tmem_ld32_request(tmem_s + 64 * half + lanes, v[0]);
            tmem_ld32_request(tmem_s + 64 * half + lanes + 32, v[1]);
            tmem_ld32_wait(v[0]);
            tmem_ld32_pass(v[1]);
        };
        auto keep_state = [&](int half, const uint32_t (&v)[2][32], float keep) {
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                uint32_t w[16];
#pragma unroll
                for (int e = 0; e < 16; ++e) w[e] = __float_as_uint(__uint_as_float(v[x >> 1][16 * (x & 1) + e]) * keep);
                tmem_st16(tmem_s + 64 * half + lanes + 16 * x, w);
            }
        };
        bool ok = true;
        for (uint32_t c = 0; c < chunks; ++c) {
            const float keep = power[min(128u, count - c * 128)];
            // the last chunk's products have written S and read its parts
            ok = (c == 0 || (mbar_wait(bar_s4, (c - 1) & 1, s_abort, p.status) && mbar_wait(bar_m2 + 8 * (DT - 1), (c - 1) & 1, s_abort, p.status))) && !*s_abort;
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            uint32_t v[2][32];
            load_state(0, v);
            stage_state(v);
            keep_state(0, v, keep);
            if (DT == 2) {
                load_state(1, v);
                keep_state(1, v, keep);
            }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            fence_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_ready);
            if (DT == 2) {
                ok = mbar_wait(bar_m2, c & 1, s_abort, p.status);
                ok = __all_sync(0xffffffffu, ok);
                if (!ok) break;
                stage_state(v);
                fence_async_smem();
                __syncwarp();
                if (lane == 0) mbar_arrive(bar_sbuf + 8);
            }
        }
        ok = ok && (chunks == 0 || mbar_wait(bar_s4, (chunks - 1) & 1, s_abort, p.status));
        ok = __all_sync(0xffffffffu, ok) && chunks != 0;
        if (ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
            for (int half = 0; half < DT; ++half) {
                uint32_t v[2][32];
                load_state(half, v);
                float4* to = reinterpret_cast<float4*>(home + (uint64_t)half * 128 * a.vdim);
#pragma unroll
                for (int x = 0; x < 16; ++x)
                    to[x] = make_float4(__uint_as_float(v[x >> 3][4 * (x & 7)]), __uint_as_float(v[x >> 3][4 * (x & 7) + 1]), __uint_as_float(v[x >> 3][4 * (x & 7) + 2]),
                                        __uint_as_float(v[x >> 3][4 * (x & 7) + 3]));
            }
        }
    } else {
        // ---------------- outputs (TMEM lane quarter = warp % 4) ----------------
        const uint32_t quarter = warp & 3u, i = quarter * 32 + lane, lanes = (quarter * 32u) << 16;
        const float* power = s_power + 127;
        bool ok = true;
        uint32_t together = 1;
        if (chunks != 0 && (*reinterpret_cast<volatile uint32_t*>(p.status) & 4u)) *s_abort = 1;      // an earlier launch gave up: store nothing
        for (uint32_t c = 0; c < chunks; ++c) {
            ok = mbar_wait(bar_o + 8 * (c & 1u), (c >> 1) & 1, s_abort, p.status) && !*s_abort;
            // the four warps go on together: they share the staging tile
            __syncwarp();
            asm volatile("{\n.reg .pred p, q;\nsetp.ne.b32 p, %1, 0;\nbarrier.red.and.pred.aligned q, 2, 128, p;\nselp.u32 %0, 1, 0, q;\n}\n"
                         : "=r"(together)
                         : "r"((uint32_t)ok)
                         : "memory");
            if (!together) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const float f = a.scale * power[i + 1];
            const uint32_t turn = (c & 1u) * 64 + lanes;
#pragma unroll
            for (uint32_t y = 0; y < 2; ++y) {
                uint32_t far[32], near[32];
                tmem_ld32_request(tmem_o1 + turn + 32 * y, far);
                tmem_ld32_request(tmem_o2 + turn + 32 * y, near);
                tmem_ld32_wait(far);
                tmem_ld32_pass(near);
                if (y == 1) {
                    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                    __syncwarp();
                    if (lane == 0) mbar_arrive(bar_oread + 8 * (c & 1u));
                }
                // the store before has read the staging tile
                if (tid == 320) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
                __syncwarp();
                asm volatile("bar.sync 2, 128;" ::: "memory");
#pragma unroll
                for (uint32_t u = 0; u < 8; ++u) {
                    float v[4];
#pragma unroll
                    for (int n = 0; n < 4; ++n) v[n] = fmaf(f, __uint_as_float(far[4 * u + n]), a.scale * __uint_as_float(near[4 * u + n]));
                    *reinterpret_cast<float4*>(sm + OFF_OUT + i * 128 + ((u ^ (i & 7u)) << 4)) = make_float4(v[0], v[1], v[2], v[3]);
                }
                fence_async_smem();
                asm volatile("bar.sync 2, 128;" ::: "memory");
                if (tid == 320) {
                    asm volatile("cp.async.bulk.tensor.2d.global.shared::cta.tile.bulk_group [%0, {%1, %2}], [%3];" ::"l"(&map_work), "r"((int)(h * a.vdim + slice * RT_W + 32 * y)),
                                 "r"((int)(c * 128)), "r"(base + OFF_OUT)
                                 : "memory");
                    asm volatile("cp.async.bulk.commit_group;" ::: "memory");
                }
                __syncwarp();
            }
        }
        if (tid == 320) asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    }
    // everyone meets here, whatever happened above, so that TMEM is always released
    __syncwarp();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
    }
}

int32_t make_map_rows(CUtensorMap* map, const void* ptr, uint64_t cols, uint64_t rows, uint64_t ld) {
    cuuint64_t dims[2] = {cols, rows};
    cuuint64_t strides[1] = {ld * 2};
    cuuint32_t box[2] = {64, 128};
    cuuint32_t es[2] = {1, 1};
    const CUresult r = encode_tiled_fn()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? HOLO_OK : holo_fail(HOLO_ERR_DISPATCH, "dispatch failed: cuTensorMapEncodeTiled (retention) returned %d", (int)r);
}

// One warp per (row, head): o over its root mean square, times the gate.
template <int PL>   // vdim <= 128 PL
__global__ void __launch_bounds__(256)
retention_finish_kernel(const HoloRetentionArgs a) {
    holo_pdl_trigger();
    const uint32_t unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, row = unit / a.heads, h = unit % a.heads;
    holo_pdl_wait();
    if (row >= min(a.rows, a.step[1])) return;
    const float4* o = reinterpret_cast<const float4*>(a.work + (uint64_t)unit * a.vdim);
    const uint2* gate = reinterpret_cast<const uint2*>((const __nv_bfloat16*)a.gate + (uint64_t)row * a.gate_ld + (uint64_t)h * a.vdim);
    float4 v[PL];
    uint2 g[PL];
    float sq = 0.0f;
#pragma unroll
    for (int x = 0; x < PL; ++x) {
        const uint32_t j = lane + 32 * x;
        v[x] = 4 * j < a.vdim ? o[j] : make_float4(0.f, 0.f, 0.f, 0.f);
        g[x] = 4 * j < a.vdim ? gate[j] : make_uint2(0, 0);
    }
#pragma unroll
    for (int x = 0; x < PL; ++x) {
        const uint32_t j = 4 * (lane + 32 * x);
        const float e[4] = {v[x].x, v[x].y, v[x].z, v[x].w};
#pragma unroll
        for (int n = 0; n < 4; ++n)
            if (j + n < a.vmean) sq = fmaf(e[n], e[n], sq);
    }
    for (int off = 16; off > 0; off >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, off);
    const float inv = 1.0f / sqrtf(sq / (float)a.vmean + a.eps);
    uint2* out = reinterpret_cast<uint2*>((__nv_bfloat16*)a.out + (uint64_t)row * a.ld + (uint64_t)h * a.vdim);
#pragma unroll
    for (int x = 0; x < PL; ++x) {
        const uint32_t j = lane + 32 * x;
        if (4 * j >= a.vdim) continue;
        const __nv_bfloat162 g0 = *reinterpret_cast<const __nv_bfloat162*>(&g[x].x), g1 = *reinterpret_cast<const __nv_bfloat162*>(&g[x].y);
        out[j] = make_uint2(pack_bf16(v[x].x * inv * __low2float(g0), v[x].y * inv * __high2float(g0)), pack_bf16(v[x].z * inv * __low2float(g1), v[x].w * inv * __high2float(g1)));
    }
}

template <int DT>
int32_t launch_tile_as(holo_b200_ctx* ctx, const HoloRetentionArgs& a) {
    constexpr uint32_t smem = (DT == 1 ? 2 : 1) * 4 * DT * TILE_CHUNK + 6 * TILE_CHUNK + 1024 + 256 + 1024;
    static_assert(smem <= 227 * 1024, "retention tile");
    static thread_local int configured_device = -1;
    if (configured_device != ctx->device) {
        HOLO_CUDA(cudaFuncSetAttribute(retention_tile_kernel<DT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        configured_device = ctx->device;
    }
    CUtensorMap mq, mk, mv;
    HOLO_TRY(make_map_rows(&mq, a.q, (uint64_t)a.heads * a.dim, a.rows, a.q_ld));
    HOLO_TRY(make_map_rows(&mk, a.k, (uint64_t)a.heads * a.dim, a.rows, a.k_ld));
    HOLO_TRY(make_map_rows(&mv, a.v, (uint64_t)a.heads * a.vdim, a.rows, a.v_ld));
    CUtensorMap mw;
    {   // stores of 32 f32 columns of 128 rows
        cuuint64_t dims[2] = {(cuuint64_t)a.heads * a.vdim, a.rows};
        cuuint64_t strides[1] = {(cuuint64_t)a.heads * a.vdim * 4};
        cuuint32_t box[2] = {32, 128};
        cuuint32_t es[2] = {1, 1};
        const CUresult r = encode_tiled_fn()(&mw, CU_TENSOR_MAP_DATA_TYPE_FLOAT32, 2, a.work, dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
        if (r != CUDA_SUCCESS) return holo_fail(HOLO_ERR_DISPATCH, "dispatch failed: cuTensorMapEncodeTiled (retention) returned %d", (int)r);
    }
    RetentionTileParams p;
    p.a = a;
    p.status = ctx->dev_status;
    HOLO_CUDA(holo_launch_kernel(ctx, retention_tile_kernel<DT>, dim3(a.vdim / RT_W, a.heads), dim3(RT_THREADS), smem, 1, mq, mk, mv, mw, p));
    const dim3 grid((a.rows * a.heads + 7) / 8);
    if (a.vdim <= 128) HOLO_CUDA(holo_launch_kernel(ctx, retention_finish_kernel<1>, grid, dim3(256), 0, 1, a));
    else if (a.vdim <= 256) HOLO_CUDA(holo_launch_kernel(ctx, retention_finish_kernel<2>, grid, dim3(256), 0, 1, a));
    else if (a.vdim <= 512) HOLO_CUDA(holo_launch_kernel(ctx, retention_finish_kernel<4>, grid, dim3(256), 0, 1, a));
    else HOLO_CUDA(holo_launch_kernel(ctx, retention_finish_kernel<8>, grid, dim3(256), 0, 1, a));
    ctx->launches += 2;
    return HOLO_OK;
}
// Launches the tile kernel, or returns with *taken false when the shape does not suit it.
int32_t try_tile(holo_b200_ctx* ctx, const HoloRetentionArgs& a, bool* taken) {
    *taken = false;
    if (a.dtype != HOLO_DTYPE_BF16 || a.rows < 128 || (a.dim != 128 && a.dim != 256) || a.vdim % RT_W || !a.work || ((uintptr_t)a.work & 15u) || a.heads > 65535 ||
        (a.q_ld | a.k_ld | a.v_ld | a.gate_ld | a.ld) % 8 || (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.gate | (uintptr_t)a.out) & 15u) ||
        encode_tiled_fn() == nullptr || getenv("HOLO_RETENTION_NO_TILE"))
        return HOLO_OK;
    *taken = true;
    return a.dim == 128 ? launch_tile_as<1>(ctx, a) : launch_tile_as<2>(ctx, a);
}

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
    if (!getenv("HOLO_RETENTION_GENERAL")) {
        bool taken = false;
        if (a.rows == 1) HOLO_TRY(a.dtype == HOLO_DTYPE_F32 ? try_token<float>(ctx, a, &taken) : try_token<__nv_bfloat16>(ctx, a, &taken));
        else HOLO_TRY(try_tile(ctx, a, &taken));
        if (!taken && a.rows > 1) HOLO_TRY(try_chunk(ctx, a, &taken));
        if (taken) return HOLO_OK;
    }
    return a.dtype == HOLO_DTYPE_F32 ? launch_sequence<float>(ctx, a) : launch_sequence<__nv_bfloat16>(ctx, a);
}
