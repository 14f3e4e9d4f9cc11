// The row-wise pieces of a decoder layer whose mixer and feed-forward run in parallel from one residual,
//
//     x <- x + (mixer(norm1(x)) + feed_forward(norm2(x))),
//
// with the residual kept in fp32:
//
//   parallel_norm   x += update (or x = embedding row), then both normalized inputs from ONE sum of squares
//   dual_proj       decode (1..8 rows): the mixer's input projection and the gated feed-forward's first half in one launch; the two
//                   read different inputs and are independent, so their blocks share a grid and fill the machine together
//   (the second halves of both branches are one projection: their inputs lie side by side in one row and their weights side by side
//   in one table, so the sum of the branches is the sum over K)
//
// Templates over the activation / weight type: bf16 for serving, fp32 for the 32-bit path.
#include "common.cuh"
#include "gemv_core.cuh"
#include "vec8.cuh"

// THREADS x REGS 8-element vectors of a row stay in registers (4096 columns either way); wider rows are read again.  Few rows: more threads
// per row, and the weights are asked for before the sum of squares is known; many rows: smaller CTAs, more of them per SM.
#define PN_FEW_ROWS 16

template <int THREADS>
__device__ __forceinline__ float pn_block_sum(float v, float* scratch) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) t += scratch[w];
    return t;
}

// One CTA per row.  `padded` columns are stored (a multiple of 8, zeros past `width`); the mean is over `width`.
template <typename T, int THREADS, int REGS>
__global__ void __launch_bounds__(THREADS)
parallel_norm_kernel(const int* __restrict__ tokens, const T* __restrict__ table, int vocab, const float* __restrict__ update,
                     float* __restrict__ residual, int width, int padded, const T* __restrict__ w1, const T* __restrict__ w2,
                     T* __restrict__ out1, T* __restrict__ out2, float eps, float table_scale, float w_offset, uint32_t* status) {
    GLMB_PDL_PROLOGUE();
    __shared__ float scratch[THREADS / 32];
    const int64_t base = (int64_t)blockIdx.x * padded;
    float* res = residual + base;
    const T* source = nullptr;
    if (tokens) {
        int id = tokens[blockIdx.x];
        if (id < 0 || id >= vocab) {
            if (threadIdx.x == 0) raise_status(status, GLMB_STATUS_BAD_INDEX);
            id = min(max(id, 0), vocab - 1);
        }
        source = table + (int64_t)id * padded;
    }
    float keep[REGS][8], wa[8], wb[8];
    constexpr bool early = REGS == 1;
    if (early && (int)threadIdx.x * 8 < padded) {  // the weights of the first vector
        load8(w1 + threadIdx.x * 8, wa);
        if (w2) load8(w2 + threadIdx.x * 8, wb);
    }
    float ss = 0.f;
    int slot = 0;
    for (int v = threadIdx.x * 8; v < padded; v += THREADS * 8, ++slot) {
        float x[8];
        if (source) {
            load8(source + v, x);
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] *= table_scale;
        } else {
            load8(res + v, x);
            if (update) {
                float u[8];
                load8(update + base + v, u);
#pragma unroll
                for (int e = 0; e < 8; ++e) x[e] = __fadd_rn(x[e], u[e]);
            }
        }
        if (source || update) store8(res + v, x);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss = fmaf(x[e], x[e], ss);
#pragma unroll
        for (int s = 0; s < REGS; ++s)
            if (s == slot)
#pragma unroll
                for (int e = 0; e < 8; ++e) keep[s][e] = x[e];
    }
    const float mean = pn_block_sum<THREADS>(ss, scratch) / (float)width;
    const float denom = sqrtf(mean + eps);
    slot = 0;
    for (int v = threadIdx.x * 8; v < padded; v += THREADS * 8, ++slot) {
        float x[8];
        if (slot < REGS) {
#pragma unroll
            for (int s = 0; s < REGS; ++s)
                if (s == slot)
#pragma unroll
                    for (int e = 0; e < 8; ++e) x[e] = keep[s][e];
        } else {
            load8(res + v, x);  // written by this same thread above
        }
        float y[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = x[e] / denom;
        if (slot || !early) load8(w1 + v, wa);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] = x[e] * (w_offset + wa[e]);
        store8(out1 + base + v, y);
        if (w2) {
            if (slot || !early) load8(w2 + v, wb);
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] = x[e] * (w_offset + wb[e]);
            store8(out2 + base + v, y);
        }
    }
}

// ---------------------------------------------------------------------------------------------------
#define DP_WARPS 8
#define DP_THREADS (DP_WARPS * 32)

__device__ __forceinline__ void dp_prefetch(const void* rows, int64_t bytes) {
    const uint32_t n = (uint32_t)(bytes & ~(int64_t)15);
    if (threadIdx.x == 0 && n) asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(rows), "r"(n) : "memory");
}

// Blocks [0, proj_blocks): out[r][n] = x1[r] . w[n]           (two output columns per warp group)
// the others:              act[r][n] = f(x2[r] . wg[n]) * (x2[r] . wu[n])
// ks warps of a CTA split K for the same outputs.  Weight rows are contiguous ([N, K]).
template <int R>
__global__ void __launch_bounds__(DP_THREADS)
dual_proj_kernel(const bf16* __restrict__ x1, const bf16* __restrict__ x2, int64_t xs, int rows, int K, const bf16* __restrict__ w, int N,
                 bf16* __restrict__ out, int64_t os, const bf16* __restrict__ wg, const bf16* __restrict__ wu, int F, bf16* __restrict__ act,
                 int64_t as, int kind, int proj_blocks, int ks) {
    asm volatile("griddepcontrol.launch_dependents;");
    const bool gated = (int)blockIdx.x >= proj_blocks;
    const int groups = DP_WARPS / ks;
    if (!gated) {
        const int first = blockIdx.x * groups * 2;
        dp_prefetch(w + (int64_t)first * K, (int64_t)min(groups * 2, N - first) * K * 2);
    } else {
        const int first = (blockIdx.x - proj_blocks) * groups, count = min(groups, F - first);
        dp_prefetch(wg + (int64_t)first * K, (int64_t)count * K * 2);
        dp_prefetch(wu + (int64_t)first * K, (int64_t)count * K * 2);
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    __shared__ float red[DP_WARPS][2][R];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int group = warp / ks, kpart = warp % ks;
    const int n = gated ? (blockIdx.x - proj_blocks) * groups + group : (blockIdx.x * groups + group) * 2;
    const bool valid = n < (gated ? F : N);
    const bf16* x = gated ? x2 : x1;
    const bf16* xr[R];
#pragma unroll
    for (int r = 0; r < R; ++r) xr[r] = x + (int64_t)(r < rows ? r : 0) * xs;
    float acc[2][R];
#pragma unroll
    for (int r = 0; r < R; ++r) acc[0][r] = acc[1][r] = 0.f;
    if (valid) {
        const bf16* wp[2] = {gated ? wg + (int64_t)n * K : w + (int64_t)n * K, gated ? wu + (int64_t)n * K : w + (int64_t)min(n + 1, N - 1) * K};
        const int kspan = K / ks;
        warp_dot_bf16<R, 2>(xr, wp, kpart * kspan, (kpart + 1) * kspan, lane, acc);
        warp_reduce_all<R, 2>(acc);
    }
    if (ks > 1) {
        if (lane == 0) {
#pragma unroll
            for (int r = 0; r < R; ++r) { red[warp][0][r] = acc[0][r]; red[warp][1][r] = acc[1][r]; }
        }
        __syncthreads();
        if (kpart == 0 && lane == 0)
            for (int p = 1; p < ks; ++p)
#pragma unroll
                for (int r = 0; r < R; ++r) { acc[0][r] += red[warp + p][0][r]; acc[1][r] += red[warp + p][1][r]; }
    }
    if (lane == 0 && kpart == 0 && valid) {
#pragma unroll
        for (int r = 0; r < R; ++r) {
            if (r >= rows) continue;
            if (gated) {
                act[(int64_t)r * as + n] = __float2bfloat16_rn(glu_activation(kind, acc[0][r]) * acc[1][r]);
            } else {
                out[(int64_t)r * os + n] = __float2bfloat16_rn(acc[0][r]);
                if (n + 1 < N) out[(int64_t)r * os + n + 1] = __float2bfloat16_rn(acc[1][r]);
            }
        }
    }
}

// ===================================================================================================
// tokens != NULL: the residual starts from the embedding `table` [vocab, padded]; update != NULL: residual += update first.
// The embedding is multiplied by table_scale; w_offset is added to the weights (1 for weights stored around zero).
// w2 / out2 may be NULL (one normalized output).  All rows are `padded` elements (a multiple of 8), 16-byte aligned.
GLMB_API int glmb_parallel_norm(const int* tokens, const void* table, int vocab, const float* update, float* residual, int rows, int width,
                                int padded, const void* w1, const void* w2, void* out1, void* out2, float eps, float table_scale, float w_offset,
                                int is_f32, uint32_t* status, void* stream) {
    if (rows < 1 || width < 1 || padded < width || (padded & 7) || (tokens && update) || (tokens && (!table || vocab < 1)) || (w2 && !out2)) return 1;
    cudaStream_t st = (cudaStream_t)stream;
#define CALL(T, THREADS, REGS)                                                                                                             \
    GLMB_LAUNCH((parallel_norm_kernel<T, THREADS, REGS>), rows, THREADS, 0, st, tokens, (const T*)table, vocab, update, residual, width, padded, \
                (const T*)w1, (const T*)w2, (T*)out1, (T*)out2, eps, table_scale, w_offset, status)
    if (rows <= PN_FEW_ROWS) {
        if (is_f32) CALL(float, 512, 1);
        else CALL(bf16, 512, 1);
    } else {
        if (is_f32) CALL(float, 256, 2);
        else CALL(bf16, 256, 2);
    }
#undef CALL
    return (int)cudaGetLastError();
}

// bf16, 1..8 rows.  F = 0: projection only.  K a multiple of 8, w [N, K] and wg / wu [F, K] contiguous.
GLMB_API int glmb_dual_proj(const void* x1, const void* x2, int64_t xs, int rows, int K, const void* w, int N, void* out, int64_t os,
                            const void* wg, const void* wu, int F, void* act, int64_t as, int kind, void* stream) {
    if (rows < 1 || rows > GLMB_MAX_ROWS || (K & 7) || K < 8 || (xs & 7) || N < 1 || F < 0 || (kind != GLU_SILU && kind != GLU_GELU_TANH)) return 1;
    const int units = ceil_div(N, 2) + F;
    int ks = 1;  // enough warps per output that about four CTAs land on every SM, with at least 512 columns per warp
    while (ks < DP_WARPS && units * ks < 148 * 4 * DP_WARPS && K % (ks * 2 * 8) == 0 && K / (ks * 2) >= 256) ks *= 2;
    const int groups = DP_WARPS / ks;
    const int proj_blocks = ceil_div(N, groups * 2), grid = proj_blocks + ceil_div(F, groups);
#define CALL(RR)                                                                                                                          \
    GLMB_LAUNCH(dual_proj_kernel<RR>, grid, DP_THREADS, 0, (cudaStream_t)stream, (const bf16*)x1, (const bf16*)x2, xs, rows, K, (const bf16*)w, N, \
                (bf16*)out, os, (const bf16*)wg, (const bf16*)wu, F, (bf16*)act, as, kind, proj_blocks, ks)
    if (rows <= 1) CALL(1);
    else if (rows <= 2) CALL(2);
    else if (rows <= 4) CALL(4);
    else CALL(8);
#undef CALL
    return (int)cudaGetLastError();
}
