// Skinny (1..8 row) weight-streaming projections for decode.
//
// With 1-8 live rows every projection of the decode step is bound by streaming the weight matrix from
// HBM once, so these kernels are organised around 16-byte streaming loads (L1 no-allocate), one warp per
// output feature (two when that shares the activation registers), fp32 accumulation and a fused epilogue:
// fp32/bf16 store, SwiGLU of a gate/up pair, or an in-kernel all-reduce over peer memory for K-split
// (tensor-parallel) projections.  The routed experts' FP8 counterparts are in moe_gemv.cu.
//
// Replaces: reference `glm_tpu/layers/linear.py:89-128` (+ psum), `layers/mlp.py:55-68`.
#include "common.cuh"
#include "gemv_core.cuh"
#include "peer.cuh"

#define SK_WARPS 8
#define SK_THREADS (SK_WARPS * 32)

// With programmatic dependent launch a kernel's CTAs become resident while its predecessor still runs and then wait for it.
// The weights do not depend on the predecessor, so before waiting a CTA asks the L2 for the rows it is about to stream: the HBM
// fetch overlaps the predecessor's tail instead of starting after it.  Tables larger than SK_PREFETCH_LIMIT are left alone (they
// would only sweep the L2).
#define SK_PREFETCH_LIMIT ((int64_t)48 << 20)
__device__ __forceinline__ void sk_prefetch_rows(const void* first_row, int rows, int64_t row_stride_elems, int K, int elem_bytes) {
    if (threadIdx.x != 0 || rows <= 0) return;
    const char* p = reinterpret_cast<const char*>(first_row);
    if (row_stride_elems == K) {
        const uint32_t bytes = (uint32_t)(((int64_t)rows * K * elem_bytes) & ~(int64_t)15);
        if (bytes && !((uintptr_t)p & 15)) asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(p), "r"(bytes) : "memory");
        return;
    }
    for (int r = 0; r < rows; ++r) {
        const char* q = p + (int64_t)r * row_stride_elems * elem_bytes;
        const uint32_t bytes = (uint32_t)(((int64_t)K * elem_bytes) & ~(int64_t)15);
        if (bytes && !((uintptr_t)q & 15)) asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(q), "r"(bytes) : "memory");
    }
}

// ---------------------------------------------------------------------------------------------------
// out[r][n] = sum_k x[r][k] * w[n][k]          (bf16 weights)
// ARGMAX compares bf16-rounded logits, ARGMAX_F32 the fp32 sums themselves.
enum { SK_OUT_F32 = 0, SK_OUT_BF16 = 1, SK_OUT_ALLREDUCE_BF16 = 2, SK_OUT_ARGMAX = 3, SK_OUT_ARGMAX_F32 = 4 };

// ks (1, 2, 4 or 8) warps of a CTA split K for the same pair of output rows and add their partial sums through
// shared memory: small-N projections then still fill the machine.  A CTA produces 16 / ks output rows.
template <int R>
__global__ void __launch_bounds__(SK_THREADS)
skinny_bf16_kernel(const bf16* __restrict__ x, int64_t xs, int rows, const bf16* __restrict__ w, int64_t ws, int N, int K,
                   void* __restrict__ out, int64_t os, int mode, int ks, int64_t xb, int64_t wb, int64_t ob, PeerComm comm,
                   int channel) {
    asm volatile("griddepcontrol.launch_dependents;");
    if ((int64_t)N * K * 2 * gridDim.y <= SK_PREFETCH_LIMIT) {
        const int first = blockIdx.x * (SK_WARPS / ks) * 2;
        sk_prefetch_rows(w + (int64_t)blockIdx.y * wb + (int64_t)first * ws, min((SK_WARPS / ks) * 2, N - first), ws, K, 2);
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    __shared__ float red[SK_WARPS][2][R];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int group = warp / ks, kpart = warp % ks, groups = SK_WARPS / ks;
    const int n0 = (blockIdx.x * groups + group) * 2;
    // blockIdx.y selects one problem of a batch (per-head projections): element offsets xb / wb / ob.
    x += (int64_t)blockIdx.y * xb;
    w += (int64_t)blockIdx.y * wb;
    out = mode == SK_OUT_F32 ? (void*)(reinterpret_cast<float*>(out) + (int64_t)blockIdx.y * ob)
                             : (void*)(reinterpret_cast<bf16*>(out) + (int64_t)blockIdx.y * ob);
    const bf16* xr[R];
#pragma unroll
    for (int r = 0; r < R; ++r) xr[r] = x + (int64_t)(r < rows ? r : 0) * xs;
    float acc[2][R];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int r = 0; r < R; ++r) acc[j][r] = 0.f;
    if (n0 < N) {
        const bf16* wp[2] = {w + (int64_t)n0 * ws, w + (int64_t)min(n0 + 1, N - 1) * ws};
        const int kspan = K / ks;
        warp_dot_bf16<R, 2>(xr, wp, kpart * kspan, (kpart + 1) * kspan, lane, acc);
        warp_reduce_all<R, 2>(acc);
    }
    if (ks > 1) {
        if (lane == 0) {
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int r = 0; r < R; ++r) red[warp][j][r] = acc[j][r];
        }
        __syncthreads();
        if (kpart == 0 && lane == 0) {
            for (int p = 1; p < ks; ++p)
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int r = 0; r < R; ++r) acc[j][r] += red[warp + p][j][r];
        }
    }
    const bool writer = lane == 0 && kpart == 0;
    if (mode == SK_OUT_ALLREDUCE_BF16) {
        __shared__ float sh[SK_WARPS * 2 * R];
        if (writer) {
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int r = 0; r < R; ++r) sh[(group * 2 + j) * R + r] = acc[j][r];
        }
        __syncthreads();
        cta_allreduce_f32(comm, channel, sh, groups * 2 * R);
        if (writer) {
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int r = 0; r < R; ++r)
                    if (n0 + j < N && r < rows)
                        reinterpret_cast<bf16*>(out)[(int64_t)r * os + n0 + j] = __float2bfloat16_rn(sh[(group * 2 + j) * R + r]);
        }
        return;
    }
    if (mode == SK_OUT_ARGMAX || mode == SK_OUT_ARGMAX_F32) {
        // out: unsigned long long best[rows]; `channel` carries the id of output column 0 (vocabulary offset).
        __shared__ unsigned long long best_s[SK_WARPS][R];
        if (lane == 0) {
#pragma unroll
            for (int r = 0; r < R; ++r) {
                unsigned long long key = 0ull;
#pragma unroll
                for (int j = 0; j < 2; ++j)
                    if (kpart == 0 && n0 + j < N) {
                        const float v = mode == SK_OUT_ARGMAX ? bf16_round(acc[j][r]) : acc[j][r];
                        if (!isfinite(v)) raise_status(comm.status, GLMB_STATUS_NONFINITE);
                        const unsigned long long k2 = candidate_key(v, channel + n0 + j);
                        key = k2 > key ? k2 : key;
                    }
                best_s[warp][r] = key;
            }
        }
        __syncthreads();
        if ((int)threadIdx.x < rows && (int)threadIdx.x < R) {
            unsigned long long key = 0ull;
#pragma unroll
            for (int w2 = 0; w2 < SK_WARPS; ++w2) key = best_s[w2][threadIdx.x] > key ? best_s[w2][threadIdx.x] : key;
            if (key) atomicMax(reinterpret_cast<unsigned long long*>(out) + threadIdx.x, key);
        }
        return;
    }
    if (writer && n0 < N) {
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int r = 0; r < R; ++r)
                if (n0 + j < N && r < rows) {
                    if (mode == SK_OUT_F32) reinterpret_cast<float*>(out)[(int64_t)r * os + n0 + j] = acc[j][r];
                    else reinterpret_cast<bf16*>(out)[(int64_t)r * os + n0 + j] = __float2bfloat16_rn(acc[j][r]);
                }
    }
}

// act[r][n] = bf16( silu(bf16(x.w_gate[n])) * bf16(x.w_up[n]) )       (bf16 weights; dense MLP / shared expert)
template <int R>
__global__ void __launch_bounds__(SK_THREADS)
skinny_bf16_swiglu_kernel(const bf16* __restrict__ x, int64_t xs, int rows, const bf16* __restrict__ wg,
                          const bf16* __restrict__ wu, int64_t ws, int N, int K, bf16* __restrict__ act, int64_t as, int ks) {
    asm volatile("griddepcontrol.launch_dependents;");
    if ((int64_t)N * K * 4 <= SK_PREFETCH_LIMIT) {
        const int first = blockIdx.x * (SK_WARPS / ks), cnt = min(SK_WARPS / ks, N - first);
        sk_prefetch_rows(wg + (int64_t)first * ws, cnt, ws, K, 2);
        sk_prefetch_rows(wu + (int64_t)first * ws, cnt, ws, K, 2);
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    __shared__ float red[SK_WARPS][2][R];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int group = warp / ks, kpart = warp % ks;
    const int n = blockIdx.x * (SK_WARPS / ks) + group;
    const bool valid = n < N;
    const bf16* xr[R];
#pragma unroll
    for (int r = 0; r < R; ++r) xr[r] = x + (int64_t)(r < rows ? r : 0) * xs;
    float acc[2][R];
#pragma unroll
    for (int r = 0; r < R; ++r) acc[0][r] = acc[1][r] = 0.f;
    if (valid) {
        const bf16* wp[2] = {wg + (int64_t)n * ws, wu + (int64_t)n * ws};
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
        for (int r = 0; r < R; ++r)
            if (r < rows) {
                const float g = bf16_round(acc[0][r]), u = bf16_round(acc[1][r]);
                act[(int64_t)r * as + n] = __float2bfloat16_rn(g * sigmoidf_precise(g) * u);
            }
    }
}

// ===================================================================================================
// Host launchers
#define DISPATCH_R(rows, CALL)                                \
    do {                                                      \
        if ((rows) <= 1) { CALL(1); }                         \
        else if ((rows) <= 2) { CALL(2); }                    \
        else if ((rows) <= 4) { CALL(4); }                    \
        else { CALL(8); }                                     \
    } while (0)

// How many warps share one unit of output (a row pair or a gate/up pair) so that about four CTAs land on every SM.
static int pick_ksplit(int units, int K) {
    int ks = 1;
    while (ks < SK_WARPS && units * ks < 148 * 4 * SK_WARPS && K % (ks * 2 * 256) == 0 && K / (ks * 2) >= 512) ks *= 2;
    return ks;
}

// x [rows<=8, K] bf16, w [N, K] bf16 -> out [rows, N] (fp32, bf16, or all-reduced bf16).  K % 8 == 0.
// batch > 1 runs `batch` independent problems whose x / w / out start xb / wb / ob elements apart.
GLMB_API int glmb_skinny_bf16(const void* x, int64_t xs, int rows, const void* w, int64_t ws, int N, int K, void* out, int64_t os,
                              int mode, int batch, int64_t xb, int64_t wb, int64_t ob, const PeerComm* comm, int channel,
                              void* stream) {
    if (rows < 1 || rows > GLMB_MAX_ROWS || (K & 7) || (xs & 7) || (ws & 7) || (xb & 7) || (wb & 7) || batch < 1) return 1;
    int ks = pick_ksplit(ceil_div(N, 2) * batch, K);
    PeerComm c = comm ? *comm : single_comm();
    // A CTA that all-reduces waits for the same CTA of every peer before it retires.  CTAs beyond the first wave would start only
    // after such a wait and then wait again: keep the grid within one wave (three CTAs per SM fit whatever the row count).
    if (mode == SK_OUT_ALLREDUCE_BF16 && c.world > 1)
        while (ks > 1 && ceil_div(N, (SK_WARPS / ks) * 2) * batch > 148 * 3) ks >>= 1;
    const dim3 grid(ceil_div(N, (SK_WARPS / ks) * 2), batch);
    if (mode == SK_OUT_ALLREDUCE_BF16 && c.world > 1 && (int)(grid.x * grid.y) > GLMB_AR_MAX_CTAS) return 2;
    if (mode == SK_OUT_ALLREDUCE_BF16 && c.world == 1) mode = SK_OUT_BF16;
#define CALL(RR)                                                                                                   \
    GLMB_LAUNCH(skinny_bf16_kernel<RR>, grid, SK_THREADS, 0, (cudaStream_t)stream, (const bf16*)x, xs, rows, (const bf16*)w, ws, N, K, \
                                                                          out, os, mode, ks, xb, wb, ob, c, channel)
    DISPATCH_R(rows, CALL);
#undef CALL
    return (int)cudaGetLastError();
}

GLMB_API int glmb_skinny_bf16_swiglu(const void* x, int64_t xs, int rows, const void* wg, const void* wu, int64_t ws, int N, int K,
                                     void* act, int64_t as, void* stream) {
    if (rows < 1 || rows > GLMB_MAX_ROWS || (K & 7) || (xs & 7) || (ws & 7)) return 1;
    const int ks = pick_ksplit(N, K);
    const int grid = ceil_div(N, SK_WARPS / ks);
#define CALL(RR)                                                                                                          \
    GLMB_LAUNCH(skinny_bf16_swiglu_kernel<RR>, grid, SK_THREADS, 0, (cudaStream_t)stream, (const bf16*)x, xs, rows, (const bf16*)wg, \
                                                                                 (const bf16*)wu, ws, N, K, (bf16*)act, as, ks)
    DISPATCH_R(rows, CALL);
#undef CALL
    return (int)cudaGetLastError();
}
