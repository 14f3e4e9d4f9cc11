// Routed experts with unquantized (bf16 or fp32) tables, where a token's weight scales the expert's input:
//
//   out_r = sum over the row's routes (e, w) of  W_down^e (f(W_gate^e (w h_r)) * (W_up^e (w h_r))) .
//
// The projections are linear, so w multiplies their fp32 sums and nothing is rounded twice.
//
//   expert_glu    decode and the 32-bit path: act[route] from the rows themselves, a warp per expert channel
//   expert_down   the same for the second half: the routes of a row are added in slot order in fp32
//   route_combine prefill: expert-sorted outputs of the grouped GEMM back to rows, added in slot order
//   gather_routes prefill: rows into expert order (zeros where there is no route)
#include "common.cuh"
#include "gemv_core.cuh"
#include "vec8.cuh"

#define MR_WARPS 8
#define MR_THREADS (MR_WARPS * 32)

template <typename T> struct ExpertDot;
template <> struct ExpertDot<bf16> {
    template <int N>
    static __device__ __forceinline__ void run(const bf16* x, const bf16* const (&w)[N], int K, int lane, float (&acc)[N]) {
        const bf16* const xr[1] = {x};
        float sum[N][1] = {};
        warp_dot_bf16<1, N>(xr, w, 0, K, lane, sum);
#pragma unroll
        for (int j = 0; j < N; ++j) acc[j] += warp_sum(sum[j][0]);
    }
};
template <> struct ExpertDot<float> {
    template <int N>
    static __device__ __forceinline__ void run(const float* x, const float* const (&w)[N], int K, int lane, float (&acc)[N]) {
        float sum[N] = {};
        for (int k = lane; k < K; k += 32)
#pragma unroll
            for (int j = 0; j < N; ++j) sum[j] = fmaf(x[k], w[j][k], sum[j]);
#pragma unroll
        for (int j = 0; j < N; ++j) acc[j] += warp_sum(sum[j]);
    }
};

// grid (pieces of MR_WARPS expert channels, routes).  gate_up [E, 2 F, K]: gate rows, then up rows.
template <typename T>
__global__ void __launch_bounds__(MR_THREADS)
expert_glu_kernel(const T* __restrict__ x, int64_t xs, int top, const int* __restrict__ ids, const float* __restrict__ weights, const T* __restrict__ gate_up,
                  int E, int F, int K, int kind, T* __restrict__ act, uint32_t* status) {
    GLMB_PDL_PROLOGUE();
    const int p = blockIdx.y, n = blockIdx.x * MR_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    int e = ids[p];
    if (e < 0 || e >= E) {
        if (threadIdx.x == 0) raise_status(status, GLMB_STATUS_BAD_INDEX);
        e = min(max(e, 0), E - 1);
    }
    if (n >= F) return;
    const T* const w[2] = {gate_up + ((int64_t)e * 2 * F + n) * K, gate_up + ((int64_t)e * 2 * F + F + n) * K};
    float acc[2] = {0.f, 0.f};
    ExpertDot<T>::template run<2>(x + (int64_t)(p / top) * xs, w, K, lane, acc);
    if (lane == 0) from_f32(glu_activation(kind, acc[0] * weights[p]) * (acc[1] * weights[p]), act[(int64_t)p * F + n]);
}

// grid (pieces of MR_WARPS output columns, rows).  down [E, N, F].
template <typename T>
__global__ void __launch_bounds__(MR_THREADS)
expert_down_kernel(const T* __restrict__ act, int top, const int* __restrict__ ids, const T* __restrict__ down, int E, int N, int F, float* __restrict__ out,
                   int64_t os) {
    GLMB_PDL_PROLOGUE();
    const int r = blockIdx.y, n = blockIdx.x * MR_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (n >= N) return;
    float total = 0.f;
    for (int s = 0; s < top; ++s) {
        const int64_t p = (int64_t)r * top + s;
        const int e = min(max(ids[p], 0), E - 1);
        const T* const w[1] = {down + ((int64_t)e * N + n) * F};
        float acc[1] = {0.f};
        ExpertDot<T>::template run<1>(act + p * F, w, F, lane, acc);
        total += acc[0];
    }
    if (lane == 0) out[(int64_t)r * os + n] = total;
}

// out[r] = sum over slots of y[place[r * top + slot]], place: route -> expert-sorted row.
__global__ void __launch_bounds__(256)
route_combine_kernel(const float* __restrict__ y, const int* __restrict__ place, int top, int routes, float* __restrict__ out, int width) {
    GLMB_PDL_PROLOGUE();
    const int r = blockIdx.x;
    for (int c = threadIdx.x * 4; c < width; c += 1024) {
        float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s = 0; s < top; ++s) {
            const int at = place[r * top + s];
            if (at < 0 || at >= routes) continue;
            const float4 v = *reinterpret_cast<const float4*>(y + (int64_t)at * width + c);
            t.x += v.x; t.y += v.y; t.z += v.z; t.w += v.w;
        }
        *reinterpret_cast<float4*>(out + (int64_t)r * width + c) = t;
    }
}

__global__ void __launch_bounds__(256)
gather_routes_kernel(const uint4* __restrict__ src, int64_t src_stride8, const int* __restrict__ perm, int top, int* __restrict__ place, uint4* __restrict__ dst,
                     int width8) {
    GLMB_PDL_PROLOGUE();
    const int i = blockIdx.x, p = perm[i];
    if (threadIdx.x == 0 && p >= 0) place[p] = i;
    for (int v = threadIdx.x; v < width8; v += 256) dst[(int64_t)i * width8 + v] = p >= 0 ? src[(int64_t)(p / top) * src_stride8 + v] : make_uint4(0, 0, 0, 0);
}

// ===================================================================================================
// x [rows, xs], ids / weights [rows, top], gate_up [E, 2 F, K], act [rows * top, F]; K and F multiples of 8.
GLMB_API int glmb_expert_glu(const void* x, int64_t xs, int rows, int top, const int* ids, const float* weights, const void* gate_up, int E, int F, int K,
                             int kind, void* act, int is_f32, uint32_t* status, void* stream) {
    if (rows < 1 || top < 1 || (int64_t)rows * top > 65535 || E < 1 || F < 1 || (K & 7) || K < 8 || (xs & 7) || (kind != GLU_SILU && kind != GLU_GELU_TANH)) return 1;
    const dim3 grid(ceil_div(F, MR_WARPS), rows * top);
    if (is_f32)
        GLMB_LAUNCH(expert_glu_kernel<float>, grid, MR_THREADS, 0, (cudaStream_t)stream, (const float*)x, xs, top, ids, weights, (const float*)gate_up, E, F, K, kind,
                    (float*)act, status);
    else
        GLMB_LAUNCH(expert_glu_kernel<bf16>, grid, MR_THREADS, 0, (cudaStream_t)stream, (const bf16*)x, xs, top, ids, weights, (const bf16*)gate_up, E, F, K, kind,
                    (bf16*)act, status);
    return (int)cudaGetLastError();
}

// out [rows, os] fp32, N columns; act [rows * top, F], down [E, N, F].
GLMB_API int glmb_expert_down(const void* act, int rows, int top, const int* ids, const void* down, int E, int N, int F, float* out, int64_t os, int is_f32,
                              void* stream) {
    if (rows < 1 || rows > 65535 || top < 1 || E < 1 || N < 1 || (F & 7) || F < 8) return 1;
    const dim3 grid(ceil_div(N, MR_WARPS), rows);
    if (is_f32)
        GLMB_LAUNCH(expert_down_kernel<float>, grid, MR_THREADS, 0, (cudaStream_t)stream, (const float*)act, top, ids, (const float*)down, E, N, F, out, os);
    else
        GLMB_LAUNCH(expert_down_kernel<bf16>, grid, MR_THREADS, 0, (cudaStream_t)stream, (const bf16*)act, top, ids, (const bf16*)down, E, N, F, out, os);
    return (int)cudaGetLastError();
}

// y [routes, width] fp32 in expert order -> out [rows, width]; width a multiple of 4, both contiguous.
GLMB_API int glmb_route_combine(const float* y, const int* place, int rows, int top, float* out, int width, void* stream) {
    if (rows < 1 || top < 1 || width < 4 || (width & 3)) return 1;
    GLMB_LAUNCH(route_combine_kernel, rows, 256, 0, (cudaStream_t)stream, y, place, top, rows * top, out, width);
    return (int)cudaGetLastError();
}

// dst [routes, width] = rows of src in the order of perm (route ids, -1: zeros); place becomes the inverse of perm.
GLMB_API int glmb_gather_routes(const void* src, int64_t src_stride, const int* perm, int routes, int top, int* place, void* dst, int width, void* stream) {
    if (routes < 1 || top < 1 || (width & 7) || width < 8 || (src_stride & 7)) return 1;
    GLMB_LAUNCH(gather_routes_kernel, routes, 256, 0, (cudaStream_t)stream, (const uint4*)src, src_stride / 8, perm, top, place, (uint4*)dst, width / 8);
    return (int)cudaGetLastError();
}
