// C[rows, N] = A[rows, K] . B[N, K]^T in plain fp32 (FMA units, no reduced-precision tensor mode): the projections of the 32-bit path,
// which exists to check a model against a 32-bit statement of it, at any row count and any size.
#include "common.cuh"

#define GF_TILE 64
#define GF_K 16

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ a, int64_t lda, const float* __restrict__ b, int64_t ldb, float* __restrict__ c, int64_t ldc, int rows, int N,
                int K) {
    GLMB_PDL_PROLOGUE();
    __shared__ float as[GF_K][GF_TILE + 4], bs[GF_K][GF_TILE + 4];
    const int m0 = blockIdx.y * GF_TILE, n0 = blockIdx.x * GF_TILE;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += GF_K) {
        for (int i = threadIdx.x; i < GF_TILE * GF_K; i += 256) {
            const int m = i / GF_K, k = i % GF_K;
            const bool in_k = k0 + k < K;
            as[k][m] = in_k && m0 + m < rows ? a[(int64_t)(m0 + m) * lda + k0 + k] : 0.f;
            bs[k][m] = in_k && n0 + m < N ? b[(int64_t)(n0 + m) * ldb + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < GF_K; ++k) {
            float x[4], y[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { x[i] = as[k][ty * 4 + i]; y[i] = bs[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (m0 + ty * 4 + i < rows && n0 + tx * 4 + j < N) c[(int64_t)(m0 + ty * 4 + i) * ldc + n0 + tx * 4 + j] = acc[i][j];
}

GLMB_API int glmb_gemm_f32(const float* a, int64_t lda, const float* b, int64_t ldb, float* c, int64_t ldc, int rows, int N, int K, void* stream) {
    if (rows < 1 || N < 1 || K < 1) return 1;
    GLMB_LAUNCH(gemm_f32_kernel, dim3(ceil_div(N, GF_TILE), ceil_div(rows, GF_TILE)), 256, 0, (cudaStream_t)stream, a, lda, b, ldb, c, ldc, rows, N, K);
    return (int)cudaGetLastError();
}
