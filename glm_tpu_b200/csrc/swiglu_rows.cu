// SwiGLU on whole rows for the prefill path: act = bf16( g * sigmoid(g) * u ) with g, u the bf16 outputs of the gate and up
// GEMMs, computed in fp32 and rounded once (the activation contract; the decode GEMVs and the grouped expert GEMM apply the
// same expression in their epilogues).  One launch instead of six elementwise library launches per layer and chunk.
//
// Reference counterpart: `glm_tpu/layers/mlp.py:21-51`.
#include "common.cuh"
#include "vec8.cuh"

__global__ void __launch_bounds__(256)
swiglu_rows_kernel(const uint4* __restrict__ gate, const uint4* __restrict__ up, uint4* __restrict__ act, int64_t n8) {
    GLMB_PDL_PROLOGUE();
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n8; i += (int64_t)gridDim.x * blockDim.x) {
        const uint4 g = gate[i], u = up[i];
        const uint32_t gw[4] = {g.x, g.y, g.z, g.w}, uw[4] = {u.x, u.y, u.z, u.w};
        uint32_t o[4];
#pragma unroll
        for (int p = 0; p < 4; ++p) {
            const float g0 = __uint_as_float(gw[p] << 16), g1 = __uint_as_float(gw[p] & 0xffff0000u);
            const float u0 = __uint_as_float(uw[p] << 16), u1 = __uint_as_float(uw[p] & 0xffff0000u);
            o[p] = pack_bf16(g0 * sigmoidf_precise(g0) * u0, g1 * sigmoidf_precise(g1) * u1);
        }
        act[i] = make_uint4(o[0], o[1], o[2], o[3]);
    }
}

// gate, up, act: contiguous bf16 arrays of n elements (n % 8 == 0), 16-byte aligned; act may alias gate.
GLMB_API int glmb_swiglu_rows(const void* gate, const void* up, void* act, int64_t n, void* stream) {
    if (n < 8 || (n & 7) || ((reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(up) | reinterpret_cast<uintptr_t>(act)) & 15)) return 1;
    const int64_t n8 = n / 8;
    const int64_t blocks = (n8 + 255) / 256;
    const int grid = blocks < 148 * 8 ? (int)blocks : 148 * 8;
    GLMB_LAUNCH(swiglu_rows_kernel, grid, 256, 0, (cudaStream_t)stream, (const uint4*)gate, (const uint4*)up, (uint4*)act, n8);
    return (int)cudaGetLastError();
}

// Gated activation of strided rows: act[r][i] = f(gate[r][i]) * up[r][i] for i < n (a multiple of 8), f by `kind` (vec8.cuh), arithmetic
// in fp32 and one rounding; with `scale`, both are first multiplied by scale[r], or by scale[scale_at[r]] (0 where that is negative).  gate and up may be the two halves of one projection's output, act the tail of a wider row.
template <typename T>
__global__ void __launch_bounds__(256)
glu_rows_kernel(const T* __restrict__ gate, const T* __restrict__ up, int64_t in_stride, T* __restrict__ act, int64_t out_stride, int rows, int n,
                int kind, const float* __restrict__ scale, const int* __restrict__ scale_at) {
    GLMB_PDL_PROLOGUE();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
    if (c >= n) return;
    for (int r = blockIdx.y; r < rows; r += gridDim.y) {
        float g[8], u[8];
        load8(gate + r * in_stride + c, g);
        load8(up + r * in_stride + c, u);
        if (scale) {
            const int at = scale_at ? scale_at[r] : r;
            const float w = at >= 0 ? scale[at] : 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) { g[e] *= w; u[e] *= w; }
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) g[e] = glu_activation(kind, g[e]) * u[e];
        store8(act + r * out_stride + c, g);
    }
}

// n and both strides multiples of 8 elements, all pointers 16-byte aligned.
GLMB_API int glmb_glu_rows(const void* gate, const void* up, int64_t in_stride, void* act, int64_t out_stride, int rows, int n, int kind, const float* scale,
                           const int* scale_at, int is_f32, void* stream) {
    if (rows < 1 || n < 8 || (n & 7) || (in_stride & 7) || (out_stride & 7) || (kind != GLU_SILU && kind != GLU_GELU_TANH)) return 1;
    if ((reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(up) | reinterpret_cast<uintptr_t>(act)) & 15) return 1;
    const dim3 grid(ceil_div(n / 8, 256), rows < 32768 ? rows : 32768);
    if (is_f32)
        GLMB_LAUNCH(glu_rows_kernel<float>, grid, 256, 0, (cudaStream_t)stream, (const float*)gate, (const float*)up, in_stride, (float*)act, out_stride,
                    rows, n, kind, scale, scale_at);
    else
        GLMB_LAUNCH(glu_rows_kernel<bf16>, grid, 256, 0, (cudaStream_t)stream, (const bf16*)gate, (const bf16*)up, in_stride, (bf16*)act, out_stride,
                    rows, n, kind, scale, scale_at);
    return (int)cudaGetLastError();
}
