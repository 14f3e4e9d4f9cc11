// Eight consecutive elements of an activation or weight row as fp32, whatever the element type (bf16: one 16-byte access, fp32: two).
// Kernels that serve both the bf16 path and the 32-bit path of a model are templates over the element type and use these.
#pragma once

#include "common.cuh"

__device__ __forceinline__ void load8(const bf16* p, float (&v)[8]) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y);
    v[4] = bf16_lo(u.z); v[5] = bf16_hi(u.z); v[6] = bf16_lo(u.w); v[7] = bf16_hi(u.w);
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void store8(bf16* p, const float (&v)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ void from_f32(float x, bf16& out) { out = __float2bfloat16_rn(x); }
__device__ __forceinline__ void from_f32(float x, float& out) { out = x; }

// Gated activations: 0 = SiLU, 1 = the tanh form of GELU.
enum { GLU_SILU = 0, GLU_GELU_TANH = 1 };
__device__ __forceinline__ float glu_activation(int kind, float z) {
    if (kind == GLU_SILU) return z * sigmoidf_precise(z);
    const float inner = 0.7978845608028654f * (z + 0.044715f * z * z * z);  // sqrt(2 / pi)
    return 0.5f * z * (1.0f + tanhf(inner));
}
