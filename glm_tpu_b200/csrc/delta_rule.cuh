// Arguments shared by the gated-delta-rule kernels (delta_rule.cu and its tensor-core and fused forms).
#pragma once

#include "common.cuh"

struct DeltaArgs {
    const void* proj; int64_t proj_stride;       // [rows, q | k | v | beta logits at off_b | ..]
    int off_b;
    const float* conv_w; int taps;               // [taps, C], C = 2 G dim + H vdim
    void* conv_state;                            // [lanes, taps, C]: slot = position mod taps
    const float* a; int64_t a_stride;            // [rows, H dim]: the decay's projection, before bias and softplus
    const void *a2, *g2; int off_a, off_g, ra, rg;  // delta_step: second halves of the low-rank projections [H dim, ra], [H vdim, rg], inputs in proj
    const float *a_rate, *dt_bias;               // [H] (positive), [H dim]
    const int *row_pos, *row_lane, *row_active;  // row_active may be NULL
    float *q, *k, *v, *lg, *beta;                // [rows, G, dimp], same, [rows, H, vdim], [rows, H, dimp] (log of the decay), [rows, H]
    float* state;                                // [lanes, H, vdim, dimp]
    float* o;                                    // [rows, H, vdim]
    const void* gate; int64_t gate_stride;       // [rows, H vdim], before the sigmoid
    const float* norm;                           // [vdim]
    void* out; int64_t out_stride;               // [rows, H vdim]
    int H, G, dim, dimp, vdim, rows, decode, lanes, capacity, rows_per_block;  // dimp: dim padded to a multiple of 32 (zeros)
    float eps;
    uint32_t* status;
};

__device__ __forceinline__ int delta_lane(const DeltaArgs& a, int row) {
    const int lane = a.row_lane[row];
    if (lane >= 0 && lane < a.lanes) return lane;
    if (threadIdx.x == 0) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
    return min(max(lane, 0), a.lanes - 1);
}
__device__ __forceinline__ bool delta_writes(const DeltaArgs& a, int row) {  // an inactive row, or one at no position, leaves the lane as it is
    if (a.row_active && a.row_active[row] == 0) return false;
    const int pos = a.row_pos[row];
    if (pos >= 0 && pos < a.capacity) return true;
    if (threadIdx.x == 0) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
    return false;
}
// log(1 + e^z) = max(z, 0) + log(1 + e), e = e^-|z| in (0, 1]; log(1 + e) = 2 artanh(e / (2 + e)) by its power series, whose argument is at most
// 1/3: the first term left out is below 2^-27 of the sum, and small results keep their relative accuracy.
__device__ __forceinline__ float delta_softplus(float z) {
    const float e = expf(-fabsf(z)), s = __fdividef(e, 2.f + e), t = s * s;
    float sum = 1.f / 15.f;
    sum = fmaf(sum, t, 1.f / 13.f);
    sum = fmaf(sum, t, 1.f / 11.f);
    sum = fmaf(sum, t, 1.f / 9.f);
    sum = fmaf(sum, t, 1.f / 7.f);
    sum = fmaf(sum, t, 1.f / 5.f);
    sum = fmaf(sum, t, 1.f / 3.f);
    sum = fmaf(sum, t, 1.f);
    return fmaf(2.f * s, sum, fmaxf(z, 0.f));
}
__device__ __forceinline__ float delta_silu(float z) { return z * sigmoidf_precise(z); }

static inline bool delta_sizes_ok(const DeltaArgs& a) {
    return a.rows >= 1 && a.H >= 1 && a.G >= 1 && a.H % a.G == 0 && a.dim >= 1 && a.dim <= 256 && a.vdim >= 1 && a.dimp >= a.dim && !(a.dimp & 31) &&
           a.dimp <= 256 && a.lanes >= 1 && a.capacity >= 1 && a.row_pos && a.row_lane;
}
