// Arguments shared by the latent-attention kernels (latent.cu, latent_decode.cu).
#pragma once

#include "common.cuh"

struct LatentArgs {
    const void* proj; int64_t proj_stride;       // [rows, query latent at 0 | key/value latent, key part at off_kv | gate logits at off_gate | ..]
    int off_kv, off_gate;
    const float *q_norm, *kv_norm;               // [q_rank], [kv_rank]
    const float2* rot;                           // [capacity, rot / 2] (cos, sin)
    const int *row_pos, *row_lane, *row_active;  // row_active may be NULL
    void* cq; int64_t cq_stride;                 // [rows, q_rank padded to cq_stride]
    void* cache;                                 // [lanes, capacity, lat + pe]
    void* q;                                     // [rows, H, dimp]: dim unrotated, rot rotated dimensions, zeros
    const void* uk;                              // [H, dim, lat]
    void* qa;                                    // [rows, H, lat + pe]
    const void* o_lat;                           // [rows, H, kv_rank]
    const void* uv;                              // [H, vdim, lat]
    void* out; int64_t out_stride;               // [rows, H vdim]
    const float* sink;                           // [H]
    float *part_o, *part_ml;                     // [rows, H, parts, lat], [rows, H, parts, 2]: partial attention of a row (latent_decode.cu)
    int parts;
    int rows, H, dim, rot_dim, dimp, vdim, q_rank, kv_rank, lat, pe, lanes, capacity;
    float eps, scale;
    uint32_t* status;
};

__device__ __forceinline__ int latent_pos(const LatentArgs& a, int row, bool& ok) {
    const int pos = a.row_pos[row];
    ok = pos >= 0 && pos < a.capacity;
    if (!ok && threadIdx.x == 0 && (!a.row_active || a.row_active[row])) raise_status(a.status, GLMB_STATUS_BAD_INDEX);  // a frozen lane may be full
    return min(max(pos, 0), a.capacity - 1);
}

static inline bool latent_ok(const LatentArgs& a) {
    return a.rows >= 1 && a.rows <= 65535 && a.H >= 1 && a.H <= 65535 && a.dim >= 1 && a.rot_dim >= 2 && !(a.rot_dim & 1) && a.dimp >= a.dim + a.rot_dim && a.vdim >= 1 && a.q_rank >= 1 &&
           a.kv_rank >= 1 && a.lat >= a.kv_rank && a.pe >= a.rot_dim && !(a.lat & 1) && !(a.pe & 1) && a.lanes >= 1 && a.capacity >= 1 && a.row_pos && a.row_lane;
}
