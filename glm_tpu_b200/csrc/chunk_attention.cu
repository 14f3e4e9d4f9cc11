// Causal attention inside chunks of the sequence, grouped query heads, a sink per query head:
//
//   query i sees key j  <=>  j <= i and j / chunk == i / chunk          (chunks counted from position 0 of the sequence)
//   out_i = sum_j exp(s_ij) v_j / (exp(sink_h) + sum_j exp(s_ij)),       s_ij = scale * q_i . k_j
//
// Prefill: the rows are consecutive positions of one sequence and every key they can see lies in linear buffers whose row 0 is position
// `base` (the lane's ring itself, or a copy of its current chunk followed by the step's rows).  Decode: one row per lane, the keys are in
// the lane's ring (slot = position mod ring; a ring holds a whole chunk, so the current chunk starts at slot 0).  Scores, exponentials and
// sums are fp32; the weights enter the product with the values as two bf16 pieces (value and remainder): 16 bits of mantissa.
//
//   chunk_attn_tc_kernel       prefill, bf16, head sizes up to 128: tcgen05, see chunk_attention_tcgen05.cu
//   chunk_attn_prefill_kernel  prefill, bf16, head sizes up to 256: 64 query rows of one head per CTA, mma.sync, cp.async double buffer
//   chunk_attn_decode_kernel   decode, bf16, head sizes up to 256: up to 16 query heads of one key head per cluster; key tiles come in by
//                              TMA and are dealt to the cluster's CTAs, the partial softmax states meet in distributed shared memory
//   chunk_attn_any_kernel      any head size and element type, one CTA per (row, head): the 32-bit path and larger heads
//
// The running maximum starts at the sink and the sum gets the sink's term once; the sink has no value.  A gate per row and head may scale
// the output.
#include <cooperative_groups.h>

#include "attention_core.cuh"
#include "chunk_attention.cuh"
#include "common.cuh"
#include "tcgen05.cuh"
#include "vec8.cuh"

namespace cg = cooperative_groups;

#define CA_LOG2E 1.4426950408889634f  // log2(e)

__device__ __forceinline__ int ca_lane(const ChunkAttnArgs& a, int row) {
    const int lane = a.row_lane[row];
    if (lane >= 0 && lane < a.lanes) return lane;
    if (threadIdx.x == 0) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
    return min(max(lane, 0), a.lanes - 1);
}
__device__ __forceinline__ int ca_pos(const ChunkAttnArgs& a, int row) {
    const int pos = a.row_pos[row];
    if (pos >= 0 && pos < a.capacity) return pos;
    if (threadIdx.x == 0 && (!a.row_active || a.row_active[row])) raise_status(a.status, GLMB_STATUS_BAD_INDEX);  // a frozen lane may be full
    return min(max(pos, 0), a.capacity - 1);
}
// bf16 value and bf16 remainder of two weights, packed as mma operands
__device__ __forceinline__ void ca_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x, y);
    lo = pack_bf16(x - bf16_lo(hi), y - bf16_hi(hi));
}
__device__ __forceinline__ void ca_store2(bf16* p, float x, float y, bool both, bool aligned) {
    if (both && aligned) {
        *reinterpret_cast<uint32_t*>(p) = pack_bf16(x, y);
    } else {
        p[0] = __float2bfloat16_rn(x);
        if (both) p[1] = __float2bfloat16_rn(y);
    }
}

template <typename T>
__device__ __forceinline__ float ca_gate(const ChunkAttnArgs& a, int row, int head) {
    return a.gate ? sigmoidf_precise(to_f32(reinterpret_cast<const T*>(a.gate)[(int64_t)row * a.gate_stride + head])) : 1.f;
}

// ---------------------------------------------------------------------------------------------------
#define CP_ROWS 64
#define CP_KEYS 64
#define CP_THREADS 128

static inline size_t chunk_prefill_smem(int dk, int dv) {  // dk, dv: head sizes rounded up to 16
    return (size_t)(CP_ROWS * (dk + 8) + 2 * CP_KEYS * (dk + 8) + 2 * CP_KEYS * (dv + 8)) * 2;
}

// DV: columns of the output accumulator (the value size rounded up to it).
template <int DV>
__global__ void __launch_bounds__(CP_THREADS) chunk_attn_prefill_kernel(ChunkAttnArgs a) {
    GLMB_PDL_PROLOGUE();
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int dk = a.dimp, dv = a.vdimp;
    const int KP = dk + 8, VP = dv + 8;  // padded rows (elements): 16-byte aligned, banks staggered for ldmatrix
    bf16* q_s = reinterpret_cast<bf16*>(smem_raw);
    bf16* k_s = q_s + CP_ROWS * KP;
    bf16* v_s = k_s + 2 * CP_KEYS * KP;
    const int head = blockIdx.y, group = head / (a.H / a.G);
    const int r0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * CP_ROWS;  // the rows with most keys (towards a chunk's end) first
    const int nrows = min(CP_ROWS, a.rows - r0);
    const int first = a.start + r0, last = first + nrows - 1;
    const int key0 = first / a.chunk * a.chunk;
    const int tiles = max((last - key0) / CP_KEYS + 1, 1);
    const bf16* k_head = reinterpret_cast<const bf16*>(a.k) + (int64_t)group * a.dimp;
    const bf16* v_head = reinterpret_cast<const bf16*>(a.v) + (int64_t)group * a.vdimp;
    const int tid = threadIdx.x;

    auto load_rows = [&](bf16* dst, int stride, int pieces, const bf16* src, int padded, int key_base) {
        for (int i = tid; i < CP_KEYS * pieces; i += CP_THREADS) {
            const int r = i / pieces, c = i % pieces, key = key_base + r;
            bf16* d = dst + r * stride + c * 8;
            if (key > last) *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
            else cp_async16(d, src + (int64_t)(key - a.base) * a.G * padded + c * 8);
        }
    };
    auto load_tile = [&](int t) {
        load_rows(k_s + (t & 1) * CP_KEYS * KP, KP, dk / 8, k_head, a.dimp, key0 + t * CP_KEYS);
        load_rows(v_s + (t & 1) * CP_KEYS * VP, VP, dv / 8, v_head, a.vdimp, key0 + t * CP_KEYS);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    {
        const bf16* q = reinterpret_cast<const bf16*>(a.q) + (int64_t)r0 * a.q_stride + (int64_t)head * a.dimp;
        const int pieces = dk / 8;
        for (int i = tid; i < CP_ROWS * pieces; i += CP_THREADS) {
            const int r = i / pieces, c = i % pieces;
            bf16* d = q_s + r * KP + c * 8;
            if (r < nrows) cp_async16(d, q + (int64_t)r * a.q_stride + c * 8);
            else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
        }
    }
    load_tile(0);

    const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int mr = lane & 7, mi = lane >> 3;
    const float scale2 = a.scale * CA_LOG2E;
    const float sink2 = a.sink ? a.sink[head] * CA_LOG2E : -INFINITY;
    float m[2] = {sink2, sink2}, l[2] = {0.f, 0.f};  // the sink's own term joins the sum at the end
    int pos[2], lo[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        pos[i] = first + warp * 16 + g + 8 * i;
        lo[i] = pos[i] / a.chunk * a.chunk;
    }
    const int warp_last = first + warp * 16 + 15, warp_lo = (first + warp * 16) / a.chunk * a.chunk;
    float o[DV / 8][4];
#pragma unroll
    for (int j = 0; j < DV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;

    for (int t = 0; t < tiles; ++t) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (t + 1 < tiles) load_tile(t + 1);
        const int key_base = key0 + t * CP_KEYS;
        if (key_base > warp_last || key_base + CP_KEYS <= warp_lo) continue;  // nothing in this tile for the warp's rows
        const bf16* kt = k_s + (t & 1) * CP_KEYS * KP;
        const bf16* vt = v_s + (t & 1) * CP_KEYS * VP;
        float s[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
        const bf16* qa = q_s + (warp * 16 + mr + 8 * (mi & 1)) * KP + 8 * (mi >> 1);
        const bf16* kb = kt + (mr + 8 * (mi >> 1)) * KP + 8 * (mi & 1);
        for (int k0 = 0; k0 < dk; k0 += 16) {
            uint32_t qf[4];
            ldmatrix_x4(qf, qa + k0);
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                uint32_t kf[4];
                ldmatrix_x4(kf, kb + j * 8 * KP + k0);
                mma_bf16_16816(s[j], qf, kf[0], kf[1]);
                mma_bf16_16816(s[j + 1], qf, kf[2], kf[3]);
            }
        }
        const bool edge = key_base < (warp_last / a.chunk * a.chunk) || key_base + CP_KEYS - 1 > first + warp * 16;
        float mx[2] = {m[0], m[1]};
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int key = key_base + j * 8 + 2 * t4 + (e & 1), i = e >> 1;
                float x = s[j][e] * scale2;
                if (edge && (key > pos[i] || key < lo[i])) x = -INFINITY;
                s[j][e] = x;
                mx[i] = fmaxf(mx[i], x);
            }
        float fix[2], base[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
            base[i] = mx[i] == -INFINITY ? 0.f : mx[i];
            fix[i] = exp2f(m[i] - base[i]);
            m[i] = mx[i];
        }
        float sum[2] = {0.f, 0.f};
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                s[j][e] = exp2f(s[j][e] - base[e >> 1]);
                sum[e >> 1] += s[j][e];
            }
        l[0] = l[0] * fix[0] + sum[0];  // this thread's keys; the four threads of a row meet at the end
        l[1] = l[1] * fix[1] + sum[1];
#pragma unroll
        for (int j = 0; j < DV / 8; ++j) { o[j][0] *= fix[0]; o[j][1] *= fix[0]; o[j][2] *= fix[1]; o[j][3] *= fix[1]; }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t hi[4], lw[4];
            ca_split(s[2 * kk][0], s[2 * kk][1], hi[0], lw[0]);
            ca_split(s[2 * kk][2], s[2 * kk][3], hi[1], lw[1]);
            ca_split(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lw[2]);
            ca_split(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lw[3]);
            const bf16* vb = vt + (kk * 16 + mr + 8 * (mi & 1)) * VP + 8 * (mi >> 1);
#pragma unroll
            for (int j = 0; j < DV / 8; j += 2)
                if (j * 8 < dv) {
                    uint32_t vf[4];
                    ldmatrix_x4_trans(vf, vb + j * 8);
                    mma_bf16_16816(o[j], hi, vf[0], vf[1]);
                    mma_bf16_16816(o[j + 1], hi, vf[2], vf[3]);
                    mma_bf16_16816(o[j], lw, vf[0], vf[1]);
                    mma_bf16_16816(o[j + 1], lw, vf[2], vf[3]);
                }
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
        if (a.sink) l[i] += exp2f(sink2 - m[i]);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = warp * 16 + g + 8 * i;
        if (r >= nrows) continue;
        bf16* dst = reinterpret_cast<bf16*>(a.out) + (int64_t)(r0 + r) * a.out_stride + (int64_t)head * a.vdim;
        const bool aligned = !(reinterpret_cast<uintptr_t>(dst) & 3);
        const float inv = ca_gate<bf16>(a, r0 + r, head) / l[i];
#pragma unroll
        for (int j = 0; j < DV / 8; ++j) {
            const int c = j * 8 + 2 * t4;
            if (c < a.vdim) ca_store2(dst + c, o[j][2 * i] * inv, o[j][2 * i + 1] * inv, c + 1 < a.vdim, aligned);
        }
    }
}

// ---------------------------------------------------------------------------------------------------
#define CD_HEADS 16
// A tile is 16 keys per warp: WARPS * 16 keys, in 64-column boxes of 128-byte rows (128-byte swizzle).

static inline int cd_boxes(int padded) { return (padded + 63) / 64; }
static inline size_t chunk_decode_smem(int dk, int dv, int stages, int warps) {
    const size_t tiles = (size_t)stages * (cd_boxes(dk) + cd_boxes(dv)) * warps * 16 * 128, merge = (size_t)warps * CD_HEADS * dv * 4;
    return 1024 + (tiles > merge ? tiles : merge) + (size_t)CD_HEADS * (dk + 8) * 2;
}

__device__ __forceinline__ uint32_t movmatrix_trans(uint32_t x) {  // 8 x 8 matrix of 16-bit elements, transposed across the warp
    uint32_t y;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
    return y;
}

// grid (splits, key heads x blocks of 16 query heads, rows), cluster (splits, 1, 1).
// A warp's 16 keys are the M of both products (scores: keys x heads; output: value columns x heads), the query heads the N (NT tiles of 8):
// with the handful of query heads that share a key head, few multiplications are spent on padding.
template <int DV, int WARPS, int NT>
__global__ void __launch_bounds__(WARPS * 32)
chunk_attn_decode_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, ChunkAttnArgs a, int stages) {
    constexpr int KEYS = WARPS * 16, BOX = KEYS * 128, HEADS = NT * 8;
    cg::cluster_group cluster = cg::this_cluster();
    extern __shared__ unsigned char smem_raw[];
    __shared__ float ml_s[WARPS][HEADS][2];  // (maximum, sum) per warp
    __shared__ __align__(8) float cta_ml[HEADS][2];
    __shared__ __align__(8) uint64_t full_bar[4];
    const int dk = a.dimp, dv = a.vdimp, KP = dk + 8;
    const int kboxes = (dk + 63) / 64, vboxes = (dv + 63) / 64;
    unsigned char* tiles_s = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const size_t stage_bytes = (size_t)(kboxes + vboxes) * BOX;
    const size_t tile_area = stages * stage_bytes, merge_area = (size_t)WARPS * HEADS * dv * 4;
    bf16* q_s = reinterpret_cast<bf16*>(tiles_s + (tile_area > merge_area ? tile_area : merge_area));
    if (threadIdx.x == 0) {
        for (int s = 0; s < stages; ++s) mbar_init(full_bar + s, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    GLMB_PDL_PROLOGUE();
    const int per = a.H / a.G, head_blocks = (per + CD_HEADS - 1) / CD_HEADS;
    const int group = blockIdx.y / head_blocks, h0 = group * per + (blockIdx.y % head_blocks) * CD_HEADS;
    const int heads = min(CD_HEADS, group * per + per - h0);
    const int row = blockIdx.z, split = blockIdx.x, splits = gridDim.x;
    const bool active = !a.row_active || a.row_active[row] != 0;
    const int pos = ca_pos(a, row), lane_id = ca_lane(a, row);
    const int keys = active ? pos % a.chunk + 1 : 0;  // slots 0 .. keys - 1 of the lane's ring
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3, mr = lane & 7, mi = lane >> 3;
    const int tiles = (keys + KEYS - 1) / KEYS, mine = tiles > split ? (tiles - split - 1) / splits + 1 : 0;  // tiles split, split + splits, ..

    auto load_tile = [&](int i) {  // the i-th tile of this CTA, by one thread
        unsigned char* dst = tiles_s + (size_t)(i % stages) * stage_bytes;
        uint64_t* bar = full_bar + i % stages;
        const int y = lane_id * a.ring + (split + i * splits) * KEYS;
        mbar_expect_tx(bar, (uint32_t)stage_bytes);
        for (int b = 0; b < kboxes; ++b) tma_load_2d(dst + b * BOX, &map_k, bar, group * dk + b * 64, y);
        for (int b = 0; b < vboxes; ++b) tma_load_2d(dst + (kboxes + b) * BOX, &map_v, bar, group * dv + b * 64, y);
    };
    if (threadIdx.x == 0)
        for (int i = 0; i < min(stages, mine); ++i) load_tile(i);
    {
        const bf16* q = reinterpret_cast<const bf16*>(a.q) + (int64_t)row * a.q_stride + (int64_t)h0 * dk;
        const int pieces = dk / 8;
        for (int i = threadIdx.x; i < HEADS * pieces; i += WARPS * 32) {
            const int r = i / pieces, c = i % pieces;
            *reinterpret_cast<uint4*>(q_s + r * KP + c * 8) = r < heads ? *reinterpret_cast<const uint4*>(q + (int64_t)r * dk + c * 8) : make_uint4(0, 0, 0, 0);
        }
    }
    __syncthreads();

    const float scale2 = a.scale * CA_LOG2E;
    float m[NT][2], l[NT][2];  // of heads 8 n + 2 t4 + e, equal on the lanes that share t4 (m) or this lane's keys (l)
    float o[DV / 16][NT][4];   // value columns 16 j + g, + 8; heads 8 n + 2 t4, + 1
#pragma unroll
    for (int n = 0; n < NT; ++n) {
        m[n][0] = m[n][1] = -INFINITY;
        l[n][0] = l[n][1] = 0.f;
#pragma unroll
        for (int j = 0; j < DV / 16; ++j) o[j][n][0] = o[j][n][1] = o[j][n][2] = o[j][n][3] = 0.f;
    }
    // this lane's rows of a key / value fragment and its 16-byte pieces of a 128-byte row, as they lie swizzled
    const int k_row = (mr + 8 * (mi & 1)) * 128, v_row = (mr + 8 * (mi >> 1)) * 128;
    int k_col[4], v_col[4];
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        k_col[c] = ((2 * c + (mi >> 1)) ^ mr) << 4;
        v_col[c] = ((2 * c + (mi & 1)) ^ mr) << 4;
    }
    const bf16* q_lane = q_s + (mr + (NT == 2 ? 8 * (mi >> 1) : 0)) * KP + 8 * (mi & 1);
    constexpr int QSTEPS = DV <= 128 ? 8 : 1;  // query fragments of head sizes up to 128 stay in registers
    uint32_t qf[QSTEPS][2 * NT];
    auto load_q = [&](uint32_t (&f)[2 * NT], int k0) {
        if constexpr (NT == 2) ldmatrix_x4(f, q_lane + k0);
        else ldmatrix_x2(f, q_lane + k0);
    };
    if constexpr (QSTEPS > 1) {
#pragma unroll
        for (int c = 0; c < QSTEPS; ++c)
            if (c * 16 < dk) load_q(qf[c], c * 16);
    }
    bool ok = true;
    for (int i = 0; i < mine; ++i) {
        const int stage = i % stages, slot0 = (split + i * splits) * KEYS;
        if (ok && !mbar_wait(full_bar + stage, (i / stages) & 1)) {
            if (lane == 0) raise_status(a.status, GLMB_STATUS_WAIT_TIMEOUT);
            ok = false;  // no more work for this warp, but it still meets the others at their barriers
        }
        unsigned char* kt = tiles_s + (size_t)stage * stage_bytes;
        unsigned char* vt = kt + kboxes * BOX;
        const int w0 = warp * 16, left = ok ? keys - slot0 - w0 : 0;  // this warp's keys of the tile, how many of them exist
        if (left > 0 && left < 16) {  // values past the last key meet zero weights: they must not be infinite or NaN
            for (int x = lane; x < (16 - left) * vboxes * 8; x += 32)
                *reinterpret_cast<uint4*>(vt + (x % (vboxes * 8) >> 3) * BOX + (w0 + left + x / (vboxes * 8)) * 128 + (x & 7) * 16) = make_uint4(0, 0, 0, 0);
            __syncwarp();
        }
        if (left > 0) {
            float s[NT][4];  // keys g, g + 8; heads 8 n + 2 t4, + 1
#pragma unroll
            for (int n = 0; n < NT; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
            const unsigned char* kb = kt + w0 * 128 + k_row;
            auto step = [&](const uint32_t (&f)[2 * NT], const unsigned char* at) {
                uint32_t kf[4];
                ldmatrix_x4(kf, at);
#pragma unroll
                for (int n = 0; n < NT; ++n) mma_bf16_16816(s[n], kf, f[2 * n], f[2 * n + 1]);
            };
            if constexpr (QSTEPS > 1) {
#pragma unroll
                for (int c = 0; c < QSTEPS; ++c)
                    if (c * 16 < dk) step(qf[c], kb + (c >> 2) * BOX + k_col[c & 3]);
            } else {
                for (int k0 = 0; k0 < dk; k0 += 64, kb += BOX)
#pragma unroll
                    for (int c = 0; c < 4; ++c)
                        if (k0 + c * 16 < dk) {
                            load_q(qf[0], k0 + c * 16);
                            step(qf[0], kb + k_col[c]);
                        }
            }
            uint32_t hi[NT][2], lw[NT][2];  // weights as the second operand: keys x heads
            float fix[NT][2];
#pragma unroll
            for (int n = 0; n < NT; ++n) {
#pragma unroll
                for (int e = 0; e < 4; ++e) s[n][e] = g + 8 * (e >> 1) >= left ? -INFINITY : s[n][e] * scale2;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float top = fmaxf(s[n][e], s[n][2 + e]);
                    top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 4));
                    top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 8));
                    top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 16));
                    top = fmaxf(top, m[n][e]);  // at least one key exists: finite
                    fix[n][e] = exp2f(m[n][e] - top);
                    m[n][e] = top;
                    s[n][e] = exp2f(s[n][e] - top);
                    s[n][2 + e] = exp2f(s[n][2 + e] - top);
                    l[n][e] = l[n][e] * fix[n][e] + s[n][e] + s[n][2 + e];
                }
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    uint32_t x, y;
                    ca_split(s[n][2 * e], s[n][2 * e + 1], x, y);
                    hi[n][e] = movmatrix_trans(x);
                    lw[n][e] = movmatrix_trans(y);
                }
            }
            bool moved = false;
#pragma unroll
            for (int n = 0; n < NT; ++n) moved |= fix[n][0] != 1.f || fix[n][1] != 1.f;
            moved = __any_sync(0xffffffffu, moved);
#pragma unroll
            for (int j = 0; j < DV / 16; ++j)
                if (j * 16 < dv) {
                    uint32_t vf[4];
                    ldmatrix_x4_trans(vf, vt + (j >> 2) * BOX + w0 * 128 + v_row + v_col[j & 3]);
#pragma unroll
                    for (int n = 0; n < NT; ++n) {
                        if (moved) { o[j][n][0] *= fix[n][0]; o[j][n][1] *= fix[n][1]; o[j][n][2] *= fix[n][0]; o[j][n][3] *= fix[n][1]; }
                        mma_bf16_16816(o[j][n], vf, hi[n][0], hi[n][1]);
                        mma_bf16_16816(o[j][n], vf, lw[n][0], lw[n][1]);
                    }
                }
        }
        if (i + stages < mine) {  // every warp has read the stage: fill it again
            __syncthreads();
            if (threadIdx.x == 0) load_tile(i + stages);
        }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            float sum = l[n][e];
            sum += __shfl_xor_sync(0xffffffffu, sum, 4);
            sum += __shfl_xor_sync(0xffffffffu, sum, 8);
            sum += __shfl_xor_sync(0xffffffffu, sum, 16);
            if (g == 0) { ml_s[warp][n * 8 + 2 * t4 + e][0] = m[n][e]; ml_s[warp][n * 8 + 2 * t4 + e][1] = sum; }
        }
    __syncthreads();  // every warp has left the tiles: the merge area takes their place
    float* o_s = reinterpret_cast<float*>(tiles_s);  // [warp][head][dv]
#pragma unroll
    for (int j = 0; j < DV / 16; ++j)
        if (j * 16 < dv)
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) o_s[((size_t)warp * HEADS + n * 8 + 2 * t4 + (e & 1)) * dv + j * 16 + g + 8 * (e >> 1)] = o[j][n][e];
    __syncthreads();
    // ---- warps of the CTA into warp 0's area ------------------------------------------------------------
    if (threadIdx.x < HEADS) {
        float top = -INFINITY, sum = 0.f;
        for (int w = 0; w < WARPS; ++w) top = fmaxf(top, ml_s[w][threadIdx.x][0]);
        for (int w = 0; w < WARPS; ++w)
            if (ml_s[w][threadIdx.x][0] != -INFINITY) sum += ml_s[w][threadIdx.x][1] * exp2f(ml_s[w][threadIdx.x][0] - top);
        cta_ml[threadIdx.x][0] = top;
        cta_ml[threadIdx.x][1] = sum;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < HEADS * dv; i += WARPS * 32) {
        const int h = i / dv;
        const float top = cta_ml[h][0];
        float v = 0.f;
        for (int w = 0; w < WARPS; ++w)
            if (ml_s[w][h][0] != -INFINITY) v += o_s[(size_t)w * HEADS * dv + i] * exp2f(ml_s[w][h][0] - top);
        o_s[i] = v;
    }
    cluster.sync();
    // ---- CTAs of the cluster: each finishes its share of the outputs, the sink joins here -----------------
    // First every CTA's (maximum, sum) of every head, all loads at once, then a weight per CTA and head.
    __shared__ float part_s[16][HEADS][2];
    for (int i = threadIdx.x; i < splits * HEADS; i += WARPS * 32) {
        const float2 ml = *reinterpret_cast<const float2*>(cluster.map_shared_rank(&cta_ml[0][0], i / HEADS) + (i % HEADS) * 2);
        part_s[i / HEADS][i % HEADS][0] = ml.x;
        part_s[i / HEADS][i % HEADS][1] = ml.y;
    }
    __syncthreads();
    if ((int)threadIdx.x < heads) {
        const int h = threadIdx.x;
        const float sink2 = a.sink ? a.sink[h0 + h] * CA_LOG2E : -INFINITY;
        float top = sink2;
        for (int p = 0; p < splits; ++p) top = fmaxf(top, part_s[p][h][0]);
        float sum = a.sink ? exp2f(sink2 - top) : 0.f;
        for (int p = 0; p < splits; ++p) {
            const float w = part_s[p][h][0] == -INFINITY ? 0.f : exp2f(part_s[p][h][0] - top);
            sum += part_s[p][h][1] * w;
            part_s[p][h][0] = w;
        }
        const float inv = sum > 0.f ? ca_gate<bf16>(a, row, h0 + h) / sum : 0.f;
        for (int p = 0; p < splits; ++p) part_s[p][h][0] *= inv;
    }
    __syncthreads();
    const int total = heads * a.vdim;
    bf16* out = reinterpret_cast<bf16*>(a.out) + (int64_t)row * a.out_stride + (int64_t)h0 * a.vdim;
    for (int i = split * WARPS * 32 + threadIdx.x; i < total; i += splits * WARPS * 32) {
        const int h = i / a.vdim, c = i % a.vdim;
        float v = 0.f;
#pragma unroll 16
        for (int p = 0; p < splits; ++p) v = fmaf(cluster.map_shared_rank(o_s, p)[h * dv + c], part_s[p][h][0], v);
        out[i] = __float2bfloat16_rn(v);
    }
    cluster.sync();  // nobody leaves while a peer may still read its shared memory
}

// ---------------------------------------------------------------------------------------------------
#define CX_THREADS 128
#define CX_KEYS 128
#define CX_COLS 8  // value columns per thread: value sizes up to 1024

template <typename T>
__global__ void __launch_bounds__(CX_THREADS) chunk_attn_any_kernel(ChunkAttnArgs a) {
    GLMB_PDL_PROLOGUE();
    extern __shared__ float q_f[];  // [dim]
    __shared__ float p_s[CX_KEYS];
    __shared__ float red[CX_THREADS / 32];
    const int row = blockIdx.x, head = blockIdx.y, group = head / (a.H / a.G);
    const bool active = !a.decode || !a.row_active || a.row_active[row] != 0;
    const int pos = a.decode ? ca_pos(a, row) : a.start + row;
    const int key0 = pos / a.chunk * a.chunk, keys = active ? pos - key0 + 1 : 0;
    const int64_t row0 = a.decode ? (int64_t)ca_lane(a, row) * a.ring : key0 - a.base;  // where the first visible key lies
    const T* q = reinterpret_cast<const T*>(a.q) + (int64_t)row * a.q_stride + (int64_t)head * a.dimp;
    for (int d = threadIdx.x; d < a.dim; d += CX_THREADS) q_f[d] = to_f32(q[d]);
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    auto at = [&](const void* table, int padded, int key) { return reinterpret_cast<const T*>(table) + ((row0 + key) * a.G + group) * padded; };
    float m = a.sink ? a.sink[head] : -INFINITY, l = a.sink ? 1.f : 0.f;
    float acc[CX_COLS];
#pragma unroll
    for (int i = 0; i < CX_COLS; ++i) acc[i] = 0.f;
    for (int t = 0; t < keys; t += CX_KEYS) {
        const int n = min(CX_KEYS, keys - t);
        for (int j = warp; j < n; j += CX_THREADS / 32) {
            const T* k = at(a.k, a.dimp, t + j);
            float s = 0.f;
            for (int d = lane; d < a.dim; d += 32) s = fmaf(q_f[d], to_f32(k[d]), s);
            s = warp_sum(s);
            if (lane == 0) p_s[j] = s * a.scale;
        }
        __syncthreads();
        const float x = (int)threadIdx.x < n ? p_s[threadIdx.x] : -INFINITY;
        float top = warp_max(x);
        if (lane == 0) red[warp] = top;
        __syncthreads();
        top = m;
#pragma unroll
        for (int w = 0; w < CX_THREADS / 32; ++w) top = fmaxf(top, red[w]);
        const float fix = expf(m - top), p = (int)threadIdx.x < n ? expf(x - top) : 0.f;
        __syncthreads();
        p_s[threadIdx.x] = p;
        const float part = warp_sum(p);
        if (lane == 0) red[warp] = part;
        __syncthreads();
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < CX_THREADS / 32; ++w) sum += red[w];
        l = l * fix + sum;
        m = top;
#pragma unroll
        for (int i = 0; i < CX_COLS; ++i) acc[i] *= fix;
        for (int j = 0; j < n; ++j) {
            const T* v = at(a.v, a.vdimp, t + j);
            const float w = p_s[j];
#pragma unroll
            for (int i = 0; i < CX_COLS; ++i) {
                const int c = threadIdx.x + i * CX_THREADS;
                if (c < a.vdim) acc[i] = fmaf(w, to_f32(v[c]), acc[i]);
            }
        }
        __syncthreads();
    }
    T* out = reinterpret_cast<T*>(a.out) + (int64_t)row * a.out_stride + (int64_t)head * a.vdim;
    const float gate = ca_gate<T>(a, row, head);
#pragma unroll
    for (int i = 0; i < CX_COLS; ++i) {
        const int c = threadIdx.x + i * CX_THREADS;
        if (c < a.vdim) from_f32(l > 0.f ? acc[i] / l * gate : 0.f, out[c]);
    }
}

// ===================================================================================================
static ChunkAttnArgs chunk_args(const ChunkAttnArgs* args) {
    ChunkAttnArgs a = *args;
    if (!a.q_stride) a.q_stride = (int64_t)a.H * a.dimp;
    return a;
}
static bool chunk_args_ok(const ChunkAttnArgs& a) {
    if (a.rows < 1 || a.H < 1 || a.G < 1 || a.H % a.G || a.dim < 1 || a.vdim < 1 || (a.dimp & 15) || (a.vdimp & 15) || a.dimp < a.dim || a.vdimp < a.vdim ||
        a.chunk < 1 || !a.q || !a.k || !a.v || !a.out || (a.q_stride & 7))
        return false;
    if (a.decode) return a.ring >= 1 && a.capacity >= 1 && a.lanes >= 1 && (a.ring == a.chunk || a.ring == a.capacity) && a.row_pos && a.row_lane;
    // every key a row can see lies in the buffers
    return a.start >= 0 && a.base >= 0 && a.start / a.chunk * a.chunk >= a.base && a.start + a.rows - a.base <= a.keys;
}

template <typename K>
static cudaError_t chunk_smem_limit(K kernel, DeviceOnce& once) {
    const int dev = once.pending();
    if (dev == DeviceOnce::SET) return cudaSuccess;
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e == cudaSuccess) once.mark(dev);
    return e;
}

template <int DV>
static int launch_chunk_prefill(const ChunkAttnArgs& a, cudaStream_t st) {
    static DeviceOnce once;
    const cudaError_t e = chunk_smem_limit(chunk_attn_prefill_kernel<DV>, once);
    if (e != cudaSuccess) return (int)e;
    const size_t smem = chunk_prefill_smem(a.dimp, a.vdimp);
    GLMB_LAUNCH(chunk_attn_prefill_kernel<DV>, dim3(ceil_div(a.rows, CP_ROWS), a.H), CP_THREADS, smem, st, a);
    return (int)cudaGetLastError();
}

template <int DV, int WARPS, int NT>
static int launch_chunk_decode(const ChunkAttnArgs& a, cudaStream_t st) {
    static DeviceOnce once;
    cudaError_t e = chunk_smem_limit(chunk_attn_decode_kernel<DV, WARPS, NT>, once);
    if (e != cudaSuccess) return (int)e;
    static DeviceOnce wide;  // clusters of 16 are beyond the portable size
    const int wide_dev = wide.pending();
    if (wide_dev != DeviceOnce::SET) {
        e = cudaFuncSetAttribute(chunk_attn_decode_kernel<DV, WARPS, NT>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        if (e != cudaSuccess) return (int)e;
        wide.mark(wide_dev);
    }
    CUtensorMap map_k, map_v;
    const uint64_t ring_rows = (uint64_t)a.lanes * a.ring;
    if (make_map(&map_k, a.k, ring_rows, (uint64_t)a.G * a.dimp, (uint64_t)a.G * a.dimp, WARPS * 16)) return 3;
    if (make_map(&map_v, a.v, ring_rows, (uint64_t)a.G * a.vdimp, (uint64_t)a.G * a.vdimp, WARPS * 16)) return 3;
    int stages = 4;
    while (stages > 2 && chunk_decode_smem(a.dimp, a.vdimp, stages, WARPS) > 200 * 1024) --stages;
    // CTAs per cluster: enough that the grid reaches every SM, at least one tile each.  A cluster of 16 only while few are launched: the
    // GPU places a handful of them at a time, and eight waited for one another (20 us before the first key, 10 us with eight per cluster).
    const int heads = a.G * ceil_div(a.H / a.G, CD_HEADS), tiles = ceil_div(a.ring, WARPS * 16), most = heads * a.rows <= 4 ? 16 : 8;
    int splits = 1;
    while (splits < most && splits * 2 <= tiles && splits * heads * a.rows < 148) splits *= 2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(splits, heads, a.rows);
    cfg.blockDim = dim3(WARPS * 32);
    cfg.dynamicSmemBytes = chunk_decode_smem(a.dimp, a.vdimp, stages, WARPS);
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = g_glmb_pdl_enabled ? 1 : 0;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = splits;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    const cudaError_t le = cudaLaunchKernelEx(&cfg, chunk_attn_decode_kernel<DV, WARPS, NT>, map_k, map_v, a, stages);
    return le != cudaSuccess ? (int)le : (int)cudaGetLastError();
}

GLMB_API size_t glmb_chunk_attn_args_sizeof(void) { return sizeof(ChunkAttnArgs); }

static int g_chunk_prefill_tc = 1;
// 1 (default): tcgen05 prefill kernel where the head sizes allow; 0: the mma.sync kernel.
GLMB_API void glmb_set_chunk_prefill_tc(int enabled) { g_chunk_prefill_tc = enabled ? 1 : 0; }

// bf16, rows of one sequence at consecutive positions; head sizes up to 256.
GLMB_API int glmb_chunk_attn_prefill(const ChunkAttnArgs* args, void* stream) {
    ChunkAttnArgs a = chunk_args(args);
    if (!chunk_args_ok(a) || a.decode || a.dimp > 256 || a.vdimp > 256) return 1;
    if (g_chunk_prefill_tc && a.dimp <= 128 && a.vdimp <= 128 && a.scale > 0.f) return launch_chunk_attn_tcgen05(a, (cudaStream_t)stream);
    if (a.vdimp <= 64) return launch_chunk_prefill<64>(a, (cudaStream_t)stream);
    if (a.vdimp <= 128) return launch_chunk_prefill<128>(a, (cudaStream_t)stream);
    return launch_chunk_prefill<256>(a, (cudaStream_t)stream);
}

// bf16, one row per sequence, every key in the ring; head sizes up to 256.
GLMB_API int glmb_chunk_attn_decode(const ChunkAttnArgs* args, void* stream) {
    ChunkAttnArgs a = chunk_args(args);
    if (!chunk_args_ok(a) || !a.decode || a.dimp > 256 || a.vdimp > 256) return 1;
    const bool few = a.H / a.G <= 8;
    cudaStream_t st = (cudaStream_t)stream;
    if (a.dimp > 128 || a.vdimp > 128) return few ? launch_chunk_decode<256, 4, 1>(a, st) : launch_chunk_decode<256, 4, 2>(a, st);
    if (a.vdimp <= 64) return few ? launch_chunk_decode<64, 8, 1>(a, st) : launch_chunk_decode<64, 8, 2>(a, st);
    return few ? launch_chunk_decode<128, 8, 1>(a, st) : launch_chunk_decode<128, 8, 2>(a, st);
}

// Any head size (values up to 1024 columns), bf16 or fp32.
GLMB_API int glmb_chunk_attn_any(const ChunkAttnArgs* args, int is_f32, void* stream) {
    ChunkAttnArgs a = chunk_args(args);
    if (!chunk_args_ok(a) || a.vdim > CX_THREADS * CX_COLS || a.dim > 8192) return 1;
    const dim3 grid(a.rows, a.H);
    const size_t smem = (size_t)a.dim * sizeof(float);
    if (is_f32) GLMB_LAUNCH(chunk_attn_any_kernel<float>, grid, CX_THREADS, smem, (cudaStream_t)stream, a);
    else GLMB_LAUNCH(chunk_attn_any_kernel<bf16>, grid, CX_THREADS, smem, (cudaStream_t)stream, a);
    return (int)cudaGetLastError();
}
