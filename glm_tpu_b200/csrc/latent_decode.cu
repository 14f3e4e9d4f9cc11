// Decode attention over cached latents (bf16, latents up to 512 wide): few query rows against long sequences of cache rows that every head
// shares, each row key and value at once.
//
//   latent_decode_kernel        up to 32 query heads of one row per cluster.  Tiles of 64 cache rows come in by TMA (64-column boxes, 128-byte
//                               swizzle) and are dealt to all CTAs of the row.  Scores: a warp takes eight keys, the heads are M; the running
//                               softmax state is per CTA; output: a warp takes 64 latent columns of every key.  Scores, exponentials and sums
//                               are fp32, the weights enter the second product as two bf16 pieces.  The CTAs of a cluster meet in
//                               distributed shared memory and leave one partial state per cluster.
//   latent_merge_value_kernel   joins a row's partial states and the sink, projects the attended latent to the head's values and applies the
//                               head's gate; a CTA serves every row with one pass over its slice of the weights
#include <cooperative_groups.h>

#include "attention_core.cuh"
#include "latent_args.cuh"
#include "tcgen05.cuh"
#include "vec8.cuh"

namespace cg = cooperative_groups;

#define LD_KEYS 64
#define LD_WARPS 8
#define LD_THREADS (LD_WARPS * 32)
#define LD_BOX (LD_KEYS * 128)
#define LD_PSTRIDE 72
#define LD_CLUSTER 4
#define LD_CLUSTERS 32  // clusters the grid aims at: all of them resident at once (of eight CTAs only fifteen were)
#define LD_LOG2E 1.4426950408889634f

static inline int ld_boxes(int W) { return (W + 63) / 64; }
static inline size_t ld_smem(int W, int heads, int stages) {
    return 1024 + (size_t)stages * ld_boxes(W) * LD_BOX + (size_t)heads * (W + 8) * 2 + 2 * (size_t)heads * LD_PSTRIDE * 2 + 2 * (size_t)LD_WARPS * heads * 4;
}

// grid (clusters x CTAs of a cluster, blocks of 16 MT heads, rows), cluster (CTAs of a cluster, 1, 1).
template <int MT>
__global__ void __launch_bounds__(LD_THREADS, 1) latent_decode_kernel(const __grid_constant__ CUtensorMap map, LatentArgs a, int stages) {
    constexpr int HEADS = 16 * MT;
    cg::cluster_group cluster = cg::this_cluster();
    extern __shared__ unsigned char smem_raw[];
    __shared__ __align__(8) float cta_ml[HEADS][2];
    __shared__ float part_s[LD_CLUSTER][HEADS][2];
    __shared__ __align__(8) uint64_t full_bar[4];
    const int W = a.lat + a.pe, KP = W + 8, boxes = (W + 63) / 64;
    unsigned char* tiles_s = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const int stage_bytes = boxes * LD_BOX;
    bf16* q_s = reinterpret_cast<bf16*>(tiles_s + stages * stage_bytes);
    bf16* p_hi = q_s + HEADS * KP;
    bf16* p_lo = p_hi + HEADS * LD_PSTRIDE;
    float* max_s = reinterpret_cast<float*>(p_lo + HEADS * LD_PSTRIDE);
    float* sum_s = max_s + LD_WARPS * HEADS;
    if (threadIdx.x == 0) {
        for (int s = 0; s < stages; ++s) mbar_init(full_bar + s, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    GLMB_PDL_PROLOGUE();
    const int row = blockIdx.z, h0 = blockIdx.y * HEADS, heads = min(HEADS, a.H - h0);
    bool in_range;
    const int pos = latent_pos(a, row, in_range);
    int seq = a.row_lane[row];
    if (seq < 0 || seq >= a.lanes) {
        if (threadIdx.x == 0) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
        seq = min(max(seq, 0), a.lanes - 1);
    }
    const int keys = !a.row_active || a.row_active[row] ? pos + 1 : 0;
    const int split = blockIdx.x, splits = gridDim.x;
    const int tiles = (keys + LD_KEYS - 1) / LD_KEYS, mine = tiles > split ? (tiles - split - 1) / splits + 1 : 0;  // tiles split, split + splits, ..
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3, mr = lane & 7, mi = lane >> 3;

    auto load_tile = [&](int i) {  // the i-th tile of this CTA, by one thread
        unsigned char* dst = tiles_s + (i % stages) * stage_bytes;
        uint64_t* bar = full_bar + i % stages;
        const int y = seq * a.capacity + (split + i * splits) * LD_KEYS;
        mbar_expect_tx(bar, (uint32_t)stage_bytes);
        for (int b = 0; b < boxes; ++b) tma_load_2d(dst + b * LD_BOX, &map, bar, b * 64, y);
    };
    if (threadIdx.x == 0)
        for (int i = 0; i < min(stages, mine); ++i) load_tile(i);
    if (mine) {
        const bf16* q = reinterpret_cast<const bf16*>(a.qa) + ((int64_t)row * a.H + h0) * W;
        const int pieces = W / 8;
        for (int i = threadIdx.x; i < HEADS * pieces; i += LD_THREADS) {
            const int r = i / pieces, c = i % pieces;
            if (r < heads) cp_async16(q_s + r * KP + c * 8, q + (int64_t)r * W + c * 8);
            else *reinterpret_cast<uint4*>(q_s + r * KP + c * 8) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();

    const float scale2 = a.scale * LD_LOG2E;
    float m[MT][2], l[MT][2], o[MT][8][4];
#pragma unroll
    for (int x = 0; x < MT; ++x) {
        m[x][0] = m[x][1] = -INFINITY;
        l[x][0] = l[x][1] = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) o[x][j][0] = o[x][j][1] = o[x][j][2] = o[x][j][3] = 0.f;
    }
    const bool values = warp * 64 < a.lat;
    bool ok = true;
    for (int i = 0; i < mine; ++i) {
        const int stage = i % stages, left = min(LD_KEYS, keys - (split + i * splits) * LD_KEYS);  // at least one key
        if (ok && !mbar_wait(full_bar + stage, (i / stages) & 1)) {
            if (lane == 0) raise_status(a.status, GLMB_STATUS_WAIT_TIMEOUT);
            ok = false;  // meaningless from here on, but every barrier is still met
        }
        unsigned char* tile = tiles_s + stage * stage_bytes;
        if (left < LD_KEYS) {  // rows past the last key meet zero weights: they must not be infinite or NaN (the lane's last tile: never refilled)
            for (int x = threadIdx.x; x < (LD_KEYS - left) * boxes * 8; x += LD_THREADS)
                *reinterpret_cast<uint4*>(tile + (x % (boxes * 8) >> 3) * LD_BOX + (left + x / (boxes * 8)) * 128 + (x & 7) * 16) = make_uint4(0, 0, 0, 0);
            __syncthreads();
        }
        // ---- scores: heads x this warp's eight keys ------------------------------------------------------
        float s[MT][2][4];
#pragma unroll
        for (int x = 0; x < MT; ++x)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[x][0][e] = s[x][1][e] = 0.f;
        const unsigned char* kb = tile + (warp * 8 + mr) * 128;
        const bf16* qb = q_s + (mr + 8 * (mi & 1)) * KP + 8 * (mi >> 1);
#pragma unroll 2
        for (int k0 = 0; k0 < W; k0 += 32) {
            const int cc = k0 / 8 + mi;
            uint32_t kf[4];
            ldmatrix_x4(kf, kb + (cc >> 3) * LD_BOX + (((cc & 7) ^ mr) << 4));
#pragma unroll
            for (int half = 0; half < 2; ++half)
                if (k0 + half * 16 < W)
#pragma unroll
                    for (int x = 0; x < MT; ++x) {
                        uint32_t qf[4];
                        ldmatrix_x4(qf, qb + x * 16 * KP + k0 + half * 16);
                        mma_bf16_16816(s[x][half], qf, kf[2 * half], kf[2 * half + 1]);
                    }
        }
#pragma unroll
        for (int x = 0; x < MT; ++x) {
            float top[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float v = warp * 8 + 2 * t4 + (e & 1) < left ? (s[x][0][e] + s[x][1][e]) * scale2 : -INFINITY;
                s[x][0][e] = v;
                top[e >> 1] = fmaxf(top[e >> 1], v);
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                top[e] = fmaxf(top[e], __shfl_xor_sync(0xffffffffu, top[e], 1));
                top[e] = fmaxf(top[e], __shfl_xor_sync(0xffffffffu, top[e], 2));
                if (t4 == 0) max_s[warp * HEADS + x * 16 + g + 8 * e] = top[e];
            }
        }
        __syncthreads();
        float fix[MT][2];
#pragma unroll
        for (int x = 0; x < MT; ++x) {
            float sum[2] = {0.f, 0.f};
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                float top = m[x][e];
#pragma unroll
                for (int w = 0; w < LD_WARPS; ++w) top = fmaxf(top, max_s[w * HEADS + x * 16 + g + 8 * e]);
                fix[x][e] = exp2f(m[x][e] - top);
                m[x][e] = top;
                const float p0 = exp2f(s[x][0][2 * e] - top), p1 = exp2f(s[x][0][2 * e + 1] - top);
                sum[e] = p0 + p1;
                const uint32_t hi = pack_bf16(p0, p1);
                const int at = (x * 16 + g + 8 * e) * LD_PSTRIDE + warp * 8 + 2 * t4;
                *reinterpret_cast<uint32_t*>(p_hi + at) = hi;
                *reinterpret_cast<uint32_t*>(p_lo + at) = pack_bf16(p0 - bf16_lo(hi), p1 - bf16_hi(hi));
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 1);
                sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 2);
                if (t4 == 0) sum_s[warp * HEADS + x * 16 + g + 8 * e] = sum[e];
            }
        }
        __syncthreads();
#pragma unroll
        for (int x = 0; x < MT; ++x)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                float sum = 0.f;
#pragma unroll
                for (int w = 0; w < LD_WARPS; ++w) sum += sum_s[w * HEADS + x * 16 + g + 8 * e];
                l[x][e] = l[x][e] * fix[x][e] + sum;
            }
        // ---- output: heads x this warp's 64 latent columns -------------------------------------------------
        if (values) {
#pragma unroll
            for (int x = 0; x < MT; ++x)
#pragma unroll
                for (int j = 0; j < 8; ++j) { o[x][j][0] *= fix[x][0]; o[x][j][1] *= fix[x][0]; o[x][j][2] *= fix[x][1]; o[x][j][3] *= fix[x][1]; }
            const unsigned char* vb = tile + warp * LD_BOX + (mr + 8 * (mi & 1)) * 128;
            const int p_at = (mr + 8 * (mi & 1)) * LD_PSTRIDE + 8 * (mi >> 1);
#pragma unroll
            for (int kk = 0; kk < LD_KEYS / 16; ++kk) {
                uint32_t hi[MT][4], lw[MT][4];
#pragma unroll
                for (int x = 0; x < MT; ++x) {
                    ldmatrix_x4(hi[x], p_hi + p_at + x * 16 * LD_PSTRIDE + kk * 16);
                    ldmatrix_x4(lw[x], p_lo + p_at + x * 16 * LD_PSTRIDE + kk * 16);
                }
#pragma unroll
                for (int j = 0; j < 8; j += 2) {
                    uint32_t vf[4];
                    ldmatrix_x4_trans(vf, vb + kk * 16 * 128 + (((j + (mi >> 1)) ^ mr) << 4));
#pragma unroll
                    for (int x = 0; x < MT; ++x) {
                        mma_bf16_16816(o[x][j], hi[x], vf[0], vf[1]);
                        mma_bf16_16816(o[x][j + 1], hi[x], vf[2], vf[3]);
                        mma_bf16_16816(o[x][j], lw[x], vf[0], vf[1]);
                        mma_bf16_16816(o[x][j + 1], lw[x], vf[2], vf[3]);
                    }
                }
            }
        }
        if (i + 1 < mine) {  // every warp has read the stage, the weights and the sums
            __syncthreads();
            if (threadIdx.x == 0 && i + stages < mine) load_tile(i + stages);
        }
    }
    __syncthreads();  // every warp has left the tiles: the merge area takes their place
    float* o_s = reinterpret_cast<float*>(tiles_s);  // [HEADS][lat]
    if (values)
#pragma unroll
        for (int x = 0; x < MT; ++x)
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const int c = warp * 64 + j * 8 + 2 * t4;
                if (c < a.lat) {
                    *reinterpret_cast<float2*>(o_s + (x * 16 + g) * a.lat + c) = make_float2(o[x][j][0], o[x][j][1]);
                    *reinterpret_cast<float2*>(o_s + (x * 16 + g + 8) * a.lat + c) = make_float2(o[x][j][2], o[x][j][3]);
                }
            }
    if (warp == 0 && t4 == 0)
#pragma unroll
        for (int x = 0; x < MT; ++x)
#pragma unroll
            for (int e = 0; e < 2; ++e) { cta_ml[x * 16 + g + 8 * e][0] = m[x][e]; cta_ml[x * 16 + g + 8 * e][1] = l[x][e]; }
    cluster.sync();
    // ---- the CTAs of the cluster: all (maximum, sum) pairs first, then each CTA its share of the columns -----
    const int size = cluster.num_blocks(), rank = cluster.block_rank(), part = blockIdx.x / size;
    for (int i = threadIdx.x; i < size * HEADS; i += LD_THREADS) {
        const float2 ml = *reinterpret_cast<const float2*>(cluster.map_shared_rank(&cta_ml[0][0], i / HEADS) + (i % HEADS) * 2);
        part_s[i / HEADS][i % HEADS][0] = ml.x;
        part_s[i / HEADS][i % HEADS][1] = ml.y;
    }
    __syncthreads();
    if ((int)threadIdx.x < heads) {
        const int h = threadIdx.x;
        float top = -INFINITY, sum = 0.f;
        for (int p = 0; p < size; ++p) top = fmaxf(top, part_s[p][h][0]);
        for (int p = 0; p < size; ++p) {
            const float w = part_s[p][h][0] == -INFINITY ? 0.f : exp2f(part_s[p][h][0] - top);
            sum += part_s[p][h][1] * w;
            part_s[p][h][0] = w;
        }
        if (rank == 0) *reinterpret_cast<float2*>(a.part_ml + (((int64_t)row * a.H + h0 + h) * a.parts + part) * 2) = make_float2(top, sum);
    }
    __syncthreads();
    const int quads = heads * a.lat / 4;
    for (int i = rank * LD_THREADS + threadIdx.x; i < quads; i += size * LD_THREADS) {
        const int h = i * 4 / a.lat, c = i * 4 % a.lat;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int p = 0; p < LD_CLUSTER; ++p)
            if (p < size) {
                const float4 x = *reinterpret_cast<const float4*>(cluster.map_shared_rank(o_s, p) + i * 4);
                const float w = part_s[p][h][0];
                v.x = fmaf(x.x, w, v.x); v.y = fmaf(x.y, w, v.y); v.z = fmaf(x.z, w, v.z); v.w = fmaf(x.w, w, v.w);
            }
        *reinterpret_cast<float4*>(a.part_o + (((int64_t)row * a.H + h0 + h) * a.parts + part) * a.lat + c) = v;
    }
    cluster.sync();  // nobody leaves while a peer may still read its shared memory
}

// ---------------------------------------------------------------------------------------------------
#define LM_WARPS 8
#define LM_COLS 32
#define LM_PARTS 32

// grid (pieces of LM_COLS value channels, H); up to R rows.  In the projection eight lanes share a value channel, a warp has four.
template <int R>
__global__ void __launch_bounds__(LM_WARPS * 32) latent_merge_value_kernel(LatentArgs a) {
    asm volatile("griddepcontrol.launch_dependents;");
    const int h = blockIdx.y, c0 = blockIdx.x * LM_COLS, cols = min(LM_COLS, a.vdim - c0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane & 7, c = warp * 4 + (lane >> 3);
    const bf16* w = reinterpret_cast<const bf16*>(a.uv) + ((int64_t)h * a.vdim + c0 + min(c, cols - 1)) * a.lat;
    uint4 wv[8];  // this lane's weights: they do not depend on the kernel before
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        wv[i] = make_uint4(0, 0, 0, 0);
        if (sub * 8 + i * 64 < a.lat) wv[i] = *reinterpret_cast<const uint4*>(w + sub * 8 + i * 64);
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    extern __shared__ __align__(16) float o_s[];  // [SPLIT][rows][lat]
    __shared__ float w_s[R][LM_PARTS], gate_s[R];
    // every partial state a thread adds up is asked for before the weights are known
    constexpr int SPLIT = R == 1 ? 2 : 1, PAIRS = R == 1 ? 1 : R / 2, MOST = R == 8 ? 8 : 16;
    const int quads = a.rows * a.lat / 4, first = R == 1 ? (threadIdx.x >> 7) * MOST : 0, thread = R == 1 ? threadIdx.x & 127 : threadIdx.x;
    float4 x[PAIRS][MOST];
#pragma unroll
    for (int k = 0; k < PAIRS; ++k) {
        const int i = thread + k * LM_WARPS * 32, r = i * 4 / a.lat, at = i * 4 % a.lat;
        const float* src = a.part_o + (((int64_t)r * a.H + h) * a.parts + first) * a.lat + at;
#pragma unroll
        for (int p = 0; p < MOST; ++p) {
            x[k][p] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i < quads && first + p < a.parts) x[k][p] = *reinterpret_cast<const float4*>(src + (int64_t)p * a.lat);
        }
    }
    if (warp < a.rows) {  // a warp per row: weights of its parts, divided by the total
        const float sink2 = a.sink ? a.sink[h] * LD_LOG2E : -INFINITY;
        float2 ml = make_float2(-INFINITY, 0.f);
        if (lane < a.parts) ml = *reinterpret_cast<const float2*>(a.part_ml + (((int64_t)warp * a.H + h) * a.parts + lane) * 2);
        if (lane == 31) gate_s[warp] = sigmoidf_precise(__bfloat162float(reinterpret_cast<const bf16*>(a.proj)[(int64_t)warp * a.proj_stride + a.off_gate + h]));
        const float top = warp_max(fmaxf(ml.x, sink2));
        const float f = ml.x == -INFINITY ? 0.f : exp2f(ml.x - top);
        const float total = warp_sum(ml.y * f) + (a.sink ? exp2f(sink2 - top) : 0.f);
        w_s[warp][lane] = total > 0.f ? f / total : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < PAIRS; ++k) {
        const int i = thread + k * LM_WARPS * 32;
        if (i >= quads) continue;
        const float* f = w_s[i * 4 / a.lat] + first;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int p = 0; p < MOST; ++p) {
            v.x = fmaf(x[k][p].x, f[p], v.x); v.y = fmaf(x[k][p].y, f[p], v.y);
            v.z = fmaf(x[k][p].z, f[p], v.z); v.w = fmaf(x[k][p].w, f[p], v.w);
        }
        reinterpret_cast<float4*>(o_s)[(R == 1 ? (threadIdx.x >> 7) * quads : 0) + i] = v;
    }
    __syncthreads();
    if constexpr (SPLIT == 2) {
        if ((int)threadIdx.x < quads) {
            const float4 u = reinterpret_cast<const float4*>(o_s)[threadIdx.x], v = reinterpret_cast<const float4*>(o_s)[quads + threadIdx.x];
            reinterpret_cast<float4*>(o_s)[threadIdx.x] = make_float4(u.x + v.x, u.y + v.y, u.z + v.z, u.w + v.w);
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
        if (r >= a.rows) break;
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int l = sub * 8 + i * 64;
            if (l < a.lat) {
                float x[8];
                load8(o_s + r * a.lat + l, x);
                const uint32_t u[4] = {wv[i].x, wv[i].y, wv[i].z, wv[i].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) sum = fmaf(bf16_hi(u[e]), x[2 * e + 1], fmaf(bf16_lo(u[e]), x[2 * e], sum));
            }
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        sum += __shfl_xor_sync(0xffffffffu, sum, 4);
        if (sub == 0 && c < cols) {
            reinterpret_cast<bf16*>(a.out)[(int64_t)r * a.out_stride + h * a.vdim + c0 + c] = __float2bfloat16_rn(sum * gate_s[r]);
        }
    }
}

// ===================================================================================================
template <int MT>
static int launch_latent_decode(const LatentArgs& a, int cluster, cudaStream_t st) {
    const int W = a.lat + a.pe;
    static DeviceOnce once;
    const int dev = once.pending();
    if (dev != DeviceOnce::SET) {
        const cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
        if (e != cudaSuccess) return (int)e;
        once.mark(dev);
    }
    int stages = 4;
    while (stages > 2 && ld_smem(W, 16 * MT, stages) > 220 * 1024) --stages;
    CUtensorMap map;
    if (make_map(&map, a.cache, (uint64_t)a.lanes * a.capacity, W, W, LD_KEYS)) return 3;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.parts * cluster, ceil_div(a.H, 16 * MT), a.rows);
    cfg.blockDim = dim3(LD_THREADS);
    cfg.dynamicSmemBytes = ld_smem(W, 16 * MT, stages);
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = g_glmb_pdl_enabled ? 1 : 0;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    const cudaError_t le = cudaLaunchKernelEx(&cfg, latent_decode_kernel<MT>, map, a, stages);
    return le != cudaSuccess ? (int)le : (int)cudaGetLastError();
}

// Attention and value projection of 1..8 rows, bf16, lat <= 512, lat + pe <= 640 (both multiples of 16): qa, cache -> out.
// part_o / part_ml hold max(rows, LD_CLUSTERS) states per head: [max(rows, 32), H, lat] and [.., 2] fp32.
GLMB_API int glmb_latent_decode(const LatentArgs* args, void* stream) {
    LatentArgs a = *args;
    if (!latent_ok(a) || a.rows > GLMB_MAX_ROWS || a.lat > 512 || a.lat + a.pe > 640 || (a.lat & 15) || (a.pe & 15) || !a.part_o || !a.part_ml) return 1;
    const int blocks = ceil_div(a.H, a.H <= 16 ? 16 : 32) * a.rows, tiles = ceil_div(a.capacity, LD_KEYS);
    int cluster = 1;
    while (cluster < LD_CLUSTER && cluster * 2 <= tiles) cluster *= 2;
    a.parts = LD_CLUSTERS / blocks;
    if (a.parts > tiles / cluster) a.parts = tiles / cluster;
    const int most = a.rows == 1 ? LM_PARTS : a.rows <= 4 ? 16 : 8;  // what the merge takes
    if (a.parts > most) a.parts = most;
    if (a.parts < 1) a.parts = 1;
    const int code = a.H <= 16 ? launch_latent_decode<1>(a, cluster, (cudaStream_t)stream) : launch_latent_decode<2>(a, cluster, (cudaStream_t)stream);
    if (code) return code;
    const dim3 grid(ceil_div(a.vdim, LM_COLS), a.H);
#define CALL(R) GLMB_LAUNCH(latent_merge_value_kernel<R>, grid, LM_WARPS * 32, (size_t)2 * a.rows * a.lat * 4, (cudaStream_t)stream, a)
    if (a.rows == 1) CALL(1);
    else if (a.rows <= 4) CALL(4);
    else CALL(8);
#undef CALL
    return (int)cudaGetLastError();
}
