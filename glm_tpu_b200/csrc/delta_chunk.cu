// The gated delta rule of delta_rule.cu for many rows of one sequence (bf16 projections, up to 128 key channels): chunks of 16 tokens, the
// products on the tensor cores.  With G_i the running sum of log g inside a chunk, S_0 the state before it and
//
//   A_ij = sum_d k_i k_j exp(G_i - G_j)  (j < i),    B_ij = sum_d q_i k_j exp(G_i - G_j)  (j <= i),    L = (1 + diag(beta) A)^-1 diag(beta),
//
// the tokens' writes and read-outs and the state after the chunk are
//
//   U = L (V - (e^G k) S_0),    O = (e^G q) S_0 + B U,    S = e^G_last S_0 + (e^(G_last - G) k)^T U.
//
// Every exponent is a sum of logarithms of decays over an interval, never positive: nothing overflows however fast a channel forgets.
//
//   delta_chunk_prep   a CTA per (chunk, head): convolution, activation, unit vectors, decays, A, B and L in fp32; leaves one record with what
//                      the scan multiplies, matrices as two bf16 pieces (value and remainder: 16 bits of mantissa)
//   delta_chunk_scan   a warp keeps the fp32 state of 16 value channels in its accumulators ([value channel, key channel]: the accumulator
//                      layout is the operand layout of the next product) and walks the chunks; records arrive by bulk copies, several chunks
//                      ahead.  Products are hi.hi + hi.lo + lo.hi with fp32 sums.
//
// A record: [6][16][dimp + 8] bf16 (e^G k, e^G q, e^(G_last - G) k, each hi and lo), [4][16][24] bf16 (L hi, lo, B hi, lo), [dimp] fp32
// (e^G_last), [vdim / 16][16][20] fp32 (V by blocks of 16 channels).  Row paddings stagger the banks for ldmatrix.
#include "attention_core.cuh"
#include "delta_rule.cuh"
#include "tcgen05.cuh"
#include "vec8.cuh"

#define DC_TOKENS 16
#define DC_THREADS 256
#define DC_TAPS 4
#define DC_LB 24      // row of L and B
#define DC_VB 20      // row of a value block
#define DC_LOG2E 1.4426950408889634f

struct DeltaChunkArgs {
    DeltaArgs d;
    unsigned char* records;  // [chunks of the segment, H] records
    int row0, count;         // the segment: rows row0 .. row0 + count - 1 of the step (row0 a multiple of 16)
    int last;                // the segment ends the step
    int warps;               // scan: blocks of 16 value channels per CTA
};

__host__ __device__ static inline int dc_mats_bytes(int dimp) { return 6 * DC_TOKENS * (dimp + 8) * 2; }
__host__ __device__ static inline int dc_head_bytes(int dimp) { return dc_mats_bytes(dimp) + 4 * DC_TOKENS * DC_LB * 2 + dimp * 4; }
__host__ __device__ static inline int dc_value_block() { return DC_TOKENS * DC_VB * 4; }
__host__ __device__ static inline int dc_record_bytes(int dimp, int vdim) { return dc_head_bytes(dimp) + (vdim + 15) / 16 * dc_value_block(); }

__device__ __forceinline__ float dc_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void dc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x, y);
    lo = pack_bf16(x - bf16_lo(hi), y - bf16_hi(hi));
}

// One step of a sum over 16 lanes that leaves every lane with a sixteenth of the values: N values become N / 2.
template <int N>
__device__ __forceinline__ void dc_fold(float (&v)[32], int lane, int offset) {
    const bool upper = lane & offset;
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
        const float keep = upper ? v[i + N / 2] : v[i], send = upper ? v[i] : v[i + N / 2];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, offset);
    }
}

// grid (chunks, H)
__global__ void __launch_bounds__(DC_THREADS) delta_chunk_prep_kernel(DeltaChunkArgs p) {
    GLMB_PDL_PROLOGUE();
    const DeltaArgs& a = p.d;
    extern __shared__ __align__(16) float smem_f[];
    const int DP = a.dimp, RS = DP + 4;
    float* q_s = smem_f;                        // [16][RS]
    float* k_s = q_s + DC_TOKENS * RS;
    float* g_s = k_s + DC_TOKENS * RS;          // log2 of the decays, then their running sum
    __shared__ float A_s[DC_TOKENS][DC_TOKENS + 1], B_s[DC_TOKENS][DC_TOKENS + 1], beta_s[DC_TOKENS];
    const int h = blockIdx.y, kvh = h / (a.H / a.G), t0 = p.row0 + blockIdx.x * DC_TOKENS, n = min(DC_TOKENS, p.row0 + p.count - t0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int C = 2 * a.G * a.dim + a.H * a.vdim, keep = a.taps - 1;
    unsigned char* record = p.records + ((int64_t)blockIdx.x * a.H + h) * dc_record_bytes(DP, a.vdim);
    float* v_out = reinterpret_cast<float*>(record + dc_head_bytes(DP));
    const bf16* proj = reinterpret_cast<const bf16*>(a.proj);
    const int start = a.row_pos[0], seq = delta_lane(a, 0);
    const bf16* state = reinterpret_cast<const bf16*>(a.conv_state) + (int64_t)seq * a.taps * C;

    // ---- decays ------------------------------------------------------------------------------------------
    const float rate = a.a_rate[h] * DC_LOG2E;
    for (int i = tid; i < DC_TOKENS * DP; i += DC_THREADS) {
        const int t = i / DP, d = i % DP;
        g_s[t * RS + d] = t < n && d < a.dim ? -rate * delta_softplus(a.a[(int64_t)(t0 + t) * a.a_stride + h * a.dim + d] + a.dt_bias[h * a.dim + d]) : 0.f;
    }
    if (tid < DC_TOKENS) beta_s[tid] = tid < n ? sigmoidf_precise(__bfloat162float(proj[(int64_t)(t0 + tid) * a.proj_stride + a.off_b + h])) : 0.f;
    // ---- convolution: a thread takes eight channels of four tokens -----------------------------------------
    const int kvec = a.dim / 8, vecs = 2 * kvec + a.vdim / 8;
    for (int i = tid; i < vecs * 4; i += DC_THREADS) {
        const int vec = i % vecs, first = i / vecs * 4;
        const int kind = vec < kvec ? 0 : vec < 2 * kvec ? 1 : 2, c = (kind == 0 ? vec : kind == 1 ? vec - kvec : vec - 2 * kvec) * 8;
        const int chan = (kind == 0 ? kvh * a.dim : kind == 1 ? (a.G + kvh) * a.dim : 2 * a.G * a.dim + h * a.vdim) + c;
        uint4 u[4 + DC_TAPS - 1];
#pragma unroll
        for (int j = 0; j < 4 + DC_TAPS - 1; ++j) {
            const int row = t0 + first + j - (DC_TAPS - 1);  // row of the step; before it: the lane's ring of projected rows
            u[j] = make_uint4(0, 0, 0, 0);
            if (row >= 0 && row < t0 + n) u[j] = *reinterpret_cast<const uint4*>(proj + (int64_t)row * a.proj_stride + chan);
            else if (row < 0 && row >= -keep && start + row >= 0) u[j] = *reinterpret_cast<const uint4*>(state + (int64_t)((start + row) % a.taps) * C + chan);
        }
        float y[4][8];
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int e = 0; e < 8; ++e) y[t][e] = 0.f;
#pragma unroll
        for (int j = 0; j < DC_TAPS; ++j) {
            const int tap = j - (DC_TAPS - a.taps);  // fewer taps: the oldest ones are not there
            if (tap < 0) continue;
            float w[8];
            load8(a.conv_w + (int64_t)tap * C + chan, w);
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const uint32_t x[4] = {u[t + j].x, u[t + j].y, u[t + j].z, u[t + j].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    y[t][2 * e] = fmaf(w[2 * e], bf16_lo(x[e]), y[t][2 * e]);
                    y[t][2 * e + 1] = fmaf(w[2 * e + 1], bf16_hi(x[e]), y[t][2 * e + 1]);
                }
            }
        }
#pragma unroll
        for (int t = 0; t < 4; ++t) {
#pragma unroll
            for (int e = 0; e < 8; ++e) y[t][e] = first + t < n ? delta_silu(y[t][e]) : 0.f;
            if (kind == 2) store8(v_out + ((int64_t)(c / 16) * DC_TOKENS + first + t) * DC_VB + c % 16, y[t]);
            else store8((kind == 0 ? q_s : k_s) + (first + t) * RS + c, y[t]);
        }
    }
    for (int i = tid; i < 2 * DC_TOKENS * (DP - a.dim); i += DC_THREADS) {  // padding of the key channels
        const int r = i / (DP - a.dim), d = a.dim + i % (DP - a.dim);
        (r < DC_TOKENS ? q_s : k_s)[(r % DC_TOKENS) * RS + d] = 0.f;
    }
    if (a.vdim % 16)  // the last value block's second half
        for (int i = tid; i < DC_TOKENS * 8; i += DC_THREADS) v_out[((int64_t)(a.vdim / 16) * DC_TOKENS + i / 8) * DC_VB + 8 + i % 8] = 0.f;
    __syncthreads();
    // ---- unit vectors (a warp per row), running sums of the decays ------------------------------------------
    for (int r = warp; r < 2 * DC_TOKENS; r += DC_THREADS / 32) {
        float* x = (r < DC_TOKENS ? q_s : k_s) + (r % DC_TOKENS) * RS;
        float ss = 0.f;
        for (int d = lane; d < DP; d += 32) ss = fmaf(x[d], x[d], ss);
        const float scale = (r < DC_TOKENS ? 1.f / sqrtf((float)a.dim) : 1.f) / sqrtf(warp_sum(ss) + 1e-6f);
        for (int d = lane; d < DP; d += 32) x[d] *= scale;
    }
    for (int d = tid; d < DP; d += DC_THREADS) {
        float sum = 0.f;
#pragma unroll
        for (int t = 0; t < DC_TOKENS; ++t) { sum += g_s[t * RS + d]; g_s[t * RS + d] = sum; }
    }
    __syncthreads();
    // ---- A and B: 4 x 4 blocks of (i, j) below the diagonal, sixteen lanes share the channels of a block ------
    for (int unit = warp; unit < 5; unit += DC_THREADS / 32) {
        const int block = unit * 2 + (lane >> 4), sub = lane & 15;
        const int bi = block < 1 ? 0 : block < 3 ? 1 : block < 6 ? 2 : 3, bj = block - bi * (bi + 1) / 2;
        float acc[32];  // A then B of the 16 pairs
#pragma unroll
        for (int x = 0; x < 32; ++x) acc[x] = 0.f;
        for (int d = sub * 2; d < DP; d += 32) {
            float2 gi[4], ki[4], qi[4], gj[4], kj[4];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                gi[x] = *reinterpret_cast<const float2*>(g_s + (bi * 4 + x) * RS + d);
                ki[x] = *reinterpret_cast<const float2*>(k_s + (bi * 4 + x) * RS + d);
                qi[x] = *reinterpret_cast<const float2*>(q_s + (bi * 4 + x) * RS + d);
                gj[x] = *reinterpret_cast<const float2*>(g_s + (bj * 4 + x) * RS + d);
                kj[x] = *reinterpret_cast<const float2*>(k_s + (bj * 4 + x) * RS + d);
            }
            if (bi != bj) {  // exp(G_i - G_j) in two factors around the end of the earlier block, both at most one
                const float2 mid = gj[3];
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const float e0 = dc_exp2(gi[x].x - mid.x), e1 = dc_exp2(gi[x].y - mid.y), f0 = dc_exp2(mid.x - gj[x].x), f1 = dc_exp2(mid.y - gj[x].y);
                    ki[x].x *= e0; ki[x].y *= e1; qi[x].x *= e0; qi[x].y *= e1;
                    kj[x].x *= f0; kj[x].y *= f1;
                }
#pragma unroll
                for (int x = 0; x < 4; ++x)
#pragma unroll
                    for (int y = 0; y < 4; ++y) {
                        acc[x * 4 + y] = fmaf(ki[x].x, kj[y].x, fmaf(ki[x].y, kj[y].y, acc[x * 4 + y]));
                        acc[16 + x * 4 + y] = fmaf(qi[x].x, kj[y].x, fmaf(qi[x].y, kj[y].y, acc[16 + x * 4 + y]));
                    }
            } else {
#pragma unroll
                for (int x = 0; x < 4; ++x)
#pragma unroll
                    for (int y = 0; y <= x; ++y) {
                        const float e0 = x == y ? kj[y].x : kj[y].x * dc_exp2(gi[x].x - gj[y].x), e1 = x == y ? kj[y].y : kj[y].y * dc_exp2(gi[x].y - gj[y].y);
                        acc[x * 4 + y] = fmaf(ki[x].x, e0, fmaf(ki[x].y, e1, acc[x * 4 + y]));
                        acc[16 + x * 4 + y] = fmaf(qi[x].x, e0, fmaf(qi[x].y, e1, acc[16 + x * 4 + y]));
                    }
            }
        }
        dc_fold<32>(acc, lane, 8);
        dc_fold<16>(acc, lane, 4);
        dc_fold<8>(acc, lane, 2);
        dc_fold<4>(acc, lane, 1);
        // lane bits from the highest choose the half at every step: this lane holds values 2 sub, 2 sub + 1
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int at = sub * 2 + x, i = bi * 4 + (at & 15) / 4, j = bj * 4 + (at & 3);
            (at < 16 ? A_s : B_s)[i][j] = j < i || (at >= 16 && j == i) ? acc[x] : 0.f;
        }
    }
    for (int i = tid; i < DC_TOKENS * DC_TOKENS; i += DC_THREADS)  // blocks above the diagonal
        if (i % DC_TOKENS / 4 > i / DC_TOKENS / 4) A_s[i / DC_TOKENS][i % DC_TOKENS] = B_s[i / DC_TOKENS][i % DC_TOKENS] = 0.f;
    __syncthreads();
    bf16* lb = reinterpret_cast<bf16*>(record + dc_mats_bytes(DP));
    if (warp == 0 && lane < DC_TOKENS) {  // column `lane` of L by forward substitution
        float x[DC_TOKENS];
#pragma unroll
        for (int i = 0; i < DC_TOKENS; ++i) {
            float sum = i == lane ? 1.f : 0.f;
#pragma unroll
            for (int j = 0; j < i; ++j) sum = fmaf(-A_s[i][j], x[j], sum);
            x[i] = beta_s[i] * sum;
            const bf16 hi = __float2bfloat16_rn(x[i]);
            lb[i * DC_LB + lane] = hi;
            lb[(DC_TOKENS + i) * DC_LB + lane] = __float2bfloat16_rn(x[i] - __bfloat162float(hi));
        }
    } else if (warp == 1) {
        for (int i = lane; i < DC_TOKENS * DC_TOKENS; i += 32) {
            const float x = B_s[i / DC_TOKENS][i % DC_TOKENS];
            const bf16 hi = __float2bfloat16_rn(x);
            lb[(2 * DC_TOKENS + i / DC_TOKENS) * DC_LB + i % DC_TOKENS] = hi;
            lb[(3 * DC_TOKENS + i / DC_TOKENS) * DC_LB + i % DC_TOKENS] = __float2bfloat16_rn(x - __bfloat162float(hi));
        }
    }
    // ---- the operands that meet the state --------------------------------------------------------------------
    uint32_t* mats = reinterpret_cast<uint32_t*>(record);
    const int words = (DP + 8) / 2;
    for (int i = tid; i < DC_TOKENS * DP / 2; i += DC_THREADS) {
        const int t = i / (DP / 2), d = i % (DP / 2) * 2;
        const float2 g = *reinterpret_cast<const float2*>(g_s + t * RS + d), end = *reinterpret_cast<const float2*>(g_s + (DC_TOKENS - 1) * RS + d);
        const float2 k = *reinterpret_cast<const float2*>(k_s + t * RS + d), q = *reinterpret_cast<const float2*>(q_s + t * RS + d);
        const float e0 = dc_exp2(g.x), e1 = dc_exp2(g.y), f0 = dc_exp2(end.x - g.x), f1 = dc_exp2(end.y - g.y);
        const float2 x[3] = {{k.x * e0, k.y * e1}, {q.x * e0, q.y * e1}, {k.x * f0, k.y * f1}};
#pragma unroll
        for (int m = 0; m < 3; ++m) dc_split(x[m].x, x[m].y, mats[((2 * m) * DC_TOKENS + t) * words + d / 2], mats[((2 * m + 1) * DC_TOKENS + t) * words + d / 2]);
    }
    float* gamma = reinterpret_cast<float*>(record + dc_mats_bytes(DP) + 4 * DC_TOKENS * DC_LB * 2);
    for (int d = tid; d < DP; d += DC_THREADS) gamma[d] = dc_exp2(g_s[(DC_TOKENS - 1) * RS + d]);
}

// ---------------------------------------------------------------------------------------------------
#define DC_STAGES 4

__device__ __forceinline__ void dc_bulk_load(void* smem_dst, const void* src, uint32_t bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(smem_u32(smem_dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}

// grid (groups of `warps` blocks of 16 value channels, H), 32 * warps threads.  KS: key channels / 16.
template <int KS>
__global__ void __launch_bounds__(128) delta_chunk_scan_kernel(DeltaChunkArgs p) {
    constexpr int DP = KS * 16, RS = DP + 8;
    const DeltaArgs& a = p.d;
    extern __shared__ __align__(128) unsigned char smem_raw[];
    __shared__ __align__(8) uint64_t full_bar[DC_STAGES];
    const int h = blockIdx.y, kvh = h / (a.H / a.G), chunks = (p.count + DC_TOKENS - 1) / DC_TOKENS;
    const int blocks = (a.vdim + 15) / 16, block0 = blockIdx.x * p.warps, here = min(p.warps, blocks - block0);
    const int head_bytes = dc_head_bytes(DP), value_bytes = here * dc_value_block(), stage_bytes = head_bytes + p.warps * dc_value_block();
    const int64_t record_bytes = dc_record_bytes(DP, a.vdim);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3, mr = lane & 7, mi = lane >> 3;
    if (threadIdx.x == 0) {
        for (int s = 0; s < DC_STAGES; ++s) mbar_init(full_bar + s, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    GLMB_PDL_PROLOGUE();
    auto load = [&](int i) {
        unsigned char* dst = smem_raw + (i % DC_STAGES) * stage_bytes;
        const unsigned char* src = p.records + ((int64_t)i * a.H + h) * record_bytes;
        uint64_t* bar = full_bar + i % DC_STAGES;
        mbar_expect_tx(bar, head_bytes + value_bytes);
        dc_bulk_load(dst, src, head_bytes, bar);
        dc_bulk_load(dst + head_bytes, src + head_bytes + (int64_t)block0 * dc_value_block(), value_bytes, bar);
    };
    if (threadIdx.x == 0)
        for (int i = 0; i < min(DC_STAGES, chunks); ++i) load(i);
    const bool mine = warp < here;
    const int c0 = (block0 + warp) * 16, seq = delta_lane(a, 0), start = a.row_pos[0] + p.row0;
    float* state = a.state + ((int64_t)seq * a.H + h) * a.vdim * DP;
    const bool writes = delta_writes(a, 0);
    // accumulators of the transposed state: value channels c0 + g, + 8; key channels 8 j + 2 t4, + 1
    float s[2 * KS][4];
#pragma unroll
    for (int j = 0; j < 2 * KS; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            float2 x = make_float2(0.f, 0.f);
            if (mine && start > 0 && c0 + g + 8 * e < a.vdim) x = *reinterpret_cast<const float2*>(state + (int64_t)(c0 + g + 8 * e) * DP + j * 8 + 2 * t4);
            s[j][2 * e] = x.x;
            s[j][2 * e + 1] = x.y;
        }
    bool ok = true;
    for (int i = 0; i < chunks; ++i) {
        const int stage = i % DC_STAGES;
        if (ok && !mbar_wait(full_bar + stage, (i / DC_STAGES) & 1)) {
            if (lane == 0) raise_status(a.status, GLMB_STATUS_WAIT_TIMEOUT);
            ok = false;  // meaningless from here on, but every barrier is still met
        }
        const unsigned char* base = smem_raw + stage * stage_bytes;
        const bf16* mats = reinterpret_cast<const bf16*>(base);
        const bf16* lb = reinterpret_cast<const bf16*>(base + dc_mats_bytes(DP));
        const float* gamma = reinterpret_cast<const float*>(base + dc_mats_bytes(DP) + 4 * DC_TOKENS * DC_LB * 2);
        const float* v_s = reinterpret_cast<const float*>(base + head_bytes + warp * dc_value_block());
        if (mine) {
            // ---- (e^G k) S and (e^G q) S, transposed: value channels x tokens ------------------------------
            float w[2][4], wl[2][4], r[2][4], rl[2][4];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) w[n][e] = wl[n][e] = r[n][e] = rl[n][e] = 0.f;
            const bf16* at = mats + (mr + 8 * (mi >> 1)) * RS + 8 * (mi & 1);
#pragma unroll
            for (int kk = 0; kk < KS; ++kk) {
                uint32_t hi[4], lo[4], kh[4], kl[4], qh[4], ql[4];
                dc_split(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
                dc_split(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
                dc_split(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
                dc_split(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
                ldmatrix_x4(kh, at + kk * 16);
                ldmatrix_x4(kl, at + kk * 16 + DC_TOKENS * RS);
                ldmatrix_x4(qh, at + kk * 16 + 2 * DC_TOKENS * RS);
                ldmatrix_x4(ql, at + kk * 16 + 3 * DC_TOKENS * RS);
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    mma_bf16_16816(w[n], hi, kh[2 * n], kh[2 * n + 1]);
                    mma_bf16_16816(r[n], hi, qh[2 * n], qh[2 * n + 1]);
                    mma_bf16_16816(wl[n], lo, kh[2 * n], kh[2 * n + 1]);
                    mma_bf16_16816(rl[n], lo, qh[2 * n], qh[2 * n + 1]);
                    mma_bf16_16816(wl[n], hi, kl[2 * n], kl[2 * n + 1]);
                    mma_bf16_16816(rl[n], hi, ql[2 * n], ql[2 * n + 1]);
                }
            }
            // ---- U = L (V - ..) -----------------------------------------------------------------------------
            uint32_t xh[4], xl[4];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float x0 = v_s[(n * 8 + 2 * t4) * DC_VB + g + 8 * e] - (w[n][2 * e] + wl[n][2 * e]);
                    const float x1 = v_s[(n * 8 + 2 * t4 + 1) * DC_VB + g + 8 * e] - (w[n][2 * e + 1] + wl[n][2 * e + 1]);
                    dc_split(x0, x1, xh[2 * n + e], xl[2 * n + e]);
                }
            uint32_t lh[4], ll[4], bh[4], bl[4];
            const bf16* lat = lb + (mr + 8 * (mi >> 1)) * DC_LB + 8 * (mi & 1);
            ldmatrix_x4(lh, lat);
            ldmatrix_x4(ll, lat + DC_TOKENS * DC_LB);
            ldmatrix_x4(bh, lat + 2 * DC_TOKENS * DC_LB);
            ldmatrix_x4(bl, lat + 3 * DC_TOKENS * DC_LB);
            uint32_t uh[4], ul[4];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                float u[4] = {0.f, 0.f, 0.f, 0.f}, ulow[4] = {0.f, 0.f, 0.f, 0.f};
                mma_bf16_16816(u, xh, lh[2 * n], lh[2 * n + 1]);
                mma_bf16_16816(ulow, xl, lh[2 * n], lh[2 * n + 1]);
                mma_bf16_16816(ulow, xh, ll[2 * n], ll[2 * n + 1]);
                dc_split(u[0] + ulow[0], u[1] + ulow[1], uh[2 * n], ul[2 * n]);
                dc_split(u[2] + ulow[2], u[3] + ulow[3], uh[2 * n + 1], ul[2 * n + 1]);
            }
            // ---- state: decay, then the chunk's writes -------------------------------------------------------
            const bf16* ke = mats + 4 * DC_TOKENS * RS + (mr + 8 * (mi & 1)) * RS + 8 * (mi >> 1);
#pragma unroll
            for (int j = 0; j < 2 * KS; j += 2) {
                uint32_t eh[4], el[4];
                ldmatrix_x4_trans(eh, ke + j * 8);
                ldmatrix_x4_trans(el, ke + j * 8 + DC_TOKENS * RS);
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const float2 f = *reinterpret_cast<const float2*>(gamma + (j + x) * 8 + 2 * t4);
                    s[j + x][0] *= f.x; s[j + x][1] *= f.y; s[j + x][2] *= f.x; s[j + x][3] *= f.y;
                    mma_bf16_16816(s[j + x], uh, eh[2 * x], eh[2 * x + 1]);
                    mma_bf16_16816(s[j + x], ul, eh[2 * x], eh[2 * x + 1]);
                    mma_bf16_16816(s[j + x], uh, el[2 * x], el[2 * x + 1]);
                }
            }
            // ---- read-out ------------------------------------------------------------------------------------
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                mma_bf16_16816(r[n], uh, bh[2 * n], bh[2 * n + 1]);
                mma_bf16_16816(rl[n], ul, bh[2 * n], bh[2 * n + 1]);
                mma_bf16_16816(rl[n], uh, bl[2 * n], bl[2 * n + 1]);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = i * DC_TOKENS + n * 8 + 2 * t4 + (e & 1), c = c0 + g + 8 * (e >> 1);
                    if (t < p.count && c < a.vdim) a.o[((int64_t)(p.row0 + t) * a.H + h) * a.vdim + c] = r[n][e] + rl[n][e];
                }
            }
        }
        if (i + 1 < chunks) {
            __syncthreads();  // every warp has read the stage
            if (threadIdx.x == 0 && i + DC_STAGES < chunks) load(i + DC_STAGES);
        }
    }
    if (!writes) return;
    if (mine)
#pragma unroll
        for (int j = 0; j < 2 * KS; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e)
                if (c0 + g + 8 * e < a.vdim) *reinterpret_cast<float2*>(state + (int64_t)(c0 + g + 8 * e) * DP + j * 8 + 2 * t4) = make_float2(s[j][2 * e], s[j][2 * e + 1]);
    if (!p.last || blockIdx.x) return;
    // the step's last rows are the convolution's history from here on (heads that share key channels write the same values)
    const bf16* proj = reinterpret_cast<const bf16*>(a.proj);
    const int C = 2 * a.G * a.dim + a.H * a.vdim, kept = min(a.taps - 1, a.rows), per = 2 * a.dim + a.vdim;
    bf16* ring = reinterpret_cast<bf16*>(a.conv_state) + (int64_t)seq * a.taps * C;
    for (int x = threadIdx.x; x < kept * per; x += blockDim.x) {
        const int row = a.rows - kept + x / per, c = x % per;
        const int chan = c < a.dim ? kvh * a.dim + c : c < 2 * a.dim ? (a.G + kvh) * a.dim + c - a.dim : 2 * a.G * a.dim + h * a.vdim + c - 2 * a.dim;
        ring[(int64_t)((a.row_pos[0] + row) % a.taps) * C + chan] = proj[(int64_t)row * a.proj_stride + chan];
    }
}

// ===================================================================================================
// 0: the sizes are not for these kernels; else the bytes of one record (one chunk of 16 tokens of one head).
GLMB_API int glmb_delta_chunk_record(int dim, int vdim, int taps) {
    if (dim < 8 || dim > 128 || (dim & 7) || vdim < 8 || (vdim & 7) || taps < 1 || taps > DC_TAPS) return 0;
    return dc_record_bytes((dim + 31) / 32 * 32, vdim);
}

template <int KS>
static int launch_chunk_scan(const DeltaChunkArgs& p, cudaStream_t st) {
    static DeviceOnce once;
    const int dev = once.pending();
    if (dev != DeviceOnce::SET) {
        const cudaError_t e = cudaFuncSetAttribute(delta_chunk_scan_kernel<KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, DC_STAGES * (dc_head_bytes(KS * 16) + 4 * dc_value_block()));
        if (e != cudaSuccess) return (int)e;
        once.mark(dev);
    }
    const size_t smem = (size_t)DC_STAGES * (dc_head_bytes(KS * 16) + p.warps * dc_value_block());
    GLMB_LAUNCH(delta_chunk_scan_kernel<KS>, dim3(ceil_div(ceil_div(p.d.vdim, 16), p.warps), p.d.H), 32 * p.warps, smem, st, p);
    return (int)cudaGetLastError();
}

// bf16, consecutive rows of one sequence: projection rows -> o, state and convolution history of the lane.  `records` holds at least H records
// and is used for as many chunks at a time as fit.
GLMB_API int glmb_delta_chunk(const DeltaArgs* args, void* records, int64_t bytes, void* stream) {
    DeltaChunkArgs p;
    p.d = *args;
    const DeltaArgs& a = p.d;
    const int record = glmb_delta_chunk_record(a.dim, a.vdim, a.taps);
    if (!delta_sizes_ok(a) || a.decode || !record || a.dimp > 128 || (a.proj_stride & 7) || a.off_b < 2 * a.G * a.dim + a.H * a.vdim || a.H > 65535) return 1;
    const int64_t chunks = bytes / ((int64_t)record * a.H);
    if (chunks < 1 || (reinterpret_cast<uintptr_t>(records) & 15)) return 2;
    cudaStream_t st = (cudaStream_t)stream;
    p.records = reinterpret_cast<unsigned char*>(records);
    const int blocks = ceil_div(a.vdim, 16);
    p.warps = blocks * a.H <= 148 ? 1 : blocks * a.H <= 2 * 148 ? 2 : 4;
    const int per_segment = (int)(chunks < ceil_div(a.rows, DC_TOKENS) ? chunks : ceil_div(a.rows, DC_TOKENS)) * DC_TOKENS;
    const size_t prep_smem = (size_t)3 * DC_TOKENS * (a.dimp + 4) * 4;
    for (p.row0 = 0; p.row0 < a.rows; p.row0 += per_segment) {
        p.count = min(per_segment, a.rows - p.row0);
        p.last = p.row0 + p.count == a.rows;
        GLMB_LAUNCH(delta_chunk_prep_kernel, dim3(ceil_div(p.count, DC_TOKENS), a.H), DC_THREADS, prep_smem, st, p);
        int code = (int)cudaGetLastError();
        if (code) return code;
        switch (a.dimp / 32) {
            case 1: code = launch_chunk_scan<2>(p, st); break;
            case 2: code = launch_chunk_scan<4>(p, st); break;
            case 3: code = launch_chunk_scan<6>(p, st); break;
            default: code = launch_chunk_scan<8>(p, st);
        }
        if (code) return code;
    }
    return 0;
}
