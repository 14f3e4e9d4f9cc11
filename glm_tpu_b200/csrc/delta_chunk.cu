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
//   delta_chunk_scan   two warps keep the fp32 state of 16 value channels in their accumulators ([value channel, key channel]: the accumulator
//                      layout is the operand layout of the next product) and walks the chunks; records arrive by bulk copies, several chunks
//                      ahead.  Products are hi.hi + hi.lo + lo.hi with fp32 sums.
//
// A record: [6][16][dimp + 8] bf16 (e^G k, e^G q, e^(G_last - G) k, each hi and lo), [4][16][24] bf16 (L hi, lo, B hi, lo), [dimp] fp32
// (e^G_last), [vdim / 16][16][20] fp32 (V by blocks of 16 channels).  Row paddings stagger the banks for ldmatrix.
#include <mutex>

#include "attention_core.cuh"
#include "delta_rule.cuh"
#include "tcgen05.cuh"
#include "vec8.cuh"

#define DC_TOKENS 16
#define DC_THREADS 256
#define DC_TAPS 4
#define DC_LB 24      // row of L and B
#define DC_VB 20      // row of a value block
#define DC_OVERLAP_CHUNKS 16  // longer steps prepare one segment while the one before is scanned
#define DC_LOG2E 1.4426950408889634f

struct DeltaChunkArgs {
    DeltaArgs d;
    unsigned char* records;  // [chunks of the segment, H] records
    int row0, count;         // the segment: rows row0 .. row0 + count - 1 of the step (row0 a multiple of 16)
    int last;                // the segment ends the step
    int blocks;              // scan: blocks of 16 value channels per CTA
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
__device__ __forceinline__ void dc_fold(float (&v)[16], int lane, int offset) {
    const bool upper = lane & offset;
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
        const float keep = upper ? v[i + N / 2] : v[i], send = upper ? v[i] : v[i + N / 2];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, offset);
    }
}

__device__ __forceinline__ float dc_silu(float z) { return __fdividef(z, 1.f + dc_exp2(-DC_LOG2E * z)); }

// Token t's rows of the three operands that meet the state, by one warp.  scale_k, scale_q: what makes the token's key and query unit vectors.
__device__ __forceinline__ void dc_operands(const float* q_s, const float* k_s, const float* g_s, int RS, int DP, int t, float scale_k, float scale_q,
                                            uint32_t* mats, int lane) {
    const int words = (DP + 8) / 2;
    for (int d = lane * 2; d < DP; d += 64) {
        const float2 g = *reinterpret_cast<const float2*>(g_s + t * RS + d), end = *reinterpret_cast<const float2*>(g_s + (DC_TOKENS - 1) * RS + d);
        float2 k = *reinterpret_cast<const float2*>(k_s + t * RS + d), q = *reinterpret_cast<const float2*>(q_s + t * RS + d);
        k.x *= scale_k; k.y *= scale_k; q.x *= scale_q; q.y *= scale_q;
        const float e0 = dc_exp2(g.x), e1 = dc_exp2(g.y), f0 = dc_exp2(end.x - g.x), f1 = dc_exp2(end.y - g.y);
        uint32_t* at = mats + t * words + d / 2;
        uint32_t hi, lo;
        dc_split(k.x * e0, k.y * e1, hi, lo);
        at[0] = hi;
        at[DC_TOKENS * words] = lo;
        dc_split(q.x * e0, q.y * e1, hi, lo);
        at[2 * DC_TOKENS * words] = hi;
        at[3 * DC_TOKENS * words] = lo;
        dc_split(k.x * f0, k.y * f1, hi, lo);
        at[4 * DC_TOKENS * words] = hi;
        at[5 * DC_TOKENS * words] = lo;
    }
}

// grid (chunks, H)
__global__ void __launch_bounds__(DC_THREADS, 4) delta_chunk_prep_kernel(DeltaChunkArgs p) {
    GLMB_PDL_PROLOGUE();
    const DeltaArgs& a = p.d;
    extern __shared__ __align__(16) float smem_f[];
    const int DP = a.dimp, RS = DP + 4;
    float* q_s = smem_f;                        // [16][RS]
    float* k_s = q_s + DC_TOKENS * RS;
    float* g_s = k_s + DC_TOKENS * RS;          // log2 of the decays, then their running sum
    __shared__ float A_s[DC_TOKENS][DC_TOKENS + 1], B_s[DC_TOKENS][DC_TOKENS + 1], beta_s[DC_TOKENS], scale_s[2 * DC_TOKENS];
    const int h = blockIdx.y, kvh = h / (a.H / a.G), t0 = p.row0 + blockIdx.x * DC_TOKENS, n = min(DC_TOKENS, p.row0 + p.count - t0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int C = 2 * a.G * a.dim + a.H * a.vdim, keep = a.taps - 1;
    unsigned char* record = p.records + ((int64_t)blockIdx.x * a.H + h) * dc_record_bytes(DP, a.vdim);
    float* v_out = reinterpret_cast<float*>(record + dc_head_bytes(DP));
    const bf16* proj = reinterpret_cast<const bf16*>(a.proj);
    const int start = a.row_pos[0], seq = delta_lane(a, 0);
    const bf16* state = reinterpret_cast<const bf16*>(a.conv_state) + (int64_t)seq * a.taps * C;

    // ---- convolution: a thread takes four channels of four tokens ------------------------------------------
    const int kvec = a.dim / 4, vecs = 2 * kvec + a.vdim / 4;
    for (int i = tid; i < vecs * 4; i += DC_THREADS) {
        const int strip = i / vecs, vec = i - strip * vecs, first = strip * 4;
        const int kind = vec < kvec ? 0 : vec < 2 * kvec ? 1 : 2, c = (kind == 0 ? vec : kind == 1 ? vec - kvec : vec - 2 * kvec) * 4;
        const int chan = (kind == 0 ? kvh * a.dim : kind == 1 ? (a.G + kvh) * a.dim : 2 * a.G * a.dim + h * a.vdim) + c;
        uint2 u[4 + DC_TAPS - 1];
#pragma unroll
        for (int j = 0; j < 4 + DC_TAPS - 1; ++j) {
            const int row = t0 + first + j - (DC_TAPS - 1);  // row of the step; before it: the lane's ring of projected rows
            u[j] = make_uint2(0, 0);
            if (row >= 0 && row < t0 + n) u[j] = *reinterpret_cast<const uint2*>(proj + (int64_t)row * a.proj_stride + chan);
            else if (row < 0 && row >= -keep && start + row >= 0) u[j] = *reinterpret_cast<const uint2*>(state + (int64_t)((start + row) % a.taps) * C + chan);
        }
        float y[4][4];
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) y[t][e] = 0.f;
#pragma unroll
        for (int j = 0; j < DC_TAPS; ++j) {
            const int tap = j - (DC_TAPS - a.taps);  // fewer taps: the oldest ones are not there
            if (tap < 0) continue;
            const float4 w = *reinterpret_cast<const float4*>(a.conv_w + (int64_t)tap * C + chan);
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                y[t][0] = fmaf(w.x, bf16_lo(u[t + j].x), y[t][0]);
                y[t][1] = fmaf(w.y, bf16_hi(u[t + j].x), y[t][1]);
                y[t][2] = fmaf(w.z, bf16_lo(u[t + j].y), y[t][2]);
                y[t][3] = fmaf(w.w, bf16_hi(u[t + j].y), y[t][3]);
            }
        }
        float* dst = kind == 2 ? v_out + ((int64_t)(c / 16) * DC_TOKENS + first) * DC_VB + c % 16 : (kind == 0 ? q_s : k_s) + first * RS + c;
        const int stride = kind == 2 ? DC_VB : RS;
#pragma unroll
        for (int t = 0; t < 4; ++t)
            *reinterpret_cast<float4*>(dst + t * stride) = first + t < n ? make_float4(dc_silu(y[t][0]), dc_silu(y[t][1]), dc_silu(y[t][2]), dc_silu(y[t][3]))
                                                                         : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (a.dim < DP)  // padding of the key channels
        for (int r = warp; r < 2 * DC_TOKENS; r += DC_THREADS / 32)
            for (int d = a.dim + lane; d < DP; d += 32) (r < DC_TOKENS ? q_s : k_s)[(r % DC_TOKENS) * RS + d] = 0.f;
    if (a.vdim % 16)  // the last value block's second half
        for (int i = tid; i < DC_TOKENS * 8; i += DC_THREADS) v_out[((int64_t)(a.vdim / 16) * DC_TOKENS + i / 8) * DC_VB + 8 + i % 8] = 0.f;
    // ---- decays ------------------------------------------------------------------------------------------
    const float rate = a.a_rate[h] * DC_LOG2E;
    for (int d = lane; d < DP; d += 32) {
        const float bias = d < a.dim ? a.dt_bias[h * a.dim + d] : 0.f;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int t = warp + x * (DC_THREADS / 32);
            g_s[t * RS + d] = t < n && d < a.dim ? -rate * delta_softplus(a.a[(int64_t)(t0 + t) * a.a_stride + h * a.dim + d] + bias) : 0.f;
        }
    }
    if (tid < DC_TOKENS) beta_s[tid] = tid < n ? sigmoidf_precise(__bfloat162float(proj[(int64_t)(t0 + tid) * a.proj_stride + a.off_b + h])) : 0.f;
    __syncthreads();
    // ---- what makes unit vectors (a warp per row), running sums of the decays --------------------------------
    {
        const float* rows = (warp < 4 ? q_s : k_s) + (warp & 3) * 4 * RS;  // four rows per warp, queries first
        float ss[4] = {0.f, 0.f, 0.f, 0.f};
        for (int d = lane; d < DP; d += 32)
#pragma unroll
            for (int x = 0; x < 4; ++x) ss[x] = fmaf(rows[x * RS + d], rows[x * RS + d], ss[x]);
        // the four sums at once: after two steps a quarter of the warp is left with each
        const bool up = lane & 16, right = lane & 8;
        const float s0 = (up ? ss[2] : ss[0]) + __shfl_xor_sync(0xffffffffu, up ? ss[0] : ss[2], 16);
        const float s1 = (up ? ss[3] : ss[1]) + __shfl_xor_sync(0xffffffffu, up ? ss[1] : ss[3], 16);
        float sum = (right ? s1 : s0) + __shfl_xor_sync(0xffffffffu, right ? s0 : s1, 8);
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        if (!(lane & 7)) scale_s[warp * 4 + lane / 8] = rsqrtf(sum + 1e-6f) * (warp < 4 ? rsqrtf((float)a.dim) : 1.f);
    }
    for (int d = tid; d < DP; d += DC_THREADS) {
        float sum = 0.f;
#pragma unroll
        for (int t = 0; t < DC_TOKENS; ++t) { sum += g_s[t * RS + d]; g_s[t * RS + d] = sum; }
    }
    __syncthreads();
    uint32_t* mats = reinterpret_cast<uint32_t*>(record);
    auto operands = [&](int t) { dc_operands(q_s, k_s, g_s, RS, DP, t, scale_s[DC_TOKENS + t], scale_s[t], mats, lane); };
    if (warp >= 5) {  // the warps that have no pairs take the operands
        for (int t = warp - 5; t < DC_TOKENS; t += 3) operands(t);
    } else {
        // ---- A and B: 4 x 4 blocks of (i, j) below the diagonal, one after the other two per warp; half of the warp makes A, half B -------
        const int sub = lane & 15;
        const float* x_s = lane < 16 ? k_s : q_s;
        for (int block = warp * 2; block < warp * 2 + 2; ++block) {
            const int bi = block < 1 ? 0 : block < 3 ? 1 : block < 6 ? 2 : 3, bj = block - bi * (bi + 1) / 2;
            float acc[16];
#pragma unroll
            for (int x = 0; x < 16; ++x) acc[x] = 0.f;
            for (int d = sub; d < DP; d += 16) {
                float gi[4], xi[4], gj[4], kj[4];
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    gi[x] = g_s[(bi * 4 + x) * RS + d];
                    xi[x] = x_s[(bi * 4 + x) * RS + d];
                    gj[x] = g_s[(bj * 4 + x) * RS + d];
                    kj[x] = k_s[(bj * 4 + x) * RS + d];
                }
                if (bi != bj) {  // exp(G_i - G_j) in two factors around the end of the earlier block, both at most one
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        xi[x] *= dc_exp2(gi[x] - gj[3]);
                        kj[x] *= dc_exp2(gj[3] - gj[x]);
                    }
#pragma unroll
                    for (int x = 0; x < 4; ++x)
#pragma unroll
                        for (int y = 0; y < 4; ++y) acc[x * 4 + y] = fmaf(xi[x], kj[y], acc[x * 4 + y]);
                } else {
#pragma unroll
                    for (int x = 0; x < 4; ++x)
#pragma unroll
                        for (int y = 0; y <= x; ++y) acc[x * 4 + y] = fmaf(xi[x], x == y ? kj[y] : kj[y] * dc_exp2(gi[x] - gj[y]), acc[x * 4 + y]);
                }
            }
            dc_fold<16>(acc, lane, 8);
            dc_fold<8>(acc, lane, 4);
            dc_fold<4>(acc, lane, 2);
            dc_fold<2>(acc, lane, 1);
            // lane bits from the highest choose the half at every step: this lane holds value `sub`
            const int i = bi * 4 + sub / 4, j = bj * 4 + (sub & 3);
            if (lane < 16) A_s[i][j] = j < i ? acc[0] * scale_s[DC_TOKENS + i] * scale_s[DC_TOKENS + j] : 0.f;
            else B_s[i][j] = j <= i ? acc[0] * scale_s[i] * scale_s[DC_TOKENS + j] : 0.f;
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
    } else if (warp == 2) {
        float* gamma = reinterpret_cast<float*>(record + dc_mats_bytes(DP) + 4 * DC_TOKENS * DC_LB * 2);
        for (int d = lane; d < DP; d += 32) gamma[d] = dc_exp2(g_s[(DC_TOKENS - 1) * RS + d]);
    }
}

// ---------------------------------------------------------------------------------------------------
#define DC_STAGES 3

__device__ __forceinline__ void dc_bulk_load(void* smem_dst, const void* src, uint32_t bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(smem_u32(smem_dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}

// grid (groups of `blocks` blocks of 16 value channels, H), 64 * blocks threads: two warps share a block, each with half of the key channels
// (the tensor pipe of one scheduler is what a single warp would wait for).  KS: key channels / 32, the 16-channel steps of a warp.
template <int KS>
__global__ void __launch_bounds__(256) delta_chunk_scan_kernel(DeltaChunkArgs p) {
    constexpr int DP = KS * 32, RS = DP + 8;
    const DeltaArgs& a = p.d;
    extern __shared__ __align__(128) unsigned char smem_raw[];
    __shared__ __align__(8) uint64_t full_bar[DC_STAGES];
    __shared__ float4 swap_s[4][2][3][32];  // [block][half]: what a warp's half of the key channels adds to the products
    const int h = blockIdx.y, kvh = h / (a.H / a.G), chunks = (p.count + DC_TOKENS - 1) / DC_TOKENS;
    const int blocks = (a.vdim + 15) / 16, block0 = blockIdx.x * p.blocks, here = min(p.blocks, blocks - block0);
    const int head_bytes = dc_head_bytes(DP), value_bytes = here * dc_value_block(), stage_bytes = head_bytes + p.blocks * dc_value_block();
    const int64_t record_bytes = dc_record_bytes(DP, a.vdim);
    const int lane = threadIdx.x & 31, block = threadIdx.x >> 6, half = (threadIdx.x >> 5) & 1;
    const int g = lane >> 2, t4 = lane & 3, mr = lane & 7, mi = lane >> 3;
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
    const bool mine = block < here;
    const int c0 = (block0 + block) * 16, k0 = half * KS * 16, seq = delta_lane(a, 0), start = a.row_pos[0] + p.row0;
    float* state = a.state + ((int64_t)seq * a.H + h) * a.vdim * DP + k0;
    const bool writes = delta_writes(a, 0);
    // accumulators of the transposed state: value channels c0 + g, + 8; key channels k0 + 8 j + 2 t4, + 1
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
        const bf16* mats = reinterpret_cast<const bf16*>(base) + k0;
        const bf16* lb = reinterpret_cast<const bf16*>(base + dc_mats_bytes(DP));
        const float* gamma = reinterpret_cast<const float*>(base + dc_mats_bytes(DP) + 4 * DC_TOKENS * DC_LB * 2) + k0;
        const float* v_s = reinterpret_cast<const float*>(base + head_bytes + block * dc_value_block());
        if (mine) {
            // ---- (e^G k) S and (e^G q) S, transposed: value channels x tokens, over this warp's key channels --------
            float w[2][4], wl[2][4], wm[2][4], r[2][4], rl[2][4], rm[2][4];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) w[n][e] = wl[n][e] = wm[n][e] = r[n][e] = rl[n][e] = rm[n][e] = 0.f;
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
                    mma_bf16_16816(wl[n], lo, kh[2 * n], kh[2 * n + 1]);
                    mma_bf16_16816(wm[n], hi, kl[2 * n], kl[2 * n + 1]);
                }
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    mma_bf16_16816(r[n], hi, qh[2 * n], qh[2 * n + 1]);
                    mma_bf16_16816(rl[n], lo, qh[2 * n], qh[2 * n + 1]);
                    mma_bf16_16816(rm[n], hi, ql[2 * n], ql[2 * n + 1]);
                }
            }
            // ---- the two halves meet: both warps go on with all of w, each with the read-out of eight tokens ---------
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) { w[n][e] += wl[n][e] + wm[n][e]; r[n][e] += rl[n][e] + rm[n][e]; }
            const int other = half ^ 1;
            swap_s[block][half][0][lane] = make_float4(w[0][0], w[0][1], w[0][2], w[0][3]);
            swap_s[block][half][1][lane] = make_float4(w[1][0], w[1][1], w[1][2], w[1][3]);
            swap_s[block][half][2][lane] = half ? make_float4(r[0][0], r[0][1], r[0][2], r[0][3]) : make_float4(r[1][0], r[1][1], r[1][2], r[1][3]);
            asm volatile("bar.sync %0, 64;" ::"r"(block + 1) : "memory");
            const float4 w0 = swap_s[block][other][0][lane], w1 = swap_s[block][other][1][lane], r0 = swap_s[block][other][2][lane];
            w[0][0] += w0.x; w[0][1] += w0.y; w[0][2] += w0.z; w[0][3] += w0.w;
            w[1][0] += w1.x; w[1][1] += w1.y; w[1][2] += w1.z; w[1][3] += w1.w;
            float out[4] = {(half ? r[1][0] : r[0][0]) + r0.x, (half ? r[1][1] : r[0][1]) + r0.y, (half ? r[1][2] : r[0][2]) + r0.z, (half ? r[1][3] : r[0][3]) + r0.w};
            // ---- U = L (V - ..) -----------------------------------------------------------------------------
            uint32_t xh[4], xl[4];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e)
                    dc_split(v_s[(n * 8 + 2 * t4) * DC_VB + g + 8 * e] - w[n][2 * e], v_s[(n * 8 + 2 * t4 + 1) * DC_VB + g + 8 * e] - w[n][2 * e + 1], xh[2 * n + e],
                             xl[2 * n + e]);
            uint32_t lh[4], ll[4], bh[2], bl[2];
            const bf16* at_l = lb + (mr + 8 * (mi >> 1)) * DC_LB + 8 * (mi & 1);
            const bf16* at_b = lb + (2 * DC_TOKENS + half * 8 + mr) * DC_LB + 8 * (mi & 1);
            ldmatrix_x4(lh, at_l);
            ldmatrix_x4(ll, at_l + DC_TOKENS * DC_LB);
            ldmatrix_x2(bh, at_b);
            ldmatrix_x2(bl, at_b + DC_TOKENS * DC_LB);
            uint32_t uh[4], ul[4];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                float u[4] = {0.f, 0.f, 0.f, 0.f}, u1[4] = {0.f, 0.f, 0.f, 0.f}, u2[4] = {0.f, 0.f, 0.f, 0.f};
                mma_bf16_16816(u, xh, lh[2 * n], lh[2 * n + 1]);
                mma_bf16_16816(u1, xl, lh[2 * n], lh[2 * n + 1]);
                mma_bf16_16816(u2, xh, ll[2 * n], ll[2 * n + 1]);
                dc_split(u[0] + (u1[0] + u2[0]), u[1] + (u1[1] + u2[1]), uh[2 * n], ul[2 * n]);
                dc_split(u[2] + (u1[2] + u2[2]), u[3] + (u1[3] + u2[3]), uh[2 * n + 1], ul[2 * n + 1]);
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
                }
#pragma unroll
                for (int x = 0; x < 2; ++x) mma_bf16_16816(s[j + x], uh, eh[2 * x], eh[2 * x + 1]);
#pragma unroll
                for (int x = 0; x < 2; ++x) mma_bf16_16816(s[j + x], ul, eh[2 * x], eh[2 * x + 1]);
#pragma unroll
                for (int x = 0; x < 2; ++x) mma_bf16_16816(s[j + x], uh, el[2 * x], el[2 * x + 1]);
            }
            // ---- read-out of this warp's eight tokens ----------------------------------------------------------
            mma_bf16_16816(out, uh, bh[0], bh[1]);
            mma_bf16_16816(out, ul, bh[0], bh[1]);
            mma_bf16_16816(out, uh, bl[0], bl[1]);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = i * DC_TOKENS + half * 8 + 2 * t4 + (e & 1), c = c0 + g + 8 * (e >> 1);
                if (t < p.count && c < a.vdim) a.o[((int64_t)(p.row0 + t) * a.H + h) * a.vdim + c] = out[e];
            }
        }
        if (i + 1 < chunks) {
            __syncthreads();  // every warp has read the stage, and its partner's sums
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
        const cudaError_t e = cudaFuncSetAttribute(delta_chunk_scan_kernel<KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, DC_STAGES * (dc_head_bytes(KS * 32) + 4 * dc_value_block()));
        if (e != cudaSuccess) return (int)e;
        once.mark(dev);
    }
    const size_t smem = (size_t)DC_STAGES * (dc_head_bytes(KS * 32) + p.blocks * dc_value_block());
    GLMB_LAUNCH(delta_chunk_scan_kernel<KS>, dim3(ceil_div(ceil_div(p.d.vdim, 16), p.blocks), p.d.H), 64 * p.blocks, smem, st, p);
    return (int)cudaGetLastError();
}

// The scan of a segment and the preparation of the next run side by side: a second stream per device, two halves of the records in turn.
struct DeltaStreams {
    cudaStream_t scan = nullptr;
    cudaEvent_t prepared = nullptr, scanned[2] = {nullptr, nullptr};
    bool ready = false;
};
static cudaError_t delta_streams(DeltaStreams** out) {
    static std::mutex mutex;
    static DeltaStreams per_device[DeviceOnce::MAX_DEVICES];
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return e;
    if (dev < 0 || dev >= DeviceOnce::MAX_DEVICES) return cudaErrorInvalidDevice;
    std::lock_guard<std::mutex> lock(mutex);
    DeltaStreams& s = per_device[dev];
    if (!s.ready) {
        int low = 0, high = 0;
        cudaDeviceGetStreamPriorityRange(&low, &high);
        if ((e = cudaStreamCreateWithPriority(&s.scan, cudaStreamNonBlocking, high)) != cudaSuccess) return e;
        for (cudaEvent_t* event : {&s.prepared, &s.scanned[0], &s.scanned[1]})
            if ((e = cudaEventCreateWithFlags(event, cudaEventDisableTiming)) != cudaSuccess) return e;
        s.ready = true;
    }
    *out = &s;
    return cudaSuccess;
}

static int launch_scan_of(const DeltaChunkArgs& p, cudaStream_t st) {
    switch (p.d.dimp / 32) {
        case 1: return launch_chunk_scan<1>(p, st);
        case 2: return launch_chunk_scan<2>(p, st);
        case 3: return launch_chunk_scan<3>(p, st);
        default: return launch_chunk_scan<4>(p, st);
    }
}

// bf16, consecutive rows of one sequence: projection rows -> o, state and convolution history of the lane.  `records` holds at least H records
// and is used for as many chunks at a time as fit (half of it, in turn, when the step does not fit at once).
GLMB_API int glmb_delta_chunk(const DeltaArgs* args, void* records, int64_t bytes, void* stream) {
    DeltaChunkArgs p;
    p.d = *args;
    const DeltaArgs& a = p.d;
    const int record = glmb_delta_chunk_record(a.dim, a.vdim, a.taps);
    if (!delta_sizes_ok(a) || a.decode || !record || a.dimp > 128 || (a.proj_stride & 7) || a.off_b < 2 * a.G * a.dim + a.H * a.vdim || a.H > 65535) return 1;
    const int64_t per_chunk = (int64_t)record * a.H, chunks = bytes / per_chunk, needed = ceil_div(a.rows, DC_TOKENS);
    if (chunks < 1 || (reinterpret_cast<uintptr_t>(records) & 15)) return 2;
    cudaStream_t st = (cudaStream_t)stream;
    unsigned char* base = reinterpret_cast<unsigned char*>(records);
    const int blocks = ceil_div(a.vdim, 16);
    p.blocks = blocks * a.H <= 148 ? 1 : blocks * a.H <= 2 * 148 ? 2 : 4;
    const size_t prep_smem = (size_t)3 * DC_TOKENS * (a.dimp + 4) * 4;
    auto prepare = [&] {
        GLMB_LAUNCH(delta_chunk_prep_kernel, dim3(ceil_div(p.count, DC_TOKENS), a.H), DC_THREADS, prep_smem, st, p);
        return (int)cudaGetLastError();
    };
    const bool halves = needed > DC_OVERLAP_CHUNKS && chunks >= 2;  // worth two streams
    const int64_t at_once = halves ? (needed + 1) / 2 < chunks / 2 ? (needed + 1) / 2 : chunks / 2 : chunks;
    const int segment = (int)(at_once < needed ? at_once : needed) * DC_TOKENS;
    if (!halves) {
        p.records = base;
        for (p.row0 = 0; p.row0 < a.rows; p.row0 += segment) {
            p.count = min(segment, a.rows - p.row0);
            p.last = p.row0 + p.count == a.rows;
            int code = prepare();
            if (!code) code = launch_scan_of(p, st);
            if (code) return code;
        }
        return 0;
    }
    DeltaStreams* side = nullptr;
    cudaError_t e = delta_streams(&side);
    if (e != cudaSuccess) return (int)e;
    int i = 0;
    for (p.row0 = 0; p.row0 < a.rows; p.row0 += segment, ++i) {
        p.count = min(segment, a.rows - p.row0);
        p.last = p.row0 + p.count == a.rows;
        p.records = base + (i & 1) * at_once * per_chunk;
        if (i >= 2 && (e = cudaStreamWaitEvent(st, side->scanned[i & 1], 0)) != cudaSuccess) return (int)e;
        int code = prepare();
        if (code) return code;
        if ((e = cudaEventRecord(side->prepared, st)) != cudaSuccess || (e = cudaStreamWaitEvent(side->scan, side->prepared, 0)) != cudaSuccess) return (int)e;
        if ((code = launch_scan_of(p, side->scan))) return code;
        if ((e = cudaEventRecord(side->scanned[i & 1], side->scan)) != cudaSuccess) return (int)e;
    }
    return (int)cudaStreamWaitEvent(st, side->scanned[(i - 1) & 1], 0);
}
