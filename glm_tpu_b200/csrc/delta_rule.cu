// Gated delta rule with one decay per head and key channel: a recurrent state S [dim, vdim] per head and sequence,
//
//   S <- diag(g_t) S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t,
//
// fp32 throughout.  q, k and v come from the layer's projection through a short causal convolution over time and SiLU; q and k are then unit
// vectors per head (q also scaled by dim^-1/2); beta = sigmoid; log g = -rate softplus(a + bias).  What is read out is normalized per head
// and gated.
//
//   delta_prep   projection -> q, k, v, log g, beta (any sizes, decode and prefill); the convolution's history moves on
//   delta_scan   the recurrence token by token: a thread keeps 4 DQ key channels of one value channel in registers, eight threads share a
//                value channel; the two sums over key channels of a token are reduced together (o_t = S'^T q_t + (q_t . k_t) u_t)
//   delta_out    root-mean-square norm per head, output gate
//
// The convolution's history is a ring of `taps` projected rows per lane (slot = position mod taps): a decode step writes a slot that none of
// its readers needs.  Prefill: the rows are consecutive tokens of one sequence.  Decode: every row is the next token of its own sequence (lane).  A sequence at
// position 0 starts from zeros whatever its lane held before.
#include "attention_core.cuh"
#include "common.cuh"
#include "delta_rule.cuh"
#include "vec8.cuh"

#define DR_THREADS 256
#define DR_WARPS (DR_THREADS / 32)
#define DR_MAX_ROWS 32     // rows of a prep block: taps - 1 may not exceed it
#define DR_CH 8            // key channels per lane held while a row's norm is found: dim up to 256

// grid (row blocks, G q-heads + G k-heads + H v-heads + H decay heads).  A warp takes a row of the block at a time.
template <typename T>
__global__ void __launch_bounds__(DR_THREADS) delta_prep_kernel(DeltaArgs a) {
    GLMB_PDL_PROLOGUE();
    const int r0 = blockIdx.x * a.rows_per_block, n = min(a.rows_per_block, a.rows - r0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y;
    if (head >= 2 * a.G + a.H) {  // decay and beta of a head
        const int h = head - 2 * a.G - a.H;
        const float rate = a.a_rate[h];
        for (int r = warp; r < n; r += DR_WARPS) {
            const int row = r0 + r;
            const float* src = a.a + (int64_t)row * a.a_stride + h * a.dim;
            float* dst = a.lg + ((int64_t)row * a.H + h) * a.dimp;
            for (int d = lane; d < a.dimp; d += 32) dst[d] = d < a.dim ? -rate * delta_softplus(src[d] + a.dt_bias[h * a.dim + d]) : 0.f;
            if (lane == 0)
                a.beta[(int64_t)row * a.H + h] = sigmoidf_precise(to_f32(reinterpret_cast<const T*>(a.proj)[(int64_t)row * a.proj_stride + a.off_b + h]));
        }
        return;
    }
    const int kind = head < a.G ? 0 : head < 2 * a.G ? 1 : 2;
    const int slot = kind == 0 ? head : kind == 1 ? head - a.G : head - 2 * a.G;
    const int hd = kind == 2 ? a.vdim : a.dim, C = 2 * a.G * a.dim + a.H * a.vdim;
    const int chan0 = kind == 0 ? slot * a.dim : kind == 1 ? (a.G + slot) * a.dim : 2 * a.G * a.dim + slot * a.vdim;
    const T* proj = reinterpret_cast<const T*>(a.proj) + chan0;
    const int state_lane = delta_lane(a, a.decode ? r0 : 0), keep = a.taps - 1;
    T* ring = reinterpret_cast<T*>(a.conv_state) + (int64_t)state_lane * a.taps * C + chan0;
    auto conv = [&](int row, int pos, int c) {
        float y = 0.f;
        for (int j = 0; j < a.taps; ++j) {
            const int back = keep - j;
            if (back > pos) continue;  // before the sequence's start
            const bool here = a.decode ? back == 0 : row >= back;
            const T u = here ? proj[(int64_t)(row - back) * a.proj_stride + c] : ring[(int64_t)((pos - back) % a.taps) * C + c];
            y = fmaf(a.conv_w[(int64_t)j * C + chan0 + c], to_f32(u), y);
        }
        return delta_silu(y);
    };
    for (int r = warp; r < n; r += DR_WARPS) {
        const int row = r0 + r, pos = a.row_pos[row];
        if (kind == 2) {
            float* dst = a.v + ((int64_t)row * a.H + slot) * a.vdim;
            for (int c = lane; c < hd; c += 32) dst[c] = conv(row, pos, c);
            continue;
        }
        float y[DR_CH], ss = 0.f;
#pragma unroll
        for (int i = 0; i < DR_CH; ++i) {
            const int c = lane + 32 * i;
            y[i] = c < hd ? conv(row, pos, c) : 0.f;
            ss = fmaf(y[i], y[i], ss);
        }
        ss = warp_sum(ss);
        const float scale = (kind == 0 ? 1.f / sqrtf((float)a.dim) : 1.f) / sqrtf(ss + 1e-6f);
        float* dst = (kind == 0 ? a.q : a.k) + ((int64_t)row * a.G + slot) * a.dimp;
#pragma unroll
        for (int i = 0; i < DR_CH; ++i)
            if (lane + 32 * i < a.dimp) dst[lane + 32 * i] = y[i] * scale;
    }
    if (!a.decode && blockIdx.x > 0) return;
    __syncthreads();  // the first rows have read the ring (no other block does: a block holds at least taps - 1 rows)
    const int first = a.decode ? r0 : 0, rows = a.decode ? 1 : a.rows, kept = min(keep, rows);
    if (!delta_writes(a, first)) return;
    for (int i = threadIdx.x; i < kept * hd; i += DR_THREADS) {
        const int row = first + rows - kept + i / hd;
        ring[(int64_t)(a.row_pos[row] % a.taps) * C + i % hd] = proj[(int64_t)row * a.proj_stride + i % hd];
    }
}

// ---------------------------------------------------------------------------------------------------
#define DS_THREADS 128
#define DS_COLS 16    // value channels per CTA
#define DS_TOKENS 8   // tokens per stage

static inline int delta_stage_floats(int dimp) { return DS_TOKENS * (3 * dimp + DS_COLS); }

// grid (blocks of DS_COLS value channels, heads, sequences).
template <int DQ>
__global__ void __launch_bounds__(DS_THREADS) delta_scan_kernel(DeltaArgs a) {
    GLMB_PDL_PROLOGUE();
    constexpr int DIMP = DQ * 32;
    extern __shared__ __align__(16) float smem_f[];
    __shared__ float qk_s[DS_TOKENS], beta_s[2][DS_TOKENS];
    const int stage_floats = DS_TOKENS * (3 * DIMP + DS_COLS);
    const int h = blockIdx.y, kvh = h / (a.H / a.G), c0 = blockIdx.x * DS_COLS;
    const int first = a.decode ? blockIdx.z : 0, total = a.decode ? 1 : a.rows;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kg = lane >> 2, col = warp * 4 + (lane & 3);
    const bool valid = c0 + col < a.vdim;
    const int seq_lane = delta_lane(a, first);
    float* state = a.state + (((int64_t)seq_lane * a.H + h) * a.vdim + min(c0 + col, a.vdim - 1)) * DIMP + kg * 4;
    float4 s[DQ];
    const bool fresh = a.row_pos[first] <= 0;
#pragma unroll
    for (int i = 0; i < DQ; ++i) s[i] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(state + 32 * i);

    auto load = [&](int t0) {  // q, k, log g and v of DS_TOKENS tokens, asynchronously
        float* q_s = smem_f + ((t0 / DS_TOKENS) & 1) * stage_floats;
        float *k_s = q_s + DS_TOKENS * DIMP, *g_s = k_s + DS_TOKENS * DIMP, *v_s = g_s + DS_TOKENS * DIMP;
        const int n = min(DS_TOKENS, total - t0);
        for (int i = threadIdx.x; i < n * (DIMP / 4); i += DS_THREADS) {
            const int t = i / (DIMP / 4), d = i % (DIMP / 4) * 4;
            const int64_t row = first + t0 + t;
            cp_async16(q_s + t * DIMP + d, a.q + (row * a.G + kvh) * DIMP + d);
            cp_async16(k_s + t * DIMP + d, a.k + (row * a.G + kvh) * DIMP + d);
            cp_async16(g_s + t * DIMP + d, a.lg + (row * a.H + h) * DIMP + d);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        for (int i = threadIdx.x; i < n * DS_COLS; i += DS_THREADS) {
            const int t = i / DS_COLS, c = c0 + i % DS_COLS;
            v_s[i] = c < a.vdim ? a.v[((int64_t)(first + t0 + t) * a.H + h) * a.vdim + c] : 0.f;
        }
        if ((int)threadIdx.x < n) beta_s[(t0 / DS_TOKENS) & 1][threadIdx.x] = a.beta[(int64_t)(first + t0 + threadIdx.x) * a.H + h];
    };
    load(0);
    for (int t0 = 0; t0 < total; t0 += DS_TOKENS) {
        const int n = min(DS_TOKENS, total - t0), buf = (t0 / DS_TOKENS) & 1;
        float* q_s = smem_f + buf * stage_floats;
        float *k_s = q_s + DS_TOKENS * DIMP, *g_s = k_s + DS_TOKENS * DIMP, *v_s = g_s + DS_TOKENS * DIMP;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the stage has arrived, and nobody reads the other one any more
        if (t0 + DS_TOKENS < total) load(t0 + DS_TOKENS);
        for (int i = threadIdx.x; i < n * DIMP; i += DS_THREADS) g_s[i] = expf(g_s[i]);
        for (int t = warp; t < n; t += DS_THREADS / 32) {
            float x = 0.f;
            for (int d = lane; d < DIMP; d += 32) x = fmaf(q_s[t * DIMP + d], k_s[t * DIMP + d], x);
            x = warp_sum(x);
            if (lane == 0) qk_s[t] = x;
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            float rk[4] = {0.f, 0.f, 0.f, 0.f}, rq[4] = {0.f, 0.f, 0.f, 0.f};
            float4 kk[DQ];
#pragma unroll
            for (int i = 0; i < DQ; ++i) {
                const float4 g = *reinterpret_cast<const float4*>(g_s + t * DIMP + 32 * i + kg * 4);
                const float4 q = *reinterpret_cast<const float4*>(q_s + t * DIMP + 32 * i + kg * 4);
                kk[i] = *reinterpret_cast<const float4*>(k_s + t * DIMP + 32 * i + kg * 4);
                s[i].x *= g.x; s[i].y *= g.y; s[i].z *= g.z; s[i].w *= g.w;
                rk[0] = fmaf(s[i].x, kk[i].x, rk[0]); rk[1] = fmaf(s[i].y, kk[i].y, rk[1]);
                rk[2] = fmaf(s[i].z, kk[i].z, rk[2]); rk[3] = fmaf(s[i].w, kk[i].w, rk[3]);
                rq[0] = fmaf(s[i].x, q.x, rq[0]); rq[1] = fmaf(s[i].y, q.y, rq[1]);
                rq[2] = fmaf(s[i].z, q.z, rq[2]); rq[3] = fmaf(s[i].w, q.w, rq[3]);
            }
            float x = (rk[0] + rk[1]) + (rk[2] + rk[3]), y = (rq[0] + rq[1]) + (rq[2] + rq[3]);
#pragma unroll
            for (int o = 4; o < 32; o <<= 1) {
                x += __shfl_xor_sync(0xffffffffu, x, o);
                y += __shfl_xor_sync(0xffffffffu, y, o);
            }
            const float u = beta_s[buf][t] * (v_s[t * DS_COLS + col] - x);
#pragma unroll
            for (int i = 0; i < DQ; ++i) {
                s[i].x = fmaf(kk[i].x, u, s[i].x); s[i].y = fmaf(kk[i].y, u, s[i].y);
                s[i].z = fmaf(kk[i].z, u, s[i].z); s[i].w = fmaf(kk[i].w, u, s[i].w);
            }
            if (kg == 0 && valid) a.o[((int64_t)(first + t0 + t) * a.H + h) * a.vdim + c0 + col] = fmaf(qk_s[t], u, y);
        }
    }
    if (valid && delta_writes(a, first))
#pragma unroll
        for (int i = 0; i < DQ; ++i) *reinterpret_cast<float4*>(state + 32 * i) = s[i];
}

// ---------------------------------------------------------------------------------------------------
// out = o / rms(o) * norm * sigmoid(gate) per (row, head).  VEC: heads up to 128 wide in whole vectors, sixteen lanes per head with eight channels
// each, DR_UNITS heads per half of a warp, everything asked for at once; otherwise a warp per (row, head), any size.
#define DR_UNITS 2
template <typename T, bool VEC>
__global__ void __launch_bounds__(DR_THREADS) delta_out_kernel(DeltaArgs a) {
    GLMB_PDL_PROLOGUE();
    const int lane = threadIdx.x & 31;
    const uint32_t units = (uint32_t)a.rows * a.H, warp = blockIdx.x * DR_WARPS + (threadIdx.x >> 5);
    if constexpr (VEC) {
        const int c = (lane & 15) * 8;
        const bool in = c < a.vdim;
        float x[DR_UNITS][8], z[DR_UNITS][8], w[8];
        uint32_t row[DR_UNITS], at[DR_UNITS];
#pragma unroll
        for (int i = 0; i < DR_UNITS; ++i) {
            const uint32_t unit = (warp * DR_UNITS + i) * 2 + (lane >> 4);
            row[i] = unit / (uint32_t)a.H;
            at[i] = (unit - row[i] * a.H) * a.vdim + c;
#pragma unroll
            for (int e = 0; e < 8; ++e) x[i][e] = z[i][e] = 0.f;
            if (in && unit < units) {
                load8(a.o + (int64_t)unit * a.vdim + c, x[i]);
                load8(reinterpret_cast<const T*>(a.gate) + (int64_t)row[i] * a.gate_stride + at[i], z[i]);
            }
        }
        if (in) load8(a.norm + c, w);
#pragma unroll
        for (int i = 0; i < DR_UNITS; ++i) {
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(x[i][e], x[i][e], ss);
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float inv = 1.f / sqrtf(ss / (float)a.vdim + a.eps);
            if (!in || (warp * DR_UNITS + i) * 2 + (lane >> 4) >= units) continue;
#pragma unroll
            for (int e = 0; e < 8; ++e) x[i][e] = x[i][e] * inv * w[e] * (sizeof(T) == 4 ? sigmoidf_precise(z[i][e]) : __fdividef(1.f, 1.f + __expf(-z[i][e])));
            store8(reinterpret_cast<T*>(a.out) + (int64_t)row[i] * a.out_stride + at[i], x[i]);
        }
    } else {
        if (warp >= units) return;
        const int row = (int)(warp / a.H), h = (int)(warp % a.H);
        const float* o = a.o + (int64_t)warp * a.vdim;
        const T* gate = reinterpret_cast<const T*>(a.gate) + (int64_t)row * a.gate_stride + h * a.vdim;
        T* out = reinterpret_cast<T*>(a.out) + (int64_t)row * a.out_stride + h * a.vdim;
        float ss = 0.f;
        for (int c = lane; c < a.vdim; c += 32) ss = fmaf(o[c], o[c], ss);
        const float denom = sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
        for (int c = lane; c < a.vdim; c += 32) from_f32(o[c] / denom * a.norm[c] * sigmoidf_precise(to_f32(gate[c])), out[c]);
    }
}

// ===================================================================================================
GLMB_API size_t glmb_delta_args_sizeof(void) { return sizeof(DeltaArgs); }
GLMB_API int glmb_delta_max_taps(void) { return DR_MAX_ROWS + 1; }

GLMB_API int glmb_delta_prep(const DeltaArgs* args, int is_f32, void* stream) {
    DeltaArgs a = *args;
    if (!delta_sizes_ok(a) || a.taps < 1 || a.taps > DR_MAX_ROWS + 1 || a.off_b < 2 * a.G * a.dim + a.H * a.vdim) return 1;
    a.rows_per_block = a.decode ? 1 : DR_MAX_ROWS;
    const dim3 grid(ceil_div(a.rows, a.rows_per_block), 2 * a.G + 2 * a.H);
    if (is_f32) GLMB_LAUNCH(delta_prep_kernel<float>, grid, DR_THREADS, 0, (cudaStream_t)stream, a);
    else GLMB_LAUNCH(delta_prep_kernel<bf16>, grid, DR_THREADS, 0, (cudaStream_t)stream, a);
    return (int)cudaGetLastError();
}

template <int DQ>
static int launch_scan(const DeltaArgs& a, cudaStream_t st) {
    const size_t smem = 2 * (size_t)delta_stage_floats(DQ * 32) * sizeof(float);
    static DeviceOnce once;
    const int dev = once.pending();
    if (dev != DeviceOnce::SET) {
        const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<DQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        once.mark(dev);
    }
    GLMB_LAUNCH(delta_scan_kernel<DQ>, dim3(ceil_div(a.vdim, DS_COLS), a.H, a.decode ? a.rows : 1), DS_THREADS, smem, st, a);
    return (int)cudaGetLastError();
}

GLMB_API int glmb_delta_scan(const DeltaArgs* args, void* stream) {
    const DeltaArgs a = *args;
    if (!delta_sizes_ok(a)) return 1;
    switch (a.dimp / 32) {
        case 1: return launch_scan<1>(a, (cudaStream_t)stream);
        case 2: return launch_scan<2>(a, (cudaStream_t)stream);
        case 3: return launch_scan<3>(a, (cudaStream_t)stream);
        case 4: return launch_scan<4>(a, (cudaStream_t)stream);
        case 5: return launch_scan<5>(a, (cudaStream_t)stream);
        case 6: return launch_scan<6>(a, (cudaStream_t)stream);
        case 7: return launch_scan<7>(a, (cudaStream_t)stream);
        default: return launch_scan<8>(a, (cudaStream_t)stream);
    }
}

GLMB_API int glmb_delta_out(const DeltaArgs* args, int is_f32, void* stream) {
    const DeltaArgs a = *args;
    if (!delta_sizes_ok(a) || (int64_t)a.rows * a.H >= (int64_t)1 << 31) return 1;
    const bool vec = !(a.vdim & 7) && a.vdim <= 128 && !(a.gate_stride & 7) && !(a.out_stride & 7);
    const int64_t per_block = DR_WARPS * (vec ? 2 * DR_UNITS : 1);
    const int grid = (int)(((int64_t)a.rows * a.H + per_block - 1) / per_block);
    cudaStream_t st = (cudaStream_t)stream;
    if (is_f32) {
        if (vec) GLMB_LAUNCH((delta_out_kernel<float, true>), grid, DR_THREADS, 0, st, a);
        else GLMB_LAUNCH((delta_out_kernel<float, false>), grid, DR_THREADS, 0, st, a);
    } else {
        if (vec) GLMB_LAUNCH((delta_out_kernel<bf16, true>), grid, DR_THREADS, 0, st, a);
        else GLMB_LAUNCH((delta_out_kernel<bf16, false>), grid, DR_THREADS, 0, st, a);
    }
    return (int)cudaGetLastError();
}
