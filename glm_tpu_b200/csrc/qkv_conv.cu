// From the fused q | k | v projection of an attention layer to what the attention reads: a short causal convolution over time on every
// channel, rotary positions on q and k, mixing of the values with an earlier layer's values, and the cache write -- one launch.
//
//   y_t[c]  = sum_j w[c][j] * u_{t - taps + 1 + j}[c]      u: projected rows, zero before the sequence; the last taps - 1 of a sequence
//                                                         live in its lane's state between steps
//   (a, b) -> (a cos - b sin, b cos + a sin)               dimensions i and i + dims/2 of every q and k head, fp32 table
//   v       = (1 - lambda) v + lambda v_first
//
// A block owns one head (of q, k or v) and RB consecutive rows.  Prefill: the rows are one sequence; the rows' own history comes from
// the projection, that of the first rows from the state, and the block of the first rows also advances the state once it has read it
// (no other block reads it: RB >= taps - 1).  Decode: every row is its own sequence (lane), RB = 1.
//
// Keys and values go to the lane's ring (slot = position mod ring size: with chunked attention a ring of one chunk holds everything a
// later token can see) and, in prefill, to linear buffers that the attention reads for the rows of this step.  Rows before `ring_from`
// stay out of the ring: their slots may still hold keys that queries of this very step need; ring_store writes them afterwards.
#include "common.cuh"
#include "vec8.cuh"

#define QC_THREADS 128
#define QC_SMEM_FLOATS 12288
#define QC_MAX_ROWS 32

struct QkvConvArgs {
    const void* proj; int64_t proj_stride;       // [rows, C]
    const float* conv_w; int taps;               // [taps, C]
    void* state;                                 // [lanes, taps - 1, C]
    const int *row_pos, *row_lane, *row_active;  // row_active may be NULL
    const float2* rot; int rot_dims;             // [capacity, rot_dims / 2] (cos, sin)
    void *q, *k_new, *v_new;                     // [rows, H, dimp], [rows, G, dimp], [rows, G, vdimp]; k_new / v_new NULL in decode
    void *k_ring, *v_ring; int ring;             // [lanes, ring, G, dimp], [lanes, ring, G, vdimp]
    void* v_first; int v_mode; float mix;        // [rows, G, vdimp]; 0: not used, 1: store this layer's values, 2: mix with them
    int H, G, dim, dimp, vdim, vdimp, rows, decode, ring_from, capacity, lanes, rows_per_block;
    uint32_t* status;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(QC_THREADS) qkv_conv_kernel(QkvConvArgs a) {
    GLMB_PDL_PROLOGUE();
    extern __shared__ float y_s[];  // [rows_per_block][hd]
    const int head = blockIdx.y;
    const int kind = head < a.H ? 0 : head < a.H + a.G ? 1 : 2;
    const int hd = kind == 2 ? a.vdim : a.dim, hdp = kind == 2 ? a.vdimp : a.dimp;
    const int slot = kind == 0 ? head : kind == 1 ? head - a.H : head - a.H - a.G;
    const int C = (a.H + a.G) * a.dim + a.G * a.vdim;
    const int chan0 = kind == 0 ? slot * a.dim : kind == 1 ? (a.H + slot) * a.dim : (a.H + a.G) * a.dim + slot * a.vdim;
    const int r0 = blockIdx.x * a.rows_per_block;
    const int n = min(a.rows_per_block, a.rows - r0);
    const T* proj = reinterpret_cast<const T*>(a.proj);
    int lane = a.row_lane[a.decode ? r0 : 0];
    if (lane < 0 || lane >= a.lanes) {
        if (threadIdx.x == 0) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
        lane = min(max(lane, 0), a.lanes - 1);
    }
    T* state = reinterpret_cast<T*>(a.state) + (int64_t)lane * (a.taps - 1) * C + chan0;
    const bool active = !a.row_active || a.row_active[a.decode ? r0 : 0] != 0;

    // ---- convolution ------------------------------------------------------------------------------------
    const int vecs = hd / VEC;
    for (int i = threadIdx.x; i < n * vecs; i += QC_THREADS) {
        const int r = i / vecs, c = (i % vecs) * VEC;
        const int row = r0 + r, pos = a.row_pos[row];
        float y[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = 0.f;
        for (int j = 0; j < a.taps; ++j) {
            const int back = a.taps - 1 - j;
            if (back > pos) continue;  // before the sequence's start
            const int from = a.decode ? -back : row - back;  // row of this step, or negative: -m = the m-th last row of the state
            const T* src = (a.decode ? back == 0 : from >= 0) ? proj + (int64_t)(row - back) * a.proj_stride + chan0
                                                              : state + (int64_t)(a.taps - 1 + from) * C;
            const float* w = a.conv_w + (int64_t)j * C + chan0 + c;
            if constexpr (VEC == 8) {
                float u[8], wv[8];
                load8(src + c, u);
                load8(w, wv);
#pragma unroll
                for (int e = 0; e < 8; ++e) y[e] = fmaf(wv[e], u[e], y[e]);
            } else {
                y[0] = fmaf(w[0], to_f32(src[c]), y[0]);
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) y_s[r * hd + c + e] = y[e];
    }
    __syncthreads();

    // ---- the state moves on: its next rows are the last taps - 1 rows up to the end of this step ----------
    if (active && (a.decode || blockIdx.x == 0) && a.row_pos[a.decode ? r0 : 0] >= 0) {
        const int seq = a.decode ? 1 : a.rows, first = a.decode ? r0 : 0, keep = a.taps - 1;
        for (int c = threadIdx.x; c < hd; c += QC_THREADS)
            for (int j = 0; j < keep; ++j)  // ascending: entry j only reads later entries
                state[(int64_t)j * C + c] = seq + j < keep ? state[(int64_t)(j + seq) * C + c]
                                                           : proj[(int64_t)(first + seq - keep + j) * a.proj_stride + chan0 + c];
    }

    // ---- rotation / value mixing, stores ------------------------------------------------------------------
    const int half = a.rot_dims / 2, outs = hdp / 8;
    for (int i = threadIdx.x; i < n * outs; i += QC_THREADS) {
        const int r = i / outs, c = (i % outs) * 8;
        const int row = r0 + r;
        int pos = a.row_pos[row];
        const bool bad = pos < 0 || pos >= a.capacity;
        if (bad) {
            if (c == 0) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
            pos = min(max(pos, 0), a.capacity - 1);
        }
        const float* y = y_s + r * hd;
        float o[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            const int d = c + e;
            float v = d < hd ? y[d] : 0.f;
            if (kind < 2 && d < a.rot_dims) {
                const bool low = d < half;
                const float2 cs = a.rot[(int64_t)pos * half + (low ? d : d - half)];
                v = low ? v * cs.x - y[d + half] * cs.y : v * cs.x + y[d - half] * cs.y;
            }
            o[e] = v;
        }
        if (kind == 0) {
            store8(reinterpret_cast<T*>(a.q) + ((int64_t)row * a.H + slot) * hdp + c, o);
            continue;
        }
        const int64_t at = ((int64_t)row * a.G + slot) * hdp + c;
        if (kind == 2 && a.v_mode) {
            T* vf = reinterpret_cast<T*>(a.v_first) + at;
            if (a.v_mode == 1) {
                store8(vf, o);
            } else {
                float f[8];
                load8(vf, f);
#pragma unroll
                for (int e = 0; e < 8; ++e) o[e] = (1.f - a.mix) * o[e] + a.mix * f[e];
            }
        }
        T* fresh = reinterpret_cast<T*>(kind == 1 ? a.k_new : a.v_new);
        if (fresh) store8(fresh + at, o);
        if (active && !bad && row >= a.ring_from) {
            T* ring = reinterpret_cast<T*>(kind == 1 ? a.k_ring : a.v_ring);
            store8(ring + (((int64_t)lane * a.ring + pos % a.ring) * a.G + slot) * hdp + c, o);
        }
    }
}

// Rows [from, rows) of the linear key / value buffers of a step into the lane's ring.
template <typename T>
__global__ void __launch_bounds__(256)
ring_store_kernel(const T* __restrict__ k_new, const T* __restrict__ v_new, const int* __restrict__ row_pos, const int* __restrict__ row_lane,
                  T* __restrict__ k_ring, T* __restrict__ v_ring, int ring, int k_row, int v_row, int from, int rows, int lanes, int capacity) {
    GLMB_PDL_PROLOGUE();
    const int lane = row_lane[0];
    if (lane < 0 || lane >= lanes) return;
    const int vecs = (k_row + v_row) / 8;
    const int64_t total = (int64_t)(rows - from) * vecs;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int row = from + (int)(i / vecs), c = (int)(i % vecs) * 8;
        const int pos = row_pos[row];
        if (pos < 0 || pos >= capacity) continue;
        const int64_t slot = (int64_t)lane * ring + pos % ring;
        float v[8];
        if (c < k_row) {
            load8(k_new + (int64_t)row * k_row + c, v);
            store8(k_ring + slot * k_row + c, v);
        } else {
            load8(v_new + (int64_t)row * v_row + c - k_row, v);
            store8(v_ring + slot * v_row + c - k_row, v);
        }
    }
}

// ===================================================================================================
GLMB_API size_t glmb_qkv_conv_args_sizeof(void) { return sizeof(QkvConvArgs); }
// The most taps a configuration of this head size may have (a block must hold taps - 1 rows).
GLMB_API int glmb_qkv_conv_max_taps(int dim) { return min(QC_MAX_ROWS, QC_SMEM_FLOATS / (dim > 0 ? dim : 1)) + 1; }

GLMB_API int glmb_qkv_conv(const QkvConvArgs* args, int is_f32, void* stream) {
    QkvConvArgs a = *args;
    const int widest = a.dim > a.vdim ? a.dim : a.vdim;
    if (a.rows < 1 || a.H < 1 || a.G < 1 || a.H % a.G || a.dim < 1 || a.vdim < 1 || (a.dimp & 7) || (a.vdimp & 7) || a.dimp < a.dim || a.vdimp < a.vdim) return 1;
    if (a.taps < 1 || a.taps > glmb_qkv_conv_max_taps(widest) || a.rot_dims < 0 || (a.rot_dims & 1) || a.rot_dims > a.dim || a.ring < 1) return 1;
    if (a.decode && (a.k_new || a.v_new)) return 1;
    if (a.v_mode && !a.v_first) return 1;
    a.rows_per_block = a.decode ? 1 : min(QC_MAX_ROWS, QC_SMEM_FLOATS / widest);
    const dim3 grid(ceil_div(a.rows, a.rows_per_block), a.H + 2 * a.G);
    const size_t smem = (size_t)a.rows_per_block * widest * sizeof(float);
    const bool vec = !(a.dim & 7) && !(a.vdim & 7) && !(a.proj_stride & 7);
    cudaStream_t st = (cudaStream_t)stream;
    if (is_f32) {
        if (vec) GLMB_LAUNCH((qkv_conv_kernel<float, 8>), grid, QC_THREADS, smem, st, a);
        else GLMB_LAUNCH((qkv_conv_kernel<float, 1>), grid, QC_THREADS, smem, st, a);
    } else {
        if (vec) GLMB_LAUNCH((qkv_conv_kernel<bf16, 8>), grid, QC_THREADS, smem, st, a);
        else GLMB_LAUNCH((qkv_conv_kernel<bf16, 1>), grid, QC_THREADS, smem, st, a);
    }
    return (int)cudaGetLastError();
}

// k_row, v_row: elements of a key / value row (all heads, padded: multiples of 8).
GLMB_API int glmb_ring_store(const void* k_new, const void* v_new, const int* row_pos, const int* row_lane, void* k_ring, void* v_ring, int ring,
                             int k_row, int v_row, int from, int rows, int lanes, int capacity, int is_f32, void* stream) {
    if (rows < 1 || from < 0 || from >= rows || ring < 1 || (k_row & 7) || (v_row & 7) || rows - from > ring) return 1;
    const int64_t blocks = ((int64_t)(rows - from) * ((k_row + v_row) / 8) + 255) / 256;
    const int grid = blocks < 148 * 8 ? (int)blocks : 148 * 8;
    if (is_f32)
        GLMB_LAUNCH(ring_store_kernel<float>, grid, 256, 0, (cudaStream_t)stream, (const float*)k_new, (const float*)v_new, row_pos, row_lane,
                    (float*)k_ring, (float*)v_ring, ring, k_row, v_row, from, rows, lanes, capacity);
    else
        GLMB_LAUNCH(ring_store_kernel<bf16>, grid, 256, 0, (cudaStream_t)stream, (const bf16*)k_new, (const bf16*)v_new, row_pos, row_lane,
                    (bf16*)k_ring, (bf16*)v_ring, ring, k_row, v_row, from, rows, lanes, capacity);
    return (int)cudaGetLastError();
}
