// From the fused q | k | v projection of an attention layer to what the attention reads: a short causal convolution over time on every
// channel, rotary positions on q and k, mixing of the values with an earlier layer's values, and the cache write -- one launch.
//
//   y_t[c]  = sum_j w[c][j] * u_{t - taps + 1 + j}[c]      u: projected rows, zero before the sequence; the last taps - 1 of a sequence
//                                                         live in its lane's state between steps
//   (a, b) -> (a cos - b sin, b cos + a sin)               dimensions i and i + dims/2 of every q and k head, fp32 table
//   v       = (1 - lambda) v + lambda v_first
//
// A block owns one head (of q, k or v) and some consecutive rows.  Prefill: the rows are one sequence; the rows' own history comes from
// the projection, that of the first rows from the state, and the block of the first rows also advances the state once it has read it (no
// other block reads it: a block holds at least taps - 1 rows).  Decode: every row is its own sequence (lane), one row per block.
//
//   qkv_conv_kernel       any sizes, decode and prefill: convolution into shared memory, then rotation / mixing / stores
//   qkv_conv_rows_kernel  prefill, head sizes in multiples of 8, up to 4 taps: a thread takes a strip of rows with two 8-channel
//                         vectors (for rotated dimensions the two halves of a pair), its taps, rows and history in registers
//
// Keys and values go to the lane's ring (slot = position mod ring size: with chunked attention a ring of one chunk holds everything a later
// token can see) or, when `k_lin` is set, to linear buffers, row by row.
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
    void* q;                                     // [rows, H, dimp]
    void *k_lin, *v_lin;                         // [rows, G, dimp], [rows, G, vdimp], or NULL: keys and values go to the ring
    void *k_ring, *v_ring; int ring;             // [lanes, ring, G, dimp], [lanes, ring, G, vdimp]
    void* v_first; int v_mode; float mix;        // [rows, G * vdim]; 0: not used, 1: store this layer's values, 2: mix with them
    int H, G, dim, dimp, vdim, vdimp, rows, decode, capacity, lanes, rows_per_block;
    uint32_t* status;
};

struct QcHead { int kind, slot, hd, hdp, chan0, C; };  // kind 0: q, 1: k, 2: v

__device__ __forceinline__ QcHead qc_head(const QkvConvArgs& a, int head) {
    QcHead h;
    h.kind = head < a.H ? 0 : head < a.H + a.G ? 1 : 2;
    h.hd = h.kind == 2 ? a.vdim : a.dim;
    h.hdp = h.kind == 2 ? a.vdimp : a.dimp;
    h.slot = h.kind == 0 ? head : h.kind == 1 ? head - a.H : head - a.H - a.G;
    h.C = (a.H + a.G) * a.dim + a.G * a.vdim;
    h.chan0 = h.kind == 0 ? h.slot * a.dim : h.kind == 1 ? (a.H + h.slot) * a.dim : (a.H + a.G) * a.dim + h.slot * a.vdim;
    return h;
}

__device__ __forceinline__ int qc_lane(const QkvConvArgs& a, int row) {
    const int lane = a.row_lane[row];
    if (lane >= 0 && lane < a.lanes) return lane;
    if (threadIdx.x == 0) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
    return min(max(lane, 0), a.lanes - 1);
}

// The state's next rows are the last taps - 1 rows up to the end of the step that starts at row `first` and has `seq` rows.
template <typename T>
__device__ __forceinline__ void qc_advance_state(const QkvConvArgs& a, const QcHead& h, T* state, int first, int seq) {
    const T* proj = reinterpret_cast<const T*>(a.proj);
    const int keep = a.taps - 1;
    for (int c = threadIdx.x; c < h.hd; c += QC_THREADS)
        for (int j = 0; j < keep; ++j)  // ascending: entry j only reads later entries
            state[(int64_t)j * h.C + c] = seq + j < keep ? state[(int64_t)(j + seq) * h.C + c]
                                                         : proj[(int64_t)(first + seq - keep + j) * a.proj_stride + h.chan0 + c];
}

// Eight finished channels of one row to where they belong; values are mixed on the way.
template <typename T>
__device__ __forceinline__ void qc_store(const QkvConvArgs& a, const QcHead& h, int row, int pos, int lane, bool keep, int c, float (&o)[8]) {
    if (h.kind == 0) {
        store8(reinterpret_cast<T*>(a.q) + ((int64_t)row * a.H + h.slot) * h.hdp + c, o);
        return;
    }
    const int64_t at = ((int64_t)row * a.G + h.slot) * h.hdp + c;
    if (h.kind == 2 && a.v_mode) {  // by channel, whatever the heads: layers may cut the same channels into other heads
        T* vf = reinterpret_cast<T*>(a.v_first) + ((int64_t)row * a.G + h.slot) * h.hd + c;
        float f[8];
        if (!(h.hd & 7)) {
            if (c < h.hd) {
                if (a.v_mode == 1) store8(vf, o);
                else load8(vf, f);
            }
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e)
                if (c + e < h.hd) {
                    if (a.v_mode == 1) from_f32(o[e], vf[e]);
                    else f[e] = to_f32(vf[e]);
                }
        }
        if (a.v_mode == 2) {
#pragma unroll
            for (int e = 0; e < 8; ++e)
                if (c + e < h.hd) o[e] = (1.f - a.mix) * o[e] + a.mix * f[e];
        }
    }
    T* lin = reinterpret_cast<T*>(h.kind == 1 ? a.k_lin : a.v_lin);
    if (lin) store8(lin + at, o);
    else if (keep) store8(reinterpret_cast<T*>(h.kind == 1 ? a.k_ring : a.v_ring) + (((int64_t)lane * a.ring + pos % a.ring) * a.G + h.slot) * h.hdp + c, o);
}

template <typename T, int VEC>
__global__ void __launch_bounds__(QC_THREADS) qkv_conv_kernel(QkvConvArgs a) {
    GLMB_PDL_PROLOGUE();
    extern __shared__ float y_s[];  // [rows_per_block][hd]
    const QcHead h = qc_head(a, blockIdx.y);
    const int hd = h.hd, C = h.C, chan0 = h.chan0;
    const int r0 = blockIdx.x * a.rows_per_block;
    const int n = min(a.rows_per_block, a.rows - r0);
    const T* proj = reinterpret_cast<const T*>(a.proj);
    const int lane = qc_lane(a, a.decode ? r0 : 0);
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

    if (active && (a.decode || blockIdx.x == 0) && a.row_pos[a.decode ? r0 : 0] >= 0) qc_advance_state(a, h, state, a.decode ? r0 : 0, a.decode ? 1 : a.rows);

    // ---- rotation / value mixing, stores ------------------------------------------------------------------
    const int half = a.rot_dims / 2, outs = h.hdp / 8;
    for (int i = threadIdx.x; i < n * outs; i += QC_THREADS) {
        const int r = i / outs, c = (i % outs) * 8;
        const int row = r0 + r;
        int pos = a.row_pos[row];
        const bool bad = pos < 0 || pos >= a.capacity;
        if (bad) {
            if (c == 0 && active) raise_status(a.status, GLMB_STATUS_BAD_INDEX);  // a frozen lane may be full
            pos = min(max(pos, 0), a.capacity - 1);
        }
        const float* y = y_s + r * hd;
        float o[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            const int d = c + e;
            float v = d < hd ? y[d] : 0.f;
            if (h.kind < 2 && d < a.rot_dims) {
                const bool low = d < half;
                const float2 cs = a.rot[(int64_t)pos * half + (low ? d : d - half)];
                v = low ? v * cs.x - y[d + half] * cs.y : v * cs.x + y[d - half] * cs.y;
            }
            o[e] = v;
        }
        qc_store<T>(a, h, row, pos, lane, active && !bad, c, o);
    }
}

// ---------------------------------------------------------------------------------------------------
#define QR_TAPS 4
#define QR_STRIP 4  // consecutive rows of a thread

// Eight elements as they come from memory.
template <typename T> struct Raw8;
template <> struct Raw8<bf16> {
    uint4 v;
    __device__ __forceinline__ void clear() { v = make_uint4(0, 0, 0, 0); }
    __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void get(float (&x)[8]) const {
        x[0] = bf16_lo(v.x); x[1] = bf16_hi(v.x); x[2] = bf16_lo(v.y); x[3] = bf16_hi(v.y);
        x[4] = bf16_lo(v.z); x[5] = bf16_hi(v.z); x[6] = bf16_lo(v.w); x[7] = bf16_hi(v.w);
    }
};
template <> struct Raw8<float> {
    float v[8];
    __device__ __forceinline__ void clear() {
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = 0.f;
    }
    __device__ __forceinline__ void load(const float* p) { load8(p, v); }
    __device__ __forceinline__ void get(float (&x)[8]) const {
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = v[e];
    }
};

template <typename T>
__global__ void __launch_bounds__(QC_THREADS) qkv_conv_rows_kernel(QkvConvArgs a) {
    GLMB_PDL_PROLOGUE();
    const QcHead h = qc_head(a, blockIdx.y);
    const T* proj = reinterpret_cast<const T*>(a.proj) + h.chan0;
    const int lane = qc_lane(a, 0), start = a.row_pos[0], keep = a.taps - 1;
    T* state = reinterpret_cast<T*>(a.state) + (int64_t)lane * keep * h.C + h.chan0;
    // pairs of channel vectors: the rotated halves of q and k first, then the rest two by two
    const int vecs = h.hd / 8, half = h.kind < 2 ? a.rot_dims / 2 : 0, rot_pairs = half / 8, plain = vecs - 2 * rot_pairs;
    const int pairs = rot_pairs + (plain + 1) / 2, strips = QC_THREADS / pairs;
    const int pair = threadIdx.x % pairs, strip = threadIdx.x / pairs;
    const bool rotated = pair < rot_pairs;
    const int c0 = rotated ? pair * 8 : half * 2 + (pair - rot_pairs) * 16, c1 = rotated ? c0 + half : c0 + 8;
    const bool both = c1 < h.hd;
    const int block_rows = strips * QR_STRIP, first = blockIdx.x * block_rows + strip * QR_STRIP, last = min(first + QR_STRIP, a.rows);
    if (strip < strips && first < a.rows) {
        // every row of the strip and its history is asked for at once: one memory round trip per strip
        Raw8<T> u0[QR_STRIP + QR_TAPS - 1], u1[QR_STRIP + QR_TAPS - 1];
#pragma unroll
        for (int i = 0; i < QR_STRIP + QR_TAPS - 1; ++i) {
            const int row = first + i - (QR_TAPS - 1);
            const T* src = nullptr;
            if (row >= 0 && row < last) src = proj + (int64_t)row * a.proj_stride;
            else if (row < 0 && row >= -keep && start + row >= 0) src = state + (int64_t)(keep + row) * h.C;
            u0[i].clear();
            u1[i].clear();
            if (src) {
                u0[i].load(src + c0);
                if (both) u1[i].load(src + c1);
            }
        }
        float w0[QR_TAPS][8], w1[QR_TAPS][8];
#pragma unroll
        for (int j = 0; j < QR_TAPS; ++j) {
            const int tap = j - (QR_TAPS - a.taps);  // fewer taps: the oldest ones are zero
#pragma unroll
            for (int e = 0; e < 8; ++e) w0[j][e] = w1[j][e] = 0.f;
            if (tap >= 0) {
                load8(a.conv_w + (int64_t)tap * h.C + h.chan0 + c0, w0[j]);
                if (both) load8(a.conv_w + (int64_t)tap * h.C + h.chan0 + c1, w1[j]);
            }
        }
        const bool bad_start = start < 0 || start + a.rows > a.capacity;
        if (bad_start) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
#pragma unroll
        for (int i = 0; i < QR_STRIP; ++i) {
            const int row = first + i;
            if (row >= last) break;
            float y0[8], y1[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) y0[e] = y1[e] = 0.f;
#pragma unroll
            for (int j = 0; j < QR_TAPS; ++j) {
                float x[8];
                u0[i + j].get(x);
#pragma unroll
                for (int e = 0; e < 8; ++e) y0[e] = fmaf(w0[j][e], x[e], y0[e]);
                u1[i + j].get(x);
#pragma unroll
                for (int e = 0; e < 8; ++e) y1[e] = fmaf(w1[j][e], x[e], y1[e]);
            }
            const int pos = min(max(start + row, 0), a.capacity - 1);
            if (rotated) {
                const float4* table = reinterpret_cast<const float4*>(a.rot + (int64_t)pos * half + c0);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float4 cs = __ldg(table + e);
                    const float p = y0[2 * e], q = y1[2 * e], r = y0[2 * e + 1], s = y1[2 * e + 1];
                    y0[2 * e] = p * cs.x - q * cs.y;
                    y1[2 * e] = q * cs.x + p * cs.y;
                    y0[2 * e + 1] = r * cs.z - s * cs.w;
                    y1[2 * e + 1] = s * cs.z + r * cs.w;
                }
            }
            qc_store<T>(a, h, row, pos, lane, !bad_start, c0, y0);
            if (both) qc_store<T>(a, h, row, pos, lane, !bad_start, c1, y1);
            if (pair == 0 && h.hdp > h.hd) {  // the padding of the head row
                float zero[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) zero[e] = 0.f;
                for (int c = h.hd; c < h.hdp; c += 8) qc_store<T>(a, h, row, pos, lane, !bad_start, c, zero);
            }
        }
    }
    if (blockIdx.x == 0) {
        __syncthreads();  // the first rows have read the state
        if (start >= 0) qc_advance_state(a, h, state, 0, a.rows);
    }
}

// ---------------------------------------------------------------------------------------------------
// Two contiguous runs of cache rows from one place to another (a ring's current chunk to a linear buffer or back): 16-byte pieces.
__global__ void __launch_bounds__(256)
kv_copy_kernel(const uint4* __restrict__ k_src, uint4* __restrict__ k_dst, int64_t k_pieces, const uint4* __restrict__ v_src, uint4* __restrict__ v_dst,
               int64_t v_pieces) {
    GLMB_PDL_PROLOGUE();
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < k_pieces + v_pieces; i += (int64_t)gridDim.x * blockDim.x) {
        if (i < k_pieces) k_dst[i] = k_src[i];
        else v_dst[i - k_pieces] = v_src[i - k_pieces];
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
    if ((a.dimp & 15) || (a.vdimp & 15) || !a.k_lin != !a.v_lin || (a.decode && a.k_lin)) return 1;
    if (a.v_mode && !a.v_first) return 1;
    const bool vec = !(a.dim & 7) && !(a.vdim & 7) && !(a.proj_stride & 7);
    cudaStream_t st = (cudaStream_t)stream;
    const int pairs = a.rot_dims / 16 + ((widest / 8 - a.rot_dims / 8) + 1) / 2;
    if (vec && !a.decode && a.taps <= QR_TAPS && !(a.rot_dims & 15) && widest <= 1024 && pairs <= QC_THREADS) {
        // strips per block differ between head kinds (their pair counts do): the grid covers the kind with the shortest block
        auto blocks_of = [&](int hd, int rot) {
            const int p = rot / 16 + ((hd / 8 - rot / 8) + 1) / 2;
            return ceil_div(a.rows, QC_THREADS / p * QR_STRIP);
        };
        const int bq = blocks_of(a.dim, a.rot_dims), bv = blocks_of(a.vdim, 0);
        const dim3 grid(bq > bv ? bq : bv, a.H + 2 * a.G);
        if (is_f32) GLMB_LAUNCH(qkv_conv_rows_kernel<float>, grid, QC_THREADS, 0, st, a);
        else GLMB_LAUNCH(qkv_conv_rows_kernel<bf16>, grid, QC_THREADS, 0, st, a);
        return (int)cudaGetLastError();
    }
    a.rows_per_block = a.decode ? 1 : min(QC_MAX_ROWS, QC_SMEM_FLOATS / widest);
    const dim3 grid(ceil_div(a.rows, a.rows_per_block), a.H + 2 * a.G);
    const size_t smem = (size_t)a.rows_per_block * widest * sizeof(float);
    if (is_f32) {
        if (vec) GLMB_LAUNCH((qkv_conv_kernel<float, 8>), grid, QC_THREADS, smem, st, a);
        else GLMB_LAUNCH((qkv_conv_kernel<float, 1>), grid, QC_THREADS, smem, st, a);
    } else {
        if (vec) GLMB_LAUNCH((qkv_conv_kernel<bf16, 8>), grid, QC_THREADS, smem, st, a);
        else GLMB_LAUNCH((qkv_conv_kernel<bf16, 1>), grid, QC_THREADS, smem, st, a);
    }
    return (int)cudaGetLastError();
}

GLMB_API int glmb_kv_copy(const void* k_src, void* k_dst, int64_t k_bytes, const void* v_src, void* v_dst, int64_t v_bytes, void* stream) {
    if (k_bytes < 16 || v_bytes < 16 || (k_bytes & 15) || (v_bytes & 15)) return 1;
    const int64_t pieces = (k_bytes + v_bytes) / 16, blocks = (pieces + 255) / 256;
    GLMB_LAUNCH(kv_copy_kernel, (unsigned)(blocks < 148 * 8 ? blocks : 148 * 8), 256, 0, (cudaStream_t)stream, (const uint4*)k_src, (uint4*)k_dst, k_bytes / 16,
                (const uint4*)v_src, (uint4*)v_dst, v_bytes / 16);
    return (int)cudaGetLastError();
}
