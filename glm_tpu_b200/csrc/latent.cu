// Attention over a shared latent: what happens around the products with keys and values.
//
//   latent_rows     projection row -> normalized query latent; normalized key/value latent and rotated key part into the lane's cache
//   latent_query    rotates the rotated part of every query head in place (keys and values are expanded per head: long prefill steps)
//   latent_absorb   query heads through the transposed key projection: [q_unrotated W_uk | rotated part], to be compared with cache rows as
//                   they are (decode, short steps); every row reads the weights of a head once per eight rows
//   latent_value    per-head value projection of the attended latent, and the head's output gate
//
// A cache row is [latent | rotated key part], both padded to a multiple of 16 columns (zeros).  Pairs (2i, 2i + 1) of the rotated part turn by
// the (cos, sin) of a fp32 table.  Templates over the element type: bf16 for serving, fp32 for the 32-bit path.
#include "common.cuh"
#include "vec8.cuh"

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
    int rows, H, dim, rot_dim, dimp, vdim, q_rank, kv_rank, lat, pe, lanes, capacity;
    float eps;
    uint32_t* status;
};

__device__ __forceinline__ int latent_pos(const LatentArgs& a, int row, bool& ok) {
    const int pos = a.row_pos[row];
    ok = pos >= 0 && pos < a.capacity;
    if (!ok && threadIdx.x == 0) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
    return min(max(pos, 0), a.capacity - 1);
}

#define LR_THREADS 128
__device__ __forceinline__ float lr_block_sum(float v, float* scratch) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < LR_THREADS / 32; ++w) t += scratch[w];
    return t;
}

// grid (rows, 2): y = 0 the query latent, y = 1 the key/value latent and the key part.
template <typename T>
__global__ void __launch_bounds__(LR_THREADS) latent_rows_kernel(LatentArgs a) {
    GLMB_PDL_PROLOGUE();
    __shared__ float scratch[LR_THREADS / 32];
    const int row = blockIdx.x;
    const bool is_q = blockIdx.y == 0;
    const int n = is_q ? a.q_rank : a.kv_rank, cols = is_q ? (int)a.cq_stride : a.lat;
    const T* src = reinterpret_cast<const T*>(a.proj) + (int64_t)row * a.proj_stride + (is_q ? 0 : a.off_kv);
    const float* w = is_q ? a.q_norm : a.kv_norm;
    bool ok = true;
    T* dst = reinterpret_cast<T*>(a.cq) + (int64_t)row * a.cq_stride;
    int pos = 0;
    if (!is_q) {
        pos = latent_pos(a, row, ok);
        int lane = a.row_lane[row];
        if (lane < 0 || lane >= a.lanes) {
            if (threadIdx.x == 0) raise_status(a.status, GLMB_STATUS_BAD_INDEX);
            ok = false;
            lane = 0;
        }
        if (a.row_active && !a.row_active[row]) ok = false;
        dst = reinterpret_cast<T*>(a.cache) + ((int64_t)lane * a.capacity + pos) * (a.lat + a.pe);
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < n; c += LR_THREADS) { const float x = to_f32(src[c]); ss = fmaf(x, x, ss); }
    const float denom = sqrtf(lr_block_sum(ss, scratch) / (float)n + a.eps);
    if (!ok) return;
    for (int c = threadIdx.x; c < cols; c += LR_THREADS) from_f32(c < n ? to_f32(src[c]) / denom * w[c] : 0.f, dst[c]);
    if (is_q) return;
    const T* pe = src + a.kv_rank;
    const int half = a.rot_dim / 2;
    for (int i = threadIdx.x; i < a.pe / 2; i += LR_THREADS) {
        float x = 0.f, y = 0.f;
        if (i < half) {
            const float2 cs = a.rot[(int64_t)pos * half + i];
            const float u = to_f32(pe[2 * i]), v = to_f32(pe[2 * i + 1]);
            x = u * cs.x - v * cs.y;
            y = v * cs.x + u * cs.y;
        }
        from_f32(x, dst[a.lat + 2 * i]);
        from_f32(y, dst[a.lat + 2 * i + 1]);
    }
}

// A thread per pair, grid (pieces of H rot / 2 pairs, rows).
template <typename T>
__global__ void __launch_bounds__(256) latent_query_kernel(LatentArgs a) {
    GLMB_PDL_PROLOGUE();
    const int half = a.rot_dim / 2, i = blockIdx.x * 256 + threadIdx.x, row = blockIdx.y;
    if (i >= a.H * half) return;
    bool ok;
    const int pos = latent_pos(a, row, ok);
    T* q = reinterpret_cast<T*>(a.q) + ((int64_t)row * a.H + i / half) * a.dimp + a.dim + i % half * 2;
    const float2 cs = a.rot[(int64_t)pos * half + i % half];
    const float u = to_f32(q[0]), v = to_f32(q[1]);
    from_f32(u * cs.x - v * cs.y, q[0]);
    from_f32(v * cs.x + u * cs.y, q[1]);
}

// grid (pieces of 8 * LA_THREADS latent columns, H, blocks of R rows): a thread owns one column.
#define LA_THREADS 64
#define LA_ROWS 8
template <typename T>
__global__ void __launch_bounds__(LA_THREADS) latent_absorb_kernel(LatentArgs a) {
    GLMB_PDL_PROLOGUE();
    extern __shared__ float q_f[];  // [LA_ROWS][dim]
    const int h = blockIdx.y, r0 = blockIdx.z * LA_ROWS, rows = min(LA_ROWS, a.rows - r0), W = a.lat + a.pe;
    const T* q = reinterpret_cast<const T*>(a.q) + ((int64_t)r0 * a.H + h) * a.dimp;
    T* qa = reinterpret_cast<T*>(a.qa) + ((int64_t)r0 * a.H + h) * W;
    for (int i = threadIdx.x; i < LA_ROWS * a.dim; i += LA_THREADS) {
        const int r = i / a.dim;
        q_f[i] = r < rows ? to_f32(q[(int64_t)r * a.H * a.dimp + i % a.dim]) : 0.f;
    }
    __syncthreads();
    const int c = (blockIdx.x * LA_THREADS + threadIdx.x) * 2;
    if (c < a.lat) {
        const T* w = reinterpret_cast<const T*>(a.uk) + (int64_t)h * a.dim * a.lat + c;
        float acc[LA_ROWS][2] = {};
#pragma unroll 8
        for (int d = 0; d < a.dim; ++d) {
            const float x = to_f32(w[(int64_t)d * a.lat]), y = to_f32(w[(int64_t)d * a.lat + 1]);
#pragma unroll
            for (int r = 0; r < LA_ROWS; ++r) {
                acc[r][0] = fmaf(q_f[r * a.dim + d], x, acc[r][0]);
                acc[r][1] = fmaf(q_f[r * a.dim + d], y, acc[r][1]);
            }
        }
#pragma unroll
        for (int r = 0; r < LA_ROWS; ++r)
            if (r < rows) {
                from_f32(acc[r][0], qa[(int64_t)r * a.H * W + c]);
                from_f32(acc[r][1], qa[(int64_t)r * a.H * W + c + 1]);
            }
    }
    if (blockIdx.x) return;
    const int half = a.rot_dim / 2;
    for (int i = threadIdx.x; i < rows * (a.pe / 2); i += LA_THREADS) {
        const int r = i / (a.pe / 2), p = i % (a.pe / 2);
        float x = 0.f, y = 0.f;
        if (p < half) {
            bool ok;
            const int pos = latent_pos(a, r0 + r, ok);
            const float2 cs = a.rot[(int64_t)pos * half + p];
            const T* src = q + (int64_t)r * a.H * a.dimp + a.dim + 2 * p;
            const float u = to_f32(src[0]), v = to_f32(src[1]);
            x = u * cs.x - v * cs.y;
            y = v * cs.x + u * cs.y;
        }
        T* dst = qa + (int64_t)r * a.H * W + a.lat + 2 * p;
        from_f32(x, dst[0]);
        from_f32(y, dst[1]);
    }
}

// grid (pieces of LV_COLS value channels, H, blocks of LA_ROWS rows); a warp per value channel at a time.
#define LV_WARPS 8
#define LV_COLS 16
template <typename T>
__global__ void __launch_bounds__(LV_WARPS * 32) latent_value_kernel(LatentArgs a) {
    GLMB_PDL_PROLOGUE();
    const int h = blockIdx.y, r0 = blockIdx.z * LA_ROWS, rows = min(LA_ROWS, a.rows - r0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const T* o = reinterpret_cast<const T*>(a.o_lat) + ((int64_t)r0 * a.H + h) * a.kv_rank;
    for (int c = blockIdx.x * LV_COLS + warp; c < min((blockIdx.x + 1) * LV_COLS, a.vdim); c += LV_WARPS) {
        const T* w = reinterpret_cast<const T*>(a.uv) + ((int64_t)h * a.vdim + c) * a.lat;
        float acc[LA_ROWS] = {};
        for (int l = lane; l < a.kv_rank; l += 32) {
            const float x = to_f32(w[l]);
#pragma unroll
            for (int r = 0; r < LA_ROWS; ++r)
                if (r < rows) acc[r] = fmaf(x, to_f32(o[(int64_t)r * a.H * a.kv_rank + l]), acc[r]);
        }
#pragma unroll
        for (int r = 0; r < LA_ROWS; ++r) {
            const float y = warp_sum(acc[r]);
            if (lane == 0 && r < rows) {
                const float z = to_f32(reinterpret_cast<const T*>(a.proj)[(int64_t)(r0 + r) * a.proj_stride + a.off_gate + h]);
                from_f32(y * sigmoidf_precise(z), reinterpret_cast<T*>(a.out)[(int64_t)(r0 + r) * a.out_stride + h * a.vdim + c]);
            }
        }
    }
}

// ===================================================================================================
static bool latent_ok(const LatentArgs& a) {
    return a.rows >= 1 && a.rows <= 65535 && a.H >= 1 && a.H <= 65535 && a.dim >= 1 && a.rot_dim >= 2 && !(a.rot_dim & 1) && a.dimp >= a.dim + a.rot_dim && a.vdim >= 1 && a.q_rank >= 1 &&
           a.kv_rank >= 1 && a.lat >= a.kv_rank && a.pe >= a.rot_dim && !(a.lat & 1) && !(a.pe & 1) && a.lanes >= 1 && a.capacity >= 1 && a.row_pos && a.row_lane;
}
#define LATENT_LAUNCH(kernel, grid, threads, smem)                                                         \
    do {                                                                                                   \
        if (is_f32) GLMB_LAUNCH(kernel<float>, grid, threads, smem, (cudaStream_t)stream, a);              \
        else GLMB_LAUNCH(kernel<bf16>, grid, threads, smem, (cudaStream_t)stream, a);                      \
        return (int)cudaGetLastError();                                                                    \
    } while (0)

GLMB_API size_t glmb_latent_args_sizeof(void) { return sizeof(LatentArgs); }

GLMB_API int glmb_latent_rows(const LatentArgs* args, int is_f32, void* stream) {
    const LatentArgs a = *args;
    if (!latent_ok(a) || a.cq_stride < a.q_rank) return 1;
    LATENT_LAUNCH(latent_rows_kernel, dim3(a.rows, 2), LR_THREADS, 0);
}
GLMB_API int glmb_latent_query(const LatentArgs* args, int is_f32, void* stream) {
    const LatentArgs a = *args;
    if (!latent_ok(a)) return 1;
    LATENT_LAUNCH(latent_query_kernel, dim3(ceil_div(a.H * (a.rot_dim / 2), 256), a.rows), 256, 0);
}
GLMB_API int glmb_latent_absorb(const LatentArgs* args, int is_f32, void* stream) {
    const LatentArgs a = *args;
    if (!latent_ok(a) || a.dim > 1024) return 1;
    LATENT_LAUNCH(latent_absorb_kernel, dim3(ceil_div(a.lat, 2 * LA_THREADS), a.H, ceil_div(a.rows, LA_ROWS)), LA_THREADS, LA_ROWS * a.dim * sizeof(float));
}
GLMB_API int glmb_latent_value(const LatentArgs* args, int is_f32, void* stream) {
    const LatentArgs a = *args;
    if (!latent_ok(a)) return 1;
    LATENT_LAUNCH(latent_value_kernel, dim3(ceil_div(a.vdim, LV_COLS), a.H, ceil_div(a.rows, LA_ROWS)), LV_WARPS * 32, 0);
}
