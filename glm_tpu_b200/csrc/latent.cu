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
#include "latent_args.cuh"
#include "vec8.cuh"

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
    if (!(n & 7) && n == cols && n <= LR_THREADS * 16) {  // whole vectors, all of them asked for before the first is used
        float x[2][8];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int c = (threadIdx.x + i * LR_THREADS) * 8;
#pragma unroll
            for (int e = 0; e < 8; ++e) x[i][e] = 0.f;
            if (c < n) load8(src + c, x[i]);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(x[i][e], x[i][e], ss);
        const float denom = sqrtf(lr_block_sum(ss, scratch) / (float)n + a.eps);
        if (!ok) return;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int c = (threadIdx.x + i * LR_THREADS) * 8;
            if (c < n) {
                float y[8];
                load8(w + c, y);
#pragma unroll
                for (int e = 0; e < 8; ++e) y[e] *= x[i][e] / denom;
                store8(dst + c, y);
            }
        }
    } else {
        for (int c = threadIdx.x; c < n; c += LR_THREADS) { const float x = to_f32(src[c]); ss = fmaf(x, x, ss); }
        const float denom = sqrtf(lr_block_sum(ss, scratch) / (float)n + a.eps);
        if (!ok) return;
        for (int c = threadIdx.x; c < cols; c += LR_THREADS) from_f32(c < n ? to_f32(src[c]) / denom * w[c] : 0.f, dst[c]);
    }
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

// A thread per VEC pairs, grid (pieces of H rot / (2 VEC) threads, rows).
template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_query_kernel(LatentArgs a) {
    GLMB_PDL_PROLOGUE();
    const int half = a.rot_dim / 2, per = half / VEC, i = blockIdx.x * 256 + threadIdx.x, row = blockIdx.y;
    if (i >= a.H * per) return;
    bool ok;
    const int pos = latent_pos(a, row, ok), p = i % per * VEC;
    T* q = reinterpret_cast<T*>(a.q) + ((int64_t)row * a.H + i / per) * a.dimp + a.dim + p * 2;
    const float2* cs = a.rot + (int64_t)pos * half + p;
    if constexpr (VEC == 4) {
        float x[8];
        load8(q, x);
        const float4 t0 = *reinterpret_cast<const float4*>(cs), t1 = *reinterpret_cast<const float4*>(cs + 2);
        const float cosine[4] = {t0.x, t0.z, t1.x, t1.z}, sine[4] = {t0.y, t0.w, t1.y, t1.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float u = x[2 * e], v = x[2 * e + 1];
            x[2 * e] = u * cosine[e] - v * sine[e];
            x[2 * e + 1] = v * cosine[e] + u * sine[e];
        }
        store8(q, x);
    } else {
        const float u = to_f32(q[0]), v = to_f32(q[1]);
        from_f32(u * cs->x - v * cs->y, q[0]);
        from_f32(v * cs->x + u * cs->y, q[1]);
    }
}

// grid (pieces of 256 latent columns, H, blocks of LA_ROWS rows): a lane owns eight columns, the warps share the unrotated dimensions.
#define LA_WARPS 8
#define LA_THREADS (LA_WARPS * 32)
#define LA_ROWS 8
template <typename T, int R>
__global__ void __launch_bounds__(LA_THREADS) latent_absorb_kernel(LatentArgs a) {
    asm volatile("griddepcontrol.launch_dependents;");
    const int h = blockIdx.y, r0 = blockIdx.z * LA_ROWS, rows = min(R, a.rows - r0), W = a.lat + a.pe;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c = (blockIdx.x * 32 + lane) * 8;
    const T* w = reinterpret_cast<const T*>(a.uk) + (int64_t)h * a.dim * a.lat + c;
    float w0[8];  // the weights do not depend on the kernel before: the first ones are asked for while it finishes
    if (c < a.lat && warp < a.dim) load8(w + (int64_t)warp * a.lat, w0);
    asm volatile("griddepcontrol.wait;" ::: "memory");
    extern __shared__ __align__(16) float la_smem[];
    float* part = la_smem;                       // [LA_WARPS][R][256]
    float* q_f = la_smem + LA_WARPS * R * 256;   // [R][dim]
    const T* q = reinterpret_cast<const T*>(a.q) + ((int64_t)r0 * a.H + h) * a.dimp;
    T* qa = reinterpret_cast<T*>(a.qa) + ((int64_t)r0 * a.H + h) * W;
    for (int i = threadIdx.x; i < R * a.dim; i += LA_THREADS) q_f[i] = i / a.dim < rows ? to_f32(q[(int64_t)(i / a.dim) * a.H * a.dimp + i % a.dim]) : 0.f;
    __syncthreads();
    float acc[R][8];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[r][e] = 0.f;
    if (c < a.lat)
#pragma unroll 4
        for (int d = warp; d < a.dim; d += LA_WARPS) {
            float x[8];
            if (d == warp) {
#pragma unroll
                for (int e = 0; e < 8; ++e) x[e] = w0[e];
            } else {
                load8(w + (int64_t)d * a.lat, x);
            }
#pragma unroll
            for (int r = 0; r < R; ++r)
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[r][e] = fmaf(q_f[r * a.dim + d], x[e], acc[r][e]);
        }
#pragma unroll
    for (int r = 0; r < R; ++r) store8(part + ((warp * R + r) * 32 + lane) * 8, acc[r]);
    __syncthreads();
    for (int i = threadIdx.x; i < R * 256; i += LA_THREADS) {
        const int r = i / 256, col = blockIdx.x * 256 + i % 256;
        if (r >= rows || col >= a.lat) continue;
        float y = 0.f;
#pragma unroll
        for (int p = 0; p < LA_WARPS; ++p) y += part[p * R * 256 + i];
        from_f32(y, qa[(int64_t)r * a.H * W + col]);
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
    const int vec = (a.dim & 7) || (a.rot_dim & 7) ? 1 : 4;
    const dim3 grid(ceil_div(a.H * (a.rot_dim / 2 / vec), 256), a.rows);
    cudaStream_t st = (cudaStream_t)stream;
    if (is_f32) {
        if (vec == 4) GLMB_LAUNCH((latent_query_kernel<float, 4>), grid, 256, 0, st, a);
        else GLMB_LAUNCH((latent_query_kernel<float, 1>), grid, 256, 0, st, a);
    } else {
        if (vec == 4) GLMB_LAUNCH((latent_query_kernel<bf16, 4>), grid, 256, 0, st, a);
        else GLMB_LAUNCH((latent_query_kernel<bf16, 1>), grid, 256, 0, st, a);
    }
    return (int)cudaGetLastError();
}
template <typename T, int R>
static int launch_absorb(const LatentArgs& a, cudaStream_t st) {
    const size_t smem = (size_t)(R * a.dim + LA_WARPS * R * 256) * sizeof(float);
    static DeviceOnce once;
    const int dev = once.pending();
    if (dev != DeviceOnce::SET) {
        const cudaError_t e = cudaFuncSetAttribute(latent_absorb_kernel<T, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (R * 1024 + LA_WARPS * R * 256) * 4);
        if (e != cudaSuccess) return (int)e;
        once.mark(dev);
    }
    GLMB_LAUNCH((latent_absorb_kernel<T, R>), dim3(ceil_div(a.lat, 256), a.H, ceil_div(a.rows, LA_ROWS)), LA_THREADS, smem, st, a);
    return (int)cudaGetLastError();
}
GLMB_API int glmb_latent_absorb(const LatentArgs* args, int is_f32, void* stream) {
    const LatentArgs a = *args;
    if (!latent_ok(a) || a.dim > 1024 || (a.lat & 15) || (a.pe & 15)) return 1;
    cudaStream_t st = (cudaStream_t)stream;
    if (is_f32) return launch_absorb<float, 8>(a, st);
    if (a.rows == 1) return launch_absorb<bf16, 1>(a, st);
    return a.rows <= 4 ? launch_absorb<bf16, 4>(a, st) : launch_absorb<bf16, 8>(a, st);
}
GLMB_API int glmb_latent_value(const LatentArgs* args, int is_f32, void* stream) {
    const LatentArgs a = *args;
    if (!latent_ok(a)) return 1;
    LATENT_LAUNCH(latent_value_kernel, dim3(ceil_div(a.vdim, LV_COLS), a.H, ceil_div(a.rows, LA_ROWS)), LV_WARPS * 32, 0);
}
