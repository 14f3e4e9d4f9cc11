// One token of the gated delta rule per sequence (decode, bf16): everything between the layer's two projections in one launch.
//
// A cluster owns a (row, head) and shares its value channels; every CTA convolves the head's queries and keys (a few hundred multiplications),
// the second halves of the low-rank projections are dealt out: a CTA makes the decays of its share of the key channels and writes them into
// every CTA of the cluster, and the gates of its own value channels.  The state's rows are asked for first and updated in registers, the sum of
// squares for the head's norm goes through the cluster, and the gated output is written once.
//
//   warp layout of the recurrence: four value channels per warp, eight lanes share a value channel's key channels (DQ float4 each)
#include <cooperative_groups.h>

#include "common.cuh"
#include "delta_rule.cuh"
#include "vec8.cuh"

namespace cg = cooperative_groups;

#define DT_THREADS 256
#define DT_WARPS 8
#define DT_CLUSTER 4
#define DT_PASS 32      // value channels a CTA updates at a time
#define DT_VALUES 256   // value channels of a CTA

// out[i] = w[i] . x for `rows` weight rows (bf16, `ld` apart, K a multiple of 8) and x in shared memory: eight lanes per row.
template <typename F>
__device__ __forceinline__ void dt_rows(const bf16* w, int64_t ld, int rows, int K, const float* x, int warp, int lane, F done) {
    const int sub = lane & 7;
    for (int base = warp * 4; base < rows; base += DT_WARPS * 4) {
        const int r = base + (lane >> 3);
        float sum = 0.f;
        if (r < rows)
            for (int k = sub * 8; k < K; k += 64) {
                float v[8];
                load8(w + (int64_t)r * ld + k, v);
#pragma unroll
                for (int e = 0; e < 8; ++e) sum = fmaf(v[e], x[k + e], sum);
            }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        sum += __shfl_xor_sync(0xffffffffu, sum, 4);
        if (sub == 0 && r < rows) done(r, sum);
    }
}

__device__ __forceinline__ void dt_prefetch(const void* p, int64_t bytes) {
    const uint32_t n = (uint32_t)(bytes & ~(int64_t)15);
    if (n) asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(p), "r"(n) : "memory");
}

// grid (CTAs of a cluster, H, rows)
template <int DQ>
__global__ void __launch_bounds__(DT_THREADS, DQ <= 4 ? 4 : 2) delta_step_kernel(DeltaArgs a) {
    constexpr int DP = DQ * 32;
    asm volatile("griddepcontrol.launch_dependents;");
    cg::cluster_group cluster = cg::this_cluster();
    extern __shared__ __align__(16) float low_s[];  // the two low-rank halves of this row
    __shared__ __align__(16) float q_s[DP], k_s[DP], g_s[DP];
    __shared__ float v_s[DT_VALUES], z_s[DT_VALUES], o_s[DT_VALUES], ss_s[DT_CLUSTER], red_s[DT_WARPS];
    const int size = gridDim.x, rank = blockIdx.x, h = blockIdx.y, row = blockIdx.z, kvh = h / (a.H / a.G);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int vb = ((a.vdim + size - 1) / size + 3) & ~3, c0 = min(rank * vb, a.vdim), cols = min(vb, a.vdim - c0);
    const int db = (a.dim + size - 1) / size, d0 = min(rank * db, a.dim), dims = min(db, a.dim - d0);
    const bf16* a2 = reinterpret_cast<const bf16*>(a.a2) + ((int64_t)h * a.dim + d0) * a.ra;
    const bf16* g2 = reinterpret_cast<const bf16*>(a.g2) + ((int64_t)h * a.vdim + c0) * a.rg;
    if (threadIdx.x == 0) {  // weights do not depend on the kernel before
        dt_prefetch(a2, (int64_t)dims * a.ra * 2);
        dt_prefetch(g2, (int64_t)cols * a.rg * 2);
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int seq = delta_lane(a, row), pos = a.row_pos[row];
    const bool writes = delta_writes(a, row);
    float* state = a.state + (((int64_t)seq * a.H + h) * a.vdim + c0) * DP;
    const int kg = lane >> 2;
    float4 s[DQ];
    auto fetch = [&](int base) {
        const int c = base + warp * 4 + (lane & 3);
#pragma unroll
        for (int i = 0; i < DQ; ++i)
            s[i] = pos > 0 && c < cols ? *reinterpret_cast<const float4*>(state + (int64_t)c * DP + 32 * i + kg * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    fetch(0);
    const bf16* proj = reinterpret_cast<const bf16*>(a.proj) + (int64_t)row * a.proj_stride;
    for (int i = threadIdx.x; i < a.ra + a.rg; i += DT_THREADS) low_s[i] = __bfloat162float(i < a.ra ? proj[a.off_a + i] : proj[a.off_g + i - a.ra]);
    // ---- convolution of the head's queries and keys and this CTA's values -----------------------------------
    const int C = 2 * a.G * a.dim + a.H * a.vdim;
    bf16* ring = reinterpret_cast<bf16*>(a.conv_state) + (int64_t)seq * a.taps * C;
    for (int i = threadIdx.x; i < 2 * DP + cols; i += DT_THREADS) {
        const int kind = i < DP ? 0 : i < 2 * DP ? 1 : 2, c = kind == 0 ? i : kind == 1 ? i - DP : i - 2 * DP;
        float y = 0.f;
        if (kind == 2 || c < a.dim) {
            const int chan = kind == 0 ? kvh * a.dim + c : kind == 1 ? (a.G + kvh) * a.dim + c : 2 * a.G * a.dim + h * a.vdim + c0 + c;
            const bf16 now = proj[chan];
            for (int j = max(0, a.taps - 1 - pos); j < a.taps - 1; ++j)
                y = fmaf(a.conv_w[(int64_t)j * C + chan], __bfloat162float(ring[(int64_t)((pos - (a.taps - 1 - j)) % a.taps) * C + chan]), y);
            y = delta_silu(fmaf(a.conv_w[(int64_t)(a.taps - 1) * C + chan], __bfloat162float(now), y));
            // this token's slot of the ring is one that no row reads; heads that share key channels leave it to the first of them
            if (writes && (kind == 2 || (rank == 0 && h % (a.H / a.G) == 0))) ring[(int64_t)(pos % a.taps) * C + chan] = now;
        }
        if (kind == 2) v_s[c] = y;
        else (kind == 0 ? q_s : k_s)[c] = y;
    }
    cluster.sync();  // also: every CTA of the cluster runs, so its shared memory may be written
    // ---- decays of this CTA's key channels for the whole cluster, gates of its value channels ------------------
    const float rate = a.a_rate[h];
    dt_rows(a2, a.ra, dims, a.ra, low_s, warp, lane, [&](int r, float x) {
        const float g = expf(-rate * delta_softplus(x + a.dt_bias[h * a.dim + d0 + r]));
        for (int p = 0; p < size; ++p) *cluster.map_shared_rank(g_s + d0 + r, p) = g;
    });
    dt_rows(g2, a.rg, cols, a.rg, low_s + a.ra, warp, lane, [&](int r, float x) { z_s[r] = sigmoidf_precise(x); });
    for (int d = a.dim + threadIdx.x; d < DP; d += DT_THREADS) g_s[d] = 0.f;  // padding: the state is zero there
    if (warp < 2) {  // unit vectors
        float* x = warp ? k_s : q_s;
        float ss = 0.f;
        for (int d = lane; d < DP; d += 32) ss = fmaf(x[d], x[d], ss);
        const float scale = (warp ? 1.f : 1.f / sqrtf((float)a.dim)) / sqrtf(warp_sum(ss) + 1e-6f);
        for (int d = lane; d < DP; d += 32) x[d] *= scale;
    }
    const float beta = sigmoidf_precise(__bfloat162float(proj[a.off_b + h]));
    cluster.sync();
    // ---- the recurrence -----------------------------------------------------------------------------------------
    float square = 0.f;
    for (int base = 0; base < cols; base += DT_PASS) {
        if (base) fetch(base);
        const int c = base + warp * 4 + (lane & 3);
        float x = 0.f, y = 0.f, qk = 0.f;
        float4 kk[DQ];
#pragma unroll
        for (int i = 0; i < DQ; ++i) {
            const float4 g = *reinterpret_cast<const float4*>(g_s + 32 * i + kg * 4), q = *reinterpret_cast<const float4*>(q_s + 32 * i + kg * 4);
            kk[i] = *reinterpret_cast<const float4*>(k_s + 32 * i + kg * 4);
            s[i].x *= g.x; s[i].y *= g.y; s[i].z *= g.z; s[i].w *= g.w;
            x = fmaf(s[i].x, kk[i].x, x); x = fmaf(s[i].y, kk[i].y, x); x = fmaf(s[i].z, kk[i].z, x); x = fmaf(s[i].w, kk[i].w, x);
            y = fmaf(s[i].x, q.x, y); y = fmaf(s[i].y, q.y, y); y = fmaf(s[i].z, q.z, y); y = fmaf(s[i].w, q.w, y);
            qk = fmaf(q.x, kk[i].x, qk); qk = fmaf(q.y, kk[i].y, qk); qk = fmaf(q.z, kk[i].z, qk); qk = fmaf(q.w, kk[i].w, qk);
        }
#pragma unroll
        for (int o = 4; o < 32; o <<= 1) {
            x += __shfl_xor_sync(0xffffffffu, x, o);
            y += __shfl_xor_sync(0xffffffffu, y, o);
            qk += __shfl_xor_sync(0xffffffffu, qk, o);
        }
        if (c < cols) {
            const float u = beta * (v_s[c] - x);
#pragma unroll
            for (int i = 0; i < DQ; ++i) {
                s[i].x = fmaf(kk[i].x, u, s[i].x); s[i].y = fmaf(kk[i].y, u, s[i].y);
                s[i].z = fmaf(kk[i].z, u, s[i].z); s[i].w = fmaf(kk[i].w, u, s[i].w);
                if (writes) *reinterpret_cast<float4*>(state + (int64_t)c * DP + 32 * i + kg * 4) = s[i];
            }
            if (kg == 0) {
                const float o = fmaf(qk, u, y);
                o_s[c] = o;
                square = fmaf(o, o, square);
            }
        }
    }
    // ---- norm over the head, gate ----------------------------------------------------------------------------------
    square = warp_sum(square);
    if (lane == 0) red_s[warp] = square;
    __syncthreads();
    if ((int)threadIdx.x < size) {
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < DT_WARPS; ++w) sum += red_s[w];
        *cluster.map_shared_rank(ss_s + rank, threadIdx.x) = sum;
    }
    cluster.sync();
    float total = 0.f;
    for (int p = 0; p < size; ++p) total += ss_s[p];
    const float denom = sqrtf(total / (float)a.vdim + a.eps);
    bf16* out = reinterpret_cast<bf16*>(a.out) + (int64_t)row * a.out_stride + h * a.vdim + c0;
    for (int c = threadIdx.x; c < cols; c += DT_THREADS) out[c] = __float2bfloat16_rn(o_s[c] / denom * a.norm[c0 + c] * z_s[c]);
}

// ===================================================================================================
template <int DQ>
static int launch_step(const DeltaArgs& a, int cluster, cudaStream_t st) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(cluster, a.H, a.rows);
    cfg.blockDim = dim3(DT_THREADS);
    cfg.dynamicSmemBytes = (size_t)(a.ra + a.rg) * sizeof(float);
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = g_glmb_pdl_enabled ? 1 : 0;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, delta_step_kernel<DQ>, a);
    return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

// bf16, one row per sequence: proj (with the low-rank first halves at off_a and off_g) -> out, state and convolution history.  ra, rg: row
// lengths of a2 and g2 (multiples of 8, up to 4096 together); value heads up to 1024 wide.
GLMB_API int glmb_delta_step(const DeltaArgs* args, void* stream) {
    const DeltaArgs a = *args;
    if (!delta_sizes_ok(a) || !a.decode || a.taps < 1 || !a.a2 || !a.g2 || a.ra < 8 || a.rg < 8 || (a.ra & 7) || (a.rg & 7) || a.ra + a.rg > 4096 || a.vdim > DT_VALUES * DT_CLUSTER) return 1;
    if ((reinterpret_cast<uintptr_t>(a.a2) | reinterpret_cast<uintptr_t>(a.g2)) & 15) return 1;
    int cluster = a.vdim >= 64 ? 4 : a.vdim >= 32 ? 2 : 1;
    while (cluster > 1 && (int64_t)cluster * a.H * a.rows > 4 * 148 && a.vdim * 2 <= cluster * DT_VALUES) cluster /= 2;  // all CTAs resident at once
    cudaStream_t st = (cudaStream_t)stream;
    switch (a.dimp / 32) {
        case 1: return launch_step<1>(a, cluster, st);
        case 2: return launch_step<2>(a, cluster, st);
        case 3: return launch_step<3>(a, cluster, st);
        case 4: return launch_step<4>(a, cluster, st);
        case 5: return launch_step<5>(a, cluster, st);
        case 6: return launch_step<6>(a, cluster, st);
        case 7: return launch_step<7>(a, cluster, st);
        default: return launch_step<8>(a, cluster, st);
    }
}
