// Routed experts of the decode step (and of short prefill chunks): FP8 weight-streaming projections on CUDA cores, the combine of routed
// and shared partial sums with its in-kernel all-reduce, and the dispatch to the mma.sync variants (moe_gemv_mma.cu).
//
// Organised like the skinny projections (gemv.cu): 16-byte streaming loads, a warp per output feature, fp32 accumulation.  FP8 weights are
// decoded with the contract formula bf16(f32(e4m3) * scale_inv[n/128][k/128]) on the fly; the product with the bf16 activation is exact
// in fp32.
//
// Replaces: reference `kernels/fp8_grouped_matmul/kernel.py:125-299` (decode routed projection, t=1 and t=2).
#include "common.cuh"
#include "gemv_core.cuh"
#include "peer.cuh"

#define SK_WARPS 8
#define SK_THREADS (SK_WARPS * 32)

// ---------------------------------------------------------------------------------------------------
// Routed experts (FP8), organised as tiles: tile t = up to RT routes of ONE expert.
//   tile_expert[t]  global expert id (< 0: empty tile)
//   tile_routes[t*RT + i]  route index p = token_row * top_k + slot, or -1
// When tile_routes == nullptr every tile is the single route t and its expert is tile_expert[t] (decode).
// A tile whose expert is not stored on this rank is skipped: expert-parallel ownership is resolved here.
template <int RT>
__global__ void __launch_bounds__(SK_THREADS)
moe_gateup_fp8_kernel(const bf16* __restrict__ x, int64_t xs, int top_k, const int* __restrict__ tile_expert,
                      const int* __restrict__ tile_routes, const int* __restrict__ n_tiles, const uint8_t* __restrict__ wg,
                      const uint8_t* __restrict__ wu, const float* __restrict__ sg, const float* __restrict__ su,
                      int expert_base, int experts_local, int I, int H, bf16* __restrict__ act) {
    GLMB_PDL_PROLOGUE();
    const int t = blockIdx.y;
    if (n_tiles && t >= *n_tiles) return;
    const int e = tile_expert[t] - expert_base;
    if (e < 0 || e >= experts_local) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n = blockIdx.x * SK_WARPS + warp;
    if (n >= I) return;
    int route[RT];
    const bf16* xr[RT];
#pragma unroll
    for (int i = 0; i < RT; ++i) {
        route[i] = tile_routes ? tile_routes[t * RT + i] : (i == 0 ? t : -1);
        xr[i] = x + (int64_t)(route[i] >= 0 ? route[i] / top_k : 0) * xs;
    }
    const int kb = (H + 127) >> 7;
    const int64_t wofs = ((int64_t)e * I + n) * H;
    const int64_t sofs = ((int64_t)e * ((I + 127) >> 7) + (n >> 7)) * kb;
    const uint8_t* wp[2] = {wg + wofs, wu + wofs};
    const float* sp[2] = {sg + sofs, su + sofs};
    float acc[2][RT];
#pragma unroll
    for (int i = 0; i < RT; ++i) acc[0][i] = acc[1][i] = 0.f;
    warp_dot_fp8<RT, 2>(xr, wp, sp, H, lane, acc);
    warp_reduce_all<RT, 2>(acc);
    if (lane == 0) {
#pragma unroll
        for (int i = 0; i < RT; ++i)
            if (route[i] >= 0) {
                const float g = bf16_round(acc[0][i]), u = bf16_round(acc[1][i]);
                act[(int64_t)route[i] * I + n] = __float2bfloat16_rn(g * sigmoidf_precise(g) * u);
            }
    }
}

// dw[p][n] = bf16( bf16(act[p] . w_down[e][n]) * bf16(route_weight[p]) )
template <int RT>
__global__ void __launch_bounds__(SK_THREADS)
moe_down_fp8_kernel(const bf16* __restrict__ act, const float* __restrict__ route_weight, const int* __restrict__ tile_expert,
                    const int* __restrict__ tile_routes, const int* __restrict__ n_tiles, const uint8_t* __restrict__ wd,
                    const float* __restrict__ sd, int expert_base, int experts_local, int I, int H, bf16* __restrict__ dw) {
    GLMB_PDL_PROLOGUE();
    const int t = blockIdx.y;
    if (n_tiles && t >= *n_tiles) return;
    const int e = tile_expert[t] - expert_base;
    if (e < 0 || e >= experts_local) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n0 = (blockIdx.x * SK_WARPS + warp) * 2;
    if (n0 >= H) return;
    int route[RT];
    const bf16* xr[RT];
#pragma unroll
    for (int i = 0; i < RT; ++i) {
        route[i] = tile_routes ? tile_routes[t * RT + i] : (i == 0 ? t : -1);
        xr[i] = act + (int64_t)(route[i] >= 0 ? route[i] : 0) * I;
    }
    const int kb = (I + 127) >> 7;
    const int n1 = min(n0 + 1, H - 1);
    const uint8_t* wp[2] = {wd + ((int64_t)e * H + n0) * I, wd + ((int64_t)e * H + n1) * I};
    const float* sp[2] = {sd + ((int64_t)e * ((H + 127) >> 7) + (n0 >> 7)) * kb, sd + ((int64_t)e * ((H + 127) >> 7) + (n1 >> 7)) * kb};
    float acc[2][RT];
#pragma unroll
    for (int i = 0; i < RT; ++i) acc[0][i] = acc[1][i] = 0.f;
    warp_dot_fp8<RT, 2>(xr, wp, sp, I, lane, acc);
    warp_reduce_all<RT, 2>(acc);
    if (lane == 0) {
#pragma unroll
        for (int i = 0; i < RT; ++i)
            if (route[i] >= 0) {
                const float wgt = bf16_round(route_weight[route[i]]);
#pragma unroll
                for (int j = 0; j < 2; ++j)
                    if (n0 + j < H) dw[(int64_t)route[i] * H + n0 + j] = __float2bfloat16_rn(bf16_round(acc[j][i]) * wgt);
            }
    }
}

// ---------------------------------------------------------------------------------------------------
// MoE combine: for row r, column n
//   routed = sum over the row's routes owned by this rank, in slot order, of dw[p][n]      (fp32)
//   shared = this rank's K-slice of the shared-expert down projection                       (fp32, given)
//   both are summed over the ranks in-kernel (peer-memory all-reduce), then
//   out = bf16( bf16( bf16(routed) * scale ) + bf16(shared) )
// plain != 0: out = bf16(sum over ranks of shared_partial)   -- dense MLP / any K-split partial.
// routed_partial != nullptr: only write the local fp32 route sums there (the caller reduces them with a
//   library collective: the NCCL baseline and prefill); no exchange, no output.
// blockIdx.y selects a chunk of GLMB_MAX_ROWS rows.
#define CB_COLS 16
__global__ void __launch_bounds__(128)
moe_combine_kernel(const bf16* __restrict__ dw, const int* __restrict__ topk_ids, const float* __restrict__ shared_partial,
                   int rows_total, int top_k, int H, int expert_base, int experts_local, float scale, int plain,
                   bf16* __restrict__ out, float* __restrict__ routed_partial, PeerComm comm, int channel) {
    GLMB_PDL_PROLOGUE();
    __shared__ float sh[2 * GLMB_MAX_ROWS * CB_COLS];
    const int n0 = blockIdx.x * CB_COLS;
    const int r0 = blockIdx.y * GLMB_MAX_ROWS;
    const int rows = min(GLMB_MAX_ROWS, rows_total - r0);
    const int per = rows * CB_COLS;
    for (int i = threadIdx.x; i < per; i += blockDim.x) {
        const int r = r0 + i / CB_COLS, n = n0 + i % CB_COLS;
        float routed = 0.f, shared = 0.f;
        if (n < H) {
            shared = shared_partial ? shared_partial[(int64_t)r * H + n] : 0.f;
            if (!plain) {
                for (int s = 0; s < top_k; ++s) {
                    const int p = r * top_k + s;
                    const int e = topk_ids[p] - expert_base;
                    if (e >= 0 && e < experts_local) routed += __bfloat162float(dw[(int64_t)p * H + n]);
                }
            }
            if (routed_partial) routed_partial[(int64_t)r * H + n] = routed;
        }
        sh[i] = shared;
        sh[per + i] = routed;
    }
    if (routed_partial) return;
    __syncthreads();
    cta_allreduce_f32(comm, channel, sh, plain ? per : 2 * per);
    for (int i = threadIdx.x; i < per; i += blockDim.x) {
        const int r = r0 + i / CB_COLS, n = n0 + i % CB_COLS;
        if (n >= H) continue;
        float v;
        if (plain) v = sh[i];
        else v = bf16_round(bf16_round(sh[per + i]) * scale) + bf16_round(sh[i]);
        out[(int64_t)r * H + n] = __float2bfloat16_rn(v);
    }
}

// Many rows, several GPUs, library all-reduce: what follows the all-reduce of the routed and the shared partial sums of a prefill
// chunk, in one launch:  out = bf16( bf16(bf16(routed) * scale) + bf16(shared) )  -- the last line of moe_combine_kernel.
__global__ void __launch_bounds__(256)
moe_finish_kernel(const float* __restrict__ routed, const float* __restrict__ shared, int64_t n, float scale, bf16* __restrict__ out) {
    GLMB_PDL_PROLOGUE();
    const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i + 3 < n) {
        const float4 r = *reinterpret_cast<const float4*>(routed + i), s = *reinterpret_cast<const float4*>(shared + i);
        uint2 packed;
        packed.x = pack_bf16(bf16_round(bf16_round(r.x) * scale) + bf16_round(s.x), bf16_round(bf16_round(r.y) * scale) + bf16_round(s.y));
        packed.y = pack_bf16(bf16_round(bf16_round(r.z) * scale) + bf16_round(s.z), bf16_round(bf16_round(r.w) * scale) + bf16_round(s.w));
        *reinterpret_cast<uint2*>(out + i) = packed;
    } else {
        for (int64_t j = i; j < n; ++j) out[j] = __float2bfloat16_rn(bf16_round(bf16_round(routed[j]) * scale) + bf16_round(shared[j]));
    }
}

GLMB_API int glmb_moe_finish(const float* routed, const float* shared, int64_t n, float scale, void* out, void* stream) {
    if (n < 1 || (reinterpret_cast<uintptr_t>(routed) & 15) || (reinterpret_cast<uintptr_t>(shared) & 15) || (reinterpret_cast<uintptr_t>(out) & 7)) return 1;
    GLMB_LAUNCH(moe_finish_kernel, (unsigned)((n / 4 + 255) / 256 + 1), 256, 0, (cudaStream_t)stream, routed, shared, n, scale, (bf16*)out);
    return (int)cudaGetLastError();
}

// ===================================================================================================
// Tensor-core variants (moe_gemv_mma.cu), used when the shapes are whole 64-wide k chunks and 16-row panels.
int glmb_launch_moe_gateup_mma(const void* x, int64_t xs, int top_k, const int* tile_expert, const int* tile_routes, const int* n_tiles,
                               int tiles, int rt, const void* wg, const void* wu, const float* sg, const float* su, int expert_base,
                               int experts_local, int I, int H, void* act, cudaStream_t stream);
int glmb_launch_moe_down_mma(const void* act, const float* route_weight, const int* tile_expert, const int* tile_routes, const int* n_tiles,
                             int tiles, int rt, const void* wd, const float* sd, int expert_base, int experts_local, int I, int H, void* dw,
                             cudaStream_t stream);
static int g_moe_mma = 1;
// The fp32-FMA kernels below serve the shapes the mma.sync kernels refuse (hidden size not a multiple of 64, intermediate not a
// multiple of 16, unaligned rows: fixtures).  The switch exists so that the tests can run BOTH families on shapes both take
// (tests/test_gpu_ops.py::test_routed_experts); nothing in the product turns it off.
GLMB_API void glmb_set_moe_mma(int enabled) { g_moe_mma = enabled ? 1 : 0; }

// Routed gate/up for `tiles` tiles of `rt` routes (rt in {1, 8}).  H % 16 == 0.
GLMB_API int glmb_moe_gateup_fp8(const void* x, int64_t xs, int top_k, const int* tile_expert, const int* tile_routes,
                                 const int* n_tiles, int tiles, int rt, const void* wg, const void* wu, const float* sg,
                                 const float* su, int expert_base, int experts_local, int I, int H, void* act, void* stream) {
    if ((H & 15) || tiles < 1) return 1;
    if (g_moe_mma && (rt == 1 || rt == 8) && !(H & 63) && !(I & 15) && !(xs & 7))
        return glmb_launch_moe_gateup_mma(x, xs, top_k, tile_expert, tile_routes, n_tiles, tiles, rt, wg, wu, sg, su, expert_base,
                                          experts_local, I, H, act, (cudaStream_t)stream);
    dim3 grid(ceil_div(I, SK_WARPS), tiles);
    if (rt == 1)
        GLMB_LAUNCH(moe_gateup_fp8_kernel<1>, grid, SK_THREADS, 0, (cudaStream_t)stream, 
            (const bf16*)x, xs, top_k, tile_expert, tile_routes, n_tiles, (const uint8_t*)wg, (const uint8_t*)wu, sg, su,
            expert_base, experts_local, I, H, (bf16*)act);
    else if (rt == 8)
        GLMB_LAUNCH(moe_gateup_fp8_kernel<8>, grid, SK_THREADS, 0, (cudaStream_t)stream, 
            (const bf16*)x, xs, top_k, tile_expert, tile_routes, n_tiles, (const uint8_t*)wg, (const uint8_t*)wu, sg, su,
            expert_base, experts_local, I, H, (bf16*)act);
    else
        return 1;
    return (int)cudaGetLastError();
}

GLMB_API int glmb_moe_down_fp8(const void* act, const float* route_weight, const int* tile_expert, const int* tile_routes,
                               const int* n_tiles, int tiles, int rt, const void* wd, const float* sd, int expert_base,
                               int experts_local, int I, int H, void* dw, void* stream) {
    if ((I & 15) || tiles < 1) return 1;
    if (g_moe_mma && (rt == 1 || rt == 8) && !(I & 63) && !(H & 15))
        return glmb_launch_moe_down_mma(act, route_weight, tile_expert, tile_routes, n_tiles, tiles, rt, wd, sd, expert_base, experts_local,
                                        I, H, dw, (cudaStream_t)stream);
    dim3 grid(ceil_div(H, SK_WARPS * 2), tiles);
    if (rt == 1)
        GLMB_LAUNCH(moe_down_fp8_kernel<1>, grid, SK_THREADS, 0, (cudaStream_t)stream, (const bf16*)act, route_weight, tile_expert, tile_routes,
                                                                             n_tiles, (const uint8_t*)wd, sd, expert_base,
                                                                             experts_local, I, H, (bf16*)dw);
    else if (rt == 8)
        GLMB_LAUNCH(moe_down_fp8_kernel<8>, grid, SK_THREADS, 0, (cudaStream_t)stream, (const bf16*)act, route_weight, tile_expert, tile_routes,
                                                                             n_tiles, (const uint8_t*)wd, sd, expert_base,
                                                                             experts_local, I, H, (bf16*)dw);
    else
        return 1;
    return (int)cudaGetLastError();
}

// Any number of rows when the exchange is off (world == 1 or routed_partial given); with the in-kernel
// all-reduce the grid must fit the per-CTA flag table.
GLMB_API int glmb_moe_combine(const void* dw, const int* topk_ids, const float* shared_partial, int rows, int top_k, int H,
                              int expert_base, int experts_local, float scale, int plain, void* out, float* routed_partial,
                              const PeerComm* comm, int channel, void* stream) {
    if (rows < 1) return 1;
    dim3 grid(ceil_div(H, CB_COLS), ceil_div(rows, GLMB_MAX_ROWS));
    PeerComm c = comm ? *comm : single_comm();
    if (c.world > 1 && !routed_partial && (int)(grid.x * grid.y) > GLMB_AR_MAX_CTAS) return 2;
    GLMB_LAUNCH(moe_combine_kernel, grid, 128, 0, (cudaStream_t)stream, (const bf16*)dw, topk_ids, shared_partial, rows, top_k, H, expert_base,
                                                               experts_local, scale, plain, (bf16*)out, routed_partial, c, channel);
    return (int)cudaGetLastError();
}
