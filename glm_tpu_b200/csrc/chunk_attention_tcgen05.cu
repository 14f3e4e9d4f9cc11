// Prefill attention inside chunks (see chunk_attention.cu) on the 5th-generation tensor cores, head sizes up to 128.
//
// A CTA owns 256 consecutive query rows of one head as two 128-row tiles that take turns on the tensor core, so one tile's softmax
// runs while the other tile's products do.  For every block of 128 keys and each tile t:
//
//   S_t = Q_t K^T        both operands K-major in shared memory (TMA, 128-byte swizzle), fp32 scores in TMEM
//   softmax              128 threads, one row each: scores from TMEM, running maximum and sum in fp32, weights back into TMEM where the
//                        scores were, as bf16 pieces: value (columns 0..63, two keys per column) and remainder (64..127)
//   O_t += P_t V         A = weights from TMEM, B = values as they lie in memory ([key, column], MN-major), both pieces into one fp32 sum
//
// The maximum is only followed when it grows by more than 2^8: the weights stay finite, the final division removes the difference, and the
// output in TMEM is rescaled rarely.
//
//   warps 0-3, 4-7   softmax and output of tile 0 and tile 1 (warp w reads TMEM lanes 32 (w % 4) ..)
//   warp 8           issues every tcgen05.mma (one lane), owns the TMEM allocation
//   warp 9           TMA producer (one lane): query tiles once, then K and V blocks through two-stage rings
//
// Every wait is bounded; a wait that runs out raises GLMB_STATUS_WAIT_TIMEOUT and the CTA still releases its TMEM.
#include "chunk_attention.cuh"
#include "tcgen05.cuh"

#define FA_TILE 128
#define FA_STAGES 2
#define FA_THREADS 320
#define FA_BOX 16384  // bytes of a 128-row, 64-column box
#define FA_LOG2E 1.4426950408889634f
#define FA_SLACK 8.0f  // log2 of how far the weights may exceed one before the maximum is followed

__device__ __forceinline__ void fa_tmem_ld32_nowait(uint32_t taddr, uint32_t* r) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
          "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]),
          "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]),
          "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
        : "r"(taddr) : "memory");
}
__device__ __forceinline__ void fa_tmem_ld16(uint32_t taddr, uint32_t (&r)[16]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
          "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(taddr) : "memory");
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void fa_tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
        "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}
// D[tmem] (+)= A[tmem] . B[shared]
__device__ __forceinline__ void fa_mma_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
        ::"r"(tmem_d), "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate) : "memory");
}
// MN-major operand, 128-byte swizzle: 64 columns (128 bytes) per K row, 8 K rows per 1024-byte group, 64-column boxes FA_BOX apart
__device__ __forceinline__ uint64_t fa_desc_mn(uint32_t smem_addr) {
    return (uint64_t)((smem_addr >> 4) & 0x3FFFu) | ((uint64_t)(FA_BOX >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ float fa_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

struct FaRange { int rows, begin, end; };  // rows of a tile, and its key blocks [begin, end)

__global__ void __launch_bounds__(FA_THREADS, 1)
chunk_attn_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                     ChunkAttnArgs a) {
    GLMB_PDL_PROLOGUE();  // before the TMEM allocation: a kernel still running may need the columns to finish
    extern __shared__ unsigned char smem_raw[];
    __shared__ __align__(8) uint64_t q_full[2], k_full[FA_STAGES], k_empty[FA_STAGES], v_full[FA_STAGES], v_empty[FA_STAGES], s_full[2], p_full[2], o_full[2];
    __shared__ uint32_t tmem_slot;
    __shared__ volatile uint32_t fail;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kboxes = (a.dimp + 63) / 64, vboxes = (a.vdimp + 63) / 64;
    unsigned char* q_s = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char* k_s = q_s + 2 * kboxes * FA_BOX;
    unsigned char* v_s = k_s + FA_STAGES * kboxes * FA_BOX;

    if (threadIdx.x == 0) {
        for (int i = 0; i < 2; ++i) { mbar_init(q_full + i, 1); mbar_init(s_full + i, 1); mbar_init(p_full + i, 4); mbar_init(o_full + i, 1); }
        for (int i = 0; i < FA_STAGES; ++i) { mbar_init(k_full + i, 1); mbar_init(k_empty + i, 1); mbar_init(v_full + i, 1); mbar_init(v_empty + i, 1); }
        fail = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 8) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_slot;  // S_0, S_1 at columns 0 and 128, O_0, O_1 at 256 and 384

    const int head = blockIdx.y, group = head / (a.H / a.G);
    const int r0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * 2 * FA_TILE;  // rows towards the end (most keys) first
    const int key0 = (a.start + r0) / a.chunk * a.chunk;
    FaRange range[2];
#pragma unroll
    for (int t = 0; t < 2; ++t) {
        const int first = r0 + t * FA_TILE;
        range[t].rows = min(FA_TILE, a.rows - first);
        range[t].begin = ((a.start + first) / a.chunk * a.chunk - key0) / FA_TILE;
        range[t].end = (a.start + first + range[t].rows - 1 - key0) / FA_TILE + 1;
        if (range[t].rows <= 0) range[t].rows = 0, range[t].begin = range[t].end = 0;
    }
    const int blocks = max(range[0].end, range[1].end);

    if (warp == 9) {
        if (lane == 0) {
            for (int t = 0; t < 2; ++t)
                if (range[t].rows) {
                    mbar_expect_tx(q_full + t, kboxes * FA_BOX);
                    for (int b = 0; b < kboxes; ++b)
                        tma_load_2d(q_s + (t * kboxes + b) * FA_BOX, &map_q, q_full + t, head * a.dimp + b * 64, r0 + t * FA_TILE);
                }
            for (int j = 0; j < blocks; ++j) {
                const int s = j % FA_STAGES, lap = j / FA_STAGES, y = key0 - a.base + j * FA_TILE;
                if (lap > 0 && !mbar_wait(k_empty + s, (lap - 1) & 1)) { fail = 1; break; }
                mbar_expect_tx(k_full + s, kboxes * FA_BOX);
                for (int b = 0; b < kboxes; ++b) tma_load_2d(k_s + (s * kboxes + b) * FA_BOX, &map_k, k_full + s, group * a.dimp + b * 64, y);
                if (lap > 0 && !mbar_wait(v_empty + s, (lap - 1) & 1)) { fail = 1; break; }
                mbar_expect_tx(v_full + s, vboxes * FA_BOX);
                for (int b = 0; b < vboxes; ++b) tma_load_2d(v_s + (s * vboxes + b) * FA_BOX, &map_v, v_full + s, group * a.vdimp + b * 64, y);
            }
        }
    } else if (warp == 8) {
        if (lane == 0) {
            const uint32_t idesc_s = umma_idesc_bf16(FA_TILE, FA_TILE), idesc_o = umma_idesc_bf16(FA_TILE, a.vdimp) | (1u << 16);  // bit 16: B is MN-major
            int done[2] = {0, 0};
            bool ok = true;
            for (int j = -1; j < blocks && ok; ++j) {
                for (int t = 0; t < 2 && ok; ++t) {
                    if (j >= range[t].begin && j < range[t].end) {  // O_t += P_t V_j
                        if (!mbar_wait(p_full + t, done[t] & 1) || !mbar_wait(v_full + j % FA_STAGES, (j / FA_STAGES) & 1) || fail) { fail = 1; ok = false; break; }
                        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                        const uint32_t v_addr = smem_u32(v_s + (j % FA_STAGES) * vboxes * FA_BOX);
                        for (int piece = 0; piece < 2; ++piece)
#pragma unroll
                            for (int k = 0; k < FA_TILE / 16; ++k)
                                fa_mma_ts(tmem + 256 + t * 128, tmem + t * 128 + piece * 64 + k * 8, fa_desc_mn(v_addr + k * 2048), idesc_o,
                                          (done[t] > 0 || piece > 0 || k > 0) ? 1u : 0u);
                        ++done[t];
                        if (j + 1 == range[t].end) umma_commit(o_full + t);
                    }
                    if (j + 1 >= range[t].begin && j + 1 < range[t].end) {  // S_t = Q_t K_{j+1}^T
                        const int n = j + 1, s = n % FA_STAGES;
                        if ((n == range[t].begin && !mbar_wait(q_full + t, 0)) || !mbar_wait(k_full + s, (n / FA_STAGES) & 1) || fail) { fail = 1; ok = false; break; }
                        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                        const uint32_t q_addr = smem_u32(q_s + t * kboxes * FA_BOX), k_addr = smem_u32(k_s + s * kboxes * FA_BOX);
                        for (int k = 0; k < a.dimp / 16; ++k) {
                            const uint32_t at = (k >> 2) * FA_BOX + (k & 3) * 32;
                            umma_bf16(tmem + t * 128, umma_desc_sw128(q_addr + at), umma_desc_sw128(k_addr + at), idesc_s, k > 0 ? 1u : 0u);
                        }
                        umma_commit(s_full + t);
                    }
                }
                if (!ok) break;
                if (j >= 0) umma_commit(v_empty + j % FA_STAGES);            // the blocks may be replaced once these products have read them
                if (j + 1 < blocks) umma_commit(k_empty + (j + 1) % FA_STAGES);
            }
        }
    } else {
        const int t = warp >> 2, quarter = warp & 3;
        const int row = quarter * 32 + lane, first = a.start + r0 + t * FA_TILE + quarter * 32, pos = first + lane;
        const int lo = pos / a.chunk * a.chunk, warp_lo = (first + 31) / a.chunk * a.chunk;
        const uint32_t lanes = (uint32_t)(quarter * 32) << 16, s_addr = tmem + t * 128 + lanes, o_addr = tmem + 256 + t * 128 + lanes;
        const float scale2 = a.scale * FA_LOG2E, sink2 = a.sink ? a.sink[head] * FA_LOG2E : -INFINITY;
        float m = sink2, l = 0.f;
        bool ok = true;
        for (int j = range[t].begin; j < range[t].end; ++j) {
            const int n = j - range[t].begin, key_base = key0 + j * FA_TILE;
            if (!mbar_wait(s_full + t, n & 1) || fail) { ok = false; break; }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            uint32_t s[128];
#pragma unroll
            for (int c = 0; c < 4; ++c) fa_tmem_ld32_nowait(s_addr + c * 32, s + c * 32);
            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
            if (key_base + FA_TILE - 1 > first || key_base < warp_lo) {  // the diagonal, or keys of an earlier chunk
#pragma unroll
                for (int i = 0; i < 128; ++i)
                    if (key_base + i > pos || key_base + i < lo) s[i] = 0xff800000u;  // -infinity
            }
            float mx0 = __uint_as_float(s[0]), mx1 = __uint_as_float(s[1]), mx2 = __uint_as_float(s[2]), mx3 = __uint_as_float(s[3]);
#pragma unroll
            for (int i = 4; i < 128; i += 4) {
                mx0 = fmaxf(mx0, __uint_as_float(s[i]));
                mx1 = fmaxf(mx1, __uint_as_float(s[i + 1]));
                mx2 = fmaxf(mx2, __uint_as_float(s[i + 2]));
                mx3 = fmaxf(mx3, __uint_as_float(s[i + 3]));
            }
            const float top = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)) * scale2;
            if (n == 0) {
                m = fmaxf(m, top);
            } else if (__any_sync(0xffffffffu, top > m + FA_SLACK)) {
                const float next = fmaxf(m, top), fix = next == -INFINITY ? 1.f : fa_exp2(m - next);
                m = next;
                l *= fix;
                for (int c = 0; c < a.vdimp; c += 16) {
                    uint32_t o[16];
                    fa_tmem_ld16(o_addr + c, o);
#pragma unroll
                    for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * fix);
                    fa_tmem_st16(o_addr + c, o);
                }
            }
            const float base = m == -INFINITY ? 0.f : m;
            float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                uint32_t hi[16], lw[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const float x = fa_exp2(fmaf(__uint_as_float(s[c * 32 + 2 * i]), scale2, -base));
                    const float y = fa_exp2(fmaf(__uint_as_float(s[c * 32 + 2 * i + 1]), scale2, -base));
                    sum0 += x;
                    sum1 += y;
                    hi[i] = pack_bf16(x, y);
                    lw[i] = pack_bf16(x - bf16_lo(hi[i]), y - bf16_hi(hi[i]));
                }
                fa_tmem_st16(s_addr + c * 16, hi);
                fa_tmem_st16(s_addr + 64 + c * 16, lw);
            }
            l += sum0 + sum1;
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full + t);
        }
        if (range[t].rows) {
            if (ok) ok = mbar_wait(o_full + t, 0) && !fail;
            if (!ok) {
                fail = 1;
                if (lane == 0) raise_status(a.status, GLMB_STATUS_WAIT_TIMEOUT);
            } else {
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (a.sink) l += fa_exp2(sink2 - m);
                float inv = 1.f / l;
                if (a.gate && row < range[t].rows)
                    inv *= sigmoidf_precise(__bfloat162float(reinterpret_cast<const bf16*>(a.gate)[(int64_t)(r0 + t * FA_TILE + row) * a.gate_stride + head]));
                bf16* dst = reinterpret_cast<bf16*>(a.out) + (int64_t)(r0 + t * FA_TILE + row) * a.out_stride + (int64_t)head * a.vdim;
                const bool vec = !(reinterpret_cast<uintptr_t>(dst) & 15);
                for (int c = 0; c < a.vdimp; c += 16) {
                    uint32_t o[16];
                    fa_tmem_ld16(o_addr + c, o);
                    if (row >= range[t].rows) continue;
                    uint32_t w[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) w[i] = pack_bf16(__uint_as_float(o[2 * i]) * inv, __uint_as_float(o[2 * i + 1]) * inv);
                    if (vec && c + 16 <= a.vdim) {
                        *reinterpret_cast<uint4*>(dst + c) = make_uint4(w[0], w[1], w[2], w[3]);
                        *reinterpret_cast<uint4*>(dst + c + 8) = make_uint4(w[4], w[5], w[6], w[7]);
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (c + i < a.vdim) dst[c + i] = __ushort_as_bfloat16((unsigned short)(i & 1 ? w[i >> 1] >> 16 : w[i >> 1] & 0xffffu));
                    }
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 8) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512) : "memory");
    }
}

int launch_chunk_attn_tcgen05(const ChunkAttnArgs& a, cudaStream_t stream) {
    CUtensorMap map_q, map_k, map_v;
    if (make_map(&map_q, a.q, (uint64_t)a.rows, (uint64_t)a.H * a.dimp, (uint64_t)a.q_stride, FA_TILE)) return 3;
    if (make_map(&map_k, a.k, (uint64_t)a.keys, (uint64_t)a.G * a.dimp, (uint64_t)a.G * a.dimp, FA_TILE)) return 3;
    if (make_map(&map_v, a.v, (uint64_t)a.keys, (uint64_t)a.G * a.vdimp, (uint64_t)a.G * a.vdimp, FA_TILE)) return 3;
    static DeviceOnce once;
    const int dev = once.pending();
    if (dev != DeviceOnce::SET) {
        const cudaError_t e = cudaFuncSetAttribute(chunk_attn_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (4 + 4 + 4) * FA_BOX + 1024);
        if (e != cudaSuccess) return (int)e;
        once.mark(dev);
    }
    const int kboxes = (a.dimp + 63) / 64, vboxes = (a.vdimp + 63) / 64;
    const size_t smem = (size_t)((2 + FA_STAGES) * kboxes + FA_STAGES * vboxes) * FA_BOX + 1024;
    GLMB_LAUNCH(chunk_attn_tc_kernel, dim3(ceil_div(a.rows, 2 * FA_TILE), a.H), FA_THREADS, smem, stream, map_q, map_k, map_v, a);
    return (int)cudaGetLastError();
}
