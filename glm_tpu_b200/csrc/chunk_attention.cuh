// Arguments shared by the chunked-attention kernels (chunk_attention.cu, chunk_attention_tcgen05.cu).
#pragma once

#include "common.cuh"

struct ChunkAttnArgs {
    const void* q; int64_t q_stride;             // [rows, H, dimp]; elements between rows (0: H * dimp)
    const void *k, *v;                           // prefill: [keys, G, dimp], [keys, G, vdimp] from position `base`; decode: the rings
    const float* sink;                           // [H], or NULL: no sink
    const int *row_pos, *row_lane, *row_active;  // decode; row_active may be NULL
    void* out; int64_t out_stride;               // [rows, H * vdim (+ more)]
    const void* gate; int64_t gate_stride;       // [rows, H]: output head h is multiplied by sigmoid(gate[h]); or NULL
    int rows, H, G, dim, dimp, vdim, vdimp;      // dimp, vdimp: head sizes padded to a multiple of 16 (zeros)
    int decode;
    int start, base, keys;                       // prefill: position of row 0, of key 0, and how many keys there are
    int chunk, ring, capacity, lanes;            // decode: rings are [lanes, ring, G, dimp] and [lanes, ring, G, vdimp]
    float scale;
    uint32_t* status;
};

int launch_chunk_attn_tcgen05(const ChunkAttnArgs& a, cudaStream_t stream);
