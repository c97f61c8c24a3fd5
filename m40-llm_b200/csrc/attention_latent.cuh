// Latent attention (internal; see attention_latent.cu).
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

struct M40LatArgs {
    const float* packed;   // of the pass's first row
    const float* c_norm;
    const void* uk;
    const void* uk_t;
    const void* uv;
    const float* sink;
    void* C;
    __nv_bfloat16* part[2];  // tensor path: hi and lo of the queries [rows][heads * dim], then of the weighted latents
    uint32_t* seq_map;
    float* qa;             // absorbed queries [rows][heads][rank]
    float* pm;             // [rows][heads][splits]
    float* pl;
    float* po;             // [rows][heads][splits][rank]
    float* out;
    uint32_t* status;
    const uint32_t* row_seq;
    const uint32_t* row_pos;
    uint32_t ld, heads, dim, vdim, rank, slot_mul, slot_add, slots, max_seq_len, rows, splits, chunk;
    uint32_t absorb_ctas, wide;
    float eps, scale;
};

// The tcgen05 form of the attention over latents (attention_latent_tc.cu): f16 cache, rank a multiple of 128 up to 512.
// Tokens per split should be a multiple of 128.
bool m40_latent_tc_takes(const M40LatArgs& a);
int m40_latent_tc(M40llmCudaContext* ctx, const M40LatArgs& a);
