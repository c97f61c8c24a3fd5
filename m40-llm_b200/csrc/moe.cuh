// Mixture of experts (internal; see m40llm_moe_async and moe.cu).
#pragma once
#include "stack_math.cuh"

struct M40MoeArgs {
    const float* x;          // [rows][K]
    const float* logits;
    const float* correction;
    const void* up;          // [experts][ff][K]
    const void* down;        // [experts][K][ff]
    const float* add;        // [rows][K] or null
    uint32_t* ids;           // [rows][top]
    float* weights;          // [rows][top]
    float* hid;              // [rows * top][ff]
    float* y;                // [rows][K]
    uint32_t rows, K, ff, experts, identity, top, groups, keep, ld_logits, wide_up, wide_down;
    int act;
    float scale;
};
