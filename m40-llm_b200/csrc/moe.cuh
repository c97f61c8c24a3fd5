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
    // tensor path: rows sorted by expert, every expert's share padded to whole tiles
    uint32_t* place;         // [rows][top]: sorted row of the slot
    struct M40GroupTile* tiles;
    uint32_t* n_tiles;
    void* xs[2];             // [sorted rows][K] hi, lo of the weights' type
    void* hs[2];             // [sorted rows][ff]
    float* ys;               // [sorted rows][K]
    uint32_t tile_rows, bf16;
    uint32_t rows, K, ff, experts, identity, top, groups, keep, ld_logits, wide_up, wide_down;
    int act;
    float scale;
};
