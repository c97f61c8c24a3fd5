// Grouped tcgen05 GEMM (internal): many weight matrices of one shape, each applied to its own rows or columns of the
// activations, in one launch. See gemm_tc_grouped.cu.
#pragma once
#include "rglru.cuh"

struct M40GroupTile {
    uint32_t group, row0, live, pad;
};

enum { M40_GROUPED_F32 = 0, M40_GROUPED_ACT_SPLIT = 1, M40_GROUPED_RG = 2, M40_GROUPED_HEADS = 3 };

// D[m][n] = sum_k X[m][group * group_k + k] * W[group * N + n][k] for the rows m of every tile.
// X is given as `parts` 16-bit arrays of the weights' type, [x_rows][ldx] each, whose sum is the activation.
struct M40GroupedCall {
    const void* w;             // [groups * N][K]
    const void* w2;            // RG: the second matrix (paired tiles)
    const void* x[3];
    uint32_t parts, bf16;
    uint32_t groups, N, K, x_rows, ldx, group_k;
    uint32_t tile_rows;        // 16, 32, 64 or 128; parts * tile_rows <= 256
    const M40GroupTile* tiles; // device table and its length (device), at most max_tiles; null: every group has all x_rows
    const uint32_t* n_tiles;
    uint32_t max_tiles;
    // result
    int kind, act;
    float* out;                // F32: [x_rows][out_ld], group g's values from column g * out_group on (0, 0: N, 0)
    uint32_t out_ld, out_group;
    void* hi;                  // ACT_SPLIT: act(D) as hi + lo of the weights' type, [x_rows][N]
    void* lo;
    __half* heads;             // HEADS: f16 [N / head_dim][x_rows][head_pitch], one row of D dealt to heads of head_dim values
    uint32_t head_dim, head_pitch;
    M40RgArgs rg;              // RG: a and b of every (row, channel)
};
// Whether the shapes and pointers are ones the kernel takes.
bool m40_gemm_tc_grouped_supported(const void* w, uint32_t N, uint32_t K, uint32_t ldx, uint32_t group_k);
int m40_gemm_tc_grouped(M40llmCudaContext* ctx, cudaStream_t s, const M40GroupedCall& c);
