// Row norms as a pass of their own (internal): what the projection kernels do not fold into themselves.
#pragma once
#include "common.cuh"

// out[r] = cap(residual[r] + norm(x[r])), rows of K values; row pitch of x ldx, of out and residual K.
struct M40NormRows {
    const float* x;
    float* out;
    const float* residual;  // may alias out
    M40llmNorm norm;
    uint32_t rows, K, ldx;
    float soft_cap;
};
// The normed value is x[r] (may be null: zeros) plus a weighted sum of `slots` rows of K values: slot j of row r adds
// weights[r][j] times row place[r][j] of `values`, or times row r of `x` when ids[r][j] >= experts.
constexpr uint32_t M40_NORM_SLOTS = 32;
struct M40NormGather {
    const float* values;
    const float* x;
    const float* weights;
    const uint32_t* ids;
    const uint32_t* place;
    uint32_t slots, experts;
};
bool m40_norm_gather_rows_takes(const M40NormRows& a, const M40NormGather& y);
int m40_norm_gather_rows(M40llmCudaContext* ctx, cudaStream_t s, const M40NormRows& a, const M40NormGather& y);

bool m40_norm_valid(const M40llmNorm& n, uint32_t K);
int m40_norm_rows(M40llmCudaContext* ctx, cudaStream_t s, const M40NormRows& a);
