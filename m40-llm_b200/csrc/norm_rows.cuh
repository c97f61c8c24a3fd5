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
bool m40_norm_valid(const M40llmNorm& n, uint32_t K);
int m40_norm_rows(M40llmCudaContext* ctx, cudaStream_t s, const M40NormRows& a);
