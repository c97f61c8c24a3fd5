// Shared pieces of the real-gated linear recurrence (internal; see rglru.cu).
#pragma once
#include "stack_math.cuh"

struct M40RgArgs {
    const float* packed;
    const float* conv_w;
    const float* conv_b;
    const void* ra;
    const float* ra_b;
    const void* ri;
    const float* ri_b;
    const float* lam;
    float* out;
    float* state;        // per slot: S [width], ring [taps][width]
    size_t slot_stride;
    float* u;            // portions: [rows][width]
    float* a;
    float* b;
    uint32_t* status;
    const uint32_t* row_seq;
    const uint32_t* row_pos;
    const uint32_t* seg;
    uint32_t ld, width, bs, taps, slot_mul, slot_add, slots, rows, wide, tensor;
    float decay;
};

__device__ __forceinline__ float m40_softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

// gate sums (biases added) -> (a, sqrt(1 - a^2) i u); sp = softplus(lam)
__device__ __forceinline__ float2 m40_rg_gated(const M40RgArgs& g, float zr, float zi, float sp, float u) {
    const float la = -g.decay * m40_sigmoid(zr) * sp;
    return make_float2(expf(la), sqrtf(-expm1f(2.0f * la)) * m40_sigmoid(zi) * u);
}
