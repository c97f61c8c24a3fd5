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
    uint32_t step;       // every row is the next token of its own sequence: whoever has a and b makes the step
    float decay;
};

__device__ __forceinline__ float m40_softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

// What one row's channel needs from memory before its step: state (0 at a sequence's start) and output gate input.
struct M40RgStep {
    float s_old, y;
    size_t slot;  // or ~0: not a valid row
};
__device__ __forceinline__ M40RgStep m40_rg_fetch(const M40RgArgs& g, uint32_t row, uint32_t c) {
    M40RgStep t = {0.0f, 0.0f, g.row_seq[row] * g.slot_mul + g.slot_add};
    if (t.slot >= g.slots) {
        if (c == 0) atomicOr(g.status, 2u);
        t.slot = ~(size_t)0;
        return t;
    }
    if (g.row_pos[row] > 0) t.s_old = g.state[t.slot * g.slot_stride + c];
    t.y = g.packed[(size_t)row * g.ld + c];
    return t;
}
__device__ __forceinline__ void m40_rg_store(const M40RgArgs& g, uint32_t row, uint32_t c, const M40RgStep& t, const float2& ab) {
    const float s = fmaf(ab.x, t.s_old, ab.y);
    const bool ok = t.slot != ~(size_t)0;
    if (ok) g.state[t.slot * g.slot_stride + c] = s;
    g.out[(size_t)row * g.width + c] = ok ? s * m40_act((int)M40LLM_ACT_GELU_TANH, t.y) : 0.0f;
}

// gate sums (biases added) -> (a, sqrt(1 - a^2) i u); sp = softplus(lam)
__device__ __forceinline__ float2 m40_rg_gated(const M40RgArgs& g, float zr, float zi, float sp, float u) {
    const float la = -g.decay * m40_sigmoid(zr) * sp;
    return make_float2(expf(la), sqrtf(-expm1f(2.0f * la)) * m40_sigmoid(zi) * u);
}
