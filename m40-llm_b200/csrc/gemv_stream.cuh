// Internal interface of the single-row weight-streaming GEMV (gemv_stream.cu).
#pragma once
#include "common.cuh"
#include "stack_math.cuh"

// One weight matrix of a grouped launch: out[n] = x . W[n] (+ bias[n]) (+ residual[n]), n < N.
// In gate/up mode W is the gate matrix and W2 the up matrix: out[n] = silu(x . W[n]) * (x . W2[n]).
struct M40GemvSeg {
    const void* W;
    const void* W2;
    float* out;
    const float* bias;
    const float* residual;
    int N;
    // M40GemvExt::tail.post == DYT: per-output weight and shift (null: 1 and 0)
    const float* post_w;
    const float* post_b;
};

// Optional norm applied to x on the fly (each CTA normalises its own copy): RMS, x <- x * rsqrt(mean(x^2)+eps) * w, or
// dynamic tanh (`dyt`), x <- tanh(alpha * x) * w + b with f32 w and b, either of which may be null (1 and 0), or (`special`)
// a PolyNorm with its four f32 coefficients in w, or the bare activation `act` (w null).
struct M40GemvNorm {
    const void* w;    // null: no normalisation
    int w_is_f32;     // 1: f32 weights, 0: f16
    float eps;
    float* xn_out;    // optional: CTA 0 also writes the normalised row here
    int dyt;
    float alpha;
    const float* b;
    int special;  // 0, M40LLM_NORM_POLY or M40LLM_NORM_ACT
    int act;
};

// What a launch does beyond the Llama layer's norm / bias / residual / SiLU: see stack_math.cuh.
struct M40GemvExt {
    int act;  // gate/up mode: M40LLM_ACT_*
    M40Tail tail;
};

enum { M40_GEMV_F16 = 0, M40_GEMV_Q80 = 1, M40_GEMV_BF16 = 2 };

// Streams up to three weight matrices that share one activation row x [K] (f32) in a single launch.
// Returns 0 when launched, 1 when the shape/alignment is not one this kernel takes (caller falls back),
// < 0 on a launch failure.
int m40_gemv_stream(M40llmCudaContext* ctx, cudaStream_t s, const float* x, int K, int fmt, int gate_up, int nseg,
                    const M40GemvSeg* segs, const M40GemvNorm* norm, const M40GemvExt* ext = nullptr);
