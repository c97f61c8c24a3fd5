// Elementwise pieces of the layer-stack mechanisms, shared by the streaming GEMV, the tensor-core GEMM, the f32 GEMM
// and the mixer kernels: activations, dynamic tanh, soft cap and 16-bit conversions.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

__device__ __forceinline__ float m40_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

__device__ __forceinline__ float m40_act(int act, float v) {
    if (act == (int)M40LLM_ACT_GELU_TANH)  // 0.5 v (1 + tanh(sqrt(2/pi) (v + 0.044715 v^3)))
        return 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    if (act == (int)M40LLM_ACT_GELU_ERF) return 0.5f * v * (1.0f + erff(0.7071067811865476f * v));
    return v / (1.0f + expf(-v));  // SiLU
}

// What follows a projection, element by element: cap(residual + post(y + bias)).
struct M40Tail {
    int post;          // M40LLM_NORM_NONE or M40LLM_NORM_DYT
    float post_alpha;
    float soft_cap;    // 0: none
};
__device__ __forceinline__ float m40_tail(const M40Tail& t, float y, float bias, float pw, float pb, float residual) {
    y += bias;
    if (t.post == (int)M40LLM_NORM_DYT) y = tanhf(t.post_alpha * y) * pw + pb;
    y += residual;
    if (t.soft_cap > 0.0f) y = t.soft_cap * tanhf(y / t.soft_cap);
    return y;
}

__device__ __forceinline__ float m40_load_elem(const float* p) { return *p; }
__device__ __forceinline__ float m40_load_elem(const __half* p) { return __half2float(*p); }
__device__ __forceinline__ float m40_load_elem(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void m40_store_elem(float* p, float v) { *p = v; }
__device__ __forceinline__ void m40_store_elem(__half* p, float v) { *p = __float2half_rn(v); }

__device__ __forceinline__ float4 m40_vec4_or(const float* p, uint32_t k, float fallback) {
    return p ? *reinterpret_cast<const float4*>(p + k) : make_float4(fallback, fallback, fallback, fallback);
}

// PolyNorm of a row with K values and sums s1 = sum z^2, s2 = sum z^4, s3 = sum z^6: (x, y, z, w) such that the result is
// x z + y z^2 + z z^3 + w.
__device__ __forceinline__ float4 m40_poly_scales(const float* coef, float s1, float s2, float s3, float K, float eps) {
    return make_float4(coef[0] / sqrtf(s1 / K + eps), coef[1] / sqrtf(s2 / K + eps), coef[2] / sqrtf(s3 / K + eps), coef[3]);
}
__device__ __forceinline__ float m40_poly(const float4& n, float z) { return fmaf(z, fmaf(z, fmaf(z, n.z, n.y), n.x), n.w); }

// Eight consecutive values of a 16-bit type (16-byte aligned), or of f32, as f32.
template <typename WT>
__device__ __forceinline__ void m40_load8(const WT* p, float* v) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const WT* h = reinterpret_cast<const WT*>(&r);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = m40_load_elem(h + i);
}
template <>
__device__ __forceinline__ void m40_load8<float>(const float* p, float* v) {
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = p[i];
}
