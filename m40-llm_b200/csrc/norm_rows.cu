// Row norms as a pass of their own, with an optional residual and soft cap. One CTA per row; all sums f32.
#include "norm_rows.cuh"

#include "stack_math.cuh"

namespace {

constexpr uint32_t MAX_GROUPS = 2048;

__device__ __forceinline__ float part_sum(const float* x, uint32_t lo, uint32_t hi, uint32_t lane) {
    float s = 0.0f;
#pragma unroll 4
    for (uint32_t k = lo + lane; k < hi; k += 32u) s = fmaf(x[k], x[k], s);
    return warp_sum(s);
}

__global__ void __launch_bounds__(256) norm_rows_kernel(M40NormRows a) {
    extern __shared__ float sh[];  // RMS: [groups * slices] partial sums, then [groups] scales
    __shared__ float red[3][8];
    pdl_wait();
    pdl_trigger();
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, K = a.K;
    const float* x = a.x + (size_t)blockIdx.x * a.ldx;
    float* o = a.out + (size_t)blockIdx.x * K;
    const float* res = a.residual ? a.residual + (size_t)blockIdx.x * K : nullptr;
    const uint32_t kind = a.norm.kind;
    const float *w = (const float*)a.norm.w, *b = (const float*)a.norm.b;
    const uint32_t G = kind == M40LLM_NORM_RMS && a.norm.groups ? a.norm.groups : 1u, L = K / G;
    float4 poly = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float* scale = sh;
    if (kind == M40LLM_NORM_RMS) {
        // a group is cut into slices when there are fewer groups than warps
        const uint32_t S = G >= 8u ? 1u : 8u / G, len = (L + S - 1u) / S;
        scale = sh + G * S;
        for (uint32_t u = warp; u < G * S; u += 8u) {
            const uint32_t g = u / S, lo = g * L + min((u % S) * len, L), hi = g * L + min((u % S + 1u) * len, L);
            const float s = part_sum(x, lo, hi, lane);
            if (lane == 0) sh[u] = s;
        }
        __syncthreads();
        for (uint32_t g = tid; g < G; g += 256u) {
            float t = 0.0f;
            for (uint32_t i = 0; i < S; ++i) t += sh[g * S + i];
            scale[g] = 1.0f / sqrtf(t / (float)L + a.norm.eps);
        }
        __syncthreads();
    } else if (kind == M40LLM_NORM_POLY) {
        float s1 = 0.0f, s2 = 0.0f, s3 = 0.0f;
#pragma unroll 4
        for (uint32_t k = tid; k < K; k += 256u) {
            const float z = x[k], q = z * z, c = q * z;
            s1 += q, s2 = fmaf(q, q, s2), s3 = fmaf(c, c, s3);
        }
        s1 = warp_sum(s1), s2 = warp_sum(s2), s3 = warp_sum(s3);
        if (lane == 0) red[0][warp] = s1, red[1][warp] = s2, red[2][warp] = s3;
        __syncthreads();
        s1 = s2 = s3 = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; ++i) s1 += red[0][i], s2 += red[1][i], s3 += red[2][i];
        poly = m40_poly_scales(w, s1, s2, s3, (float)K, a.norm.eps);
    }
#pragma unroll 4
    for (uint32_t k = tid; k < K; k += 256u) {
        float v = x[k];
        if (kind == M40LLM_NORM_RMS) v = v * scale[G == 1u ? 0u : k / L] * w[k];
        else if (kind == M40LLM_NORM_DYT) v = tanhf(a.norm.alpha * v) * (w ? w[k] : 1.0f) + (b ? b[k] : 0.0f);
        else if (kind == M40LLM_NORM_POLY) v = m40_poly(poly, v);
        else if (kind == M40LLM_NORM_ACT) v = m40_act((int)a.norm.act, v);
        if (res) v += res[k];
        if (a.soft_cap > 0.0f) v = a.soft_cap * tanhf(v / a.soft_cap);
        o[k] = v;
    }
}

}  // namespace

bool m40_norm_valid(const M40llmNorm& n, uint32_t K) {
    if (n.kind > M40LLM_NORM_ACT) return false;
    if (n.kind == M40LLM_NORM_RMS && (!n.w || (n.groups && (K % n.groups != 0 || n.groups > MAX_GROUPS)))) return false;
    if (n.kind == M40LLM_NORM_POLY && !n.w) return false;
    return n.kind != M40LLM_NORM_ACT || n.act <= M40LLM_ACT_GELU_ERF;
}

int m40_norm_rows(M40llmCudaContext* ctx, cudaStream_t s, const M40NormRows& a) {
    const uint32_t G = a.norm.groups ? a.norm.groups : 1u;
    const size_t smem = a.norm.kind == M40LLM_NORM_RMS ? (size_t)G * ((G >= 8u ? 1u : 8u / G) + 1u) * sizeof(float) : 0;
    const cudaError_t e = m40_launch_dependent(norm_rows_kernel, dim3(a.rows), dim3(256), smem, s, a);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}
