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

// The usual shapes (K a multiple of 128 per part, up to 8192): a row is read once and stays in registers, and everything the
// result needs is requested before the sums are known. A warp's 16-byte loads cover 128 values of one part.
template <int V>
__global__ void __launch_bounds__(256) norm_rows_wide_kernel(M40NormRows a, M40NormGather y) {
    __shared__ float part[64];
    __shared__ float sw[M40_NORM_SLOTS];
    __shared__ const float* sp[M40_NORM_SLOTS];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, K = a.K, row = blockIdx.x;
    const float *w = (const float*)a.norm.w, *b = (const float*)a.norm.b;
    const uint32_t kind = a.norm.kind;
    float4 x[V], wv[V], res[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const uint32_t k = tid * 4u + 1024u * i;
        wv[i] = w && k < K ? *reinterpret_cast<const float4*>(w + k) : make_float4(1.f, 1.f, 1.f, 1.f);
    }
    pdl_wait();
    pdl_trigger();
    if (y.slots) {
        if (tid < y.slots) {
            const size_t j = (size_t)row * y.slots + tid;
            sw[tid] = y.weights[j];
            sp[tid] = y.ids[j] < y.experts ? y.values + (size_t)y.place[j] * K : y.x + (size_t)row * K;
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const uint32_t k = tid * 4u + 1024u * i;
        x[i] = res[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (k >= K) continue;
        if (a.x) x[i] = *reinterpret_cast<const float4*>(a.x + (size_t)row * a.ldx + k);
        if (a.residual) res[i] = *reinterpret_cast<const float4*>(a.residual + (size_t)row * K + k);
#pragma unroll 4
        for (uint32_t j = 0; j < y.slots; ++j) {
            const float4 v = *reinterpret_cast<const float4*>(sp[j] + k);
            x[i].x = fmaf(sw[j], v.x, x[i].x), x[i].y = fmaf(sw[j], v.y, x[i].y);
            x[i].z = fmaf(sw[j], v.z, x[i].z), x[i].w = fmaf(sw[j], v.w, x[i].w);
        }
    }
    float scale[V];
#pragma unroll
    for (int i = 0; i < V; ++i) scale[i] = 1.0f;
    if (kind == M40LLM_NORM_RMS) {
        const uint32_t G = a.norm.groups ? a.norm.groups : 1u, chunks = K / G / 128u;  // 128-value chunks per part
#pragma unroll
        for (int i = 0; i < V; ++i) {
            const float s = warp_sum(x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w);
            if (lane == 0) part[i * 8 + warp] = s;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < V; ++i) {
            const uint32_t first = (i * 8u + warp) / chunks * chunks;
            if ((i * 8u + warp) * 128u >= K) continue;
            float t = 0.0f;
            for (uint32_t c = 0; c < chunks; ++c) t += part[first + c];
            scale[i] = 1.0f / sqrtf(t / (float)(chunks * 128u) + a.norm.eps);
        }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const uint32_t k = tid * 4u + 1024u * i;
        if (k >= K) continue;
        float v[4] = {x[i].x, x[i].y, x[i].z, x[i].w};
        const float wk[4] = {wv[i].x, wv[i].y, wv[i].z, wv[i].w}, rk[4] = {res[i].x, res[i].y, res[i].z, res[i].w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if (kind == M40LLM_NORM_RMS) v[j] = v[j] * scale[i] * wk[j];
            else if (kind == M40LLM_NORM_DYT) v[j] = tanhf(a.norm.alpha * v[j]) * wk[j] + (b ? b[k + j] : 0.0f);
            v[j] += rk[j];
            if (a.soft_cap > 0.0f) v[j] = a.soft_cap * tanhf(v[j] / a.soft_cap);
        }
        *reinterpret_cast<float4*>(a.out + (size_t)row * K + k) = make_float4(v[0], v[1], v[2], v[3]);
    }
}

bool wide_takes(const M40NormRows& a) {
    const uint32_t G = a.norm.kind == M40LLM_NORM_RMS && a.norm.groups ? a.norm.groups : 1u;
    const uintptr_t all = (uintptr_t)a.x | (uintptr_t)a.out | (uintptr_t)a.residual | (uintptr_t)a.norm.w;
    return a.norm.kind <= M40LLM_NORM_DYT && a.K <= 8192 && a.K % (G * 128u) == 0 && a.ldx % 4 == 0 && (all & 15u) == 0;
}

int launch_wide(M40llmCudaContext* ctx, cudaStream_t s, const M40NormRows& a, const M40NormGather& y) {
    const dim3 grid(a.rows), block(256);
    const cudaError_t e = a.K <= 2048   ? m40_launch_dependent(norm_rows_wide_kernel<2>, grid, block, 0, s, a, y)
                          : a.K <= 4096 ? m40_launch_dependent(norm_rows_wide_kernel<4>, grid, block, 0, s, a, y)
                                        : m40_launch_dependent(norm_rows_wide_kernel<8>, grid, block, 0, s, a, y);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

}  // namespace

bool m40_norm_valid(const M40llmNorm& n, uint32_t K) {
    if (n.kind > M40LLM_NORM_ACT) return false;
    if (n.kind == M40LLM_NORM_RMS && (!n.w || (n.groups && (K % n.groups != 0 || n.groups > MAX_GROUPS)))) return false;
    if (n.kind == M40LLM_NORM_POLY && !n.w) return false;
    return n.kind != M40LLM_NORM_ACT || n.act <= M40LLM_ACT_GELU_ERF;
}

bool m40_norm_gather_rows_takes(const M40NormRows& a, const M40NormGather& y) {
    return wide_takes(a) && y.slots > 0 && y.slots <= M40_NORM_SLOTS && (((uintptr_t)y.values | (uintptr_t)y.x) & 15u) == 0;
}

int m40_norm_gather_rows(M40llmCudaContext* ctx, cudaStream_t s, const M40NormRows& a, const M40NormGather& y) {
    return launch_wide(ctx, s, a, y);
}

int m40_norm_rows(M40llmCudaContext* ctx, cudaStream_t s, const M40NormRows& a) {
    if (wide_takes(a)) return launch_wide(ctx, s, a, M40NormGather{});
    const uint32_t G = a.norm.groups ? a.norm.groups : 1u;
    const size_t smem = a.norm.kind == M40LLM_NORM_RMS ? (size_t)G * ((G >= 8u ? 1u : 8u / G) + 1u) * sizeof(float) : 0;
    const cudaError_t e = m40_launch_dependent(norm_rows_kernel, dim3(a.rows), dim3(256), smem, s, a);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}
