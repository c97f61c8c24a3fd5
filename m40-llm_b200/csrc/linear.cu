// m40llm_linear_async: one projection with its norm before and its elementwise tail after, for any of three routes:
//   one row      the weight-streaming GEMV (gemv_stream.cu), norm, activation and tail folded into the launch;
//   more rows    the tcgen05 GEMM (gemm_tc.cu), norm folded into the 16-bit hi/lo split, tail into the epilogue;
//   f32          the kernels below: f32 multiply-adds only. They are the exact mode and take every shape and alignment.
// Norms that a route does not fold in (grouped RMS; any norm on the f32 route) and an RMS norm of the result, which needs
// whole rows, run as passes of norm_rows.cu.
#include "common.cuh"
#include "gemm.cuh"
#include "gemm_tc.cuh"
#include "gemv_stream.cuh"
#include "norm_rows.cuh"
#include "stack_math.cuh"

namespace {

struct F32Args {
    const float* x;
    const void* w;
    const void* w2;
    float* out;
    const float* bias;
    const float* residual;
    const float* post_w;
    const float* post_b;
    uint32_t M, N, K, ldx;
    int act;
    M40Tail tail;
};

__device__ __forceinline__ void f32_finish(const F32Args& a, uint32_t m, uint32_t n, float y, float y2) {
    if (a.w2) y = m40_act(a.act, y) * y2;
    const size_t at = (size_t)m * a.N + n;
    a.out[at] = m40_tail(a.tail, y, a.bias ? a.bias[n] : 0.0f, a.post_w ? a.post_w[n] : 1.0f, a.post_b ? a.post_b[n] : 0.0f,
                         a.residual ? a.residual[at] : 0.0f);
}

// A few rows: one warp per weight row (pair), lanes stride K.
template <typename WT, int MT>
__global__ void __launch_bounds__(256) linear_f32_rows_kernel(F32Args a) {
    pdl_wait();
    pdl_trigger();
    const uint32_t n = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31u;
    if (n >= a.N) return;
    const WT* w = reinterpret_cast<const WT*>(a.w) + (size_t)n * a.K;
    const WT* w2 = a.w2 ? reinterpret_cast<const WT*>(a.w2) + (size_t)n * a.K : nullptr;
    const uint32_t m0 = blockIdx.y * MT;
    float acc[MT] = {}, acc2[MT] = {};
    for (uint32_t k = lane; k < a.K; k += 32u) {
        const float wk = m40_load_elem(w + k), uk = w2 ? m40_load_elem(w2 + k) : 0.0f;
#pragma unroll
        for (int i = 0; i < MT; ++i) {
            const float xv = a.x[(size_t)min(m0 + i, a.M - 1u) * a.ldx + k];
            acc[i] = fmaf(xv, wk, acc[i]);
            acc2[i] = fmaf(xv, uk, acc2[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < MT; ++i) {
        const float y = warp_sum(acc[i]), y2 = w2 ? warp_sum(acc2[i]) : 0.0f;
        if (lane == 0 && m0 + i < a.M) f32_finish(a, m0 + i, n, y, y2);
    }
}

// Many rows: 64 x 64 output tile, 16-deep k tiles in shared memory, 4 x 4 outputs per thread. A k tile is summed on its own
// before it joins the running sum, so that the rounding error grows with K / 16, not K.
template <typename WT>
__global__ void __launch_bounds__(256) linear_f32_tile_kernel(F32Args a) {
    constexpr int BM = 64, BN = 64, BK = 16;
    __shared__ float sx[BK][BM + 4], sw[BK][BN + 4], su[BK][BN + 4];
    pdl_wait();
    pdl_trigger();
    const uint32_t tid = threadIdx.x, m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
    const uint32_t tm = (tid >> 4) * 4u, tn = (tid & 15u) * 4u;
    const WT* w = reinterpret_cast<const WT*>(a.w);
    const WT* w2 = reinterpret_cast<const WT*>(a.w2);
    float acc[4][4] = {}, acc2[4][4] = {};
    for (uint32_t k0 = 0; k0 < a.K; k0 += BK) {
#pragma unroll
        for (int i = 0; i < (BM * BK) / 256; ++i) {
            const uint32_t e = tid + i * 256u, r = e / BK, kk = e % BK, k = k0 + kk;
            sx[kk][r] = (m0 + r < a.M && k < a.K) ? a.x[(size_t)(m0 + r) * a.ldx + k] : 0.0f;
            const bool in = n0 + r < a.N && k < a.K;
            sw[kk][r] = in ? m40_load_elem(w + (size_t)(n0 + r) * a.K + k) : 0.0f;
            if (w2) su[kk][r] = in ? m40_load_elem(w2 + (size_t)(n0 + r) * a.K + k) : 0.0f;
        }
        __syncthreads();
        float part[4][4] = {}, part2[4][4] = {};
#pragma unroll
        for (int kk = 0; kk < BK; ++kk) {
            const float4 xv = *reinterpret_cast<const float4*>(&sx[kk][tm]);
            const float4 wv = *reinterpret_cast<const float4*>(&sw[kk][tn]);
            const float xa[4] = {xv.x, xv.y, xv.z, xv.w}, wa[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) part[i][j] = fmaf(xa[i], wa[j], part[i][j]);
            if (w2) {
                const float4 uv = *reinterpret_cast<const float4*>(&su[kk][tn]);
                const float ua[4] = {uv.x, uv.y, uv.z, uv.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) part2[i][j] = fmaf(xa[i], ua[j], part2[i][j]);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j], acc2[i][j] += part2[i][j];
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (m0 + tm + i < a.M && n0 + tn + j < a.N) f32_finish(a, m0 + tm + i, n0 + tn + j, acc[i][j], acc2[i][j]);
}

template <typename WT>
int launch_f32(M40llmCudaContext* ctx, cudaStream_t s, const F32Args& a) {
    cudaError_t e;
    if (a.M <= 8) {
        const dim3 grid((a.N + 7) / 8, (a.M + 3) / 4);
        e = a.M == 1 ? m40_launch_dependent(linear_f32_rows_kernel<WT, 1>, grid, dim3(256), 0, s, a)
                     : m40_launch_dependent(linear_f32_rows_kernel<WT, 4>, grid, dim3(256), 0, s, a);
    } else {
        e = m40_launch_dependent(linear_f32_tile_kernel<WT>, dim3((a.N + 63) / 64, (a.M + 63) / 64), dim3(256), 0, s, a);
    }
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

bool al16(const void* p) { return (((uintptr_t)p) & 15u) == 0u; }

bool tc_takes(const M40llmLinear& c) {
    const void* wp[2] = {c.w, c.w2};
    const bool tail_used = c.post.kind != M40LLM_NORM_NONE || c.soft_cap > 0.0f || c.bias || c.residual;
    return c.rows >= 2 && (!c.w2 || !tail_used) && al16(c.x) && c.ldx % 4 == 0 &&
           m40_gemm_tc_supported(c.rows > 256 ? 256 : (int)c.rows, (int)c.K, c.w2 ? 2 : 1, wp);
}

// Whether the route the call takes applies its norm of x itself. (The streaming kernel declines a few shapes only when it is
// called; project() then runs the norm as a pass.)
bool folds_norm(const M40llmLinear& c) {
    if (c.exact || c.w_dtype == M40LLM_DT_F32 || (c.pre.kind == M40LLM_NORM_RMS && c.pre.groups > 1)) return false;
    if (c.pre.kind <= M40LLM_NORM_DYT && (!al16(c.pre.w) || !al16(c.pre.b))) return false;
    return c.rows == 1 ? c.K % 8 == 0 && al16(c.x) : tc_takes(c);
}

// The projection itself: pre is NONE or one that the route folds in, post NONE or DYT.
int project(M40llmCudaContext* ctx, cudaStream_t s, uint32_t stream_kind, const M40llmLinear& c) {
    const M40Tail tail = {(int)c.post.kind, c.post.alpha, c.soft_cap};
    const float *post_w = (const float*)c.post.w, *post_b = (const float*)c.post.b;
    const float *bias = (const float*)c.bias, *residual = (const float*)c.residual;
    M40GemvNorm norm = {};
    norm.w = c.pre.kind == M40LLM_NORM_ACT ? nullptr : c.pre.w;
    norm.w_is_f32 = 1;
    norm.eps = c.pre.eps;
    norm.dyt = c.pre.kind == M40LLM_NORM_DYT ? 1 : 0;
    norm.alpha = c.pre.alpha;
    norm.b = (const float*)c.pre.b;
    norm.special = c.pre.kind >= M40LLM_NORM_POLY ? (int)c.pre.kind : 0;
    norm.act = (int)c.pre.act;
    const M40GemvNorm* np = c.pre.kind != M40LLM_NORM_NONE ? &norm : nullptr;
    const bool fast = !c.exact && c.w_dtype != M40LLM_DT_F32;

    if (fast && c.rows == 1) {
        const M40GemvSeg seg = {c.w, c.w2, (float*)c.out, bias, residual, (int)c.N, post_w, post_b};
        const M40GemvExt ext = {(int)c.act, tail};
        const int rc = m40_gemv_stream(ctx, s, (const float*)c.x, (int)c.K,
                                       c.w_dtype == M40LLM_DT_BF16 ? M40_GEMV_BF16 : M40_GEMV_F16, c.w2 ? 1 : 0, 1, &seg, np, &ext);
        if (rc != 1) return rc;
    }
    if (fast && tc_takes(c)) {
        M40TcExt ext = {};
        ext.bf16 = c.w_dtype == M40LLM_DT_BF16 ? 1 : 0;
        ext.ldx = (int)c.ldx;
        ext.act = (int)c.act;
        ext.tail = tail;
        ext.post_w = post_w;
        ext.post_b = post_b;
        const __half* w[2] = {(const __half*)c.w, (const __half*)c.w2};
        const int n[2] = {(int)c.N, (int)c.N};
        float* o[2] = {(float*)c.out, nullptr};
        const float* b[2] = {bias, nullptr};
        const float* r[2] = {residual, nullptr};
        return m40_gemm_tc_f16(ctx, s, stream_kind, (const float*)c.x, (int)c.rows, (int)c.K, c.w2 ? 2 : 1, w, n, o, b, r,
                               c.w2 ? 1 : 0, np, nullptr, &ext);
    }

    F32Args a = {};
    a.x = (const float*)c.x;
    a.ldx = c.ldx;
    if (np) {
        float* xn = (float*)m40_ensure_scratch(ctx, stream_kind, (size_t)c.rows * c.K * sizeof(float));
        if (!xn) return -5;
        const M40NormRows first = {a.x, xn, nullptr, c.pre, c.rows, c.K, c.ldx, 0.0f};
        const int rc = m40_norm_rows(ctx, s, first);
        if (rc != 0) return rc;
        a.x = xn;
        a.ldx = c.K;
    }
    a.w = c.w;
    a.w2 = c.w2;
    a.out = (float*)c.out;
    a.bias = bias;
    a.residual = residual;
    a.post_w = post_w;
    a.post_b = post_b;
    a.M = c.rows;
    a.N = c.N;
    a.K = c.K;
    a.act = (int)c.act;
    a.tail = tail;
    if (c.w_dtype == M40LLM_DT_F32) return launch_f32<float>(ctx, s, a);
    return c.w_dtype == M40LLM_DT_BF16 ? launch_f32<__nv_bfloat16>(ctx, s, a) : launch_f32<__half>(ctx, s, a);
}

}  // namespace

extern "C" int m40llm_linear_async(M40llmCudaContext* ctx, const M40llmLinear* call, uint32_t stream_kind) {
    if (!ctx || !call || !call->x || !call->w || !call->out || stream_kind > 1) return -1;
    if (call->rows == 0 || call->K == 0 || call->N == 0) return -2;
    if (call->w_dtype > M40LLM_DT_BF16 || call->act > M40LLM_ACT_GELU_ERF) return -3;
    if (!m40_norm_valid(call->pre, call->K) || !m40_norm_valid(call->post, call->N)) return -4;
    if (call->post.kind > M40LLM_NORM_DYT) return -4;
    M40llmLinear c = *call;
    if (c.ldx == 0) c.ldx = c.K;
    if (c.ldx < c.K) return -2;
    if (m40_ensure_device(ctx) != 0) return -1;
    cudaStream_t s = m40_stream(ctx, stream_kind);

    // passes of their own: rows of pre(x), rows of the plain result (level-1 arena: this is a composite call)
    const bool rms_after = c.post.kind == M40LLM_NORM_RMS;
    const bool norm_first = c.pre.kind != M40LLM_NORM_NONE && !folds_norm(c);
    const size_t pre_elems = norm_first ? ((size_t)c.rows * c.K + 3) & ~(size_t)3 : 0;
    const size_t post_elems = rms_after ? (size_t)c.rows * c.N : 0;
    float* work = nullptr;
    if (pre_elems + post_elems) {
        work = (float*)m40_ensure_scratch(ctx, stream_kind, (pre_elems + post_elems) * sizeof(float), 1);
        if (!work) return -5;
    }
    if (norm_first) {
        const M40NormRows first = {(const float*)c.x, work, nullptr, c.pre, c.rows, c.K, c.ldx, 0.0f};
        const int rc = m40_norm_rows(ctx, s, first);
        if (rc != 0) return rc;
        c.x = work;
        c.ldx = c.K;
        c.pre = M40llmNorm{};
    }
    if (!rms_after) return project(ctx, s, stream_kind, c);
    const M40NormRows after = {work + pre_elems, (float*)c.out, (const float*)c.residual, c.post, c.rows, c.N, c.N, c.soft_cap};
    c.out = work + pre_elems;
    c.residual = nullptr;
    c.post = M40llmNorm{};
    c.soft_cap = 0.0f;
    const int rc = project(ctx, s, stream_kind, c);
    return rc != 0 ? rc : m40_norm_rows(ctx, s, after);
}
