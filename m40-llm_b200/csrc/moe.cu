// Mixture of experts: m40llm_moe_async.
//
//   moe_route_kernel   warp = row: softmax over all outputs, group-limited choice on the corrected scores, weights;
//   moe_up_kernel      hid[row, slot] = act(up_e x), moe_down_kernel y[row] = sum_slot weight * down_e hid + identity + add:
//                      f32 multiply-adds on streamed weight rows, any shape. They serve one row (every chosen expert's weights
//                      are read once), the exact mode and the shapes the tensor path does not take;
//   then post norm and residual (norm_rows.cu).
#include "moe.cuh"

#include "norm_rows.cuh"

namespace {

constexpr uint32_t MAX_OUTPUTS = 1024, MAX_TOP = 32;
constexpr int ROUTE_WARPS = 4;

// Largest value of v[0 .. n) and the lowest index that holds it, over the warp.
__device__ __forceinline__ uint32_t warp_argmax(const float* v, uint32_t n, uint32_t lane) {
    float best = -INFINITY;
    uint32_t at = n;
    for (uint32_t i = lane; i < n; i += 32u)
        if (v[i] > best) best = v[i], at = i;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float b2 = __shfl_xor_sync(0xffffffffu, best, o);
        const uint32_t a2 = __shfl_xor_sync(0xffffffffu, at, o);
        if (b2 > best || (b2 == best && a2 < at)) best = b2, at = a2;
    }
    return min(at, n - 1u);
}

__global__ void __launch_bounds__(32 * ROUTE_WARPS) moe_route_kernel(M40MoeArgs a) {
    extern __shared__ float sh[];  // per warp: scores [n], choice [n], groups [groups]
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, row = blockIdx.x * ROUTE_WARPS + warp;
    const uint32_t n = a.experts + a.identity, G = a.groups > 1u ? a.groups : 1u;
    float* s = sh + warp * (2u * n + G);
    float* choice = s + n;
    float* best = choice + n;
    pdl_wait();
    pdl_trigger();
    if (row >= a.rows) return;
    const float* z = a.logits + (size_t)row * a.ld_logits;
    float mx = -INFINITY;
    for (uint32_t i = lane; i < n; i += 32u) mx = fmaxf(mx, s[i] = z[i]);
    mx = warp_max(mx);
    float sum = 0.0f;
    for (uint32_t i = lane; i < n; i += 32u) sum += s[i] = expf(s[i] - mx);
    sum = warp_sum(sum);
    for (uint32_t i = lane; i < n; i += 32u) {
        s[i] = s[i] / sum;
        choice[i] = s[i] + (a.correction ? a.correction[i] : 0.0f);
    }
    __syncwarp();
    if (G > 1u) {
        const uint32_t per = n / G;
        for (uint32_t g = lane; g < G; g += 32u) {
            float m = -INFINITY;
            for (uint32_t i = 0; i < per; ++i) m = fmaxf(m, choice[g * per + i]);
            best[g] = m;
        }
        __syncwarp();
        // kept groups are marked by +inf, which no score reaches; the marking does not disturb the order of the others
        for (uint32_t k = 0; k < a.keep; ++k) {
            float b = -INFINITY;
            uint32_t at = G;
            for (uint32_t g = lane; g < G; g += 32u)
                if (best[g] < INFINITY && best[g] > b) b = best[g], at = g;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float b2 = __shfl_xor_sync(0xffffffffu, b, o);
                const uint32_t a2 = __shfl_xor_sync(0xffffffffu, at, o);
                if (b2 > b || (b2 == b && a2 < at)) b = b2, at = a2;
            }
            if (lane == 0 && at < G) best[at] = INFINITY;
            __syncwarp();
        }
        for (uint32_t i = lane; i < n; i += 32u)
            if (best[i / per] < INFINITY) choice[i] = -INFINITY;
        __syncwarp();
    }
    float w_own = 0.0f, total = 0.0f;
    uint32_t id_own = 0;
    for (uint32_t k = 0; k < a.top; ++k) {
        const uint32_t e = warp_argmax(choice, n, lane);
        const float w = s[e];
        total += w;
        if (lane == k) w_own = w, id_own = e;
        __syncwarp();
        if (lane == 0) choice[e] = -INFINITY;
        __syncwarp();
    }
    if (lane < a.top) {
        a.ids[(size_t)row * a.top + lane] = id_own;
        a.weights[(size_t)row * a.top + lane] = w_own / (total + 1e-20f) * a.scale;
    }
}

// dot of one weight row with x (f32, in shared or global memory), the warp's lanes striding K
template <typename WT, int NR>
__device__ __forceinline__ void row_dots(const WT* w, size_t pitch, const float* x, uint32_t K, bool wide, uint32_t lane, float* acc) {
    if (wide) {
#pragma unroll 2
        for (uint32_t k = lane * 8u; k < K; k += 256u) {
            float wv[NR][8];
#pragma unroll
            for (int j = 0; j < NR; ++j) m40_load8(w + (size_t)j * pitch + k, wv[j]);
            const float4 x0 = *reinterpret_cast<const float4*>(x + k), x1 = *reinterpret_cast<const float4*>(x + k + 4);
            const float xv[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
            for (int j = 0; j < NR; ++j) {
                float p = 0.0f;
#pragma unroll
                for (int i = 0; i < 8; ++i) p = fmaf(wv[j][i], xv[i], p);
                acc[j] += p;
            }
        }
    } else {
        for (uint32_t k = lane; k < K; k += 32u)
#pragma unroll
            for (int j = 0; j < NR; ++j) acc[j] = fmaf(m40_load_elem(w + (size_t)j * pitch + k), x[k], acc[j]);
    }
}

// grid (ff / 8 warps / NR rows, rows * top)
template <typename WT, int NR>
__global__ void __launch_bounds__(256) moe_up_kernel(M40MoeArgs a) {
    pdl_wait();
    pdl_trigger();
    const uint32_t slot = blockIdx.y, e = a.ids[slot], lane = threadIdx.x & 31u;
    const uint32_t n0 = (blockIdx.x * 8u + (threadIdx.x >> 5)) * NR;
    if (e >= a.experts || n0 >= a.ff) return;
    const float* x = a.x + (size_t)(slot / a.top) * a.K;
    const WT* w = reinterpret_cast<const WT*>(a.up) + (size_t)e * a.ff * a.K;
    if (n0 + NR <= a.ff) {
        float acc[NR] = {};
        row_dots<WT, NR>(w + (size_t)n0 * a.K, a.K, x, a.K, a.wide_up, lane, acc);
#pragma unroll
        for (int j = 0; j < NR; ++j) {
            const float v = warp_sum(acc[j]);
            if (lane == 0) a.hid[(size_t)slot * a.ff + n0 + j] = m40_act(a.act, v);
        }
    } else {
        for (uint32_t n = n0; n < a.ff; ++n) {
            float acc = 0.0f;
            row_dots<WT, 1>(w + (size_t)n * a.K, a.K, x, a.K, a.wide_up, lane, &acc);
            const float v = warp_sum(acc);
            if (lane == 0) a.hid[(size_t)slot * a.ff + n] = m40_act(a.act, v);
        }
    }
}

// grid (K / 8 warps, rows): warp = output
template <typename WT>
__global__ void __launch_bounds__(256) moe_down_kernel(M40MoeArgs a) {
    pdl_wait();
    pdl_trigger();
    const uint32_t row = blockIdx.y, n = blockIdx.x * 8u + (threadIdx.x >> 5), lane = threadIdx.x & 31u;
    if (n >= a.K) return;
    const size_t at = (size_t)row * a.K + n;
    float y = 0.0f, own = 0.0f;
#pragma unroll 2
    for (uint32_t k = 0; k < a.top; ++k) {
        const uint32_t slot = row * a.top + k, e = a.ids[slot];
        const float w = a.weights[slot];
        if (e >= a.experts) {
            own += w;
            continue;
        }
        float acc = 0.0f;
        row_dots<WT, 1>(reinterpret_cast<const WT*>(a.down) + ((size_t)e * a.K + n) * a.ff, 0, a.hid + (size_t)slot * a.ff, a.ff,
                        a.wide_down, lane, &acc);
        y = fmaf(w, acc, y);
    }
    y = warp_sum(y);
    if (lane == 0) a.y[at] = fmaf(own, a.x[at], y) + (a.add ? a.add[at] : 0.0f);
}

template <typename WT>
int run_rows(M40llmCudaContext* ctx, cudaStream_t s, const M40MoeArgs& a) {
    constexpr int NR = 2;
    cudaError_t e = m40_launch_dependent(moe_up_kernel<WT, NR>, dim3((a.ff + 8 * NR - 1) / (8 * NR), a.rows * a.top), dim3(256), 0, s, a);
    M40_COUNT_LAUNCH(ctx);
    if (e != cudaSuccess) return -6;
    e = m40_launch_dependent(moe_down_kernel<WT>, dim3((a.K + 7) / 8, a.rows), dim3(256), 0, s, a);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

bool al16(const void* p) { return (((uintptr_t)p) & 15u) == 0u; }

}  // namespace

extern "C" int m40llm_moe_async(M40llmCudaContext* ctx, const M40llmMoe* c, uint32_t stream_kind) {
    if (!ctx || !c || !c->x || !c->logits || !c->up || !c->down || !c->out || stream_kind > 1) return -1;
    const uint64_t n = (uint64_t)c->experts + c->identity, G = c->groups > 1 ? c->groups : 1;
    if (c->rows == 0 || c->K == 0 || c->ff == 0 || c->experts == 0 || n > MAX_OUTPUTS || c->ld_logits < n) return -2;
    if (c->top == 0 || c->top > MAX_TOP || (uint64_t)c->rows * c->top > 65535u * 64ull) return -2;
    if (n % G != 0 || (G > 1 && (c->keep == 0 || c->keep > G)) || c->top > (G > 1 ? c->keep * (n / G) : n)) return -2;
    if (c->w_dtype > M40LLM_DT_BF16 || c->act > M40LLM_ACT_GELU_ERF) return -3;
    if (c->post.kind > M40LLM_NORM_DYT || !m40_norm_valid(c->post, c->K)) return -4;
    if (m40_ensure_device(ctx) != 0) return -1;
    cudaStream_t s = m40_stream(ctx, stream_kind);

    M40MoeArgs a = {};
    a.x = (const float*)c->x;
    a.logits = (const float*)c->logits;
    a.correction = (const float*)c->correction;
    a.up = c->up;
    a.down = c->down;
    a.add = (const float*)c->add;
    a.K = c->K;
    a.ff = c->ff;
    a.experts = c->experts;
    a.identity = c->identity;
    a.top = c->top;
    a.groups = (uint32_t)G;
    a.keep = c->keep;
    a.ld_logits = c->ld_logits;
    a.act = (int)c->act;
    a.scale = c->scale;
    a.wide_up = c->w_dtype != M40LLM_DT_F32 && c->K % 8 == 0 && al16(c->up) && al16(c->x);
    a.wide_down = c->w_dtype != M40LLM_DT_F32 && c->ff % 8 == 0 && al16(c->down);
    a.rows = c->rows;

    // level-1 arena: chosen ids, weights, sums, hidden values (16-byte aligned pieces). Rows go in passes whose slots fit the
    // grid.
    const uint32_t pass = 65535u / c->top < c->rows ? 65535u / c->top : c->rows;
    auto pad = [](size_t v) { return (v + 3) & ~(size_t)3; };
    const size_t n_sel = pad((size_t)c->rows * c->top), n_y = pad((size_t)c->rows * c->K), n_hid = (size_t)pass * c->top * c->ff;
    float* work = (float*)m40_ensure_scratch(ctx, stream_kind, (2 * n_sel + n_y + n_hid) * sizeof(float), 1);
    if (!work) return -5;
    a.ids = (uint32_t*)work;
    a.weights = work + n_sel;
    a.y = work + 2 * n_sel;
    a.hid = a.y + n_y;

    const size_t smem = (size_t)ROUTE_WARPS * (2 * n + G) * sizeof(float);
    cudaError_t e = m40_launch_dependent(moe_route_kernel, dim3((c->rows + ROUTE_WARPS - 1) / ROUTE_WARPS), dim3(32 * ROUTE_WARPS), smem, s, a);
    M40_COUNT_LAUNCH(ctx);
    if (e != cudaSuccess) return -6;
    for (uint32_t at = 0; at < c->rows; at += pass) {
        M40MoeArgs p = a;
        p.rows = c->rows - at < pass ? c->rows - at : pass;
        p.x += (size_t)at * c->K;
        if (p.add) p.add += (size_t)at * c->K;
        p.y += (size_t)at * c->K;
        p.ids += (size_t)at * c->top;
        p.weights += (size_t)at * c->top;
        const int rc = c->w_dtype == M40LLM_DT_F32 ? run_rows<float>(ctx, s, p)
                       : c->w_dtype == M40LLM_DT_BF16 ? run_rows<__nv_bfloat16>(ctx, s, p) : run_rows<__half>(ctx, s, p);
        if (rc != 0) return rc;
    }
    const M40NormRows after = {a.y, (float*)c->out, (const float*)c->residual, c->post, c->rows, c->K, c->K, 0.0f};
    return m40_norm_rows(ctx, s, after);
}
