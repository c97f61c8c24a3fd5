// Mixture of experts: m40llm_moe_async.
//
//   moe_route_kernel   warp = row: softmax over all outputs, group-limited choice on the corrected scores, weights;
//   moe_up_kernel      hid[row, slot] = act(up_e x), moe_down_kernel y[row] = sum_slot weight * down_e hid + identity + add:
//                      f32 multiply-adds on streamed weight rows, any shape. They serve one row (every chosen expert's weights
//                      are read once), the exact mode and the shapes the tensor path does not take;
//   tensor path          moe_sort_kernel deals the chosen slots to experts (rows sorted by expert, each expert's share padded to
//                      whole tiles) and writes the tile table, moe_scatter_kernel copies the rows there as hi + lo, two grouped
//                      GEMMs (gemm_tc_grouped.cu; act and the next split in the first one's epilogue). No host round trip: the table
//                      and its length stay on the device;
//   then post norm and residual (norm_rows.cu), after the tensor path together with adding a row's slots up (or, for shapes
//   that pass does not take, after moe_gather_kernel).
#include "moe.cuh"

#include <math.h>

#include "gemm_tc_grouped.cuh"
#include "norm_rows.cuh"

namespace {

constexpr uint32_t MAX_OUTPUTS = 1024, MAX_TOP = 32;
constexpr int ROUTE_WARPS = 4;
constexpr uint32_t TENSOR_ROWS = 2;               // rows from which the tensor path is taken
constexpr uint64_t PASS_SLOTS = 32768;            // slots of one pass of it

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

// One CTA. Slots are counted per expert, shares padded to tiles, tiles listed; then every slot draws its place. The order
// within a share follows from atomics, which changes no result: a row's values do not depend on its place.
__global__ void __launch_bounds__(1024) moe_sort_kernel(M40MoeArgs a) {
    extern __shared__ uint32_t count[];  // [experts] counts, then next places
    __shared__ uint32_t warp_sum_tiles[32], total_tiles;
    pdl_wait();
    pdl_trigger();
    const uint32_t tid = threadIdx.x, lane = tid & 31u, warp = tid >> 5, slots = a.rows * a.top, E = a.experts;
    for (uint32_t e = tid; e < E; e += 1024u) count[e] = 0u;
    __syncthreads();
    for (uint32_t i = tid; i < slots; i += 1024u) {
        const uint32_t e = a.ids[i];
        if (e < E) atomicAdd(&count[e], 1u);
    }
    __syncthreads();
    // exclusive sum of the experts' tiles; experts <= 1024: one per thread
    const uint32_t n = tid < E ? count[tid] : 0u, t = (n + a.tile_rows - 1u) / a.tile_rows;
    uint32_t inc = t;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const uint32_t v = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= (uint32_t)o) inc += v;
    }
    if (lane == 31u) warp_sum_tiles[warp] = inc;
    __syncthreads();
    if (warp == 0) {
        uint32_t w = warp_sum_tiles[lane], own = w;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const uint32_t v = __shfl_up_sync(0xffffffffu, w, o);
            if (lane >= (uint32_t)o) w += v;
        }
        warp_sum_tiles[lane] = w - own;
        if (lane == 31u) total_tiles = w;
    }
    __syncthreads();
    const uint32_t first = warp_sum_tiles[warp] + inc - t;
    if (tid < E) {
        count[tid] = first * a.tile_rows;
        for (uint32_t i = 0; i < t; ++i)
            a.tiles[first + i] = M40GroupTile{tid, (first + i) * a.tile_rows, min(a.tile_rows, n - i * a.tile_rows), 0u};
    }
    if (tid == 0) *a.n_tiles = total_tiles;
    __syncthreads();
    for (uint32_t i = tid; i < slots; i += 1024u) {
        const uint32_t e = a.ids[i];
        if (e < E) a.place[i] = atomicAdd(&count[e], 1u);
    }
}

// CTA = row: its hi and lo parts to every place that reads it.
template <typename T>
__global__ void __launch_bounds__(256) moe_scatter_kernel(M40MoeArgs a) {
    pdl_wait();
    pdl_trigger();
    const uint32_t row = blockIdx.x;
    const float* x = a.x + (size_t)row * a.K;
    for (uint32_t k = threadIdx.x * 4u; k < a.K; k += 1024u) {
        const float4 v = *reinterpret_cast<const float4*>(x + k);
        const float y[4] = {v.x, v.y, v.z, v.w};
        T h[4], l[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            h[i] = (T)y[i];
            l[i] = (T)(y[i] - m40_load_elem(&h[i]));
        }
        for (uint32_t j = 0; j < a.top; ++j) {
            if (a.ids[(size_t)row * a.top + j] >= a.experts) continue;
            const size_t at = (size_t)a.place[(size_t)row * a.top + j] * a.K + k;
            *reinterpret_cast<uint2*>(reinterpret_cast<T*>(a.xs[0]) + at) = *reinterpret_cast<const uint2*>(h);
            *reinterpret_cast<uint2*>(reinterpret_cast<T*>(a.xs[1]) + at) = *reinterpret_cast<const uint2*>(l);
        }
    }
}

// CTA = (row, 1024 columns): y = sum of the slots' results (in the slots' order) + identity + add.
__global__ void __launch_bounds__(256) moe_gather_kernel(M40MoeArgs a) {
    __shared__ float sw[MAX_TOP];
    __shared__ uint32_t sp[MAX_TOP];
    pdl_wait();
    pdl_trigger();
    const uint32_t row = blockIdx.y, k = blockIdx.x * 1024u + threadIdx.x * 4u;
    if (threadIdx.x < a.top) {
        const size_t i = (size_t)row * a.top + threadIdx.x;
        sw[threadIdx.x] = a.weights[i];
        sp[threadIdx.x] = a.ids[i] < a.experts ? a.place[i] : 0xffffffffu;
    }
    __syncthreads();
    if (k >= a.K) return;
    const size_t at = (size_t)row * a.K + k;
    const float4 x = *reinterpret_cast<const float4*>(a.x + at);
    float4 y = a.add ? *reinterpret_cast<const float4*>(a.add + at) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (uint32_t j = 0; j < a.top; ++j) {
        const float4 v = sp[j] == 0xffffffffu ? x : *reinterpret_cast<const float4*>(a.ys + (size_t)sp[j] * a.K + k);
        y.x = fmaf(sw[j], v.x, y.x), y.y = fmaf(sw[j], v.y, y.y), y.z = fmaf(sw[j], v.z, y.z), y.w = fmaf(sw[j], v.w, y.w);
    }
    *reinterpret_cast<float4*>(a.y + at) = y;
}

// Rows of a tile: the rows that all but the most crowded experts get (their mean and two standard deviations of an even
// routing), dealt to as few tiles of at most 64 as hold them. (128-row tiles measured no faster: three CTAs with small tiles
// hide each other's prologues and epilogues better than two with large ones.)
uint32_t pick_tile_rows(uint64_t slots, uint32_t outputs) {
    const double avg = (double)slots / outputs, most = avg + 2.0 * sqrt(avg);
    const uint32_t n = (uint32_t)ceil(most), tiles = (n + 63u) / 64u;
    const uint32_t rows = ((n + tiles - 1u) / tiles + 15u) / 16u * 16u;
    return rows < 16u ? 16u : (rows > 64u ? 64u : rows);
}

// `after`: the norm of these rows.
int run_tensor(M40llmCudaContext* ctx, cudaStream_t s, const M40MoeArgs& a, uint32_t max_tiles, M40NormRows after) {
    cudaError_t e = m40_launch_dependent(moe_sort_kernel, dim3(1), dim3(1024), a.experts * sizeof(uint32_t), s, a);
    M40_COUNT_LAUNCH(ctx);
    if (e != cudaSuccess) return -6;
    e = a.bf16 ? m40_launch_dependent(moe_scatter_kernel<__nv_bfloat16>, dim3(a.rows), dim3(256), 0, s, a)
               : m40_launch_dependent(moe_scatter_kernel<__half>, dim3(a.rows), dim3(256), 0, s, a);
    M40_COUNT_LAUNCH(ctx);
    if (e != cudaSuccess) return -6;
    M40GroupedCall c = {};
    c.w = a.up;
    c.x[0] = a.xs[0], c.x[1] = a.xs[1];
    c.parts = 2;
    c.bf16 = a.bf16;
    c.groups = a.experts;
    c.N = a.ff;
    c.K = c.ldx = a.K;
    c.x_rows = max_tiles * a.tile_rows;
    c.tile_rows = a.tile_rows;
    c.tiles = a.tiles;
    c.n_tiles = a.n_tiles;
    c.max_tiles = max_tiles;
    c.kind = M40_GROUPED_ACT_SPLIT;
    c.act = a.act;
    c.hi = a.hs[0], c.lo = a.hs[1];
    int rc = m40_gemm_tc_grouped(ctx, s, c);
    if (rc != 0) return rc;
    c.w = a.down;
    c.x[0] = a.hs[0], c.x[1] = a.hs[1];
    c.N = a.K;
    c.K = c.ldx = a.ff;
    c.kind = M40_GROUPED_F32;
    c.out = a.ys;
    if ((rc = m40_gemm_tc_grouped(ctx, s, c)) != 0) return rc;
    after.x = a.add;
    const M40NormGather y = {a.ys, a.x, a.weights, a.ids, a.place, a.top, a.experts};
    if (m40_norm_gather_rows_takes(after, y)) return m40_norm_gather_rows(ctx, s, after, y);
    e = m40_launch_dependent(moe_gather_kernel, dim3((a.K + 1023) / 1024, a.rows), dim3(256), 0, s, a);
    M40_COUNT_LAUNCH(ctx);
    if (e != cudaSuccess || cudaGetLastError() != cudaSuccess) return -6;
    after.x = a.y;
    return m40_norm_rows(ctx, s, after);
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

    a.bf16 = c->w_dtype == M40LLM_DT_BF16;
    const bool tensor = !c->exact && c->rows >= TENSOR_ROWS && c->w_dtype != M40LLM_DT_F32 && al16(c->x) && al16(c->add) &&
                        m40_gemm_tc_grouped_supported(c->up, c->ff, c->K, c->K, 0) &&
                        m40_gemm_tc_grouped_supported(c->down, c->K, c->ff, c->ff, 0);

    // level-1 arena: chosen ids, weights, sums; hidden values, or the sorted rows and their results (256-byte aligned pieces).
    // Rows go in passes whose slots fit the grid and whose sorted rows stay within a fixed work space.
    uint64_t pass = 65535u / c->top;
    if (tensor && pass > PASS_SLOTS / c->top) pass = PASS_SLOTS / c->top;
    if (pass > c->rows) pass = c->rows;
    const uint64_t slots = pass * c->top;
    a.tile_rows = pick_tile_rows(slots, (uint32_t)n);
    const uint32_t max_tiles = (uint32_t)(slots / a.tile_rows + (c->experts < slots ? c->experts : slots));
    const uint64_t sorted = (uint64_t)max_tiles * a.tile_rows;
    size_t used = 0;
    auto take = [&](size_t bytes) {
        const size_t at = used;
        used += (bytes + 255) & ~(size_t)255;
        return at;
    };
    const size_t at_ids = take((size_t)c->rows * c->top * 4), at_weights = take((size_t)c->rows * c->top * 4);
    const size_t at_y = take((size_t)c->rows * c->K * 4), at_hid = take(tensor ? 0 : slots * c->ff * 4);
    size_t at_place = 0, at_tiles = 0, at_n = 0, at_x[2] = {}, at_h[2] = {}, at_ys = 0;
    if (tensor) {
        at_place = take(slots * 4), at_tiles = take((size_t)max_tiles * sizeof(M40GroupTile)), at_n = take(4);
        for (int p = 0; p < 2; ++p) at_x[p] = take(sorted * c->K * 2), at_h[p] = take(sorted * c->ff * 2);
        at_ys = take(sorted * c->K * 4);
    }
    unsigned char* work = (unsigned char*)m40_ensure_scratch(ctx, stream_kind, used + 256, 1);
    if (!work) return -5;
    work = (unsigned char*)(((uintptr_t)work + 255) & ~(uintptr_t)255);
    a.ids = (uint32_t*)(work + at_ids);
    a.weights = (float*)(work + at_weights);
    a.y = (float*)(work + at_y);
    a.hid = (float*)(work + at_hid);
    a.place = (uint32_t*)(work + at_place);
    a.tiles = (M40GroupTile*)(work + at_tiles);
    a.n_tiles = (uint32_t*)(work + at_n);
    for (int p = 0; p < 2; ++p) a.xs[p] = work + at_x[p], a.hs[p] = work + at_h[p];
    a.ys = (float*)(work + at_ys);

    const size_t smem = (size_t)ROUTE_WARPS * (2 * n + G) * sizeof(float);
    cudaError_t e = m40_launch_dependent(moe_route_kernel, dim3((c->rows + ROUTE_WARPS - 1) / ROUTE_WARPS), dim3(32 * ROUTE_WARPS), smem, s, a);
    M40_COUNT_LAUNCH(ctx);
    if (e != cudaSuccess) return -6;
    for (uint32_t at = 0; at < c->rows; at += (uint32_t)pass) {
        M40MoeArgs p = a;
        p.rows = c->rows - at < pass ? c->rows - at : (uint32_t)pass;
        p.x += (size_t)at * c->K;
        if (p.add) p.add += (size_t)at * c->K;
        p.y += (size_t)at * c->K;
        p.ids += (size_t)at * c->top;
        p.weights += (size_t)at * c->top;
        const M40NormRows after = {p.y, (float*)c->out + (size_t)at * c->K, c->residual ? (const float*)c->residual + (size_t)at * c->K : nullptr,
                             c->post, p.rows, c->K, c->K, 0.0f};
        if (tensor) {
            const int rc = run_tensor(ctx, s, p, max_tiles, after);
            if (rc != 0) return rc;
            continue;
        }
        int rc = c->w_dtype == M40LLM_DT_F32 ? run_rows<float>(ctx, s, p)
                       : c->w_dtype == M40LLM_DT_BF16 ? run_rows<__nv_bfloat16>(ctx, s, p) : run_rows<__half>(ctx, s, p);
        if (rc == 0) rc = m40_norm_rows(ctx, s, after);
        if (rc != 0) return rc;
    }
    return 0;
}
