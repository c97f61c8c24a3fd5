// Generalised delta rule: a recurrent mixer whose state is one matrix per head,
//   S <- diag(w) S - (a * u) (u^T S) + k v^T,   o = S^T r,
// with a decay w and a removal rate a per head and key channel, u the unit key. All of it is f32.
//
// With k = n u (n the key's length) the update of one value column s of S is
//   d = u . s,   s_i <- w_i s_i + u_i (n v - a_i d),   o = r . s,
// so columns are independent and a token costs one dot product, one update and one dot product per column. Four lanes
// share a column (16-byte pieces of the key dimension dealt round-robin), the state stays in registers, and the only
// serial chain is d: 4 * NI / 4 multiply-adds, two shuffles, the update. The second dot product of token t overlaps the
// first of token t + 1.
//
//   delta_scan_kernel    portions of several tokens: CTA = (32 columns, head, segment), four consumer warps walk the tokens
//                        while four producer warps make the next chunk's vectors (gates, decays, unit keys) in shared
//                        memory and fetch the raw values of the one after it; delta_finish_kernel then applies the per-head norm and the output gate.
//   delta_decode_kernel  one token per sequence: CTA = (head, row) does everything, the low-rank decay projection
//                        included, in one launch; bound by reading and writing the state once.
// A chunked (matrix-product) form is not used: its products of decays and of removals would have to leave f32, or lose the
// property that the result does not depend on where a portion was cut.
#include <stdlib.h>

#include "common.cuh"
#include "stack_math.cuh"

struct M40llmStateCache {
    int device_id;
    uint32_t slots, heads, dim;
    float* d_state;  // [slot][head][value][key]
};

namespace {

constexpr int LANES = 4;             // lanes per column
constexpr int SCAN_COLS = 32;        // columns per scan CTA
constexpr int SCAN_CONSUMERS = SCAN_COLS * LANES;
constexpr int SCAN_PRODUCERS = 128;
constexpr int CHUNK = 16;            // tokens per ring buffer

struct DeltaArgs {
    const float* packed;
    const void* w2;
    const float* w0;
    const float* a_bias;
    const float* norm;
    const float* decay_in;
    float* out;
    float* state;
    uint32_t* status;
    const uint32_t* row_seq;
    const uint32_t* row_pos;
    const uint32_t* seg;
    uint32_t ld, rank, w2_dtype, heads, dim, slots, slot_mul, slot_add, rows;
    float decay_scale, unit_eps, eps;
};

__device__ __forceinline__ float w2_elem(const DeltaArgs& a, size_t i) {
    if (a.w2_dtype == M40LLM_DT_BF16) return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(a.w2)[i]);
    if (a.w2_dtype == M40LLM_DT_F16) return __half2float(reinterpret_cast<const __half*>(a.w2)[i]);
    return reinterpret_cast<const float*>(a.w2)[i];
}
__device__ __forceinline__ float decay_of(const DeltaArgs& a, float z) { return expf(a.decay_scale * m40_sigmoid(z)); }

// State of one column: elements 4 (lane4 + LANES i) .. + 3 of the key dimension.
template <int NI>
__device__ __forceinline__ void load_column(const float* col, uint32_t dim, uint32_t l4, bool zero, float4 (&s)[NI]) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const uint32_t k = 4u * (l4 + LANES * i);
        s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (zero || k >= dim) continue;
        if (dim % 4u == 0u) {
            s[i] = *reinterpret_cast<const float4*>(col + k);
        } else {
            s[i].x = col[k];
            if (k + 1 < dim) s[i].y = col[k + 1];
            if (k + 2 < dim) s[i].z = col[k + 2];
            if (k + 3 < dim) s[i].w = col[k + 3];
        }
    }
}
template <int NI>
__device__ __forceinline__ void store_column(float* col, uint32_t dim, uint32_t l4, const float4 (&s)[NI]) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const uint32_t k = 4u * (l4 + LANES * i);
        if (k >= dim) continue;
        if (dim % 4u == 0u) {
            *reinterpret_cast<float4*>(col + k) = s[i];
        } else {
            col[k] = s[i].x;
            if (k + 1 < dim) col[k + 1] = s[i].y;
            if (k + 2 < dim) col[k + 2] = s[i].z;
            if (k + 3 < dim) col[k + 3] = s[i].w;
        }
    }
}

// One token on one column: vec = [w | u | a | r], each DP floats (zero beyond dim); nv = n * v of this column. Returns o,
// the same in all LANES lanes.
template <int NI>
__device__ __forceinline__ float delta_token(const float* vec, uint32_t l4, float nv, float4 (&s)[NI]) {
    constexpr int DP = NI * LANES * 4;
    const float4* w = reinterpret_cast<const float4*>(vec) + l4;
    const float4* u = reinterpret_cast<const float4*>(vec + DP) + l4;
    const float4* a = reinterpret_cast<const float4*>(vec + 2 * DP) + l4;
    const float4* r = reinterpret_cast<const float4*>(vec + 3 * DP) + l4;
    float4 uu[NI];
    float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        uu[i] = u[LANES * i];
        d0 = fmaf(uu[i].x, s[i].x, d0), d1 = fmaf(uu[i].y, s[i].y, d1);
        d2 = fmaf(uu[i].z, s[i].z, d2), d3 = fmaf(uu[i].w, s[i].w, d3);
    }
    float d = (d0 + d1) + (d2 + d3);
    d += __shfl_xor_sync(0xffffffffu, d, 1);
    d += __shfl_xor_sync(0xffffffffu, d, 2);
    float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const float4 wi = w[LANES * i], ai = a[LANES * i], ri = r[LANES * i];
        s[i].x = fmaf(uu[i].x, fmaf(-ai.x, d, nv), wi.x * s[i].x);
        s[i].y = fmaf(uu[i].y, fmaf(-ai.y, d, nv), wi.y * s[i].y);
        s[i].z = fmaf(uu[i].z, fmaf(-ai.z, d, nv), wi.z * s[i].z);
        s[i].w = fmaf(uu[i].w, fmaf(-ai.w, d, nv), wi.w * s[i].w);
        o0 = fmaf(ri.x, s[i].x, o0), o1 = fmaf(ri.y, s[i].y, o1);
        o2 = fmaf(ri.z, s[i].z, o2), o3 = fmaf(ri.w, s[i].w, o3);
    }
    float o = (o0 + o1) + (o2 + o3);
    o += __shfl_xor_sync(0xffffffffu, o, 1);
    o += __shfl_xor_sync(0xffffffffu, o, 2);
    return o;
}

// grid (column blocks, heads, segments), block SCAN_CONSUMERS + SCAN_PRODUCERS; dynamic smem 2 * CHUNK * (4 DP + SCAN_COLS).
template <int NI>
__global__ void __launch_bounds__(SCAN_CONSUMERS + SCAN_PRODUCERS) delta_scan_kernel(DeltaArgs a) {
    constexpr int DP = NI * LANES * 4;
    constexpr int TOK = 4 * DP + SCAN_COLS;  // floats per staged token
    constexpr int CPL = (DP + 31) / 32;      // channels per producer lane
    extern __shared__ __align__(16) float ring[];
    pdl_wait();
    pdl_trigger();
    const uint32_t head = blockIdx.y, col0 = blockIdx.x * SCAN_COLS, D = a.dim, HD = a.heads * D;
    const uint32_t row0 = a.seg[4 * blockIdx.z], n = a.seg[4 * blockIdx.z + 1];
    const uint32_t slot = a.seg[4 * blockIdx.z + 2] * a.slot_mul + a.slot_add, pos0 = a.seg[4 * blockIdx.z + 3];
    if (slot >= a.slots || (uint64_t)row0 + n > a.rows || n == 0) {
        if (threadIdx.x == 0 && blockIdx.x == 0 && head == 0) atomicOr(a.status, 2u);
        return;
    }
    const uint32_t tid = threadIdx.x;
    const bool consumer = tid < SCAN_CONSUMERS;
    const uint32_t c = (tid % SCAN_CONSUMERS) / LANES, l4 = tid % LANES, col = col0 + c;
    float* colp = a.state + (((size_t)slot * a.heads + head) * D + (col < D ? col : 0u)) * D;
    float4 s[NI];
    if (consumer) load_column<NI>(colp, D, l4, pos0 == 0 || col >= D, s);

    // Producers: a warp owns tokens pw, pw + 4, ... of every chunk. The raw values of its tokens of one chunk are fetched
    // into registers a whole chunk ahead (the loads fly while the consumers work), then turned into the staged vectors.
    constexpr int TPW = CHUNK / (SCAN_PRODUCERS / 32);  // tokens per producer warp and chunk
    const uint32_t pw = (tid - SCAN_CONSUMERS) >> 5, lane = tid & 31u;
    float raw[TPW][4 * CPL + 1], w0[CPL], ab[CPL];
    auto fetch = [&](uint32_t chunk) {
#pragma unroll
        for (int j = 0; j < TPW; ++j) {
            const uint32_t row = chunk * CHUNK + pw + j * (SCAN_PRODUCERS / 32);
            const size_t at = row0 + (row < n ? row : n - 1u);
            const float* p = a.packed + at * a.ld + head * D;
#pragma unroll
            for (int i = 0; i < CPL; ++i) {
                const uint32_t ch = lane + 32u * i, cc = ch < D ? ch : D - 1u;  // clamped: every load is unconditional
                raw[j][4 * i] = p[cc];
                raw[j][4 * i + 1] = p[HD + cc];
                raw[j][4 * i + 2] = p[4 * (size_t)HD + cc];
                raw[j][4 * i + 3] = a.decay_in ? a.decay_in[at * HD + head * D + cc] : 0.0f;
            }
            raw[j][4 * CPL] = p[2 * (size_t)HD + (col0 + lane < D ? col0 + lane : D - 1u)];  // SCAN_COLS == 32
        }
    };
    auto stage = [&](uint32_t chunk) {
        float* buf = ring + (size_t)(chunk & 1u) * CHUNK * TOK;
#pragma unroll
        for (int j = 0; j < TPW; ++j) {
            const uint32_t t = pw + j * (SCAN_PRODUCERS / 32), row = chunk * CHUNK + t;
            if (row >= n) break;
            float* dst = buf + (size_t)t * TOK;
            float ss = 0.0f;
#pragma unroll
            for (int i = 0; i < CPL; ++i) {
                const float k = lane + 32u * i < D ? raw[j][4 * i + 1] : 0.0f;
                ss = fmaf(k, k, ss);
            }
            ss = warp_sum(ss) + a.unit_eps;
            const float len = sqrtf(ss), inv = 1.0f / len;
#pragma unroll
            for (int i = 0; i < CPL; ++i) {
                const uint32_t ch = lane + 32u * i;
                if (ch >= DP) break;
                const bool in = ch < D;
                float z = raw[j][4 * i + 3];
                if (!a.decay_in && in) {
                    const float* zp = a.packed + (size_t)(row0 + row) * a.ld + 5 * (size_t)HD;
                    for (uint32_t q = 0; q < a.rank; ++q)
                        z = fmaf(w2_elem(a, (size_t)(head * D + ch) * a.rank + q), tanhf(zp[q]), z);
                }
                dst[ch] = in ? decay_of(a, z + w0[i]) : 0.0f;
                dst[DP + ch] = in ? raw[j][4 * i + 1] * inv : 0.0f;
                dst[2 * DP + ch] = in ? m40_sigmoid(raw[j][4 * i + 2] + ab[i]) : 0.0f;
                dst[3 * DP + ch] = in ? raw[j][4 * i] : 0.0f;
            }
            dst[4 * DP + lane] = col0 + lane < D ? len * raw[j][4 * CPL] : 0.0f;
        }
    };
    const uint32_t chunks = (n + CHUNK - 1) / CHUNK;
    if (!consumer) {
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            const uint32_t ch = lane + 32u * i, cc = ch < D ? ch : D - 1u;
            w0[i] = a.w0[head * D + cc];
            ab[i] = a.a_bias[head * D + cc];
        }
        fetch(0);
        stage(0);
        if (chunks > 1) fetch(1);
    }
    __syncthreads();
    for (uint32_t ch = 0; ch < chunks; ++ch) {
        if (consumer) {
            const float* buf = ring + (size_t)(ch & 1u) * CHUNK * TOK;
            const uint32_t left = n - ch * CHUNK, m = left < CHUNK ? left : CHUNK;
            float* o = a.out + (size_t)(row0 + ch * CHUNK) * HD + head * D + col;
#pragma unroll 2
            for (uint32_t t = 0; t < m; ++t) {
                const float v = delta_token<NI>(buf + (size_t)t * TOK, l4, buf[(size_t)t * TOK + 4 * DP + c], s);
                if (l4 == 0 && col < D) o[(size_t)t * HD] = v;
            }
        } else if (ch + 1 < chunks) {
            stage(ch + 1);
            if (ch + 2 < chunks) fetch(ch + 2);
        }
        __syncthreads();
    }
    if (consumer && col < D) store_column<NI>(colp, D, l4, s);
}

// out <- (out / rms per head) * norm * sigmoid(g). One warp per (row, head).
__global__ void __launch_bounds__(256) delta_finish_kernel(DeltaArgs a) {
    pdl_wait();
    pdl_trigger();
    const uint32_t wid = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31u;
    if (wid >= a.rows * a.heads) return;
    const uint32_t row = wid / a.heads, head = wid % a.heads, D = a.dim, HD = a.heads * D;
    float* o = a.out + (size_t)row * HD + head * D;
    const float* g = a.packed + (size_t)row * a.ld + 3 * (size_t)HD + head * D;
    float v[8], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const uint32_t ch = lane + 32u * i;
        v[i] = ch < D ? o[ch] : 0.0f;
        ss = fmaf(v[i], v[i], ss);
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)D + a.eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const uint32_t ch = lane + 32u * i;
        if (ch < D) o[ch] = v[i] * inv * a.norm[head * D + ch] * m40_sigmoid(g[ch]);
    }
}

// grid (heads, rows), block = dim * LANES rounded up to a warp.
template <int NI>
__global__ void __launch_bounds__(NI * LANES * 4 * LANES) delta_decode_kernel(DeltaArgs a) {
    constexpr int DP = NI * LANES * 4;
    __shared__ __align__(16) float vec[4 * DP];
    __shared__ float sv[DP], so[DP], sz[1024];
    pdl_wait();
    pdl_trigger();
    const uint32_t head = blockIdx.x, row = blockIdx.y, D = a.dim, HD = a.heads * D, tid = threadIdx.x;
    const uint32_t lane = tid & 31u;
    const uint32_t slot = a.row_seq[row] * a.slot_mul + a.slot_add;
    if (slot >= a.slots) {
        if (tid == 0 && head == 0) atomicOr(a.status, 2u);
        for (uint32_t ch = tid; ch < D; ch += blockDim.x) a.out[(size_t)row * HD + head * D + ch] = 0.0f;
        return;
    }
    const uint32_t col = tid / LANES, l4 = tid % LANES;
    float* colp = a.state + (((size_t)slot * a.heads + head) * D + (col < D ? col : 0u)) * D;
    float4 s[NI];
    load_column<NI>(colp, D, l4, a.row_pos[row] == 0 || col >= D, s);

    const float* p = a.packed + (size_t)row * a.ld + head * D;
    float ss = 0.0f;
    for (uint32_t ch = lane; ch < D; ch += 32u) ss = fmaf(p[HD + ch], p[HD + ch], ss);
    const float len = sqrtf(warp_sum(ss) + a.unit_eps), inv = 1.0f / len;  // every warp, redundantly
    if (!a.decay_in) {
        const float* zp = a.packed + (size_t)row * a.ld + 5 * (size_t)HD;
        for (uint32_t q = tid; q < a.rank; q += blockDim.x) sz[q] = tanhf(zp[q]);
        __syncthreads();
    }
    // the low-rank product: LANES lanes per channel
    float z = 0.0f;
    if (!a.decay_in) {
        if (col < D)
            for (uint32_t q = l4; q < a.rank; q += LANES) z = fmaf(w2_elem(a, (size_t)(head * D + col) * a.rank + q), sz[q], z);
        z += __shfl_xor_sync(0xffffffffu, z, 1);
        z += __shfl_xor_sync(0xffffffffu, z, 2);
    } else if (col < D) {
        z = a.decay_in[(size_t)row * HD + head * D + col];
    }
    if (l4 == 0 && col < DP) {
        const bool in = col < D;
        vec[col] = in ? decay_of(a, z + a.w0[head * D + col]) : 0.0f;
        vec[DP + col] = in ? p[HD + col] * inv : 0.0f;
        vec[2 * DP + col] = in ? m40_sigmoid(p[4 * (size_t)HD + col] + a.a_bias[head * D + col]) : 0.0f;
        vec[3 * DP + col] = in ? p[col] : 0.0f;
        sv[col] = in ? len * p[2 * (size_t)HD + col] : 0.0f;
    }
    // channels beyond the block's columns (block = dim * LANES rounded up to a warp, vectors padded to DP)
    for (uint32_t ch = blockDim.x / LANES + tid; ch < DP; ch += blockDim.x)
        vec[ch] = vec[DP + ch] = vec[2 * DP + ch] = vec[3 * DP + ch] = 0.0f;
    __syncthreads();
    const float o = delta_token<NI>(vec, l4, col < DP ? sv[col] : 0.0f, s);
    if (col < D) store_column<NI>(colp, D, l4, s);
    if (l4 == 0 && col < D) so[col] = o;
    __syncthreads();
    ss = 0.0f;
    for (uint32_t ch = lane; ch < D; ch += 32u) ss = fmaf(so[ch], so[ch], ss);
    const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)D + a.eps);
    for (uint32_t ch = tid; ch < D; ch += blockDim.x)
        a.out[(size_t)row * HD + head * D + ch] =
            so[ch] * rs * a.norm[head * D + ch] * m40_sigmoid(p[3 * (size_t)HD + ch]);
}

template <int NI>
int run(M40llmCudaContext* ctx, const DeltaArgs& a, uint32_t segments, uint32_t max_segment_rows) {
    cudaStream_t s = ctx->decode_stream;
    if (max_segment_rows == 1) {
        const uint32_t threads = (a.dim * LANES + 31u) & ~31u;
        const cudaError_t e =
            m40_launch_dependent(delta_decode_kernel<NI>, dim3(a.heads, a.rows), dim3(threads), 0, s, a);
        M40_COUNT_LAUNCH(ctx);
        return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
    }
    constexpr size_t smem = (size_t)2 * CHUNK * (4 * NI * LANES * 4 + SCAN_COLS) * sizeof(float);
    static unsigned long long configured = 0ull;
    const unsigned long long bit = 1ull << (ctx->device_id & 63);
    if (!(configured & bit)) {
        if (cudaFuncSetAttribute(delta_scan_kernel<NI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return -6;
        configured |= bit;
    }
    const dim3 grid((a.dim + SCAN_COLS - 1) / SCAN_COLS, a.heads, segments);
    cudaError_t e = m40_launch_dependent(delta_scan_kernel<NI>, grid, dim3(SCAN_CONSUMERS + SCAN_PRODUCERS), smem, s, a);
    M40_COUNT_LAUNCH(ctx);
    if (e != cudaSuccess) return -6;
    e = m40_launch_dependent(delta_finish_kernel, dim3((a.rows * a.heads + 7) / 8), dim3(256), 0, s, a);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

}  // namespace

extern "C" {

M40llmStateCache* m40llm_statecache_create(M40llmCudaContext* ctx, uint32_t slots, uint32_t heads, uint32_t dim) {
    if (!ctx || slots == 0 || heads == 0 || dim == 0 || dim > 256) return nullptr;
    if (m40_ensure_device(ctx) != 0) return nullptr;
    M40llmStateCache* st = (M40llmStateCache*)calloc(1, sizeof(M40llmStateCache));
    if (!st) return nullptr;
    st->device_id = ctx->device_id;
    st->slots = slots;
    st->heads = heads;
    st->dim = dim;
    const size_t bytes = (size_t)slots * heads * dim * dim * sizeof(float);
    if (cudaMalloc((void**)&st->d_state, bytes) != cudaSuccess || cudaMemset(st->d_state, 0, bytes) != cudaSuccess ||
        cudaStreamSynchronize(cudaStreamLegacy) != cudaSuccess) {
        cudaGetLastError();
        m40llm_statecache_destroy(st);
        return nullptr;
    }
    return st;
}

void m40llm_statecache_destroy(M40llmStateCache* st) {
    if (!st) return;
    cudaSetDevice(st->device_id);
    if (st->d_state) cudaFree(st->d_state);
    free(st);
}

int m40llm_statecache_debug_read(M40llmCudaContext* ctx, M40llmStateCache* st, uint32_t slot, float* out_host) {
    if (!ctx || !st || !out_host) return -1;
    if (slot >= st->slots) return -2;
    if (m40_ensure_device(ctx) != 0) return -1;
    const size_t per = (size_t)st->heads * st->dim * st->dim;
    float* tmp = (float*)malloc(per * sizeof(float));
    if (!tmp) return -5;
    int rc = 0;
    if (cudaMemcpyAsync(tmp, st->d_state + slot * per, per * sizeof(float), cudaMemcpyDeviceToHost, ctx->decode_stream) !=
            cudaSuccess ||
        cudaStreamSynchronize(ctx->decode_stream) != cudaSuccess)
        rc = -4;
    for (size_t h = 0; rc == 0 && h < st->heads; ++h)
        for (size_t v = 0; v < st->dim; ++v)
            for (size_t k = 0; k < st->dim; ++k)
                out_host[(h * st->dim + k) * st->dim + v] = tmp[(h * st->dim + v) * st->dim + k];
    free(tmp);
    return rc;
}

int m40llm_delta_rule_async(M40llmCudaContext* ctx, M40llmStateCache* st, const M40llmDeltaRule* c,
                            const M40llmStepRows* rows) {
    if (!ctx || !st || !c || !rows || !c->packed || !c->w0 || !c->a_bias || !c->norm || !c->out) return -1;
    if (!c->decay_in && (!c->w2 || c->rank == 0 || c->rank > 1024)) return -2;
    if (rows->rows == 0 || rows->segments == 0 || rows->max_segment_rows == 0) return -2;
    if (rows->max_segment_rows == 1 ? (!rows->row_seq || !rows->row_pos) : !rows->seg) return -1;
    if (c->w_dtype > M40LLM_DT_BF16) return -3;
    const uint64_t need = 5ull * st->heads * st->dim + (c->decay_in ? 0u : c->rank);
    if (c->ld < need) return -2;
    if (m40_ensure_device(ctx) != 0) return -1;
    DeltaArgs a = {};
    a.packed = (const float*)c->packed;
    a.w2 = c->w2;
    a.w0 = (const float*)c->w0;
    a.a_bias = (const float*)c->a_bias;
    a.norm = (const float*)c->norm;
    a.decay_in = (const float*)c->decay_in;
    a.out = (float*)c->out;
    a.state = st->d_state;
    a.status = ctx->d_status;
    a.row_seq = rows->row_seq;
    a.row_pos = rows->row_pos;
    a.seg = rows->seg;
    a.ld = c->ld;
    a.rank = c->rank;
    a.w2_dtype = c->w_dtype;
    a.heads = st->heads;
    a.dim = st->dim;
    a.slots = st->slots;
    a.slot_mul = rows->slot_mul;
    a.slot_add = rows->slot_add;
    a.rows = rows->rows;
    a.decay_scale = c->decay_scale;
    a.unit_eps = c->unit_eps;
    a.eps = c->eps;
    const uint32_t sg = rows->segments, mx = rows->max_segment_rows;
    switch ((st->dim + 15) / 16) {  // 16-channel pieces per lane group
        case 1: return run<1>(ctx, a, sg, mx);
        case 2: return run<2>(ctx, a, sg, mx);
        case 3: return run<3>(ctx, a, sg, mx);
        case 4: return run<4>(ctx, a, sg, mx);
        case 5: return run<5>(ctx, a, sg, mx);
        case 6: return run<6>(ctx, a, sg, mx);
        case 7: case 8: return run<8>(ctx, a, sg, mx);
        case 9: case 10: case 11: case 12: return run<12>(ctx, a, sg, mx);
        default: return run<16>(ctx, a, sg, mx);
    }
}

}  // extern "C"
