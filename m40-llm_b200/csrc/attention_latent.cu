// Attention over a cache of latents, without positions: m40llm_attention_latent_async.
//
// A head's key and value are uk c and uv c of the cached latent c, so  q . k = (uk^T q) . c  and  sum p v = uv (sum p c):
// with uk folded into the query every head attends the same rows c, which are key and value at once.
//
//   latent_prepare_kernel  uk^T q per head (absorbed query), and the latent's norm and append;
//   attention over latents latent_rows_kernel: any rank, f16 or f32 cache, f32 arithmetic, CTA = (head, row, token split);
//   latent_merge_kernel    merges the token splits and the sink, then uv.
#include "attention.cuh"
#include "stack_math.cuh"

namespace {

constexpr uint32_t MAX_RANK = 1024;
constexpr uint32_t COLS = 64;        // latent columns per absorbing CTA
constexpr uint32_t RUN_ROWS = 512;   // rows per pass of the absorbed form (bounds the work space)

struct LatArgs {
    const float* packed;   // of the pass's first row
    const float* c_norm;
    const void* uk;
    const void* uv;
    const float* sink;
    void* C;
    uint32_t* seq_map;
    float* qa;             // absorbed queries [rows][heads][rank]
    float* pm;             // [rows][heads][splits]
    float* pl;
    float* po;             // [rows][heads][splits][rank]
    float* out;
    uint32_t* status;
    const uint32_t* row_seq;
    const uint32_t* row_pos;
    uint32_t ld, heads, dim, vdim, rank, slot_mul, slot_add, slots, max_seq_len, rows, splits, chunk;
    uint32_t absorb_ctas, wide;
    float eps, scale;
};

__device__ __forceinline__ float block_sum_256(float v, float* red) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31u) == 0u) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) t += red[i];
    return t;
}

// grid (absorb_ctas + 1 or 0, row groups of RG). CTAs below absorb_ctas: (head, 64 latent columns) of the absorbed query;
// the last one, when present: norm and append of the group's latents.
template <typename WT, typename ET, int RG>
__global__ void __launch_bounds__(256) latent_prepare_kernel(LatArgs a) {
    extern __shared__ __align__(16) float sq[];  // [RG][dim]
    __shared__ float part[8][RG][COLS];
    __shared__ float red[8];
    pdl_wait();
    pdl_trigger();
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, row0 = blockIdx.y * RG;
    if (blockIdx.x >= a.absorb_ctas) {
        for (uint32_t r = 0; r < RG && row0 + r < a.rows; ++r) {
            const uint32_t row = row0 + r, pos = a.row_pos[row], slot = a.row_seq[row] * a.slot_mul + a.slot_add;
            if (slot >= a.slots || pos >= a.max_seq_len) {
                if (tid == 0) atomicOr(a.status, 2u);
                continue;
            }
            const float* c = a.packed + (size_t)row * a.ld + (size_t)a.heads * a.dim;
            float v[MAX_RANK / 256], ss = 0.0f;
#pragma unroll
            for (int i = 0; i < (int)MAX_RANK / 256; ++i) {
                const uint32_t k = tid + 256u * i;
                v[i] = k < a.rank ? c[k] : 0.0f;
                ss = fmaf(v[i], v[i], ss);
            }
            const float n = 1.0f / sqrtf(block_sum_256(ss, red) / (float)a.rank + a.eps);
            ET* dst = reinterpret_cast<ET*>(a.C) + ((size_t)slot * a.max_seq_len + pos) * a.rank;
#pragma unroll
            for (int i = 0; i < (int)MAX_RANK / 256; ++i) {
                const uint32_t k = tid + 256u * i;
                if (k < a.rank) m40_store_elem(dst + k, v[i] * n * a.c_norm[k]);
            }
            if (tid == 0 && a.seq_map) a.seq_map[slot] = pos + 1u;
        }
        return;
    }
    const uint32_t slices = (a.rank + COLS - 1u) / COLS, head = blockIdx.x / slices, c0 = (blockIdx.x % slices) * COLS;
    for (uint32_t i = tid; i < RG * a.dim; i += 256u) {
        const uint32_t row = min(row0 + i / a.dim, a.rows - 1u);
        sq[i] = a.packed[(size_t)row * a.ld + (size_t)head * a.dim + i % a.dim];
    }
    __syncthreads();
    const uint32_t cg = c0 + (lane & 7u) * 8u, kg = warp * 4u + (lane >> 3);
    const WT* w = reinterpret_cast<const WT*>(a.uk) + (size_t)head * a.dim * a.rank;
    float acc[RG][8] = {};
    if (cg < a.rank) {
#pragma unroll 4
        for (uint32_t d = kg; d < a.dim; d += 32u) {
            float wv[8];
            if (a.wide) {
                m40_load8(w + (size_t)d * a.rank + cg, wv);
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) wv[i] = cg + i < a.rank ? m40_load_elem(w + (size_t)d * a.rank + cg + i) : 0.0f;
            }
#pragma unroll
            for (int r = 0; r < RG; ++r)
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[r][i] = fmaf(sq[r * a.dim + d], wv[i], acc[r][i]);
        }
    }
#pragma unroll
    for (int r = 0; r < RG; ++r)
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            float v = acc[r][i];
            v += __shfl_xor_sync(0xffffffffu, v, 8);
            v += __shfl_xor_sync(0xffffffffu, v, 16);
            if (lane < 8u) part[warp][r][lane * 8u + i] = v;
        }
    __syncthreads();
    for (uint32_t i = tid; i < RG * COLS; i += 256u) {
        const uint32_t r = i / COLS, c = i % COLS;
        if (row0 + r >= a.rows || c0 + c >= a.rank) continue;
        float t = 0.0f;
#pragma unroll
        for (int k = 0; k < 8; ++k) t += part[k][r][c];
        a.qa[((size_t)(row0 + r) * a.heads + head) * a.rank + c0 + c] = t;
    }
}

// grid (heads, rows, splits), block 128: a thread scores one token of a 128-token tile, the softmax is online over tiles,
// then a thread owns latent columns tid, tid + 128, ...
template <typename ET>
__global__ void __launch_bounds__(128) latent_rows_kernel(LatArgs a) {
    __shared__ float q[MAX_RANK], sp[128], red[4], red2[4];
    pdl_wait();
    pdl_trigger();
    const uint32_t head = blockIdx.x, row = blockIdx.y, split = blockIdx.z, tid = threadIdx.x, lane = tid & 31u, warp = tid >> 5;
    const uint32_t pos = a.row_pos[row], slot = a.row_seq[row] * a.slot_mul + a.slot_add;
    const size_t pi = ((size_t)row * a.heads + head) * a.splits + split;
    const uint32_t lo = split * a.chunk, hi = min(lo + a.chunk, pos + 1u);
    if (slot >= a.slots || pos >= a.max_seq_len || lo >= hi) {  // an empty partial
        if (tid == 0) a.pm[pi] = -INFINITY, a.pl[pi] = 0.0f;
        return;
    }
    const ET* C = reinterpret_cast<const ET*>(a.C) + (size_t)slot * a.max_seq_len * a.rank;
    for (uint32_t d = tid; d < a.rank; d += 128u) q[d] = a.qa[((size_t)row * a.heads + head) * a.rank + d];
    __syncthreads();
    float acc[MAX_RANK / 128] = {}, M = -INFINITY, L = 0.0f;
    for (uint32_t t0 = lo; t0 < hi; t0 += 128u) {
        float s = -INFINITY;
        if (t0 + tid < hi) {
            const ET* cr = C + (size_t)(t0 + tid) * a.rank;
            float d0 = 0.0f, d1 = 0.0f, d2 = 0.0f, d3 = 0.0f;
            uint32_t d = 0;
            for (; d + 4u <= a.rank; d += 4u) {
                d0 = fmaf(q[d], m40_load_elem(cr + d), d0), d1 = fmaf(q[d + 1], m40_load_elem(cr + d + 1), d1);
                d2 = fmaf(q[d + 2], m40_load_elem(cr + d + 2), d2), d3 = fmaf(q[d + 3], m40_load_elem(cr + d + 3), d3);
            }
            for (; d < a.rank; ++d) d0 = fmaf(q[d], m40_load_elem(cr + d), d0);
            s = ((d0 + d1) + (d2 + d3)) * a.scale;
        }
        const float mx = warp_max(s);
        if (lane == 0) red[warp] = mx;
        __syncthreads();
        const float m_new = fmaxf(M, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
        const float corr = expf(M - m_new), p = expf(s - m_new);  // token t0 is always visible: m_new is finite
        M = m_new;
        sp[tid] = p;
        const float ps = warp_sum(p);
        if (lane == 0) red2[warp] = ps;
        __syncthreads();
        L = L * corr + ((red2[0] + red2[1]) + (red2[2] + red2[3]));
        const uint32_t m = min(hi - t0, 128u);
#pragma unroll
        for (int i = 0; i < (int)MAX_RANK / 128; ++i) {
            const uint32_t d = tid + 128u * i;
            if (d >= a.rank) break;
            float x0 = 0.0f, x1 = 0.0f;
            const ET* cp = C + (size_t)t0 * a.rank + d;
            uint32_t t = 0;
            for (; t + 2u <= m; t += 2u) {
                x0 = fmaf(sp[t], m40_load_elem(cp + (size_t)t * a.rank), x0);
                x1 = fmaf(sp[t + 1u], m40_load_elem(cp + (size_t)(t + 1u) * a.rank), x1);
            }
            if (t < m) x0 = fmaf(sp[t], m40_load_elem(cp + (size_t)t * a.rank), x0);
            acc[i] = fmaf(acc[i], corr, x0 + x1);
        }
        __syncthreads();  // sp, red and red2 are rewritten by the next tile
    }
    if (tid == 0) a.pm[pi] = M, a.pl[pi] = L;
#pragma unroll
    for (int i = 0; i < (int)MAX_RANK / 128; ++i) {
        const uint32_t d = tid + 128u * i;
        if (d < a.rank) a.po[pi * a.rank + d] = acc[i];
    }
}

// grid (heads, row groups of RG, slices of the values): splits and sink -> the head's weighted latent, then uv.
template <typename WT, int RG>
__global__ void __launch_bounds__(256) latent_merge_kernel(LatArgs a) {
    extern __shared__ __align__(16) float so[];  // [RG][rank padded to 4], then [RG][splits] weights
    pdl_wait();
    pdl_trigger();
    const uint32_t head = blockIdx.x, row0 = blockIdx.y * RG, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    const uint32_t rp = (a.rank + 3u) & ~3u, live = min((uint32_t)RG, a.rows - row0);
    float* sw = so + RG * rp;
    if (warp < RG && warp < live) {  // one warp per row: the splits' weights
        const size_t base = ((size_t)(row0 + warp) * a.heads + head) * a.splits;
        const float sink = a.sink ? a.sink[head] : -INFINITY;
        float M = sink;
        for (uint32_t s = lane; s < a.splits; s += 32u)
            if (a.pl[base + s] > 0.0f) M = fmaxf(M, a.pm[base + s]);
        M = warp_max(M);
        float L = 0.0f;
        for (uint32_t s = lane; s < a.splits; s += 32u) {
            const float l = a.pl[base + s], e = l > 0.0f ? expf(a.pm[base + s] - M) : 0.0f;
            sw[warp * a.splits + s] = e;
            L = fmaf(l, e, L);
        }
        L = warp_sum(L);
        if (a.sink) L += expf(sink - M);
        const float inv = 1.0f / (L > 0.0f ? L : 1.0f);
        for (uint32_t s = lane; s < a.splits; s += 32u) sw[warp * a.splits + s] *= inv;
    }
    __syncthreads();
    for (uint32_t i = tid; i < RG * rp; i += 256u) {
        const uint32_t r = i / rp, c = i % rp;
        float t = 0.0f;
        if (r < live && c < a.rank) {
            const float* w = sw + r * a.splits;
            const float* o = a.po + ((size_t)(row0 + r) * a.heads + head) * a.splits * a.rank + c;
#pragma unroll 8
            for (uint32_t s = 0; s < a.splits; ++s) {
                const float ws = w[s], x = ws != 0.0f ? o[(size_t)s * a.rank] : 0.0f;  // empty splits may hold anything
                t = fmaf(ws, x, t);
            }
        }
        so[i] = t;
    }
    __syncthreads();
    const uint32_t per = (a.vdim + gridDim.z - 1u) / gridDim.z, n1 = min((blockIdx.z + 1u) * per, a.vdim);
    const WT* uv = reinterpret_cast<const WT*>(a.uv) + (size_t)head * a.vdim * a.rank;
#pragma unroll 2
    for (uint32_t n = blockIdx.z * per + warp; n < n1; n += 8u) {
        const WT* w = uv + (size_t)n * a.rank;
        float acc[RG] = {};
        if (a.wide) {
#pragma unroll 2
            for (uint32_t k = lane * 8u; k < a.rank; k += 256u) {
                float wv[8];
                m40_load8(w + k, wv);
#pragma unroll
                for (int r = 0; r < RG; ++r)
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[r] = fmaf(wv[i], so[r * rp + k + i], acc[r]);
            }
        } else {
            for (uint32_t k = lane; k < a.rank; k += 32u)
#pragma unroll
                for (int r = 0; r < RG; ++r) acc[r] = fmaf(m40_load_elem(w + k), so[r * rp + k], acc[r]);
        }
#pragma unroll
        for (int r = 0; r < RG; ++r) {
            const float v = warp_sum(acc[r]);
            if (lane == 0 && (uint32_t)r < live) a.out[((size_t)(row0 + r) * a.heads + head) * a.vdim + n] = v;
        }
    }
}

template <typename WT, typename ET>
cudaError_t launch_prepare(cudaStream_t s, const LatArgs& a, bool append) {
    const uint32_t x = a.absorb_ctas + (append ? 1u : 0u);
    if (a.rows == 1) return m40_launch_dependent(latent_prepare_kernel<WT, ET, 1>, dim3(x, 1), dim3(256), a.dim * sizeof(float), s, a);
    return m40_launch_dependent(latent_prepare_kernel<WT, ET, 4>, dim3(x, (a.rows + 3) / 4), dim3(256), 4 * a.dim * sizeof(float), s, a);
}

template <typename WT>
cudaError_t launch_merge(M40llmCudaContext* ctx, const LatArgs& a) {
    const uint32_t rp = (a.rank + 3u) & ~3u, rg = a.rows == 1 ? 1u : 4u, groups = (a.rows + rg - 1) / rg;
    uint32_t z = (uint32_t)ctx->sm_count / (a.heads * groups);
    const uint32_t z_max = (a.vdim + 15u) / 16u;
    z = z < 1u ? 1u : (z > z_max ? z_max : z);
    const size_t smem = (size_t)rg * (rp + a.splits) * sizeof(float);
    const dim3 grid(a.heads, groups, z);
    return rg == 1 ? m40_launch_dependent(latent_merge_kernel<WT, 1>, grid, dim3(256), smem, ctx->decode_stream, a)
                   : m40_launch_dependent(latent_merge_kernel<WT, 4>, grid, dim3(256), smem, ctx->decode_stream, a);
}

template <typename WT>
cudaError_t prepare(cudaStream_t s, const LatArgs& a, bool f32, bool append) {
    return f32 ? launch_prepare<WT, float>(s, a, append) : launch_prepare<WT, __half>(s, a, append);
}

template <typename WT>
int run(M40llmCudaContext* ctx, const M40llmKVCache* kv, const LatArgs& all, uint32_t bound) {
    cudaStream_t s = ctx->decode_stream;
    const uint32_t slices = (all.rank + COLS - 1) / COLS;
    cudaError_t e;
    // one pass does everything in one prepare launch; several append first, so that every pass sees the whole step
    const bool one = all.rows <= RUN_ROWS;
    if (!one) {
        LatArgs a = all;
        a.absorb_ctas = 0;
        e = prepare<WT>(s, a, kv->elem_f32, true);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess) return -6;
    }
    for (uint32_t at = 0; at < all.rows; at += RUN_ROWS) {
        LatArgs a = all;
        a.rows = all.rows - at < RUN_ROWS ? all.rows - at : RUN_ROWS;
        a.packed += (size_t)at * a.ld;
        a.out += (size_t)at * a.heads * a.vdim;
        a.row_seq += at;
        a.row_pos += at;
        m40_attn_pick_chunk(ctx, a.rows, a.heads, bound, &a.chunk, &a.splits);
        const size_t nh = (size_t)a.rows * a.heads, np = nh * a.splits;
        auto pad = [](size_t v) { return (v + 3) & ~(size_t)3; };
        float* work = (float*)m40_ensure_scratch(ctx, 1, (pad(nh * a.rank) + pad(np * a.rank) + 2 * np) * sizeof(float), 1);
        if (!work) return -5;
        a.qa = work;
        a.po = work + pad(nh * a.rank);
        a.pm = a.po + pad(np * a.rank);
        a.pl = a.pm + np;
        a.absorb_ctas = a.heads * slices;
        e = prepare<WT>(s, a, kv->elem_f32, one);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess) return -6;
        const dim3 grid(a.heads, a.rows, a.splits);
        e = kv->elem_f32 ? m40_launch_dependent(latent_rows_kernel<float>, grid, dim3(128), 0, s, a)
                         : m40_launch_dependent(latent_rows_kernel<__half>, grid, dim3(128), 0, s, a);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess) return -6;
        e = launch_merge<WT>(ctx, a);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess || cudaGetLastError() != cudaSuccess) return -6;
    }
    return 0;
}

}  // namespace

extern "C" int m40llm_attention_latent_async(M40llmCudaContext* ctx, M40llmKVCache* kv, const M40llmLatentAttention* c,
                                             const M40llmStepRows* r) {
    if (!ctx || !kv || !c || !r || !c->packed || !c->c_norm || !c->uk || !c->uv || !c->out || !r->row_seq || !r->row_pos) return -1;
    if (r->rows == 0 || r->segments == 0 || r->max_segment_rows == 0 || r->rows > 65535u) return -2;
    if (!kv->d_typed_k || kv->d_typed_v || kv->num_heads != 1) return -4;
    if (c->heads == 0 || c->dim == 0 || c->vdim == 0 || kv->head_dim > MAX_RANK || c->dim > 2048 || c->w_dtype > M40LLM_DT_BF16) return -3;
    if (c->ld < (uint64_t)c->heads * c->dim + kv->head_dim) return -2;
    if (m40_ensure_device(ctx) != 0) return -1;
    LatArgs a = {};
    a.packed = (const float*)c->packed;
    a.c_norm = (const float*)c->c_norm;
    a.uk = c->uk;
    a.uv = c->uv;
    a.sink = (const float*)c->sink;
    a.C = kv->d_typed_k;
    a.seq_map = kv->d_seq_map;
    a.out = (float*)c->out;
    a.status = ctx->d_status;
    a.row_seq = r->row_seq;
    a.row_pos = r->row_pos;
    a.ld = c->ld;
    a.heads = c->heads;
    a.dim = c->dim;
    a.vdim = c->vdim;
    a.rank = kv->head_dim;
    a.slot_mul = r->slot_mul;
    a.slot_add = r->slot_add;
    a.slots = kv->max_batch_size;
    a.max_seq_len = kv->max_seq_len;
    a.rows = r->rows;
    a.eps = c->eps;
    a.scale = c->scale;
    a.wide = c->w_dtype != M40LLM_DT_F32 && a.rank % 8 == 0 && (((uintptr_t)c->uk | (uintptr_t)c->uv) & 15u) == 0;
    const uint32_t bound = r->max_len && r->max_len < kv->max_seq_len ? r->max_len : kv->max_seq_len;
    if (c->w_dtype == M40LLM_DT_F32) return run<float>(ctx, kv, a, bound);
    return c->w_dtype == M40LLM_DT_BF16 ? run<__nv_bfloat16>(ctx, kv, a, bound) : run<__half>(ctx, kv, a, bound);
}
