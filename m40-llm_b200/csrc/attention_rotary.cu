// Softmax attention with whole-projection query / key norms, partial rotary keys with a scaled frequency table, rotary
// values and a per-head output gate: m40llm_attention_rotary_async.
//
//   rotary_prepare_kernel  CTA = (row, share of the heads): both norms, all rotations, the cache append, and the row's
//                          value-rotation table (cos, sin), which the last step needs to turn the output back. With few
//                          rows the heads are dealt to many CTAs, each summing the squares of the whole projection itself.
//   attention              one of
//     decode tiles  (attention_tiled.cu)   f16 cache, head sizes 64 / 128, few rows: token splits over the whole GPU, then
//                                          rotary_merge_kernel merges them and finishes (turn back, gate);
//     prompt tiles  (attention_prefill.cu) same caches, longer portions: finished in the kernel;
//     rotary_rows_kernel                   every other size and the f32 cache: f32 arithmetic, CTA = (row, q head).
#include "attention.cuh"
#include "common.cuh"
#include "stack_math.cuh"

namespace {

constexpr int TILE_ROWS_MAX = 16;  // rows up to which the decode tiles are used
constexpr int MAX_VDIM = 512;

struct RotArgs {
    const float* packed;
    const float* q_norm;
    const float* k_norm;
    const double* k_turns;
    const double* v_turns;
    void* K;
    void* V;
    uint32_t* seq_map;
    float* q;          // [rows][q_heads * kd]
    float2* turn;      // [rows][vd / 2]
    float* out;
    uint32_t* status;
    const uint32_t* row_seq;
    const uint32_t* row_pos;
    uint32_t ld, q_heads, kv_heads, kd, vd, k_pairs, has_gate, slot_mul, slot_add, slots, max_seq_len, rows;
    float eps, k_amp, scale;
};

// sum of squares of x[0 .. n), this thread's share; eight loads in flight
__device__ __forceinline__ float squares_256(const float* __restrict__ x, uint32_t n) {
    float s0 = 0.0f, s1 = 0.0f;
    uint32_t i = threadIdx.x;
    for (; i + 7u * 256u < n; i += 8u * 256u) {
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = x[i + 256u * j];
#pragma unroll
        for (int j = 0; j < 8; j += 2) s0 = fmaf(v[j], v[j], s0), s1 = fmaf(v[j + 1], v[j + 1], s1);
    }
    for (; i < n; i += 256u) s0 = fmaf(x[i], x[i], s0);
    return s0 + s1;
}

// sine and cosine of `pos * turns` full turns; the whole turns are dropped in double, where the product is exact enough
__device__ __forceinline__ float2 turn_cs(uint32_t pos, double turns) {
    const double t = (double)pos * turns;
    float s, c;
    sincospif(2.0f * (float)(t - rint(t)), &s, &c);
    return make_float2(c, s);
}

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

template <typename ET>
__global__ void __launch_bounds__(256) rotary_prepare_kernel(RotArgs a) {
    extern __shared__ float2 tables[];  // [k_pairs] keys, [vd / 2] values
    __shared__ float red[8];
    pdl_wait();
    pdl_trigger();
    const uint32_t row = blockIdx.x, tid = threadIdx.x;
    const uint32_t pos = a.row_pos[row], slot = a.row_seq[row] * a.slot_mul + a.slot_add;
    if (slot >= a.slots || pos >= a.max_seq_len) {
        if (tid == 0 && blockIdx.y == 0) atomicOr(a.status, 2u);
        return;
    }
    const uint32_t QD = a.q_heads * a.kd, KD = a.kv_heads * a.kd, VD = a.kv_heads * a.vd, half_v = a.vd / 2u;
    const float* q = a.packed + (size_t)row * a.ld;
    const float* k = q + QD;
    const float* v = k + KD;
    float2* tk = tables;
    float2* tv = tables + a.k_pairs;
    for (uint32_t i = tid; i < a.k_pairs; i += 256u) {
        const float2 cs = turn_cs(pos, a.k_turns[i]);
        tk[i] = make_float2(cs.x * a.k_amp, cs.y * a.k_amp);
    }
    if (a.v_turns)
        for (uint32_t i = tid; i < half_v; i += 256u) {
            tv[i] = turn_cs(pos, a.v_turns[i]);
            if (blockIdx.y == 0) a.turn[(size_t)row * half_v + i] = tv[i];
        }
    float sq = a.q_norm ? squares_256(q, QD) : 0.0f, sk = a.k_norm ? squares_256(k, KD) : 0.0f;
    sq = block_sum_256(sq, red);  // its barriers also publish the tables
    sk = block_sum_256(sk, red);
    const float nq = a.q_norm ? 1.0f / sqrtf(sq / (float)QD + a.eps) : 1.0f;
    const float nk = a.k_norm ? 1.0f / sqrtf(sk / (float)KD + a.eps) : 1.0f;
    // element e of a projection, normalised and turned
    auto turned = [&](const float* x, const float* w, float n, uint32_t e) {
        const uint32_t d = e % a.kd;
        const float own = x[e] * n * (w ? w[e] : 1.0f);
        if (d >= 2u * a.k_pairs) return own;
        const bool low = d < a.k_pairs;
        const uint32_t e2 = low ? e + a.k_pairs : e - a.k_pairs;
        const float other = x[e2] * n * (w ? w[e2] : 1.0f);
        const float2 cs = tk[low ? d : d - a.k_pairs];
        return low ? own * cs.x - other * cs.y : own * cs.x + other * cs.y;
    };
    // this CTA's share of the elements of each projection
    const uint32_t step = gridDim.y * 256u, first = blockIdx.y * 256u + tid;
#pragma unroll 2
    for (uint32_t e = first; e < QD; e += step) a.q[(size_t)row * QD + e] = turned(q, a.q_norm, nq, e);
    ET* K = reinterpret_cast<ET*>(a.K);
    ET* V = reinterpret_cast<ET*>(a.V);
    for (uint32_t e = first; e < KD; e += step)
        m40_store_elem(K + kv_row_offset(slot, e / a.kd, pos, a.kv_heads, a.max_seq_len, a.kd) + e % a.kd,
                       turned(k, a.k_norm, nk, e));
    for (uint32_t e = first; e < VD; e += step) {
        const uint32_t d = e % a.vd;
        float y = v[e];
        if (a.v_turns && d < 2u * half_v) {
            const bool low = d < half_v;
            const float other = v[low ? e + half_v : e - half_v];
            const float2 cs = tv[low ? d : d - half_v];
            y = low ? y * cs.x - other * cs.y : y * cs.x + other * cs.y;
        }
        m40_store_elem(V + kv_row_offset(slot, e / a.vd, pos, a.kv_heads, a.max_seq_len, a.vd) + d, y);
    }
    if (tid == 0 && blockIdx.y == 0 && a.seq_map) a.seq_map[slot] = pos + 1u;
}

// Output element d of one head, given the head's attention output o[vd] in shared memory.
__device__ __forceinline__ float finished(const RotArgs& a, const float* o, uint32_t row, uint32_t head, uint32_t d, float gate) {
    float y = o[d];
    const uint32_t half_v = a.vd / 2u;
    if (a.v_turns && d < 2u * half_v) {
        const bool low = d < half_v;
        const float2 cs = a.turn[(size_t)row * half_v + (low ? d : d - half_v)];
        y = low ? y * cs.x + o[d + half_v] * cs.y : y * cs.x - o[d - half_v] * cs.y;
    }
    return y * gate;
}
__device__ __forceinline__ float gate_of(const RotArgs& a, uint32_t row, uint32_t head) {
    if (!a.has_gate) return 1.0f;
    return m40_sigmoid(a.packed[(size_t)row * a.ld + (size_t)a.q_heads * a.kd + (size_t)a.kv_heads * (a.kd + a.vd) + head]);
}

// Merge of the decode tiles' partials [row][head][split] (splits <= 128, vd 64 or 128), then the finish.
// grid (q_heads, rows), block 256: eight groups of 32 float4 lanes share the splits.
__global__ void __launch_bounds__(256) rotary_merge_kernel(RotArgs a, const float* __restrict__ pm, const float* __restrict__ pl,
                                                           const float* __restrict__ po, uint32_t splits) {
    __shared__ __align__(16) float so[128];
    __shared__ float sw[128], red[4], red2[4];
    __shared__ float4 sacc[8][32];
    pdl_wait();
    pdl_trigger();
    const uint32_t head = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, lane = tid & 31u, warp = tid >> 5;
    const size_t base = ((size_t)row * a.q_heads + head) * splits;
    const float gate = gate_of(a, row, head);
    const float l = tid < splits ? pl[base + tid] : 0.0f;
    const float m = l > 0.0f ? pm[base + tid] : -INFINITY;
    const float wm = warp_max(m);
    if (lane == 0 && warp < 4u) red[warp] = wm;
    __syncthreads();
    const float M = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    const float e = l > 0.0f ? expf(m - M) : 0.0f;
    if (tid < 128u) sw[tid] = e;
    const float part = warp_sum(l * e);
    if (lane == 0 && warp < 4u) red2[warp] = part;
    __syncthreads();
    const float L = (red2[0] + red2[1]) + (red2[2] + red2[3]);
    const float inv = 1.0f / (L > 0.0f ? L : 1.0f);
    const uint32_t vl = a.vd / 4u;
    float4 acc = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (lane < vl) {
#pragma unroll 4
        for (uint32_t s = warp; s < splits; s += 8u) {
            const float w = sw[s];
            const float4 x = *reinterpret_cast<const float4*>(po + (base + s) * a.vd + 4u * lane);
            if (w != 0.0f) {  // empty splits may hold anything
                acc.x = fmaf(w, x.x, acc.x), acc.y = fmaf(w, x.y, acc.y);
                acc.z = fmaf(w, x.z, acc.z), acc.w = fmaf(w, x.w, acc.w);
            }
        }
    }
    sacc[warp][lane] = acc;
    __syncthreads();
    if (warp == 0 && lane < vl) {
        float4 t = sacc[0][lane];
#pragma unroll
        for (int i = 1; i < 8; ++i) {
            const float4 u = sacc[i][lane];
            t.x += u.x, t.y += u.y, t.z += u.z, t.w += u.w;
        }
        *reinterpret_cast<float4*>(so + 4u * lane) = make_float4(t.x * inv, t.y * inv, t.z * inv, t.w * inv);
    }
    __syncthreads();
    if (tid < a.vd) a.out[((size_t)row * a.q_heads + head) * a.vd + tid] = finished(a, so, row, head, tid, gate);
}

// Any head sizes, f16 or f32 cache, f32 arithmetic. grid (q_heads, rows), block 128: a thread scores one key of a
// 128-key tile, the softmax is online over tiles, then a thread owns output dims tid, tid + 128, ...
template <typename ET>
__global__ void __launch_bounds__(128) rotary_rows_kernel(RotArgs a) {
    extern __shared__ __align__(16) float sq[];  // [kd] the query, scaled
    __shared__ float sp[128], so[MAX_VDIM], red[4], red2[4];
    pdl_wait();
    pdl_trigger();
    const uint32_t head = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, lane = tid & 31u, warp = tid >> 5;
    const uint32_t pos = a.row_pos[row], slot = a.row_seq[row] * a.slot_mul + a.slot_add;
    float* out = a.out + ((size_t)row * a.q_heads + head) * a.vd;
    if (slot >= a.slots || pos >= a.max_seq_len) {  // the prepare kernel has raised the status bit
        for (uint32_t d = tid; d < a.vd; d += 128u) out[d] = 0.0f;
        return;
    }
    const uint32_t kvh = head / (a.q_heads / a.kv_heads);
    const ET* K = reinterpret_cast<const ET*>(a.K) + kv_row_offset(slot, kvh, 0, a.kv_heads, a.max_seq_len, a.kd);
    const ET* V = reinterpret_cast<const ET*>(a.V) + kv_row_offset(slot, kvh, 0, a.kv_heads, a.max_seq_len, a.vd);
    for (uint32_t d = tid; d < a.kd; d += 128u) sq[d] = a.q[((size_t)row * a.q_heads + head) * a.kd + d];
    __syncthreads();
    float acc[MAX_VDIM / 128] = {}, M = -INFINITY, L = 0.0f;
    const uint32_t n = pos + 1u;
    for (uint32_t t0 = 0; t0 < n; t0 += 128u) {
        float s = -INFINITY;
        if (t0 + tid < n) {
            const ET* kr = K + (size_t)(t0 + tid) * a.kd;
            float d0 = 0.0f, d1 = 0.0f, d2 = 0.0f, d3 = 0.0f;
            uint32_t d = 0;
            for (; d + 4u <= a.kd; d += 4u) {
                d0 = fmaf(sq[d], m40_load_elem(kr + d), d0), d1 = fmaf(sq[d + 1], m40_load_elem(kr + d + 1), d1);
                d2 = fmaf(sq[d + 2], m40_load_elem(kr + d + 2), d2), d3 = fmaf(sq[d + 3], m40_load_elem(kr + d + 3), d3);
            }
            for (; d < a.kd; ++d) d0 = fmaf(sq[d], m40_load_elem(kr + d), d0);
            s = ((d0 + d1) + (d2 + d3)) * a.scale;
        }
        float mx = warp_max(s);
        if (lane == 0) red[warp] = mx;
        __syncthreads();
        const float m_new = fmaxf(M, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
        const float corr = expf(M - m_new), p = expf(s - m_new);  // key t0 is always visible: m_new is finite
        M = m_new;
        sp[tid] = p;
        const float ps = warp_sum(p);
        if (lane == 0) red2[warp] = ps;
        __syncthreads();
        L = L * corr + ((red2[0] + red2[1]) + (red2[2] + red2[3]));
        const uint32_t m = n - t0 < 128u ? n - t0 : 128u;
#pragma unroll
        for (int i = 0; i < MAX_VDIM / 128; ++i) {
            const uint32_t d = tid + 128u * i;
            if (d >= a.vd) break;
            // the tile's sum on its own, in two chains, before it meets the running one: fewer roundings in a row
            float x0 = 0.0f, x1 = 0.0f;
            const ET* vp = V + (size_t)t0 * a.vd + d;
            uint32_t t = 0;
            for (; t + 2u <= m; t += 2u) {
                x0 = fmaf(sp[t], m40_load_elem(vp + (size_t)t * a.vd), x0);
                x1 = fmaf(sp[t + 1u], m40_load_elem(vp + (size_t)(t + 1u) * a.vd), x1);
            }
            if (t < m) x0 = fmaf(sp[t], m40_load_elem(vp + (size_t)t * a.vd), x0);
            acc[i] = fmaf(acc[i], corr, x0 + x1);
        }
        __syncthreads();  // sp, red and red2 are rewritten by the next tile
    }
#pragma unroll
    for (int i = 0; i < MAX_VDIM / 128; ++i) {
        const uint32_t d = tid + 128u * i;
        if (d < a.vd) so[d] = acc[i] / L;
    }
    __syncthreads();
    const float gate = gate_of(a, row, head);
    for (uint32_t d = tid; d < a.vd; d += 128u) out[d] = finished(a, so, row, head, d, gate);
}

}  // namespace

extern "C" int m40llm_attention_rotary_async(M40llmCudaContext* ctx, M40llmKVCache* kv, const M40llmRotaryAttention* c,
                                             const M40llmStepRows* r) {
    if (!ctx || !kv || !c || !r || !c->packed || !c->out || !c->k_turns || !r->row_seq || !r->row_pos || !r->row_len) return -1;
    if (r->rows == 0 || r->segments == 0 || r->max_segment_rows == 0) return -2;
    if (c->q_heads == 0 || kv->num_heads == 0 || c->q_heads % kv->num_heads != 0) return -3;
    const bool typed = kv->d_typed_k != nullptr;
    if (kv->compressed || (typed ? !kv->d_typed_v : (!kv->d_k || !kv->d_v))) return -4;
    const uint32_t kd = kv->head_dim, vd = typed && kv->v_dim ? kv->v_dim : kd;
    if (2u * c->k_pairs > kd || kd > 1024u || vd > (uint32_t)MAX_VDIM) return -3;
    const uint64_t need = (uint64_t)c->q_heads * kd + (uint64_t)kv->num_heads * (kd + vd) + (c->has_gate ? c->q_heads : 0u);
    if (c->ld < need) return -2;
    if (r->max_segment_rows > 1 && !r->seg) return -1;
    if (m40_ensure_device(ctx) != 0) return -1;
    cudaStream_t s = ctx->decode_stream;

    RotArgs a = {};
    a.packed = (const float*)c->packed;
    a.q_norm = (const float*)c->q_norm;
    a.k_norm = (const float*)c->k_norm;
    a.k_turns = (const double*)c->k_turns;
    a.v_turns = (const double*)c->v_turns;
    a.K = typed ? kv->d_typed_k : (void*)kv->d_k;
    a.V = typed ? kv->d_typed_v : (void*)kv->d_v;
    a.seq_map = kv->d_seq_map;
    a.out = (float*)c->out;
    a.status = ctx->d_status;
    a.row_seq = r->row_seq;
    a.row_pos = r->row_pos;
    a.ld = c->ld;
    a.q_heads = c->q_heads;
    a.kv_heads = kv->num_heads;
    a.kd = kd;
    a.vd = vd;
    a.k_pairs = c->k_pairs;
    a.has_gate = c->has_gate;
    a.slot_mul = r->slot_mul;
    a.slot_add = r->slot_add;
    a.slots = kv->max_batch_size;
    a.max_seq_len = kv->max_seq_len;
    a.rows = r->rows;
    a.eps = c->eps;
    a.k_amp = c->k_amp;
    a.scale = c->scale;

    const bool tiles = !typed && (kd == 64 || kd == 128) && c->q_heads / kv->num_heads <= 16;
    const bool decode = tiles && r->rows <= (uint32_t)TILE_ROWS_MAX + (r->max_segment_rows == 1 ? 0xffffu : 0u);
    uint32_t chunk = 0, splits = 0;
    const uint32_t bound = r->max_len ? r->max_len : kv->max_seq_len;
    // level-1 arena: turned queries and rotation tables; level-0 arena: the splits' partials
    const size_t q_elems = (size_t)r->rows * c->q_heads * kd, turn_elems = (size_t)r->rows * (vd / 2u);
    unsigned char* work = (unsigned char*)m40_ensure_scratch(ctx, 1, q_elems * sizeof(float) + turn_elems * sizeof(float2) + 16, 1);
    if (!work) return -5;
    a.q = (float*)work;
    a.turn = (float2*)(work + ((q_elems * sizeof(float) + 15) & ~(size_t)15));
    float* part = nullptr;
    if (decode) {
        m40_attn_pick_chunk(ctx, r->rows, kv->num_heads, bound, &chunk, &splits);
        // o first (16-byte aligned rows for the merge), then m and l
        part = (float*)m40_ensure_scratch(ctx, 1, (size_t)r->rows * c->q_heads * splits * (2 + (size_t)vd) * sizeof(float), 0);
        if (!part) return -5;
    }

    const size_t table_bytes = ((size_t)c->k_pairs + vd / 2u) * sizeof(float2);
    const uint32_t shares_max = (c->q_heads * kd + 255u) / 256u, shares_want = (uint32_t)ctx->sm_count / r->rows;
    const dim3 pgrid(r->rows, shares_want < 1u ? 1u : (shares_want < shares_max ? shares_want : shares_max));
    cudaError_t e = kv->elem_f32 ? m40_launch_dependent(rotary_prepare_kernel<float>, pgrid, dim3(256), table_bytes, s, a)
                                 : m40_launch_dependent(rotary_prepare_kernel<__half>, pgrid, dim3(256), table_bytes, s, a);
    M40_COUNT_LAUNCH(ctx);
    if (e != cudaSuccess) return -6;

    if (decode) {
        DenseAttnArgs d = {};
        d.K = kv->d_k;
        d.V = kv->d_v;
        d.q = a.q;
        d.seq_ids = r->row_seq;
        d.seq_lens = r->row_len;
        const size_t n = (size_t)r->rows * c->q_heads * splits;
        d.part_o = part;
        d.part_m = part + n * vd;
        d.part_l = d.part_m + n;
        d.status = ctx->d_status;
        d.max_seq_len = kv->max_seq_len;
        d.max_batch = kv->max_batch_size;
        d.kv_heads = kv->num_heads;
        d.q_heads = c->q_heads;
        d.hd = kd;
        d.splits = splits;
        d.chunk = chunk;
        d.write_partials = 1u;
        d.inv_sqrt = c->scale;
        d.slot_mul = r->slot_mul;
        d.slot_add = r->slot_add;
        const int rc = m40_attention_dense_tiled(ctx, d, r->rows);
        if (rc != 0) return rc < 0 ? rc : -6;
        e = m40_launch_dependent(rotary_merge_kernel, dim3(c->q_heads, r->rows), dim3(256), 0, s, a, d.part_m, d.part_l, d.part_o,
                                 splits);
        M40_COUNT_LAUNCH(ctx);
        return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
    }
    if (tiles) {
        const float* gate = c->has_gate ? a.packed + (size_t)c->q_heads * kd + (size_t)kv->num_heads * (kd + vd) : nullptr;
        M40PrefillCall p = {};
        p.K = kv->d_k;
        p.V = kv->d_v;
        p.q = a.q;
        p.out = a.out;
        p.seg = r->seg;
        p.turn_back = a.v_turns ? a.turn : nullptr;
        p.gate = gate;
        p.gate_ld = c->ld;
        p.segments = r->segments;
        p.max_segment_rows = r->max_segment_rows;
        p.rows = r->rows;
        p.hd = p.q_dim = p.v_dim = kd;
        p.q_heads = c->q_heads;
        p.kv_heads = kv->num_heads;
        p.q_ld = p.out_ld = c->q_heads * kd;
        p.slot_mul = r->slot_mul;
        p.slot_add = r->slot_add;
        p.slots = kv->max_batch_size;
        p.max_seq_len = kv->max_seq_len;
        p.scale = c->scale;
        const int rc = m40_attention_prefill(ctx, p);
        if (rc <= 0) return rc;
    }
    const size_t smem = (size_t)kd * sizeof(float);
    const dim3 grid(c->q_heads, r->rows);
    e = kv->elem_f32 ? m40_launch_dependent(rotary_rows_kernel<float>, grid, dim3(128), smem, s, a)
                     : m40_launch_dependent(rotary_rows_kernel<__half>, grid, dim3(128), smem, s, a);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}
