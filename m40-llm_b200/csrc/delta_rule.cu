// Generalised delta rule: a recurrent mixer whose state is one matrix per head,
//   S <- diag(w) S - (a * u) (u^T S) + k v^T,   o = S^T r,
// with a decay w and a removal rate a per head and key channel, u the unit key. All of it is f32.
//
// With k = n u (n the key's length) the update of one value column s of S is
//   d = u . s,   s_i <- w_i s_i + u_i (n v - a_i d),   o = r . s,
// so columns are independent and a token costs one dot product, one update and one dot product per column. A column's key
// dimension is shared by a few lanes (16-byte pieces dealt round-robin) and stays in registers; the only serial chain is d,
// and the second dot product of a token overlaps the first of the next.
//
//   portions of several tokens, in passes of rows whose records stay in L2:
//     delta_prepare_kernel  warp = (row, head): gates, decays, unit key -> one record [w | u | a | r | n v] per (head, row);
//     delta_scan_kernel     CTA = (32 columns, head, segment) walks the tokens; the records of 32 or 16 tokens arrive by one bulk
//                           copy (cp.async.bulk + mbarrier) several chunks ahead. Eight lanes share two columns, because
//                           the limit is shared-memory reads: every vector piece read serves both;
//     delta_finish_kernel   the per-head norm and the output gate.
//   delta_decode_kernel     one token per sequence: CTA = (head, row) does everything, the low-rank decay projection
//                           included, in one launch; bound by reading and writing the state once.
// A chunked (matrix-product) form is not used: its products of decays and of removals would have to leave f32, or lose the
// property that the result does not depend on where a portion was cut.
//
// The scan's waits are bounded like the tensor-core kernels': a wait that runs out raises status bit 4, the CTA stops,
// waits (bounded) for its copies in flight and returns.
#include "common.cuh"
#include "stack_math.cuh"
#include "state_cache.cuh"
#include "tc_ptx.cuh"

namespace {

constexpr int LANES = 4;          // decode: lanes per column
constexpr int SCAN_LANES = 8;     // scan: lanes per pair of columns
constexpr int SCAN_COLS = 32;     // columns per scan CTA
constexpr int SCAN_THREADS = SCAN_COLS / 2 * SCAN_LANES;
constexpr size_t PASS_BYTES = (size_t)96 << 20;  // records of one pass: inside L2
// Tokens per bulk copy, and copies in flight, for records of 5 * DP floats.
__host__ __device__ constexpr int scan_chunk(int dp) { return dp <= 128 ? 32 : 16; }
__host__ __device__ constexpr size_t scan_stage_bytes(int dp) { return (size_t)scan_chunk(dp) * 5 * dp * sizeof(float); }
__host__ __device__ constexpr uint32_t scan_stages(int dp) {
    return (size_t)4 * scan_stage_bytes(dp) <= 196608u ? 4u : (uint32_t)(196608u / scan_stage_bytes(dp));
}

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
    uint32_t ld, rank, w2_dtype, w2_wide, heads, dim, slots, slot_mul, slot_add, rows;
    float decay_scale, unit_eps, eps;
};

__device__ __forceinline__ float w2_elem(const DeltaArgs& a, size_t i) {
    if (a.w2_dtype == M40LLM_DT_BF16) return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(a.w2)[i]);
    if (a.w2_dtype == M40LLM_DT_F16) return __half2float(reinterpret_cast<const __half*>(a.w2)[i]);
    return reinterpret_cast<const float*>(a.w2)[i];
}
__device__ __forceinline__ float decay_of(const DeltaArgs& a, float z) { return expf(a.decay_scale * m40_sigmoid(z)); }

// State of one column: elements 4 (l4 + LANES i) .. + 3 of the key dimension.
template <int NI, int LANES>
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
template <int NI, int LANES>
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

// Rows [base, base + count) of every segment (relative to its start) -> records. One warp per (row, head); `rec` holds, per
// head, n_rec records of 5 * DP floats, the record of row r of the step at r - base.
template <int DP>
__global__ void __launch_bounds__(256) delta_prepare_kernel(DeltaArgs a, float* __restrict__ rec, uint32_t n_rec, uint32_t base,
                                                            uint32_t count) {
    constexpr int CPL = DP / 32;  // channels per lane
    pdl_wait();
    pdl_trigger();
    const uint32_t wid = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31u;
    if (wid >= count * a.heads) return;
    const uint32_t head = wid % a.heads, row = base + wid / a.heads, D = a.dim, HD = a.heads * D;
    const float* p = a.packed + (size_t)row * a.ld + head * D;
    float r[CPL], k[CPL], v[CPL], rate[CPL], z[CPL], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        const uint32_t ch = lane + 32u * i, cc = ch < D ? ch : D - 1u;  // clamped: every load is unconditional
        r[i] = p[cc];
        k[i] = p[HD + cc];
        v[i] = p[2 * (size_t)HD + cc];
        rate[i] = p[4 * (size_t)HD + cc] + a.a_bias[head * D + cc];
        z[i] = (a.decay_in ? a.decay_in[(size_t)row * HD + head * D + cc] : 0.0f) + a.w0[head * D + cc];
    }
    if (!a.decay_in) {
        const float* zp = a.packed + (size_t)row * a.ld + 5 * (size_t)HD;
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
            const uint32_t ch = lane + 32u * i, cc = ch < D ? ch : D - 1u;
            float acc = 0.0f;
            for (uint32_t q = 0; q < a.rank; ++q) acc = fmaf(w2_elem(a, (size_t)(head * D + cc) * a.rank + q), tanhf(zp[q]), acc);
            z[i] += acc;
        }
    }
#pragma unroll
    for (int i = 0; i < CPL; ++i) ss = lane + 32u * i < D ? fmaf(k[i], k[i], ss) : ss;
    const float len = sqrtf(warp_sum(ss) + a.unit_eps), inv = 1.0f / len;
    float* dst = rec + ((size_t)head * n_rec + (row - base)) * (5 * DP);
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
        const uint32_t ch = lane + 32u * i;
        const bool in = ch < D;
        dst[ch] = in ? decay_of(a, z[i]) : 0.0f;
        dst[DP + ch] = in ? k[i] * inv : 0.0f;
        dst[2 * DP + ch] = in ? m40_sigmoid(rate[i]) : 0.0f;
        dst[3 * DP + ch] = in ? r[i] : 0.0f;
        dst[4 * DP + ch] = in ? len * v[i] : 0.0f;
    }
}

// Four sums over the eight lanes of a column pair at once: the shuffles of one level are independent of each other.
__device__ __forceinline__ void sum_lanes8(float& a, float& b, float& c, float& d) {
#pragma unroll
    for (int o = 1; o < SCAN_LANES; o <<= 1) {
        const float ta = __shfl_xor_sync(0xffffffffu, a, o), tb = __shfl_xor_sync(0xffffffffu, b, o);
        const float tc_ = __shfl_xor_sync(0xffffffffu, c, o), td = __shfl_xor_sync(0xffffffffu, d, o);
        a += ta, b += tb, c += tc_, d += td;
    }
}
// This lane's pieces of one token's record.
template <int NI>
struct TokenVec {
    float4 u[NI], w[NI], a[NI], r[NI];
    float2 nv;
    __device__ __forceinline__ void load(const float* rec, uint32_t l, uint32_t col) {
        constexpr int DP = NI * SCAN_LANES * 4;
        const float4* v4 = reinterpret_cast<const float4*>(rec) + l;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            w[i] = v4[SCAN_LANES * i];
            u[i] = v4[DP / 4 + SCAN_LANES * i];
            a[i] = v4[2 * (DP / 4) + SCAN_LANES * i];
            r[i] = v4[3 * (DP / 4) + SCAN_LANES * i];
        }
        nv = *reinterpret_cast<const float2*>(rec + 4 * DP + col);
    }
};
__device__ __forceinline__ float dot4(const float4& x, const float4& y) {
    return fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, x.w * y.w)));
}
__device__ __forceinline__ void update4(float4& s, const float4& w, const float4& u, const float4& a, float d, float nv) {
    s.x = fmaf(u.x, fmaf(-a.x, d, nv), w.x * s.x);
    s.y = fmaf(u.y, fmaf(-a.y, d, nv), w.y * s.y);
    s.z = fmaf(u.z, fmaf(-a.z, d, nv), w.z * s.z);
    s.w = fmaf(u.w, fmaf(-a.w, d, nv), w.w * s.w);
}

// grid (column blocks, heads, segments). Rows [base, base + count) of the segment, counted from its start.
template <int NI>
__global__ void __launch_bounds__(SCAN_THREADS) delta_scan_kernel(DeltaArgs a, const float* __restrict__ rec, uint32_t n_rec,
                                                                  uint32_t rec_base, uint32_t base, uint32_t count) {
    constexpr int DP = NI * SCAN_LANES * 4, CHUNK = scan_chunk(DP);
    constexpr uint32_t stages = scan_stages(DP);
    constexpr uint32_t REC = 5 * DP;
    extern __shared__ __align__(128) float ring[];
    __shared__ uint64_t full[4];
    __shared__ uint32_t stop;
    const uint32_t tid = threadIdx.x;
    if (tid == 0) {
        for (uint32_t s = 0; s < stages; ++s) tc::mbar_init(&full[s], 1);
        stop = 0u;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    pdl_trigger();
    const uint32_t head = blockIdx.y, col0 = blockIdx.x * SCAN_COLS, D = a.dim, HD = a.heads * D;
    const uint32_t seg0 = a.seg[4 * blockIdx.z], seg_n = a.seg[4 * blockIdx.z + 1];
    const uint32_t slot = a.seg[4 * blockIdx.z + 2] * a.slot_mul + a.slot_add, pos0 = a.seg[4 * blockIdx.z + 3];
    if (slot >= a.slots || (uint64_t)seg0 + seg_n > a.rows) {
        if (tid == 0 && blockIdx.x == 0 && head == 0) atomicOr(a.status, 2u);
        return;
    }
    if (base >= seg_n) return;
    const uint32_t n = seg_n - base < count ? seg_n - base : count, row0 = seg0 + base;
    const float* src = rec + ((size_t)head * n_rec + (row0 - rec_base)) * REC;
    const uint32_t chunks = (n + CHUNK - 1) / CHUNK;
    auto request = [&](uint32_t ch) {  // thread 0
        const uint32_t m = n - ch * CHUNK < CHUNK ? n - ch * CHUNK : CHUNK, bytes = m * REC * 4u, s = ch % stages;
        tc::mbar_expect_tx(&full[s], bytes);
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                     ::"r"(tc::smem_u32(ring + (size_t)s * CHUNK * REC)), "l"(src + (size_t)ch * CHUNK * REC), "r"(bytes),
                     "r"(tc::smem_u32(&full[s])) : "memory");
    };
    if (tid == 0)
        for (uint32_t ch = 0; ch < chunks && ch < stages; ++ch) request(ch);

    const uint32_t l = tid % SCAN_LANES, c = tid / SCAN_LANES * 2u, ca = col0 + c, cb = ca + 1u;
    float* state = a.state + ((size_t)slot * a.heads + head) * D * D;
    float4 sa[NI], sb[NI];
    const bool fresh = pos0 == 0 && base == 0;
    load_column<NI, SCAN_LANES>(state + (size_t)(ca < D ? ca : 0u) * D, D, l, fresh || ca >= D, sa);
    load_column<NI, SCAN_LANES>(state + (size_t)(cb < D ? cb : 0u) * D, D, l, fresh || cb >= D, sb);
    float* out = a.out + (size_t)row0 * HD + head * D + (l == 0 ? ca : cb);
    const bool store = l == 0 ? ca < D : (l == 1 && cb < D);

    // Software pipeline: a token's pieces are read while the previous token is worked on (within a chunk), and the two
    // outputs of the previous token are summed over the lanes together with this token's two d.
    float oa = 0.0f, ob = 0.0f;
    uint32_t ch = 0;
    for (; ch < chunks; ++ch) {
        const uint32_t s = ch % stages;
        if (!tc::mbar_wait(&full[s], (ch / stages) & 1u)) stop = 1u;
        const float* buf = ring + (size_t)s * CHUNK * REC;
        const uint32_t m = n - ch * CHUNK < CHUNK ? n - ch * CHUNK : CHUNK;
        TokenVec<NI> cur;
        cur.load(buf, l, col0 + c);
#pragma unroll 2
        for (uint32_t t = 0; t < m; ++t) {
            TokenVec<NI> nxt;
            nxt.load(buf + (size_t)(t + 1u < m ? t + 1u : t) * REC, l, col0 + c);
            float da = 0.0f, db = 0.0f;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                da += dot4(cur.u[i], sa[i]);
                db += dot4(cur.u[i], sb[i]);
            }
            sum_lanes8(da, db, oa, ob);
            const uint32_t row = ch * CHUNK + t;
            if (store && row > 0u) out[(size_t)(row - 1u) * HD] = l == 0 ? oa : ob;
            oa = ob = 0.0f;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                update4(sa[i], cur.w[i], cur.u[i], cur.a[i], da, cur.nv.x);
                update4(sb[i], cur.w[i], cur.u[i], cur.a[i], db, cur.nv.y);
                oa += dot4(cur.r[i], sa[i]);
                ob += dot4(cur.r[i], sb[i]);
            }
            cur = nxt;
        }
        __syncthreads();  // everyone is done with this slot
        if (stop) break;
        if (tid == 0 && ch + stages < chunks) request(ch + stages);
    }
    if (ch < chunks) {  // a wait ran out: the copies still in flight must land before this CTA's memory goes away
        if (tid == 0) {
            atomicOr(a.status, 4u);
            for (uint32_t i = ch; i < chunks && i < ch + stages; ++i) tc::mbar_wait(&full[i % stages], (i / stages) & 1u);
        }
        return;
    }
    float x0 = 0.0f, x1 = 0.0f;
    sum_lanes8(oa, ob, x0, x1);
    if (store) out[(size_t)(n - 1u) * HD] = l == 0 ? oa : ob;
    if (ca < D) store_column<NI, SCAN_LANES>(state + (size_t)ca * D, D, l, sa);
    if (cb < D) store_column<NI, SCAN_LANES>(state + (size_t)cb * D, D, l, sb);
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
__global__ void __launch_bounds__(NI * LANES * 4 * LANES, NI <= 4 ? 16 / NI : 1) delta_decode_kernel(DeltaArgs a) {
    constexpr int DP = NI * LANES * 4;
    __shared__ __align__(16) float vec[4 * DP];
    __shared__ __align__(16) float sz[1024];
    __shared__ float sv[DP], so[DP];
    const uint32_t head = blockIdx.x, row = blockIdx.y, D = a.dim, HD = a.heads * D, tid = threadIdx.x;
    const uint32_t lane = tid & 31u, col = tid / LANES, l4 = tid % LANES;
    const uint32_t cc = head * D + (col < D ? col : D - 1u);  // this thread's channel (clamped)
    // The low-rank rows of this channel do not depend on the previous kernel: 16-byte pieces l4, l4 + 4, ... of a 16-bit
    // row, up to four per lane, are requested before the dependency wait.
    const bool wide = a.w2_wide != 0u;
    uint4 wq[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const uint32_t q8 = l4 + LANES * j;
        wq[j] = make_uint4(0u, 0u, 0u, 0u);
        if (wide && q8 < a.rank / 8u)
            wq[j] = *reinterpret_cast<const uint4*>(reinterpret_cast<const uint16_t*>(a.w2) + (size_t)cc * a.rank + 8u * q8);
    }
    const float w0 = a.w0[cc], ab = a.a_bias[cc];
    pdl_wait();
    pdl_trigger();
    const uint32_t slot = a.row_seq[row] * a.slot_mul + a.slot_add;
    if (slot >= a.slots) {
        if (tid == 0 && head == 0) atomicOr(a.status, 2u);
        for (uint32_t ch = tid; ch < D; ch += blockDim.x) a.out[(size_t)row * HD + head * D + ch] = 0.0f;
        return;
    }
    float* colp = a.state + (((size_t)slot * a.heads + head) * D + (col < D ? col : 0u)) * D;
    float4 s[NI];
    load_column<NI, LANES>(colp, D, l4, a.row_pos[row] == 0 || col >= D, s);
    const float* prow = a.packed + (size_t)row * a.ld;
    const float* p = prow + head * D;
    const float pr = prow[cc], pk = prow[HD + cc], pv = prow[2 * (size_t)HD + cc], pa = prow[4 * (size_t)HD + cc];
    float z = a.decay_in ? a.decay_in[(size_t)row * HD + cc] : 0.0f;
    float ss = 0.0f;
    for (uint32_t ch = lane; ch < D; ch += 32u) ss = fmaf(p[HD + ch], p[HD + ch], ss);
    if (!a.decay_in) {
        const float* zp = prow + 5 * (size_t)HD;
        for (uint32_t q = tid; q < a.rank; q += blockDim.x) sz[q] = tanhf(zp[q]);
    }
    const float len = sqrtf(warp_sum(ss) + a.unit_eps), inv = 1.0f / len;  // every warp, redundantly
    if (!a.decay_in) {
        __syncthreads();
        // the low-rank product: LANES lanes per channel
        if (wide) {
            const bool bf = a.w2_dtype == M40LLM_DT_BF16;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const uint32_t q8 = l4 + LANES * j;
                if (q8 >= a.rank / 8u) break;
                const uint32_t u[4] = {wq[j].x, wq[j].y, wq[j].z, wq[j].w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float2 h = __half22float2(*reinterpret_cast<const __half2*>(&u[i]));
                    z = fmaf(bf ? __uint_as_float(u[i] << 16) : h.x, sz[8u * q8 + 2 * i], z);
                    z = fmaf(bf ? __uint_as_float(u[i] & 0xffff0000u) : h.y, sz[8u * q8 + 2 * i + 1], z);
                }
            }
        } else {
            for (uint32_t q = l4; q < a.rank; q += LANES) z = fmaf(w2_elem(a, (size_t)cc * a.rank + q), sz[q], z);
        }
        z += __shfl_xor_sync(0xffffffffu, z, 1);
        z += __shfl_xor_sync(0xffffffffu, z, 2);
    }
    if (l4 == 0 && col < DP) {
        const bool in = col < D;
        vec[col] = in ? decay_of(a, z + w0) : 0.0f;
        vec[DP + col] = in ? pk * inv : 0.0f;
        vec[2 * DP + col] = in ? m40_sigmoid(pa + ab) : 0.0f;
        vec[3 * DP + col] = in ? pr : 0.0f;
        sv[col] = in ? len * pv : 0.0f;
    }
    const float gate = m40_sigmoid(prow[3 * (size_t)HD + cc]) * a.norm[cc];
    // channels beyond the block's columns (block = dim * LANES rounded up to a warp, vectors padded to DP)
    for (uint32_t ch = blockDim.x / LANES + tid; ch < DP; ch += blockDim.x)
        vec[ch] = vec[DP + ch] = vec[2 * DP + ch] = vec[3 * DP + ch] = 0.0f;
    __syncthreads();
    const float o = delta_token<NI>(vec, l4, col < DP ? sv[col] : 0.0f, s);
    if (col < D) store_column<NI, LANES>(colp, D, l4, s);
    if (l4 == 0 && col < D) so[col] = o;
    __syncthreads();
    ss = 0.0f;
    for (uint32_t ch = lane; ch < D; ch += 32u) ss = fmaf(so[ch], so[ch], ss);
    const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)D + a.eps);
    if (l4 == 0 && col < D) a.out[(size_t)row * HD + cc] = so[col] * rs * gate;
}

template <int NI>
int run_decode(M40llmCudaContext* ctx, const DeltaArgs& a) {
    const uint32_t threads = (a.dim * LANES + 31u) & ~31u;
    const cudaError_t e =
        m40_launch_dependent(delta_decode_kernel<NI>, dim3(a.heads, a.rows), dim3(threads), 0, ctx->decode_stream, a);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

template <int NI>
int run_scan(M40llmCudaContext* ctx, const DeltaArgs& a, uint32_t segments, uint32_t max_segment_rows) {
    constexpr int DP = NI * SCAN_LANES * 4;
    constexpr uint32_t CHUNK = (uint32_t)scan_chunk(DP);
    cudaStream_t s = ctx->decode_stream;
    constexpr size_t smem = scan_stages(DP) * scan_stage_bytes(DP);
    static_assert(scan_stages(DP) >= 2, "the ring needs two slots");
    static unsigned long long configured = 0ull;
    const unsigned long long bit = 1ull << (ctx->device_id & 63);
    if (!(configured & bit)) {
        if (cudaFuncSetAttribute(delta_scan_kernel<NI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return -6;
        configured |= bit;
    }
    // One segment is walked in passes of rows whose records fit PASS_BYTES; several segments take one pass.
    const size_t per_row = (size_t)a.heads * 5 * DP * sizeof(float);
    uint32_t pass = max_segment_rows;
    if (segments == 1) {
        const size_t fit = PASS_BYTES / per_row / CHUNK * CHUNK;
        pass = fit < CHUNK ? CHUNK : (fit < pass ? (uint32_t)fit : pass);
    }
    const uint32_t n_rec = segments == 1 ? pass : a.rows;
    float* rec = (float*)m40_ensure_scratch(ctx, 1, n_rec * per_row, 1);
    if (!rec) return -5;
    const dim3 grid((a.dim + SCAN_COLS - 1) / SCAN_COLS, a.heads, segments);
    cudaError_t e;
    for (uint32_t base = 0; base < max_segment_rows; base += pass) {
        // `rows` of the step from `base` on: with one segment the pass's rows, with several all of them
        const uint32_t rows = segments == 1 ? (a.rows - base < pass ? a.rows - base : pass) : a.rows;
        e = m40_launch_dependent(delta_prepare_kernel<DP>, dim3((rows * a.heads + 7) / 8), dim3(256), 0, s, a, rec, n_rec, base, rows);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess) return -6;
        e = m40_launch_dependent(delta_scan_kernel<NI>, grid, dim3(SCAN_THREADS), smem, s, a, (const float*)rec, n_rec, base, base,
                                 pass);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess) return -6;
    }
    e = m40_launch_dependent(delta_finish_kernel, dim3((a.rows * a.heads + 7) / 8), dim3(256), 0, s, a);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

}  // namespace

extern "C" {

int m40llm_delta_rule_async(M40llmCudaContext* ctx, M40llmStateCache* st, const M40llmDeltaRule* c,
                            const M40llmStepRows* rows) {
    if (!ctx || !st || !c || !rows || !c->packed || !c->w0 || !c->a_bias || !c->norm || !c->out) return -1;
    if (!c->decay_in && (!c->w2 || c->rank == 0 || c->rank > 1024)) return -2;
    if (st->dim == 0) return -3;  // a cache of plain values
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
    a.w2_wide = !c->decay_in && c->w_dtype != M40LLM_DT_F32 && c->rank % 8 == 0 && c->rank <= 128 && ((uintptr_t)c->w2 & 15u) == 0;
    a.heads = st->heads;
    a.dim = st->dim;
    a.slots = st->slots;
    a.slot_mul = rows->slot_mul;
    a.slot_add = rows->slot_add;
    a.rows = rows->rows;
    a.decay_scale = c->decay_scale;
    a.unit_eps = c->unit_eps;
    a.eps = c->eps;
    if (rows->max_segment_rows > 1) {
        // rows outside the segment's range must not be prepared: with one segment it must start at row 0 and span the step
        const uint32_t sg = rows->segments, mx = rows->max_segment_rows;
        if (sg == 1 && mx != rows->rows) return -2;
        switch ((st->dim + 31) / 32) {  // 32-channel pieces per lane group
            case 1: return run_scan<1>(ctx, a, sg, mx);
            case 2: return run_scan<2>(ctx, a, sg, mx);
            case 3: return run_scan<3>(ctx, a, sg, mx);
            case 4: return run_scan<4>(ctx, a, sg, mx);
            case 5: case 6: return run_scan<6>(ctx, a, sg, mx);
            default: return run_scan<8>(ctx, a, sg, mx);
        }
    }
    switch ((st->dim + 15) / 16) {  // 16-channel pieces per lane group
        case 1: return run_decode<1>(ctx, a);
        case 2: return run_decode<2>(ctx, a);
        case 3: return run_decode<3>(ctx, a);
        case 4: return run_decode<4>(ctx, a);
        case 5: return run_decode<5>(ctx, a);
        case 6: return run_decode<6>(ctx, a);
        case 7: case 8: return run_decode<8>(ctx, a);
        case 9: case 10: case 11: case 12: return run_decode<12>(ctx, a);
        default: return run_decode<16>(ctx, a);
    }
}

}  // extern "C"
