// Attention over a cache of latents, without positions: m40llm_attention_latent_async.
//
// A head's key and value are uk c and uv c of the cached latent c, so  q . k = (uk^T q) . c  and  sum p v = uv (sum p c):
// with uk folded into the query every head attends the same rows c, which are key and value at once.
//
//   latent_prepare_kernel  uk^T q per head (absorbed query), and the latent's norm and append; with several rows on the tensor
//                          path latent_append_kernel (append, and the queries cut into hi + lo) and a grouped tcgen05 GEMM;
//   attention over latents, one of
//     latent_tc_kernel     (attention_latent_tc.cu) f16 cache, rank a multiple of 128 up to 512: tcgen05, CTA = (row, 32 heads,
//                          token split);
//     latent_tiles_kernel  f16 cache, rank a multiple of 16 up to 512: mma.sync, CTA = (row, 16 heads, token split). In both the
//                          tokens' latents stream once through shared memory and serve all the heads, as keys and as values;
//     latent_rows_kernel   any rank, f16 or f32 cache, f32 arithmetic: CTA = (head, row, token split);
//   latent_merge_kernel    merges the token splits and the sink, then uv (itself, or as a grouped GEMM of several rows).
// Long portions (segments of EXPAND_ROWS rows or more, f16 cache) do less work with the heads' keys and values in hand: they
// are made once per portion from the cached latents by the grouped tcgen05 GEMM, f16 and head-major, and the prompt kernel of
// attention_prefill.cu attends them.
#include "attention_latent.cuh"

#include "attention.cuh"
#include "attention_mma.cuh"
#include "gemm_tc_grouped.cuh"
#include "stack_math.cuh"
#include "tc_ptx.cuh"

namespace {

constexpr uint32_t MAX_RANK = 1024;
constexpr uint32_t RUN_ROWS = 512;   // rows per pass of the absorbed form (bounds the work space)
constexpr uint32_t EXPAND_ROWS = 64;
constexpr uint32_t TEAM_ROWS = 4;       // rows from which a CTA takes 32 heads
constexpr uint32_t GROUPED_ROWS = 8;    // rows from which uk and uv go through the grouped GEMM
constexpr size_t EXPAND_BYTES = (size_t)1 << 30;  // work space for one portion's keys and values

using LatArgs = M40LatArgs;

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

// Norm and append of one row's latent by the whole CTA.
template <typename ET>
__device__ __forceinline__ void append_row(const LatArgs& a, uint32_t row, float* red) {
    const uint32_t tid = threadIdx.x, pos = a.row_pos[row], slot = a.row_seq[row] * a.slot_mul + a.slot_add;
    if (slot >= a.slots || pos >= a.max_seq_len) {
        if (tid == 0) atomicOr(a.status, 2u);
        return;
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

__device__ __forceinline__ void split_store4(__nv_bfloat16* hi, __nv_bfloat16* lo, size_t at, const float4& x) {
    const float v[4] = {x.x, x.y, x.z, x.w};
    __nv_bfloat16 h[4], l[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        h[i] = __float2bfloat16_rn(v[i]);
        l[i] = __float2bfloat16_rn(v[i] - __bfloat162float(h[i]));
    }
    *reinterpret_cast<uint2*>(hi + at) = *reinterpret_cast<const uint2*>(h);
    *reinterpret_cast<uint2*>(lo + at) = *reinterpret_cast<const uint2*>(l);
}

// grid (rows, 1 + shares of the query): CTA (row, 0) appends the row's latent (when asked to), the others cut its queries.
__global__ void __launch_bounds__(256) latent_append_kernel(LatArgs a, uint32_t append) {
    __shared__ float red[8];
    pdl_wait();
    pdl_trigger();
    const uint32_t row = blockIdx.x, n = a.heads * a.dim;
    if (blockIdx.y == 0) {
        if (append) append_row<__half>(a, row, red);
        return;
    }
    for (uint32_t k = ((blockIdx.y - 1u) * 256u + threadIdx.x) * 4u; k < n; k += (gridDim.y - 1u) * 1024u)
        split_store4(a.part[0], a.part[1], (size_t)row * n + k, *reinterpret_cast<const float4*>(a.packed + (size_t)row * a.ld + k));
}

__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

// grid (absorb_ctas + RG or 0, row groups of RG). CTAs below absorb_ctas: (head, COLS latent columns) of the group's absorbed
// queries; the others, when present: norm and append of one row's latent.
template <typename WT, typename ET, int RG, int COLS>
__global__ void __launch_bounds__(256) latent_prepare_kernel(LatArgs a) {
    extern __shared__ __align__(16) float sq[];  // [RG][dim]
    constexpr uint32_t CG = COLS / 8, KG = 256 / CG;  // groups of 8 columns, groups of query dimensions
    __shared__ float part[8][RG][COLS];
    __shared__ float red[8];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u, row0 = blockIdx.y * RG;
    const uint32_t slices = (a.rank + COLS - 1u) / COLS, head = blockIdx.x / slices, c0 = (blockIdx.x % slices) * COLS;
    const WT* w = reinterpret_cast<const WT*>(a.uk) + (size_t)head * a.dim * a.rank;
    if (blockIdx.x < a.absorb_ctas)  // the weights do not depend on the previous kernel
        for (uint32_t d = tid; d < a.dim; d += 256u) prefetch_l2(w + (size_t)d * a.rank + c0);
    pdl_wait();
    pdl_trigger();
    if (blockIdx.x >= a.absorb_ctas) {
        const uint32_t row = row0 + blockIdx.x - a.absorb_ctas;
        if (row < a.rows) append_row<ET>(a, row, red);
        return;
    }
    for (uint32_t i = tid; i < RG * a.dim; i += 256u) {
        const uint32_t row = min(row0 + i / a.dim, a.rows - 1u);
        sq[i] = a.packed[(size_t)row * a.ld + (size_t)head * a.dim + i % a.dim];
    }
    __syncthreads();
    const uint32_t cg = c0 + (lane % CG) * 8u, kg = warp * (32u / CG) + lane / CG;
    float acc[RG][8] = {};
    if (cg < a.rank) {
#pragma unroll 4
        for (uint32_t d = kg; d < a.dim; d += KG) {
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
#pragma unroll
            for (uint32_t o = CG; o < 32u; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            acc[r][i] = v;
        }
    if (lane < CG) {
#pragma unroll
        for (int r = 0; r < RG; ++r) {
            *reinterpret_cast<float4*>(&part[warp][r][lane * 8u]) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
            *reinterpret_cast<float4*>(&part[warp][r][lane * 8u + 4u]) = make_float4(acc[r][4], acc[r][5], acc[r][6], acc[r][7]);
        }
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

// Tensor-core form. Eight warps; warp w owns UW units of 16 latent columns. Per tile of 64 or 32 tokens: every warp multiplies the
// absorbed queries of 16 heads with the tile over its own columns (mma.sync, query split into f16 hi + lo), the eight partial
// score tiles are added in shared memory, two heads per warp run the online softmax (base 2), and every warp adds P c for its
// columns. So a latent is read from shared memory once as key and once as value, whatever the number of heads.
// Two CTAs, or two teams of warps, share an SM, so that one's barriers and softmax hide behind the other's products. The ring
// of tiles is handed over by mbarriers (every thread copies its pieces with cp.async, every warp releases a tile when it has
// used it), so that the teams need not keep step. Every wait is bounded: one that runs out raises status bit 4, and from then
// on nothing waits.
template <int UW>
struct LatTile {
    static constexpr int TOKENS = UW <= 2 ? 64 : 32;
    static constexpr int PITCH = TOKENS + 8;  // of scores (f32) and weights (f16): no bank conflicts
    static constexpr size_t FIXED = ((size_t)8 * 16 * PITCH * 4 + (size_t)16 * PITCH * 2 + 16 * 4 + 127) / 128 * 128;
    static constexpr size_t bytes(uint32_t rank) { return (size_t)TOKENS * (rank + 8u) * 2u; }
};
constexpr uint32_t MAX_STAGES = 6;
constexpr size_t TILE_SMEM = 112u * 1024u, TILE_SMEM_ALONE = 200u * 1024u;

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }
__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src));
}

// RANK: the latent size when it is 128 * UW (addresses are then constants), or 0 for any other. TEAMS = 2: two teams of eight
// warps with 16 heads each share one ring (one CTA per SM), so that the latents are fetched once for 32 heads.
template <int UW, int RANK, int TEAMS>
__global__ void __launch_bounds__(256 * TEAMS, TEAMS == 2 ? 1 : 2) latent_tiles_kernel(LatArgs a, uint32_t stages) {
    using namespace attn_mma;
    constexpr int LT = LatTile<UW>::TOKENS, PITCH = LatTile<UW>::PITCH, TPL = LT / 32;
    extern __shared__ __align__(128) unsigned char lt_smem[];
    constexpr uint32_t NT = 256u * TEAMS;
    const uint32_t team = TEAMS == 2 ? threadIdx.x >> 8 : 0u;
    __shared__ uint64_t full[MAX_STAGES], empty[MAX_STAGES];
    __shared__ volatile uint32_t abort_flag;
    float* sc = reinterpret_cast<float*>(lt_smem + team * LatTile<UW>::FIXED);  // [8][16][PITCH]
    __half* sp = reinterpret_cast<__half*>(sc + 8 * 16 * PITCH);    // [16][PITCH]
    float* scorr = reinterpret_cast<float*>(sp + 16 * PITCH);       // [16]
    const uint32_t ring = (uint32_t)__cvta_generic_to_shared(lt_smem + TEAMS * LatTile<UW>::FIXED);
    auto team_barrier = [&]() {
        if (TEAMS == 1) __syncthreads();
        else asm volatile("bar.sync %0, 256;" ::"r"(team + 1u) : "memory");
    };
    if (threadIdx.x == 0) {
        for (uint32_t i = 0; i < stages; ++i) {
            tc::mbar_init(&full[i], NT);
            tc::mbar_init(&empty[i], NT / 32u);
        }
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    pdl_trigger();
    const uint32_t rank = RANK ? (uint32_t)RANK : a.rank;
    const uint32_t split = blockIdx.x, h0 = (blockIdx.y * TEAMS + team) * 16u, row = blockIdx.z;
    const uint32_t tid = threadIdx.x & 255u, warp = tid >> 5, lane = tid & 31u;
    const uint32_t g = lane >> 2, t4 = lane & 3u, jm = lane >> 3, NU = rank / 16u, pitch = (rank + 8u) * 2u, tile_bytes = LT * pitch;
    const uint32_t pos = a.row_pos[row], slot = a.row_seq[row] * a.slot_mul + a.slot_add;
    const uint32_t lo = split * a.chunk, hi = min(lo + a.chunk, pos + 1u), heads = h0 < a.heads ? min(16u, a.heads - h0) : 0u;
    if (slot >= a.slots || pos >= a.max_seq_len || lo >= hi) {  // empty partials
        if (tid < heads) {
            const size_t pi = ((size_t)row * a.heads + h0 + tid) * a.splits + split;
            a.pm[pi] = -INFINITY, a.pl[pi] = 0.0f;
        }
        return;
    }
    const __half* C = reinterpret_cast<const __half*>(a.C) + (size_t)slot * a.max_seq_len * rank;
    const uint32_t n_tiles = (hi - lo + LT - 1u) / LT, pieces = rank / 8u;
    // this thread's 16-byte pieces of a tile: every NT-th, as (token, piece) pairs that are stepped, not divided for
    const uint32_t r_first = threadIdx.x / pieces, ch_first = threadIdx.x % pieces, r_step = NT / pieces, ch_step = NT % pieces;
    auto load_tile = [&](uint32_t tile, uint32_t slot_of_ring) {
        const uint32_t dst = ring + slot_of_ring * tile_bytes, base = lo + tile * LT;
        const __half* src = C + (size_t)base * rank;
        if (RANK && base + LT <= hi) {
            constexpr uint32_t RS = RANK ? NT * 8u / RANK : 1u;  // tokens per NT pieces
            const __half* p = src + (size_t)r_first * rank + ch_first * 8u;
            const uint32_t d = dst + r_first * pitch + ch_first * 16u;
#pragma unroll
            for (uint32_t i = 0; i < LT / RS; ++i) cp16(d + i * RS * pitch, p + (size_t)i * RS * rank);
            return;
        }
        const uint32_t last = hi - 1u - base;
        for (uint32_t r = r_first, ch = ch_first; r < LT;) {
            // rows past the end repeat the last visible one: masked below, and their bytes are finite
            cp16(dst + r * pitch + ch * 16u, src + min(r, last) * rank + ch * 8u);
            r += r_step, ch += ch_step;
            if (ch >= pieces) ch -= pieces, ++r;
        }
    };
    auto wait = [&](uint64_t* bar, uint32_t parity) {
        if (!abort_flag && !tc::mbar_wait(bar, parity)) {
            abort_flag = 1;
            atomicOr(a.status, 4u);
        }
    };
    auto landed_on = [&](uint64_t* bar) {  // this thread's copies so far arrive on the barrier when they have landed
        asm volatile("cp.async.mbarrier.arrive.noinc.shared::cta.b64 [%0];" ::"r"(tc::smem_u32(bar)) : "memory");
    };
    // tiles in flight ahead of the one in use; with four slots or more, one stays free so that a team may lag by a tile
    const uint32_t ahead = stages >= 4u ? stages - 2u : stages - 1u;
    for (uint32_t t = 0; t < ahead && t < n_tiles; ++t) {
        load_tile(t, t);
        landed_on(&full[t]);
    }
    // query fragments of this warp's columns
    uint32_t qhi[UW][4], qlo[UW][4];
    const float qs = a.scale * LOG2E;
#pragma unroll
    for (int i = 0; i < UW; ++i) {
        const uint32_t u = warp * UW + i, k0 = u * 16u + 2u * t4;
#pragma unroll
        for (int j = 0; j < 4; ++j) {  // rows g, g + 8 of columns k0, then of k0 + 8
            const uint32_t h = g + (j & 1) * 8u;
            const float2 x = (RANK || u < NU) && h < heads
                                 ? *reinterpret_cast<const float2*>(a.qa + ((size_t)row * a.heads + h0 + h) * rank + k0 + (j >> 1) * 8u)
                                 : make_float2(0.f, 0.f);
            split_h2(x.x * qs, x.y * qs, &qhi[i][j], &qlo[i][j]);
        }
    }
    float o[UW][2][4];
#pragma unroll
    for (int i = 0; i < UW; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) o[i][j >> 2][j & 3] = 0.0f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};  // heads 2 * warp and 2 * warp + 1
    const uint32_t busy = RANK ? 8u : (NU + UW - 1u) / UW;             // warps that own columns
    // this lane's ldmatrix rows: tokens (jm / 2) * 8 + lane % 8 as keys, (jm % 2) * 8 + lane % 8 as values, P's row lane % 16
    const uint32_t key_at = ((jm >> 1) * 8u + (lane & 7u)) * pitch + (jm & 1u) * 16u + warp * UW * 32u;
    const uint32_t val_at = ((jm & 1u) * 8u + (lane & 7u)) * pitch + (jm >> 1) * 16u + warp * UW * 32u;
    const uint32_t p_at = (uint32_t)__cvta_generic_to_shared(sp) + ((lane & 15u) * PITCH + (lane >> 4) * 8u) * 2u;
    float* sc_out = sc + ((size_t)warp * 16 + g) * PITCH + 2 * t4;
    const float* sc_in = sc + 2u * warp * PITCH + lane;

    // ring slots and use numbers of this tile and of the one to be requested
    uint32_t here = 0, here_use = 0, next = ahead % stages, next_use = ahead / stages;
    for (uint32_t tile = 0; tile < n_tiles; ++tile) {
        if (tile + ahead < n_tiles) {
            if (next_use > 0u) wait(&empty[next], (next_use - 1u) & 1u);
            load_tile(tile + ahead, next);
            landed_on(&full[next]);
        }
        if (++next == stages) next = 0, ++next_use;
        wait(&full[here], here_use & 1u);
        const uint32_t tile_at = ring + here * tile_bytes;
        if (warp < busy) {
            float s[LT / 8][4];
#pragma unroll
            for (int j = 0; j < LT / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.0f;
#pragma unroll
            for (int i = 0; i < UW; ++i) {
                if (!RANK && warp * UW + i >= NU) break;
#pragma unroll
                for (int p = 0; p < LT / 16; ++p) {
                    uint32_t b[4];
                    ldsm4(b, tile_at + key_at + p * 16u * pitch + i * 32u);
                    mma16816(s[2 * p], qhi[i][0], qhi[i][1], qhi[i][2], qhi[i][3], b[0], b[1]);
                    mma16816(s[2 * p + 1], qhi[i][0], qhi[i][1], qhi[i][2], qhi[i][3], b[2], b[3]);
                    mma16816(s[2 * p], qlo[i][0], qlo[i][1], qlo[i][2], qlo[i][3], b[0], b[1]);
                    mma16816(s[2 * p + 1], qlo[i][0], qlo[i][1], qlo[i][2], qlo[i][3], b[2], b[3]);
                }
            }
#pragma unroll
            for (int j = 0; j < LT / 8; ++j) {
                *reinterpret_cast<float2*>(sc_out + j * 8) = make_float2(s[j][0], s[j][1]);
                *reinterpret_cast<float2*>(sc_out + 8 * PITCH + j * 8) = make_float2(s[j][2], s[j][3]);
            }
        }
        team_barrier();
        {
            float v[2][TPL] = {}, mx[2], ps[2] = {0.0f, 0.0f};
#pragma unroll
            for (uint32_t w = 0; w < 8u; ++w)
                if (RANK || w < busy) {
#pragma unroll
                    for (int e = 0; e < 2; ++e)
#pragma unroll
                        for (int j = 0; j < TPL; ++j) v[e][j] += sc_in[(w * 16 + e) * PITCH + 32 * j];
                }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                mx[e] = -INFINITY;
#pragma unroll
                for (int j = 0; j < TPL; ++j) {
                    if (lo + tile * LT + lane + 32u * j >= hi) v[e][j] = -INFINITY;
                    mx[e] = fmaxf(mx[e], v[e][j]);
                }
            }
#pragma unroll
            for (int d = 16; d > 0; d >>= 1)  // the two heads' chains side by side
#pragma unroll
                for (int e = 0; e < 2; ++e) mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], d));
            float corr[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const float m_new = fmaxf(m_run[e], mx[e]);  // the tile's first token is visible: finite
                corr[e] = fast_exp2(m_run[e] - m_new);
                m_run[e] = m_new;
#pragma unroll
                for (int j = 0; j < TPL; ++j) {
                    const float p = fast_exp2(v[e][j] - m_new);
                    ps[e] += p;
                    sp[(2u * warp + e) * PITCH + lane + 32u * j] = __float2half_rn(p);
                }
            }
            // a lane keeps its own share of the sum; the shares meet at the end
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                l_run[e] = l_run[e] * corr[e] + ps[e];
                if (lane == 0) scorr[2u * warp + e] = corr[e];
            }
        }
        team_barrier();
        if (warp < busy) {
            const float ca = scorr[g], cb = scorr[g + 8];
            if (!__all_sync(0xffffffffu, ca == 1.0f && cb == 1.0f)) {
#pragma unroll
                for (int i = 0; i < UW; ++i)
#pragma unroll
                    for (int n = 0; n < 2; ++n) o[i][n][0] *= ca, o[i][n][1] *= ca, o[i][n][2] *= cb, o[i][n][3] *= cb;
            }
#pragma unroll
            for (int kk = 0; kk < LT / 16; ++kk) {
                uint32_t pa[4];
                ldsm4(pa, p_at + kk * 32u);
#pragma unroll
                for (int i = 0; i < UW; ++i) {
                    if (!RANK && warp * UW + i >= NU) break;
                    uint32_t b[4];
                    ldsm4_trans(b, tile_at + val_at + kk * 16u * pitch + i * 32u);
                    mma16816(o[i][0], pa[0], pa[1], pa[2], pa[3], b[0], b[1]);
                    mma16816(o[i][1], pa[0], pa[1], pa[2], pa[3], b[2], b[3]);
                }
            }
        }
        __syncwarp();
        if (lane == 0) tc::mbar_arrive(&empty[here]);
        if (++here == stages) here = 0, ++here_use;
    }
    cp_async_wait_all();
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const uint32_t h = 2u * warp + e;
        const float l = warp_sum(l_run[e]);
        if (lane == 0 && h < heads) {
            const size_t pi = ((size_t)row * a.heads + h0 + h) * a.splits + split;
            a.pm[pi] = m_run[e] * LN2;  // natural-log domain, as in the other form
            a.pl[pi] = l;
        }
    }
#pragma unroll
    for (int i = 0; i < UW; ++i) {
        const uint32_t u = warp * UW + i;
        if (!RANK && u >= NU) break;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const uint32_t h = g + 8u * j;
            if (h >= heads) continue;
            float* dst = a.po + (((size_t)row * a.heads + h0 + h) * a.splits + split) * rank + u * 16u + 2u * t4;
#pragma unroll
            for (int n = 0; n < 2; ++n) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[i][n][2 * j], o[i][n][2 * j + 1]);
        }
    }
}

// Cached f16 latents -> hi + lo in bf16 (exact: 8 + 8 significant bits cover 11).
__global__ void __launch_bounds__(256) latent_split_kernel(const __half* __restrict__ c, __nv_bfloat16* __restrict__ hi,
                                                           __nv_bfloat16* __restrict__ lo, size_t n) {
    pdl_wait();
    pdl_trigger();
    for (size_t i = ((size_t)blockIdx.x * 256u + threadIdx.x) * 8u; i < n; i += (size_t)gridDim.x * 2048u) {
        float v[8];
        m40_load8(c + i, v);
        __nv_bfloat16 h[8], l[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            h[j] = __float2bfloat16_rn(v[j]);
            l[j] = __float2bfloat16_rn(v[j] - __bfloat162float(h[j]));
        }
        *reinterpret_cast<uint4*>(hi + i) = *reinterpret_cast<const uint4*>(h);
        *reinterpret_cast<uint4*>(lo + i) = *reinterpret_cast<const uint4*>(l);
    }
}

// grid (heads, row groups of RG, slices of the values): splits and sink -> the head's weighted latent, then uv. Every slice
// merges for itself: the partials are in L2. SPLIT: the weighted latents are the result, as hi + lo (the caller applies uv).
template <typename WT, int RG, bool SPLIT>
__global__ void __launch_bounds__(256) latent_merge_kernel(LatArgs a) {
    extern __shared__ __align__(16) float so[];  // [RG][rank padded to 8], [RG][splits] weights, [256][RG] float4
    const uint32_t head = blockIdx.x, row0 = blockIdx.y * RG, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    const uint32_t rp = (a.rank + 7u) & ~7u, live = min((uint32_t)RG, a.rows - row0);
    float* sw = so + RG * rp;
    const uint32_t per = (a.vdim + gridDim.z - 1u) / gridDim.z, n_lo = blockIdx.z * per, n_hi = min(n_lo + per, a.vdim);
    const WT* uv = reinterpret_cast<const WT*>(a.uv) + (size_t)head * a.vdim * a.rank;
    // The weights do not depend on the previous kernel. One row of 16-bit weights: a warp's first four rows of uv go to
    // registers (their part of columns below 512), everything else to L2.
    constexpr bool HOLD = RG == 1 && !SPLIT && sizeof(WT) == 2;
    uint4 held[HOLD ? 4 : 1][2];
    if (!SPLIT && n_lo < n_hi) {
        if (HOLD && a.wide) {
#pragma unroll
            for (int j = 0; j < (HOLD ? 4 : 0); ++j) {
                const WT* w = uv + (size_t)min(n_lo + 2u * warp + (j >> 1) * 16u + (j & 1), n_hi - 1u) * a.rank;
#pragma unroll
                for (int i = 0; i < 2; ++i) held[j][i] = *reinterpret_cast<const uint4*>(w + min(lane * 8u + 256u * i, a.rank - 8u));
            }
        }
        const char* p = reinterpret_cast<const char*>(uv + (size_t)n_lo * a.rank);
        const size_t bytes = (size_t)(n_hi - n_lo) * a.rank * sizeof(WT);
        for (size_t i = (size_t)tid * 128u; i < bytes; i += 256u * 128u) prefetch_l2(p + i);
    }
    pdl_wait();
    pdl_trigger();
    if (warp < RG && warp < live) {  // one warp per row: the splits' weights (at most 128 splits)
        const size_t base = ((size_t)(row0 + warp) * a.heads + head) * a.splits;
        const float sink = a.sink ? a.sink[head] : -INFINITY;
        float l[4], m[4], M = sink, L = 0.0f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const uint32_t s = lane + 32u * i;
            l[i] = s < a.splits ? a.pl[base + s] : 0.0f;
            m[i] = s < a.splits ? a.pm[base + s] : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (l[i] > 0.0f) M = fmaxf(M, m[i]);
        M = warp_max(M);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            m[i] = l[i] > 0.0f ? expf(m[i] - M) : 0.0f;
            L = fmaf(l[i], m[i], L);
        }
        L = warp_sum(L);
        if (a.sink) L += expf(sink - M);
        const float inv = 1.0f / (L > 0.0f ? L : 1.0f);
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (lane + 32u * i < a.splits) sw[warp * a.splits + lane + 32u * i] = m[i] * inv;
    }
    // where column k of the weighted latent lies: the halves of every 8 columns apart, so that 16-byte reads of neighbouring
    // lanes fall into different banks
    auto place = [&](uint32_t k) { return ((k & 4u) ? rp / 2u : 0u) + (k >> 3) * 4u + (k & 3u); };
    if (a.rank % 4u == 0u) {
        const uint32_t c4 = a.rank / 4u, teams = 256u / c4, team = tid / c4, col = tid % c4;  // rank <= 1024
        const bool busy = team < teams;
        float4* st = reinterpret_cast<float4*>(sw + ((RG * a.splits + 3u) & ~3u));
        constexpr int AHEAD = RG == 1 ? 16 : 4;  // partials requested before the weights are known, per row
        float4 x[RG][AHEAD];
        const float4* o0 = reinterpret_cast<const float4*>(a.po + ((size_t)row0 * a.heads + head) * a.splits * a.rank) + (busy ? col : 0u);
        const size_t row_step = (size_t)a.heads * a.splits * c4;
#pragma unroll
        for (int r = 0; r < RG; ++r)
#pragma unroll
            for (int i = 0; i < AHEAD; ++i)
                x[r][i] = o0[min((uint32_t)r, live - 1u) * row_step + (size_t)min((busy ? team : 0u) + i * teams, a.splits - 1u) * c4];
        __syncthreads();
        auto add = [](float4& t, float w, const float4& v) {
            if (w != 0.0f)  // empty splits may hold anything
                t.x = fmaf(w, v.x, t.x), t.y = fmaf(w, v.y, t.y), t.z = fmaf(w, v.z, t.z), t.w = fmaf(w, v.w, t.w);
        };
#pragma unroll
        for (int r = 0; r < RG; ++r) {
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            if (busy && (uint32_t)r < live) {
                const float* w = sw + r * a.splits;
#pragma unroll
                for (int i = 0; i < AHEAD; ++i)
                    if (team + i * teams < a.splits) add(acc, w[team + i * teams], x[r][i]);
#pragma unroll 8
                for (uint32_t s = team + AHEAD * teams; s < a.splits; s += teams) add(acc, w[s], o0[r * row_step + (size_t)s * c4]);
            }
            st[tid * RG + r] = acc;
        }
        __syncthreads();
        for (uint32_t i = tid; i < RG * c4; i += 256u) {
            const uint32_t r = i / c4, c = i % c4;
            float4 t = st[c * RG + r];
            for (uint32_t k = 1; k < teams; ++k) {
                const float4 u = st[(k * c4 + c) * RG + r];
                t.x += u.x, t.y += u.y, t.z += u.z, t.w += u.w;
            }
            if (!SPLIT) *reinterpret_cast<float4*>(so + r * rp + place(4u * c)) = t;
            else if (r < live) split_store4(a.part[0], a.part[1], ((size_t)(row0 + r) * a.heads + head) * a.rank + 4u * c, t);
        }
    } else {
        __syncthreads();
        for (uint32_t i = tid; i < RG * rp; i += 256u) {
            const uint32_t r = i / rp, c = i % rp;
            float t = 0.0f;
            if (r < live && c < a.rank) {
                const float* w = sw + r * a.splits;
                const float* o = a.po + ((size_t)(row0 + r) * a.heads + head) * a.splits * a.rank + c;
                for (uint32_t s = 0; s < a.splits; ++s) {
                    const float ws = w[s], x = ws != 0.0f ? o[(size_t)s * a.rank] : 0.0f;
                    t = fmaf(ws, x, t);
                }
            }
            so[r * rp + place(c)] = t;
        }
    }
    if (SPLIT) return;
    __syncthreads();
    for (uint32_t n0 = n_lo + 2u * warp, it = 0; n0 < n_hi; n0 += 16u, ++it) {  // two values at a time
        const uint32_t n1 = min(n0 + 1u, n_hi - 1u);
        const WT *w0 = uv + (size_t)n0 * a.rank, *w1 = uv + (size_t)n1 * a.rank;
        float acc[2][RG] = {};
        if (a.wide) {
            auto piece = [&](uint32_t k, const float* v0, const float* v1) {
#pragma unroll
                for (int r = 0; r < RG; ++r) {
                    const float4 x0 = *reinterpret_cast<const float4*>(so + r * rp + (k >> 1));
                    const float4 x1 = *reinterpret_cast<const float4*>(so + r * rp + rp / 2u + (k >> 1));
                    const float x[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[0][r] = fmaf(v0[i], x[i], acc[0][r]), acc[1][r] = fmaf(v1[i], x[i], acc[1][r]);
                }
            };
            uint32_t k = lane * 8u;
            if (HOLD && it < 2u) {
#pragma unroll
                for (int i = 0; i < 2; ++i, k += 256u) {
                    if (k >= a.rank) break;
                    float v0[8], v1[8];
                    const uint4 h0 = it == 0u ? held[0][i] : held[HOLD ? 2 : 0][i], h1 = it == 0u ? held[HOLD ? 1 : 0][i] : held[HOLD ? 3 : 0][i];
                    m40_load8(reinterpret_cast<const WT*>(&h0), v0);
                    m40_load8(reinterpret_cast<const WT*>(&h1), v1);
                    piece(k, v0, v1);
                }
            }
#pragma unroll 2
            for (; k < a.rank; k += 256u) {
                float v0[8], v1[8];
                m40_load8(w0 + k, v0);
                m40_load8(w1 + k, v1);
                piece(k, v0, v1);
            }
        } else {
            for (uint32_t k = lane; k < a.rank; k += 32u) {
                const float v0 = m40_load_elem(w0 + k), v1 = m40_load_elem(w1 + k);
#pragma unroll
                for (int r = 0; r < RG; ++r) {
                    const float x = so[r * rp + place(k)];
                    acc[0][r] = fmaf(v0, x, acc[0][r]), acc[1][r] = fmaf(v1, x, acc[1][r]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int r = 0; r < RG; ++r) {
                const float v = warp_sum(acc[j][r]);
                if (lane == 0 && (uint32_t)r < live && n0 + j < n_hi) a.out[((size_t)(row0 + r) * a.heads + head) * a.vdim + n0 + j] = v;
            }
    }
}

// Rows per prepare CTA: 8 when there are several (their queries fit shared memory), and the latent columns that go with it.
uint32_t prepare_rows(const LatArgs& a) { return a.rows > 1 && a.dim <= 256 ? 8u : 1u; }
uint32_t absorb_ctas(const LatArgs& a) {
    const uint32_t cols = prepare_rows(a) == 8 ? 128u : 64u;
    return a.heads * ((a.rank + cols - 1) / cols);
}

template <typename WT, typename ET>
cudaError_t launch_prepare(cudaStream_t s, const LatArgs& a, bool append) {
    const uint32_t rg = prepare_rows(a);
    const dim3 grid(a.absorb_ctas + (append ? rg : 0u), (a.rows + rg - 1) / rg);
    const size_t smem = (size_t)rg * a.dim * sizeof(float);
    return rg == 8 ? m40_launch_dependent(latent_prepare_kernel<WT, ET, 8, 128>, grid, dim3(256), smem, s, a)
                   : m40_launch_dependent(latent_prepare_kernel<WT, ET, 1, 64>, grid, dim3(256), smem, s, a);
}

template <typename WT>
cudaError_t launch_merge(M40llmCudaContext* ctx, const LatArgs& a, bool split) {
    const uint32_t rp = (a.rank + 7u) & ~7u, rg = a.rows == 1 ? 1u : 4u, groups = (a.rows + rg - 1) / rg;
    uint32_t z = (uint32_t)ctx->sm_count / (a.heads * groups);
    const uint32_t z_max = (a.vdim + 15u) / 16u;
    z = z < 1u ? 1u : (z > z_max ? z_max : z);
    const size_t smem = ((size_t)rg * rp + (((size_t)rg * a.splits + 3) & ~(size_t)3) + (size_t)256 * 4 * rg) * sizeof(float);
    const dim3 grid(a.heads, groups, split ? 1 : z);
    if (split) return m40_launch_dependent(latent_merge_kernel<WT, 4, true>, grid, dim3(256), smem, ctx->decode_stream, a);
    return rg == 1 ? m40_launch_dependent(latent_merge_kernel<WT, 1, false>, grid, dim3(256), smem, ctx->decode_stream, a)
                   : m40_launch_dependent(latent_merge_kernel<WT, 4, false>, grid, dim3(256), smem, ctx->decode_stream, a);
}

template <typename WT>
cudaError_t prepare(cudaStream_t s, const LatArgs& a, bool f32, bool append) {
    return f32 ? launch_prepare<WT, float>(s, a, append) : launch_prepare<WT, __half>(s, a, append);
}

template <int UW, int RANK, int TEAMS>
cudaError_t launch_tiles_as(M40llmCudaContext* ctx, const LatArgs& a) {
    static unsigned long long configured = 0ull;
    const unsigned long long bit = 1ull << (ctx->device_id & 63);
    auto kernel = latent_tiles_kernel<UW, RANK, TEAMS>;
    if (!(configured & bit)) {
        const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TILE_SMEM_ALONE);
        if (e != cudaSuccess) return e;
        configured |= bit;
    }
    const dim3 grid(a.splits, (a.heads + 16 * TEAMS - 1) / (16 * TEAMS), a.rows);
    // a launch that gives every SM at most one CTA lets it have the shared memory of two: a deeper ring
    const bool alone = TEAMS == 2 || (uint64_t)grid.x * grid.y * grid.z <= (uint64_t)ctx->sm_count;
    constexpr size_t fixed = TEAMS * LatTile<UW>::FIXED;
    size_t stages = ((alone ? TILE_SMEM_ALONE : TILE_SMEM) - fixed) / LatTile<UW>::bytes(a.rank);
    if (stages > MAX_STAGES) stages = MAX_STAGES;
    return m40_launch_dependent(kernel, grid, dim3(256 * TEAMS), fixed + stages * LatTile<UW>::bytes(a.rank), ctx->decode_stream, a,
                                (uint32_t)stages);
}
template <int UW>
cudaError_t launch_tiles(M40llmCudaContext* ctx, const LatArgs& a, uint32_t teams) {
    if (teams == 2) return a.rank == 128u * UW ? launch_tiles_as<UW, 128 * UW, 2>(ctx, a) : launch_tiles_as<UW, 0, 2>(ctx, a);
    return a.rank == 128u * UW ? launch_tiles_as<UW, 128 * UW, 1>(ctx, a) : launch_tiles_as<UW, 0, 1>(ctx, a);
}
static_assert(LatTile<2>::FIXED + 2 * LatTile<2>::bytes(256) <= TILE_SMEM && LatTile<4>::FIXED + 2 * LatTile<4>::bytes(512) <= TILE_SMEM,
              "two tiles of the largest rank");
static_assert(2 * LatTile<4>::FIXED + 2 * LatTile<4>::bytes(512) <= TILE_SMEM_ALONE, "two teams");

// Tokens per split: as many splits as keep every CTA of the launch resident (`slots` of them), at least 128 tokens each; at most
// 1024, because the bound may be the cache's capacity when the lengths are not known.
// A split is a multiple of `unit` tokens.
void pick_splits(uint32_t slots, uint32_t ctas_per_split, uint32_t bound, uint32_t unit, uint32_t* chunk, uint32_t* splits) {
    uint32_t n = slots / ctas_per_split;
    if (n <= 1u) {  // rows enough: no splits, whatever the length
        *chunk = bound;
        *splits = 1u;
        return;
    }
    n = n > 128u ? 128u : n;
    auto whole = [&](uint32_t v) { return (v + unit - 1) / unit * unit; };
    uint32_t c = whole((bound + n - 1) / n);
    c = c < 128u ? 128u : (c > 1024u ? 1024u : c);
    if ((bound + c - 1) / c > 128u) c = whole((bound + 127u) / 128u);
    *chunk = c;
    *splits = (bound + c - 1) / c;
}

// Whether uk and uv of several rows go through the grouped GEMM.
bool takes_grouped(const M40llmKVCache* kv, const LatArgs& a, uint32_t w_dtype) {
    return !kv->elem_f32 && w_dtype == M40LLM_DT_BF16 && a.uk_t && a.ld % 4 == 0 && (((uintptr_t)a.packed | (uintptr_t)a.out) & 15u) == 0 &&
           m40_gemm_tc_grouped_supported(a.uk_t, a.rank, a.dim, a.heads * a.dim, a.dim) &&
           m40_gemm_tc_grouped_supported(a.uv, a.vdim, a.rank, a.heads * a.rank, a.rank);
}

// out[row][head * N ..] = the head's matrix [N][K] times x[row][head * K ..], x as hi + lo.
int per_head(M40llmCudaContext* ctx, const LatArgs& a, const void* w, uint32_t N, uint32_t K, float* out) {
    M40GroupedCall c = {};
    c.w = w;
    c.x[0] = a.part[0], c.x[1] = a.part[1];
    c.parts = 2;
    c.bf16 = 1;
    c.groups = a.heads;
    c.N = N;
    c.K = c.group_k = K;
    c.x_rows = a.rows;
    c.ldx = a.heads * K;
    c.tile_rows = a.rows <= 16 ? 16 : (a.rows <= 32 ? 32 : (a.rows <= 64 ? 64 : 128));
    c.kind = M40_GROUPED_F32;
    c.out = out;
    c.out_ld = a.heads * N;
    c.out_group = N;
    return m40_gemm_tc_grouped(ctx, ctx->decode_stream, c);
}

// Absorbed form over the rows of `all`; append: the latents are not in the cache yet.
template <typename WT>
int run_absorbed(M40llmCudaContext* ctx, const M40llmKVCache* kv, const LatArgs& all, uint32_t bound, bool append, uint32_t w_dtype) {
    cudaStream_t s = ctx->decode_stream;
    const bool tiles = !kv->elem_f32 && all.rank % 16 == 0 && all.rank <= 512;
    cudaError_t e;
    for (uint32_t at = 0; at < all.rows; at += RUN_ROWS) {
        LatArgs a = all;
        a.rows = all.rows - at < RUN_ROWS ? all.rows - at : RUN_ROWS;
        a.packed += (size_t)at * a.ld;
        a.out += (size_t)at * a.heads * a.vdim;
        a.row_seq += at;
        a.row_pos += at;
        const bool grouped = a.rows >= GROUPED_ROWS && takes_grouped(kv, a, w_dtype);
        // a few rows: smaller CTAs start sooner; else tcgen05, or two teams per CTA where there are heads for them
        const bool tc = tiles && a.rows >= TEAM_ROWS && m40_latent_tc_takes(a);
        const uint32_t teams = tiles && a.heads > 16 && a.rows >= TEAM_ROWS ? 2 : 1, sms = (uint32_t)ctx->sm_count;
        const uint32_t g16 = (a.heads + 15) / 16, g32 = (a.heads + 31) / 32;
        if (tc || teams == 2) pick_splits(sms, a.rows * g32, bound, tc ? 128u : 64u, &a.chunk, &a.splits);
        else pick_splits(2u * sms, a.rows * (tiles ? g16 : a.heads), bound, 64u, &a.chunk, &a.splits);
        const size_t nh = (size_t)a.rows * a.heads, np = nh * a.splits;
        auto pad = [](size_t v) { return (v + 63) & ~(size_t)63; };
        const size_t part = grouped ? pad(nh * (a.rank > a.dim ? a.rank : a.dim)) : 0;  // 16-bit values
        float* work = (float*)m40_ensure_scratch(ctx, 1, (pad(nh * a.rank) + pad(np * a.rank) + 2 * pad(np) + part) * sizeof(float) + 256, 1);
        if (!work) return -5;
        work = (float*)(((uintptr_t)work + 255) & ~(uintptr_t)255);
        a.qa = work;
        a.po = work + pad(nh * a.rank);
        a.pm = a.po + pad(np * a.rank);
        a.pl = a.pm + pad(np);
        a.part[0] = (__nv_bfloat16*)(a.pl + pad(np));
        a.part[1] = a.part[0] + part;
        int rc;
        if (grouped) {
            const uint32_t shares = (a.heads * a.dim + 1023) / 1024;
            e = m40_launch_dependent(latent_append_kernel, dim3(a.rows, 1 + (shares < 4 ? shares : 4)), dim3(256), 0, s, a, append ? 1u : 0u);
            M40_COUNT_LAUNCH(ctx);
            if (e != cudaSuccess) return -6;
            if ((rc = per_head(ctx, a, a.uk_t, a.rank, a.dim, a.qa)) != 0) return rc;
        } else {
            a.absorb_ctas = absorb_ctas(a);
            e = prepare<WT>(s, a, kv->elem_f32, append);
            M40_COUNT_LAUNCH(ctx);
            if (e != cudaSuccess) return -6;
        }
        const dim3 grid(a.heads, a.rows, a.splits);
        if (tc) {
            if ((rc = m40_latent_tc(ctx, a)) != 0) return rc;
        } else if (tiles) {
            e = a.rank <= 128 ? launch_tiles<1>(ctx, a, teams)
                              : (a.rank <= 256 ? launch_tiles<2>(ctx, a, teams) : launch_tiles<4>(ctx, a, teams));
            M40_COUNT_LAUNCH(ctx);
        } else {
            e = kv->elem_f32 ? m40_launch_dependent(latent_rows_kernel<float>, grid, dim3(128), 0, s, a)
                             : m40_launch_dependent(latent_rows_kernel<__half>, grid, dim3(128), 0, s, a);
            M40_COUNT_LAUNCH(ctx);
        }
        if (e != cudaSuccess) return -6;
        e = launch_merge<WT>(ctx, a, grouped);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess || cudaGetLastError() != cudaSuccess) return -6;
        if (grouped && (rc = per_head(ctx, a, a.uv, a.vdim, a.rank, a.out)) != 0) return rc;
    }
    return 0;
}

bool takes_expanded(const M40llmKVCache* kv, const LatArgs& a, uint32_t w_dtype) {
    return !kv->elem_f32 && w_dtype != M40LLM_DT_F32 && a.dim <= 128 && a.vdim <= 128 && a.dim % 2 == 0 && a.vdim % 2 == 0 &&
           a.ld % 2 == 0 && (((uintptr_t)a.packed | (uintptr_t)a.out) & 7u) == 0 && (a.heads * a.vdim) % 2 == 0 &&
           m40_gemm_tc_grouped_supported(a.uk, a.heads * a.dim, a.rank, a.rank, 0) &&
           m40_gemm_tc_grouped_supported(a.uv, a.heads * a.vdim, a.rank, a.rank, 0);
}
size_t expanded_bytes(const LatArgs& a, uint32_t kv_len, uint32_t hd) {
    return (size_t)kv_len * ((size_t)a.heads * hd * 4 + (size_t)a.rank * 4) + 1024;
}

// One portion (its latents are in the cache): the heads' keys and values, then the prompt kernel. seg is on the device.
int run_expanded(M40llmCudaContext* ctx, const LatArgs& a, uint32_t w_dtype, const uint32_t* seg, const uint32_t* seg_host) {
    cudaStream_t s = ctx->decode_stream;
    const uint32_t hd = a.dim <= 64 && a.vdim <= 64 ? 64u : 128u, n = seg_host[3] + seg_host[1];
    const uint32_t slot = seg_host[2] * a.slot_mul + a.slot_add;
    const __half* C = reinterpret_cast<const __half*>(a.C) + (size_t)slot * a.max_seq_len * a.rank;
    const size_t kv_elems = (size_t)n * a.heads * hd, c_elems = (size_t)n * a.rank;
    unsigned char* work = (unsigned char*)m40_ensure_scratch(ctx, 1, expanded_bytes(a, n, hd), 1);
    if (!work) return -5;
    work = (unsigned char*)(((uintptr_t)work + 255) & ~(uintptr_t)255);
    __half *K = (__half*)work, *V = K + kv_elems;
    const bool bf16 = w_dtype == M40LLM_DT_BF16;
    M40GroupedCall c = {};
    c.x[0] = C;
    c.parts = 1;
    cudaError_t e;
    if (bf16) {
        __nv_bfloat16 *hi = (__nv_bfloat16*)(((uintptr_t)(V + kv_elems) + 127) & ~(uintptr_t)127), *lo = hi + c_elems;
        const size_t blocks = (c_elems + 2047) / 2048;
        e = m40_launch_dependent(latent_split_kernel, dim3((unsigned)(blocks < 4096 ? blocks : 4096)), dim3(256), 0, s, C, hi, lo, c_elems);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess) return -6;
        c.x[0] = hi, c.x[1] = lo;
        c.parts = 2;
    }
    // dimensions beyond a head's own are zeros
    if (a.dim < hd && cudaMemsetAsync(K, 0, kv_elems * 2, s) != cudaSuccess) return -6;
    if (a.vdim < hd && cudaMemsetAsync(V, 0, kv_elems * 2, s) != cudaSuccess) return -6;
    c.bf16 = bf16;
    c.groups = 1;
    c.K = c.ldx = a.rank;
    c.x_rows = n;
    c.tile_rows = 128;
    c.kind = M40_GROUPED_HEADS;
    c.head_pitch = hd;
    c.w = a.uk;
    c.N = a.heads * a.dim;
    c.head_dim = a.dim;
    c.heads = K;
    int rc = m40_gemm_tc_grouped(ctx, s, c);
    if (rc != 0) return rc;
    c.w = a.uv;
    c.N = a.heads * a.vdim;
    c.head_dim = a.vdim;
    c.heads = V;
    if ((rc = m40_gemm_tc_grouped(ctx, s, c)) != 0) return rc;
    M40PrefillCall p = {};
    p.K = K;
    p.V = V;
    p.q = a.packed;
    p.out = a.out;
    p.seg = seg;
    p.sink = a.sink;
    p.segments = 1;
    p.max_segment_rows = seg_host[1];
    p.rows = a.rows;
    p.hd = hd;
    p.q_heads = p.kv_heads = a.heads;
    p.q_ld = a.ld;
    p.q_dim = a.dim;
    p.out_ld = a.heads * a.vdim;
    p.v_dim = a.vdim;
    p.slots = 1;
    p.max_seq_len = n;
    p.scale = a.scale;
    rc = m40_attention_prefill(ctx, p);
    return rc > 0 ? -6 : rc;
}

template <typename WT>
int run(M40llmCudaContext* ctx, const M40llmKVCache* kv, const LatArgs& all, uint32_t bound, uint32_t w_dtype, const M40llmStepRows& r) {
    const uint32_t hd = all.dim <= 64 && all.vdim <= 64 ? 64u : 128u;
    // the portion's host copy decides its form; out-of-range portions take the absorbed form, which checks them on the device
    auto expands = [&](const uint32_t* sg) {
        return sg[1] >= EXPAND_ROWS && (uint64_t)sg[0] + sg[1] <= all.rows && (uint64_t)sg[3] + sg[1] <= all.max_seq_len &&
               (uint64_t)sg[2] * all.slot_mul + all.slot_add < all.slots && expanded_bytes(all, sg[3] + sg[1], hd) <= EXPAND_BYTES;
    };
    bool any = false;
    if (r.seg_host && r.seg && r.max_segment_rows >= EXPAND_ROWS && takes_expanded(kv, all, w_dtype))
        for (uint32_t i = 0; i < r.segments; ++i) any = any || expands(r.seg_host + 4 * i);
    // several launches read the cache: every latent of the step is appended first
    const bool first = any || all.rows > RUN_ROWS;
    if (first) {
        LatArgs a = all;
        a.absorb_ctas = 0;
        const cudaError_t e = prepare<WT>(ctx->decode_stream, a, kv->elem_f32, true);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess) return -6;
    }
    if (!any) return run_absorbed<WT>(ctx, kv, all, bound, !first, w_dtype);
    uint32_t run0 = 0;  // first row of the absorbed run that is being gathered
    for (uint32_t i = 0; i <= r.segments; ++i) {
        const uint32_t* sg = i < r.segments ? r.seg_host + 4 * i : nullptr;
        if (sg && !expands(sg)) continue;
        const uint32_t end = sg ? sg[0] : all.rows;
        if (end > run0) {
            LatArgs a = all;
            a.rows = end - run0;
            a.packed += (size_t)run0 * a.ld;
            a.out += (size_t)run0 * a.heads * a.vdim;
            a.row_seq += run0;
            a.row_pos += run0;
            const int rc = run_absorbed<WT>(ctx, kv, a, bound, false, w_dtype);
            if (rc != 0) return rc;
        }
        if (!sg) break;
        const int rc = run_expanded(ctx, all, w_dtype, r.seg + 4 * i, sg);
        if (rc != 0) return rc;
        run0 = sg[0] + sg[1];
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
    a.uk_t = c->uk_t;
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
    if (c->w_dtype == M40LLM_DT_F32) return run<float>(ctx, kv, a, bound, c->w_dtype, *r);
    return c->w_dtype == M40LLM_DT_BF16 ? run<__nv_bfloat16>(ctx, kv, a, bound, c->w_dtype, *r) : run<__half>(ctx, kv, a, bound, c->w_dtype, *r);
}
