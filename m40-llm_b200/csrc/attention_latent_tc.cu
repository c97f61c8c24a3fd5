// Decode attention over latents on the 5th-generation tensor cores: CTA = (row, 16 or 32 heads, token split).
//
// The heads' absorbed queries are one small matrix, and the cached latents are its only other operand, as keys and as values.
// A tile is 128 tokens; its latents lie in shared memory once, 128-byte swizzled, in pairs of 64-column chunks:
//
//   scores   S[128 tokens][2 HP]  = C Q^T     A = the tile, K-major; B = the queries as f16 hi over lo rows (HP heads each), so
//                                             that hi + lo of a score are two columns of one accumulator lane;
//   softmax  thread = token = accumulator lane: 32 scores in registers. Maxima over the tokens meet by a transposing butterfly
//            (31 shuffles for 32 heads) and shared memory. A head's reference moves only when its maximum has grown by 2^8 or
//            more (weights stay in f16 range below that), so the accumulated output is rarely rescaled;
//   values   O^T[rank][HP]       += C^T P     A = the same bytes, MN-major, 128 latent columns at a time; B = the weights.
//
// Warp 0 loads by TMA, warp 1 issues the MMAs, warps 2..5 are the tokens. A pair is released when its value product has been
// committed, so the next tile arrives while this one's values are being multiplied. Every wait is bounded: a wait that runs
// out raises status bit 4; nothing waits any more from then on, the CTA's copies are drained and its TMEM is freed.
#include "attention_latent.cuh"
#include "attention_mma.cuh"
#include "gemm_tc.cuh"
#include "tc_ptx.cuh"

namespace {

using namespace tc;
using attn_mma::fast_exp2;
using attn_mma::LN2;
using attn_mma::LOG2E;

constexpr uint32_t TOKENS = 128, PAIR_BYTES = 2 * TOKENS * 128, CHUNK_BYTES = TOKENS * 128;
constexpr uint32_t MAX_SLOTS = 6;
constexpr size_t SMEM_BUDGET = 226 * 1024;

// MN-major, 128-byte-swizzled operand: 64-element chunks along MN are lbo bytes apart, groups of 8 along K 1024 bytes.
__device__ __forceinline__ uint64_t make_desc_mn_sw128(uint32_t smem_addr, uint32_t lbo) {
    uint64_t d = 0;
    d |= (uint64_t)((smem_addr & 0x3FFFFu) >> 4);
    d |= (uint64_t)(lbo >> 4) << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
constexpr uint32_t IDESC_A_MN = 1u << 15;

template <int HP>
struct Layout {
    static constexpr uint32_t Q_CHUNK = 2 * HP * 128;  // hi and lo rows of 64 columns
    static constexpr uint32_t P_CHUNK = HP * 128;      // weights of 64 tokens
    static constexpr size_t fixed(uint32_t rank) { return (size_t)(rank / 64) * Q_CHUNK + 2 * P_CHUNK + 6 * HP * 4 + 256; }
    static uint32_t slots(uint32_t rank) {
        const size_t n = (SMEM_BUDGET - 1024 - fixed(rank)) / PAIR_BYTES;
        return (uint32_t)(n < MAX_SLOTS ? n : MAX_SLOTS);
    }
};

// N values of 32 lanes -> each lane holds the reduction of one: value (lane % N). OP(a, b).
template <int N, typename Op>
__device__ __forceinline__ float transposed_reduce(float (&v)[N], uint32_t lane, Op op) {
    if (N == 16) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = op(v[i], __shfl_xor_sync(0xffffffffu, v[i], 16));
    }
#pragma unroll
    for (int w = N / 2; w > 0; w >>= 1) {
        const bool up = (lane & (uint32_t)w) != 0u;
#pragma unroll
        for (int i = 0; i < w; ++i) {
            const float send = up ? v[i] : v[i + w], keep = up ? v[i + w] : v[i];
            v[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, w));
        }
    }
    return v[0];
}

template <int HP>
__device__ __forceinline__ void tmem_ld_hp(uint32_t addr, float (&v)[HP]) {
    uint32_t r[HP];
    if constexpr (HP == 32) tmem_ld_x32(addr, r);
    else tmem_ld_x16(addr, r);
    tmem_ld_wait();
#pragma unroll
    for (int i = 0; i < HP; ++i) v[i] = __uint_as_float(r[i]);
}

template <int HP>
__global__ void __launch_bounds__(192, 1) latent_tc_kernel(const __grid_constant__ CUtensorMap tmC, M40LatArgs a, uint32_t slots) {
    extern __shared__ unsigned char smem_unaligned[];
    unsigned char* smem = smem_unaligned + ((1024u - (smem_u32(smem_unaligned) & 1023u)) & 1023u);
    __shared__ uint64_t full[MAX_SLOTS], empty[MAX_SLOTS], q_ready, s_done, p_ready, o_done;
    __shared__ uint32_t tmem_slot;
    __shared__ volatile uint32_t abort_flag;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, NP = a.rank / 128u;
    unsigned char* ring = smem;
    unsigned char* sq = ring + slots * PAIR_BYTES;
    unsigned char* sp = sq + (a.rank / 64u) * Layout<HP>::Q_CHUNK;
    float* s_max = reinterpret_cast<float*>(sp + 2 * Layout<HP>::P_CHUNK);  // [4][HP]
    float* s_ref = s_max + 4 * HP;                                          // [HP]
    float* s_corr = s_ref + HP;                                             // [HP]
    __shared__ uint32_t s_rescale;

    if (threadIdx.x == 0) {
        for (uint32_t i = 0; i < slots; ++i) {
            mbar_init(&full[i], 1);
            mbar_init(&empty[i], 1);
        }
        mbar_init(&q_ready, 128);
        mbar_init(&s_done, 1);
        mbar_init(&p_ready, 128);
        mbar_init(&o_done, 1);
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    pdl_wait();
    const uint32_t split = blockIdx.x, h0 = blockIdx.y * HP, row = blockIdx.z;
    const uint32_t pos = a.row_pos[row], slot = a.row_seq[row] * a.slot_mul + a.slot_add;
    const uint32_t lo = split * a.chunk, hi = min(lo + a.chunk, pos + 1u), heads = min((uint32_t)HP, a.heads - h0);
    const size_t part0 = ((size_t)row * a.heads + h0) * a.splits + split;  // head h: + h * splits
    if (slot >= a.slots || pos >= a.max_seq_len || lo >= hi) {             // empty partials
        pdl_trigger();
        if (threadIdx.x < heads) a.pm[part0 + (size_t)threadIdx.x * a.splits] = -INFINITY, a.pl[part0 + (size_t)threadIdx.x * a.splits] = 0.0f;
        return;
    }
    constexpr uint32_t S_COLS = 2 * HP;
    const uint32_t used_cols = S_COLS + NP * HP;
    uint32_t tmem_cols = 32;
    while (tmem_cols < used_cols) tmem_cols <<= 1;
    if (warp == 1) tmem_alloc(&tmem_slot, tmem_cols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_s = tmem_slot, tmem_o = tmem_s + S_COLS;
    pdl_trigger();
    const uint32_t n_tiles = (hi - lo + TOKENS - 1u) / TOKENS;
    auto wait = [&](uint64_t* bar, uint32_t parity) {
        if (abort_flag) return false;
        if (mbar_wait(bar, parity)) return true;
        abort_flag = 1;
        atomicOr(a.status, 4u);
        return false;
    };

    if (warp == 0) {
        if (lane == 0) {
            const int row0 = (int)(slot * a.max_seq_len + lo);
            uint32_t s = 0, use = 0, issued = 0;
            const uint32_t total = n_tiles * NP;
            for (; issued < total; ++issued) {
                if (use > 0 && !wait(&empty[s], (use - 1u) & 1u)) break;
                const uint32_t t = issued / NP, b = issued % NP;
                unsigned char* dst = ring + s * PAIR_BYTES;
                mbar_expect_tx(&full[s], PAIR_BYTES);
                tma_load_2d(dst, &tmC, &full[s], (int)(b * 128u), row0 + (int)(t * TOKENS));
                tma_load_2d(dst + CHUNK_BYTES, &tmC, &full[s], (int)(b * 128u + 64u), row0 + (int)(t * TOKENS));
                if (++s == slots) s = 0, ++use;
            }
            if (abort_flag)  // copies in flight land (bounded) before the CTA goes away
                for (uint32_t i = issued > slots ? issued - slots : 0u; i < issued; ++i) mbar_wait(&full[i % slots], (i / slots) & 1u);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_s = make_idesc(S_COLS), idesc_o = make_idesc(HP) | IDESC_A_MN;
            const uint32_t ring_at = smem_u32(ring), q_at = smem_u32(sq), p_at = smem_u32(sp);
            bool ok = wait(&q_ready, 0);
            uint32_t s0 = 0, use0 = 0;  // ring slot and use of the tile's first pair
            for (uint32_t t = 0; t < n_tiles && ok; ++t) {
                uint32_t s = s0, use = use0;
                for (uint32_t b = 0; b < NP && ok; ++b) {
                    ok = wait(&full[s], use & 1u);
                    if (!ok) break;
                    tc_fence_after();
#pragma unroll
                    for (uint32_t j = 0; j < 8; ++j)  // chunk j / 4 of the pair, 16 columns each
                        umma_f16(tmem_s, make_desc_sw128(ring_at + s * PAIR_BYTES + (j >> 2) * CHUNK_BYTES + (j & 3u) * 32u),
                                 make_desc_sw128(q_at + (2u * b + (j >> 2)) * Layout<HP>::Q_CHUNK + (j & 3u) * 32u), idesc_s, (b | j) != 0u);
                    if (++s == slots) s = 0, ++use;
                }
                if (!ok) break;
                umma_commit(&s_done);
                ok = wait(&p_ready, t & 1u);
                if (!ok) break;
                tc_fence_after();
                s = s0;
                for (uint32_t b = 0; b < NP; ++b) {
#pragma unroll
                    for (uint32_t k = 0; k < 8; ++k)  // 16 tokens each
                        umma_f16(tmem_o + b * HP, make_desc_mn_sw128(ring_at + s * PAIR_BYTES + k * 2048u, CHUNK_BYTES),
                                 make_desc_sw128(p_at + (k >> 2) * Layout<HP>::P_CHUNK + (k & 3u) * 32u), idesc_o, (t | k) != 0u);
                    umma_commit(&empty[s]);
                    if (++s == slots) s = 0;
                }
                for (uint32_t b = 0; b < NP; ++b)
                    if (++s0 == slots) s0 = 0, ++use0;
            }
            if (ok) umma_commit(&o_done);
        }
    } else {
        const uint32_t group = warp & 3u, tok = group * 32u + lane, tid = threadIdx.x - 64u;
        const uint32_t lane_addr = (group * 32u) << 16;
        // ---- the queries, scaled to base 2, as f16 hi rows 0 .. HP - 1 and lo rows HP .. 2 HP - 1
        {
            const float qs = a.scale * LOG2E;
            const uint32_t pieces = a.rank / 8u;
#pragma unroll 8
            for (uint32_t i = tid; i < HP * pieces; i += 128u) {
                const uint32_t h = i / pieces, pc = i % pieces;
                float4 x0 = make_float4(0.f, 0.f, 0.f, 0.f), x1 = x0;
                if (h < heads) {
                    const float4* q = reinterpret_cast<const float4*>(a.qa + ((size_t)row * a.heads + h0 + h) * a.rank + pc * 8u);
                    x0 = q[0], x1 = q[1];
                }
                uint32_t hi4[4], lo4[4];
                attn_mma::split_h2(x0.x * qs, x0.y * qs, &hi4[0], &lo4[0]);
                attn_mma::split_h2(x0.z * qs, x0.w * qs, &hi4[1], &lo4[1]);
                attn_mma::split_h2(x1.x * qs, x1.y * qs, &hi4[2], &lo4[2]);
                attn_mma::split_h2(x1.z * qs, x1.w * qs, &hi4[3], &lo4[3]);
                // rows h and HP + h share h % 8 (HP is a multiple of 8)
                unsigned char* dst = sq + (pc >> 3) * Layout<HP>::Q_CHUNK + h * 128u + (((pc & 7u) ^ (h & 7u)) << 4);
                *reinterpret_cast<uint4*>(dst) = make_uint4(hi4[0], hi4[1], hi4[2], hi4[3]);
                *reinterpret_cast<uint4*>(dst + HP * 128u) = make_uint4(lo4[0], lo4[1], lo4[2], lo4[3]);
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            mbar_arrive(&q_ready);
        }
        if (tid < HP) s_ref[tid] = -INFINITY;
        float l[HP];
#pragma unroll
        for (int h = 0; h < HP; ++h) l[h] = 0.0f;
        unsigned char* p_out = sp + (tok >> 6) * Layout<HP>::P_CHUNK + (tok & 7u) * 2u;  // + row and swizzled piece
        const uint32_t p_piece = (tok & 63u) >> 3;
        for (uint32_t t = 0; t < n_tiles; ++t) {
            const bool ok = __all_sync(0xffffffffu, wait(&s_done, t & 1u));  // tensor-memory loads are warp-collective
            tc_fence_after();
            float s[HP], v[HP];
            tmem_ld_hp<HP>(tmem_s + lane_addr, s);
            tmem_ld_hp<HP>(tmem_s + lane_addr + HP, v);
            const bool seen = ok && lo + t * TOKENS + tok < hi;
#pragma unroll
            for (int h = 0; h < HP; ++h) v[h] = s[h] = seen ? s[h] + v[h] : -INFINITY;
            const float top = transposed_reduce<HP>(v, lane, [](float x, float y) { return fmaxf(x, y); });
            if (lane < HP) s_max[group * HP + lane] = top;
            if (tid == 0) s_rescale = 0;
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (tid < HP) {
                const float m = fmaxf(fmaxf(s_max[tid], s_max[HP + tid]), fmaxf(s_max[2 * HP + tid], s_max[3 * HP + tid]));
                const float ref = s_ref[tid];
                float corr = 1.0f;
                if (m > ref + 8.0f) {  // also the first tile: the reference is -inf
                    s_ref[tid] = m;
                    corr = fast_exp2(ref - m);
                    s_rescale = 1;
                }
                s_corr[tid] = corr;
            }
            asm volatile("bar.sync 1, 128;" ::: "memory");
            if (t > 0 && s_rescale) {
                float corr[HP];
#pragma unroll
                for (int h = 0; h < HP; h += 4) {
                    const float4 c = *reinterpret_cast<const float4*>(s_corr + h);
                    corr[h] = c.x, corr[h + 1] = c.y, corr[h + 2] = c.z, corr[h + 3] = c.w;
                }
#pragma unroll
                for (int h = 0; h < HP; ++h) l[h] *= corr[h];
                for (uint32_t b = 0; b < NP; ++b) {
#pragma unroll
                    for (int part = 0; part < HP; part += 16) {
                        uint32_t r[16];
                        tmem_ld_x16(tmem_o + b * HP + part + lane_addr, r);
                        tmem_ld_wait();
#pragma unroll
                        for (int h = 0; h < 16; ++h) r[h] = __float_as_uint(__uint_as_float(r[h]) * corr[part + h]);
                        tmem_st_x16(tmem_o + b * HP + part + lane_addr, r);
                    }
                }
                tmem_st_wait();
            }
#pragma unroll
            for (int h = 0; h < HP; h += 4) {
                const float4 ref = *reinterpret_cast<const float4*>(s_ref + h);
                const float r4[4] = {ref.x, ref.y, ref.z, ref.w};
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float p = fast_exp2(s[h + j] - r4[j]);
                    l[h + j] += p;
                    *reinterpret_cast<__half*>(p_out + (h + j) * 128u + ((p_piece ^ ((h + j) & 7u)) << 4)) = __float2half_rn(p);
                }
            }
            tc_fence_before();
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            mbar_arrive(&p_ready);
        }
        // ---- sums over the tokens, then the accumulated output: lane = latent column of a 128-column block
        const float sum = transposed_reduce<HP>(l, lane, [](float x, float y) { return x + y; });
        if (lane < HP) s_max[group * HP + lane] = sum;
        asm volatile("bar.sync 1, 128;" ::: "memory");
        const bool ok = __all_sync(0xffffffffu, wait(&o_done, 0));
        tc_fence_after();
        if (tid < heads) {
            a.pm[part0 + (size_t)tid * a.splits] = s_ref[tid] * LN2;  // natural-log domain, as in the other forms
            a.pl[part0 + (size_t)tid * a.splits] = ok ? (s_max[tid] + s_max[HP + tid]) + (s_max[2 * HP + tid] + s_max[3 * HP + tid]) : 0.0f;
        }
        for (uint32_t b = 0; b < NP; ++b) {
            float o[HP];
            tmem_ld_hp<HP>(tmem_o + b * HP + lane_addr, o);
            float* dst = a.po + part0 * a.rank + b * 128u + tok;
#pragma unroll
            for (int h = 0; h < HP; ++h)
                if ((uint32_t)h < heads) dst[(size_t)h * a.splits * a.rank] = o[h];
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_s, tmem_cols);
    }
}

template <int HP>
int launch(M40llmCudaContext* ctx, const M40LatArgs& a) {
    static unsigned long long configured = 0ull;
    const unsigned long long bit = 1ull << (ctx->device_id & 63);
    if (!(configured & bit)) {
        if (cudaFuncSetAttribute(latent_tc_kernel<HP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_BUDGET) != cudaSuccess) return -6;
        configured |= bit;
    }
    CUtensorMap map;
    if (!m40_tc_map(&map, a.C, (uint64_t)a.slots * a.max_seq_len, a.rank, TOKENS, false)) return -6;
    const uint32_t slots = Layout<HP>::slots(a.rank);
    const size_t smem = 1024 + slots * (size_t)PAIR_BYTES + Layout<HP>::fixed(a.rank);
    const cudaError_t e = m40_launch_dependent(latent_tc_kernel<HP>, dim3(a.splits, (a.heads + HP - 1) / HP, a.rows), dim3(192), smem,
                                               ctx->decode_stream, map, a, slots);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

}  // namespace

bool m40_latent_tc_takes(const M40LatArgs& a) {
    const void* w[1] = {a.C};
    return a.rank % 128 == 0 && a.rank <= 512 && (uint64_t)a.slots * a.max_seq_len < 0x7fffff00ull &&
           m40_gemm_tc_supported(2, (int)a.rank, 1, w);
}

int m40_latent_tc(M40llmCudaContext* ctx, const M40LatArgs& a) { return a.heads > 16 ? launch<32>(ctx, a) : launch<16>(ctx, a); }
