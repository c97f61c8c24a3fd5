// Grouped GEMM on the 5th-generation tensor cores: the experts of a mixture (each applied to the rows routed to it) and
// block-diagonal maps (each block applied to its own columns of every row).
//
// As in gemm_tc.cu the weight tile (128 rows) is the MMA's A operand and the activation rows are B; D[128 x rows] accumulates
// in tensor memory. The parts of the activations (hi + lo, or three bf16 parts, whose sum is the f32 value exactly) are
// stacked along B's rows, so one MMA of width parts * tile_rows takes a weight tile against all of them, and the epilogue adds
// the slices. No K split: there are as many tiles as groups need.
//
// CTA (n tile, row tile [, group]): warp 0 loads by TMA, warp 1 issues the MMAs and owns tensor memory, warps 2..5 finish.
// With a tile table (made on the device) CTAs beyond its length leave at once, before they take any resource.
// Every wait is bounded, as in gemm_tc.cu: a wait that runs out sets bit 2 of the status word, and the CTA winds down.
#include "gemm_tc_grouped.cuh"

#include "gemm_tc.cuh"
#include "tc_ptx.cuh"

namespace {

using namespace tc;

struct GArgs {
    const M40GroupTile* tiles;
    const uint32_t* n_tiles;
    float* out;
    void* hi;
    void* lo;
    uint32_t* status;
    uint32_t N, K, x_rows, group_k, tile_rows, parts, kblocks, stages, fmt_bits, bf16;
    int act;
    uint32_t out_ld, out_group;
    __half* heads;
    uint32_t head_dim, head_pitch;
    M40RgArgs rg;
};

template <typename T>
__device__ __forceinline__ void store_split(T* hi, T* lo, size_t at, float v);
template <>
__device__ __forceinline__ void store_split<__half>(__half* hi, __half* lo, size_t at, float v) {
    const __half h = __float2half_rn(v);
    hi[at] = h;
    lo[at] = __float2half_rn(v - __half2float(h));
}
template <>
__device__ __forceinline__ void store_split<__nv_bfloat16>(__nv_bfloat16* hi, __nv_bfloat16* lo, size_t at, float v) {
    const __nv_bfloat16 h = __float2bfloat16_rn(v);
    hi[at] = h;
    lo[at] = __float2bfloat16_rn(v - __bfloat162float(h));
}

template <int KIND>
__global__ void __launch_bounds__(192, 1) gemm_tc_grouped_kernel(const __grid_constant__ CUtensorMap tmW,
                                                                 const __grid_constant__ CUtensorMap tmW2,
                                                                 const __grid_constant__ CUtensorMap tmX0,
                                                                 const __grid_constant__ CUtensorMap tmX1,
                                                                 const __grid_constant__ CUtensorMap tmX2, GArgs a) {
    extern __shared__ unsigned char smem_unaligned[];
    unsigned char* smem = smem_unaligned + ((1024u - (smem_u32(smem_unaligned) & 1023u)) & 1023u);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
    constexpr bool PAIRED = KIND == M40_GROUPED_RG;
    constexpr uint32_t N_TILE = PAIRED ? BLOCK_N / 2 : BLOCK_N;
    uint32_t group = blockIdx.z, m_base = blockIdx.y * a.tile_rows, m_live = 0;
    if (a.tiles) {  // every thread waits: the table comes from the previous kernels
        pdl_wait();
        if (blockIdx.y >= *a.n_tiles) {
            pdl_trigger();
            return;
        }
        const M40GroupTile t = a.tiles[blockIdx.y];
        group = t.group, m_base = t.row0, m_live = t.live;
    } else {
        m_live = min(a.tile_rows, a.x_rows - m_base);
    }
    const uint32_t n0 = blockIdx.x * N_TILE, w_row = group * a.N + n0, x_col = group * a.group_k;
    const uint32_t a_bytes = BLOCK_N * BLOCK_K * 2, b_bytes = a.tile_rows * BLOCK_K * 2;
    const uint32_t stage_bytes = a_bytes + a.parts * b_bytes, acc_cols = a.parts * a.tile_rows;
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + a.stages * stage_bytes);
    uint64_t *full = bars, *empty = bars + a.stages, *accum = bars + 2 * a.stages;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * a.stages + 1);
    volatile uint32_t* abort_flag = tmem_slot + 1;
    uint32_t tmem_cols = 32;
    while (tmem_cols < acc_cols) tmem_cols <<= 1;

    if (threadIdx.x == 0) {
        for (uint32_t s = 0; s < a.stages; ++s) {
            mbar_init(&full[s], 1);
            mbar_init(&empty[s], 1);
        }
        mbar_init(accum, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(tmem_slot, tmem_cols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    pdl_trigger();

    if (warp == 0) {
        if (lane == 0) {
            auto load_w = [&](uint32_t i) {
                unsigned char* st = smem + (i % a.stages) * stage_bytes;
                uint64_t* bar = &full[i % a.stages];
                mbar_expect_tx(bar, stage_bytes);
                tma_load_2d(st, &tmW, bar, (int)(i * BLOCK_K), (int)w_row);
                if (PAIRED) tma_load_2d(st + a_bytes / 2, &tmW2, bar, (int)(i * BLOCK_K), (int)w_row);
            };
            auto load_x = [&](uint32_t i) {
                unsigned char* st = smem + (i % a.stages) * stage_bytes + a_bytes;
                uint64_t* bar = &full[i % a.stages];
                const int kx = (int)(x_col + i * BLOCK_K);
                tma_load_2d(st, &tmX0, bar, kx, (int)m_base);
                if (a.parts > 1) tma_load_2d(st + b_bytes, &tmX1, bar, kx, (int)m_base);
                if (a.parts > 2) tma_load_2d(st + 2 * b_bytes, &tmX2, bar, kx, (int)m_base);
            };
            const uint32_t pre = min(a.kblocks, a.stages);
            for (uint32_t i = 0; i < pre; ++i) load_w(i);
            pdl_wait();
            for (uint32_t i = 0; i < pre; ++i) load_x(i);
            uint32_t issued = pre;
            for (; issued < a.kblocks; ++issued) {
                if (!mbar_wait(&empty[issued % a.stages], (issued / a.stages - 1u) & 1u)) { *abort_flag = 1; break; }
                if (*abort_flag) break;
                load_w(issued);
                load_x(issued);
            }
            if (*abort_flag)  // copies still in flight land (bounded wait) before the CTA goes away
                for (uint32_t i = issued > a.stages ? issued - a.stages : 0u; i < issued; ++i)
                    mbar_wait(&full[i % a.stages], (i / a.stages) & 1u);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = make_idesc(acc_cols) | a.fmt_bits;
            bool ok = true;
            for (uint32_t i = 0; i < a.kblocks && ok; ++i) {
                const uint32_t s = i % a.stages;
                if (!mbar_wait(&full[s], (i / a.stages) & 1u)) { *abort_flag = 1; ok = false; break; }
                tc_fence_after();
                const uint32_t sa = smem_u32(smem + s * stage_bytes), sb = sa + a_bytes;
#pragma unroll
                for (uint32_t k = 0; k < BLOCK_K / UMMA_K; ++k)
                    umma_f16(tmem_base, make_desc_sw128(sa + k * UMMA_K * 2), make_desc_sw128(sb + k * UMMA_K * 2), idesc, (i | k) != 0u);
                umma_commit(&empty[s]);
            }
            if (ok) umma_commit(accum);
        }
    } else {
        const uint32_t lane_group = warp & 3u, row_of_tile = lane_group * 32u + lane;  // weight row of the tile
        pdl_wait();
        bool ok = mbar_wait(accum, 0);
        if (!ok) *abort_flag = 1;
        ok = __all_sync(0xffffffffu, ok);
        tc_fence_after();
        // columns c .. c + 7 of this thread's weight row, the parts added
        auto sums = [&](uint32_t c, float* v) {
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = 0.0f;
            if (!ok) return;
            for (uint32_t p = 0; p < a.parts; ++p) {
                float w[8];
                tmem_ld8(tmem_base + ((lane_group * 32u) << 16) + p * a.tile_rows + c, w);
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] += w[j];
            }
        };
        if constexpr (PAIRED) {
            // lanes 0..63 hold r sums, 64..127 the i sums of the same channels. Each half finishes half of the rows and hands
            // the other half's sums over through shared memory (the ring is free).
            float* xs = reinterpret_cast<float*>(smem);  // [tile_rows][64]
            const uint32_t ch = row_of_tile & 63u, n = n0 + ch, half = a.tile_rows / 2u;
            const bool is_i = row_of_tile >= 64u;
            const uint32_t mine = is_i ? half : 0u, other = is_i ? 0u : half;
            for (uint32_t c = other; c < other + half; c += 8) {
                float v[8];
                sums(c, v);
#pragma unroll
                for (int j = 0; j < 8; ++j) xs[(c + j) * 64u + ch] = v[j];
            }
            asm volatile("bar.sync 1, 128;" ::: "memory");
            const M40RgArgs& g = a.rg;
            const bool n_ok = n < a.N;
            const uint32_t chan = x_col + (n_ok ? n : 0u);
            const float sp = m40_softplus(g.lam[chan]), rb = g.ra_b[chan], ib = g.ri_b[chan];
            for (uint32_t c = mine; c < mine + half; c += 8) {
                float v[8], u[8];
                sums(c, v);
#pragma unroll
                for (int j = 0; j < 8; ++j) u[j] = g.u[(size_t)(m_base + min(c + j, m_live - 1u)) * g.width + chan];
                if (g.step) {
                    M40RgStep st[8];
#pragma unroll
                    for (int j = 0; j < 8; ++j) st[j] = m40_rg_fetch(g, m_base + min(c + j, m_live - 1u), chan);
#pragma unroll
                    for (int j = 0; j < 8; ++j) {
                        if (!n_ok || c + j >= m_live) continue;
                        const float o = xs[(c + j) * 64u + ch];
                        m40_rg_store(g, m_base + c + j, chan, st[j],
                                     m40_rg_gated(g, (is_i ? o : v[j]) + rb, (is_i ? v[j] : o) + ib, sp, u[j]));
                    }
                    continue;
                }
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    if (!n_ok || c + j >= m_live) continue;
                    const float o = xs[(c + j) * 64u + ch];
                    const float2 ab = m40_rg_gated(g, (is_i ? o : v[j]) + rb, (is_i ? v[j] : o) + ib, sp, u[j]);
                    const size_t at = (size_t)(m_base + c + j) * g.width + chan;
                    g.a[at] = ab.x;
                    g.b[at] = ab.y;
                }
            }
        } else {
            const uint32_t n = n0 + row_of_tile;
            __half* heads = KIND == M40_GROUPED_HEADS
                                ? a.heads + (size_t)(n / a.head_dim) * a.x_rows * a.head_pitch + n % a.head_dim : nullptr;
            for (uint32_t c = 0; c < a.tile_rows && c < m_live; c += 8) {
                float v[8];
                sums(c, v);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    if (n >= a.N || c + j >= m_live) continue;
                    const size_t at = (size_t)(m_base + c + j) * a.N + n;
                    if (KIND == M40_GROUPED_F32) a.out[(size_t)(m_base + c + j) * a.out_ld + group * a.out_group + n] = v[j];
                    else if (KIND == M40_GROUPED_HEADS) heads[(size_t)(m_base + c + j) * a.head_pitch] = __float2half_rn(v[j]);
                    else if (a.bf16) store_split((__nv_bfloat16*)a.hi, (__nv_bfloat16*)a.lo, at, m40_act(a.act, v[j]));
                    else store_split((__half*)a.hi, (__half*)a.lo, at, m40_act(a.act, v[j]));
                }
            }
        }
    }
    if (*abort_flag && threadIdx.x == 64) atomicOr(a.status, 4u);
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, tmem_cols);
    }
}

template <int KIND>
int launch(M40llmCudaContext* ctx, cudaStream_t s, dim3 grid, size_t smem, const CUtensorMap* m, const GArgs& a) {
    static unsigned long long configured = 0ull;
    const unsigned long long bit = 1ull << (ctx->device_id & 63);
    if (!(configured & bit)) {
        if (cudaFuncSetAttribute(gemm_tc_grouped_kernel<KIND>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
            return -2;
        configured |= bit;
    }
    const cudaError_t e = m40_launch_dependent(gemm_tc_grouped_kernel<KIND>, grid, dim3(192), smem, s, m[0], m[1], m[2], m[3], m[4], a);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace

bool m40_gemm_tc_grouped_supported(const void* w, uint32_t N, uint32_t K, uint32_t ldx, uint32_t group_k) {
    const void* wp[1] = {w};
    return N > 0 && ldx % 8 == 0 && group_k % 8 == 0 && m40_gemm_tc_supported(2, (int)K, 1, wp);
}

int m40_gemm_tc_grouped(M40llmCudaContext* ctx, cudaStream_t s, const M40GroupedCall& c) {
    if (c.parts < 1 || c.parts > 3 || c.tile_rows * c.parts > 256 || c.tile_rows % 16 != 0 || c.K == 0 || c.x_rows == 0) return -2;
    const bool paired = c.kind == M40_GROUPED_RG;
    CUtensorMap m[5];
    const uint32_t box = paired ? tc::BLOCK_N / 2 : tc::BLOCK_N;
    if (!m40_tc_map(&m[0], c.w, (uint64_t)c.groups * c.N, c.K, box, c.bf16)) return -2;
    if (!m40_tc_map(&m[1], paired ? c.w2 : c.w, (uint64_t)c.groups * c.N, c.K, box, c.bf16)) return -2;
    for (uint32_t p = 0; p < 3; ++p)
        if (!m40_tc_map(&m[2 + p], c.x[p < c.parts ? p : 0], c.x_rows, c.ldx, c.tile_rows, c.bf16)) return -2;
    GArgs a = {};
    a.tiles = c.tiles;
    a.n_tiles = c.n_tiles;
    a.out = c.out;
    a.hi = c.hi;
    a.lo = c.lo;
    a.status = ctx->d_status;
    a.N = c.N;
    a.K = c.K;
    a.x_rows = c.x_rows;
    a.group_k = c.group_k;
    a.tile_rows = c.tile_rows;
    a.parts = c.parts;
    a.kblocks = (c.K + tc::BLOCK_K - 1) / tc::BLOCK_K;
    a.fmt_bits = c.bf16 ? tc::idesc_bf16() : 0u;
    a.bf16 = c.bf16;
    a.act = c.act;
    a.out_ld = c.out_ld ? c.out_ld : c.N;
    a.out_group = c.out_group;
    a.heads = c.heads;
    a.head_dim = c.head_dim;
    a.head_pitch = c.head_pitch;
    a.rg = c.rg;
    const uint32_t stage = tc::BLOCK_N * tc::BLOCK_K * 2 + c.parts * c.tile_rows * tc::BLOCK_K * 2;
    // a short ring and three CTAs per SM where the tile allows it: their prologues and epilogues cover one another
    uint32_t stages = 66u * 1024u / stage;
    if (stages < 2) stages = 2;
    if (stages > a.kblocks) stages = a.kblocks;
    // the paired epilogue passes tile_rows * 64 f32 through the ring
    const uint32_t least = paired ? (c.tile_rows * 64u * 4u + stage - 1) / stage : 1u;
    a.stages = stages < least ? least : stages;
    const size_t smem = (size_t)a.stages * stage + (2 * a.stages + 1) * 8 + 16 + 1024;
    const uint32_t n_tile = paired ? tc::BLOCK_N / 2 : tc::BLOCK_N;
    const dim3 grid((c.N + n_tile - 1) / n_tile, c.tiles ? c.max_tiles : (c.x_rows + c.tile_rows - 1) / c.tile_rows, c.tiles ? 1 : c.groups);
    switch (c.kind) {
        case M40_GROUPED_F32: return launch<M40_GROUPED_F32>(ctx, s, grid, smem, m, a);
        case M40_GROUPED_ACT_SPLIT: return launch<M40_GROUPED_ACT_SPLIT>(ctx, s, grid, smem, m, a);
        case M40_GROUPED_HEADS: return launch<M40_GROUPED_HEADS>(ctx, s, grid, smem, m, a);
        default: return launch<M40_GROUPED_RG>(ctx, s, grid, smem, m, a);
    }
}
