// Real-gated linear recurrence (a diagonal state) with its causal convolution: m40llm_rglru_async.
//
//   S <- a S + sqrt(1 - a^2) i u,  log a = -decay r softplus(lam),  r, i = sigmoid of block-diagonal maps of u.
//
//   rglru_decode_kernel   one token: CTA = 32 channels of a block does the convolution, the gates, the state and the output
//                         gate in one launch.
//   several rows:
//     short convolution   u (short_conv.cu);
//     gates               a and b = sqrt(1 - a^2) i u per (row, channel). The block-diagonal products run on the tensor cores
//                         (gemm_tc_grouped.cu) with u cut into three bf16 parts, whose sum is the f32 value and whose products
//                         with bf16 weights are exact in f32, or on f32 multiply-adds: 32-bit arithmetic either way;
//     one token per sequence: the gates' epilogue makes the step and the output;
//     portions: rglru_scan_kernel, CTA = (32 channels, segment), a warp per piece of the portion: every piece is folded into one
//                         (product of a, sum) pair, the pairs are chained from the slot's state, and the pieces are walked
//                         again from their starting states.
// 1 - a^2 is taken as -expm1(2 log a), which keeps its accuracy when a is close to one.
#include "rglru.cuh"

#include "gemm_tc_grouped.cuh"
#include "short_conv.cuh"

namespace {

constexpr uint32_t SLICE = 32;  // output channels per decode CTA

using RgArgs = M40RgArgs;

template <typename WT>
__global__ void __launch_bounds__(256) rglru_decode_kernel(RgArgs g) {
    extern __shared__ __align__(16) float su[];  // [bs padded to 8]
    __shared__ float sz[2][SLICE];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;
    const uint32_t slices = (g.bs + SLICE - 1u) / SLICE, blk = blockIdx.x / slices, o0 = (blockIdx.x % slices) * SLICE;
    const uint32_t bsp = (g.bs + 7u) & ~7u;
    const WT* ra = reinterpret_cast<const WT*>(g.ra) + (size_t)blk * g.bs * g.bs;
    const WT* ri = reinterpret_cast<const WT*>(g.ri) + (size_t)blk * g.bs * g.bs;
    // this warp's first weight pieces do not depend on the previous kernel
    constexpr int PER = SLICE / 8;  // output channels per warp
    const uint32_t ow = o0 + warp * PER;
    float wr[PER][8], wi[PER][8];
    if (g.wide && lane * 8u < g.bs) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const uint32_t o = min(ow + j, g.bs - 1u);
            m40_load8(ra + (size_t)o * g.bs + lane * 8u, wr[j]);
            m40_load8(ri + (size_t)o * g.bs + lane * 8u, wi[j]);
        }
    }
    pdl_wait();
    pdl_trigger();
    const uint32_t slot = g.row_seq[0] * g.slot_mul + g.slot_add, pos = g.row_pos[0];
    const bool ok = slot < g.slots;
    // the finishing warp's inputs
    const uint32_t fo = o0 + lane, fc = blk * g.bs + fo;
    const bool mine = warp == 0 && fo < g.bs;
    M40RgStep step = {0.0f, 0.0f, ~(size_t)0};
    float fx = 0.0f;
    if (mine) {
        step = m40_rg_fetch(g, 0, fc);
        fx = g.packed[g.width + fc];
    }
    // u of the whole block
    for (uint32_t ch = tid; ch < bsp; ch += 256u) {
        float y = 0.0f;
        if (ch < g.bs && ok) {
            const uint32_t c = blk * g.bs + ch;
            const float* w = g.conv_w + (size_t)c * g.taps;
            const float* ring = g.state + slot * g.slot_stride + g.width + c;
            y = g.conv_b ? g.conv_b[c] : 0.0f;
#pragma unroll 4
            for (uint32_t back = g.taps - 1u; back > 0u; --back)
                if (back <= pos) y = fmaf(w[g.taps - 1u - back], ring[(size_t)((pos - back) % g.taps) * g.width], y);
            y = fmaf(w[g.taps - 1u], g.packed[g.width + c], y);
        }
        su[ch] = y;
    }
    __syncthreads();
    float ar[PER] = {}, ai[PER] = {};
    if (g.wide) {
        for (uint32_t k = lane * 8u; k < g.bs; k += 256u) {
            if (k >= 256u) {
#pragma unroll
                for (int j = 0; j < PER; ++j) {
                    const uint32_t o = min(ow + j, g.bs - 1u);
                    m40_load8(ra + (size_t)o * g.bs + k, wr[j]);
                    m40_load8(ri + (size_t)o * g.bs + k, wi[j]);
                }
            }
            const float4 x0 = *reinterpret_cast<const float4*>(su + k), x1 = *reinterpret_cast<const float4*>(su + k + 4);
            const float x[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
            for (int j = 0; j < PER; ++j)
#pragma unroll
                for (int i = 0; i < 8; ++i) ar[j] = fmaf(wr[j][i], x[i], ar[j]), ai[j] = fmaf(wi[j][i], x[i], ai[j]);
        }
    } else {
        for (uint32_t k = lane; k < g.bs; k += 32u)
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const uint32_t o = min(ow + j, g.bs - 1u);
                ar[j] = fmaf(m40_load_elem(ra + (size_t)o * g.bs + k), su[k], ar[j]);
                ai[j] = fmaf(m40_load_elem(ri + (size_t)o * g.bs + k), su[k], ai[j]);
            }
    }
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const float zr = warp_sum(ar[j]), zi = warp_sum(ai[j]);
        if (lane == 0) sz[0][warp * PER + j] = zr, sz[1][warp * PER + j] = zi;
    }
    __syncthreads();
    if (!mine) return;
    m40_rg_store(g, 0, fc, step,
                 m40_rg_gated(g, sz[0][lane] + g.ra_b[fc], sz[1][lane] + g.ri_b[fc], m40_softplus(g.lam[fc]), su[fo]));
    if (ok && g.taps > 1u) g.state[slot * g.slot_stride + g.width + (size_t)(pos % g.taps) * g.width + fc] = fx;
}

// a and b of 64 rows x 64 channels of one block, f32 multiply-adds. A k tile is summed on its own before it joins the
// running sum.
template <typename WT>
__global__ void __launch_bounds__(256) rglru_gates_f32_kernel(RgArgs g) {
    constexpr int BM = 64, BN = 64, BK = 16;
    __shared__ float sx[BK][BM + 4], sr[BK][BN + 4], si[BK][BN + 4];
    pdl_wait();
    pdl_trigger();
    const uint32_t tid = threadIdx.x, m0 = blockIdx.y * BM, n0 = blockIdx.x * BN, c0 = blockIdx.z * g.bs;
    const uint32_t tm = (tid >> 4) * 4u, tn = (tid & 15u) * 4u;
    const WT* ra = reinterpret_cast<const WT*>(g.ra) + (size_t)blockIdx.z * g.bs * g.bs;
    const WT* ri = reinterpret_cast<const WT*>(g.ri) + (size_t)blockIdx.z * g.bs * g.bs;
    float ar[4][4] = {}, ai[4][4] = {};
    for (uint32_t k0 = 0; k0 < g.bs; k0 += BK) {
#pragma unroll
        for (int i = 0; i < (BM * BK) / 256; ++i) {
            const uint32_t e = tid + i * 256u, r = e / BK, kk = e % BK, k = k0 + kk;
            sx[kk][r] = (m0 + r < g.rows && k < g.bs) ? g.u[(size_t)(m0 + r) * g.width + c0 + k] : 0.0f;
            const bool in = n0 + r < g.bs && k < g.bs;
            sr[kk][r] = in ? m40_load_elem(ra + (size_t)(n0 + r) * g.bs + k) : 0.0f;
            si[kk][r] = in ? m40_load_elem(ri + (size_t)(n0 + r) * g.bs + k) : 0.0f;
        }
        __syncthreads();
        float pr[4][4] = {}, pi[4][4] = {};
#pragma unroll
        for (int kk = 0; kk < BK; ++kk) {
            const float4 xv = *reinterpret_cast<const float4*>(&sx[kk][tm]);
            const float4 rv = *reinterpret_cast<const float4*>(&sr[kk][tn]), iv = *reinterpret_cast<const float4*>(&si[kk][tn]);
            const float xa[4] = {xv.x, xv.y, xv.z, xv.w}, rr[4] = {rv.x, rv.y, rv.z, rv.w}, ii[4] = {iv.x, iv.y, iv.z, iv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) pr[i][j] = fmaf(xa[i], rr[j], pr[i][j]), pi[i][j] = fmaf(xa[i], ii[j], pi[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) ar[i][j] += pr[i][j], ai[i][j] += pi[i][j];
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const uint32_t o = n0 + tn + j;
        if (o >= g.bs) continue;
        const uint32_t c = c0 + o;
        const float sp = m40_softplus(g.lam[c]), rb = g.ra_b[c], ib = g.ri_b[c];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const uint32_t m = m0 + tm + i;
            if (m >= g.rows) continue;
            const size_t at = (size_t)m * g.width + c;
            const float2 ab = m40_rg_gated(g, ar[i][j] + rb, ai[i][j] + ib, sp, g.u[at]);
            if (g.step) {
                m40_rg_store(g, m, c, m40_rg_fetch(g, m, c), ab);
                continue;
            }
            g.a[at] = ab.x;
            g.b[at] = ab.y;
        }
    }
}

// grid (channel groups of 32, segments), block 1024: warp = piece of the portion, lane = channel.
__global__ void __launch_bounds__(1024) rglru_scan_kernel(RgArgs g) {
    __shared__ float sa[32][33], sb[32][33];
    pdl_wait();
    pdl_trigger();
    const uint32_t lane = threadIdx.x & 31u, piece = threadIdx.x >> 5, c = blockIdx.x * 32u + lane;
    const uint32_t* sg = g.seg + 4u * blockIdx.y;
    const uint32_t row0 = sg[0], n = sg[1], slot = sg[2] * g.slot_mul + g.slot_add, p0 = sg[3];
    const bool live = c < g.width;
    if (slot >= g.slots || (uint64_t)row0 + n > g.rows) {
        if (threadIdx.x == 0) atomicOr(g.status, 2u);
        return;
    }
    const uint32_t len = (n + 31u) / 32u, lo = min(piece * len, n), hi = min(lo + len, n);
    const size_t at0 = (size_t)row0 * g.width + c;
    float A = 1.0f, B = 0.0f;
    if (live) {
        uint32_t t = lo;
        for (; t + 8u <= hi; t += 8u) {
            float av[8], bv[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) av[i] = g.a[at0 + (size_t)(t + i) * g.width], bv[i] = g.b[at0 + (size_t)(t + i) * g.width];
#pragma unroll
            for (int i = 0; i < 8; ++i) B = fmaf(av[i], B, bv[i]), A *= av[i];
        }
        for (; t < hi; ++t) {
            const float av = g.a[at0 + (size_t)t * g.width];
            B = fmaf(av, B, g.b[at0 + (size_t)t * g.width]);
            A *= av;
        }
    }
    sa[piece][lane] = A;
    sb[piece][lane] = B;
    __syncthreads();
    if (piece == 0 && live) {
        float* st = g.state + slot * g.slot_stride + c;
        float s = p0 > 0u ? *st : 0.0f;
#pragma unroll
        for (int k = 0; k < 32; ++k) {
            const float next = fmaf(sa[k][lane], s, sb[k][lane]);
            sa[k][lane] = s;  // the piece's starting state
            s = next;
        }
        *st = s;
    }
    __syncthreads();
    if (!live) return;
    float s = sa[piece][lane];
    const float* y = g.packed + (size_t)row0 * g.ld + c;
    uint32_t t = lo;
    for (; t + 4u <= hi; t += 4u) {
        float av[4], bv[4], yv[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            av[i] = g.a[at0 + (size_t)(t + i) * g.width], bv[i] = g.b[at0 + (size_t)(t + i) * g.width];
            yv[i] = y[(size_t)(t + i) * g.ld];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            s = fmaf(av[i], s, bv[i]);
            g.out[at0 + (size_t)(t + i) * g.width] = s * m40_act((int)M40LLM_ACT_GELU_TANH, yv[i]);
        }
    }
    for (; t < hi; ++t) {
        s = fmaf(g.a[at0 + (size_t)t * g.width], s, g.b[at0 + (size_t)t * g.width]);
        g.out[at0 + (size_t)t * g.width] = s * m40_act((int)M40LLM_ACT_GELU_TANH, y[(size_t)t * g.ld]);
    }
}

template <typename WT>
int run_one(M40llmCudaContext* ctx, const RgArgs& g, uint32_t blocks) {
    const uint32_t bsp = (g.bs + 7u) & ~7u, slices = (g.bs + SLICE - 1) / SLICE;
    const cudaError_t e =
        m40_launch_dependent(rglru_decode_kernel<WT>, dim3(blocks * slices), dim3(256), bsp * sizeof(float), ctx->decode_stream, g);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

template <typename WT>
int run_rows(M40llmCudaContext* ctx, RgArgs g, uint32_t blocks, const M40llmStepRows& rows) {
    cudaStream_t s = ctx->decode_stream;
    const size_t n = ((size_t)g.rows * g.width + 3) & ~(size_t)3;
    const bool tensor = g.tensor && m40_gemm_tc_grouped_supported(g.ra, g.bs, g.bs, g.width, g.bs) &&
                        m40_gemm_tc_grouped_supported(g.ri, g.bs, g.bs, g.width, g.bs);
    const size_t part = (n * 2 + 255) / 256 * 256;
    float* work = (float*)m40_ensure_scratch(ctx, 1, 3 * n * sizeof(float) + (tensor ? 256 + 3 * part : 0), 1);
    if (!work) return -5;
    unsigned char* parts = (unsigned char*)(((uintptr_t)(work + 3 * n) + 255) & ~(uintptr_t)255);
    g.u = work, g.a = work + n, g.b = work + 2 * n;
    M40ConvArgs c = {};
    c.x = g.packed + g.width;
    c.w = g.conv_w;
    c.bias = g.conv_b;
    c.out = g.u;
    c.ring = g.state + g.width;
    c.slot_stride = g.slot_stride;
    c.status = g.status;
    c.row_seq = g.row_seq, c.row_pos = g.row_pos, c.seg = g.seg;
    c.ldx = g.ld, c.dim = g.width, c.taps = g.taps;
    c.slot_mul = g.slot_mul, c.slot_add = g.slot_add, c.slots = g.slots, c.rows = g.rows;
    for (int p = 0; tensor && p < 3; ++p) c.parts[p] = parts + p * part;
    int rc = m40_short_conv(ctx, s, c, rows);
    if (rc != 0) return rc;
    cudaError_t e;
    if (tensor) {
        M40GroupedCall q = {};
        q.w = g.ra;
        q.w2 = g.ri;
        for (int p = 0; p < 3; ++p) q.x[p] = c.parts[p];
        q.parts = 3;
        q.bf16 = 1;
        q.groups = blocks;
        q.N = q.K = q.group_k = g.bs;
        q.x_rows = g.rows;
        q.ldx = g.width;
        q.tile_rows = 32;
        q.kind = M40_GROUPED_RG;
        q.rg = g;
        if ((rc = m40_gemm_tc_grouped(ctx, s, q)) != 0) return rc;
    } else {
        const dim3 grid((g.bs + 63) / 64, (g.rows + 63) / 64, blocks);
        e = m40_launch_dependent(rglru_gates_f32_kernel<WT>, grid, dim3(256), 0, s, g);
        M40_COUNT_LAUNCH(ctx);
        if (e != cudaSuccess) return -6;
    }
    if (g.step) return cudaGetLastError() == cudaSuccess ? 0 : -6;
    e = m40_launch_dependent(rglru_scan_kernel, dim3((g.width + 31) / 32, rows.segments), dim3(1024), 0, s, g);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

template <typename WT>
int run(M40llmCudaContext* ctx, const RgArgs& g, uint32_t blocks, const M40llmStepRows& rows) {
    return g.step && g.rows == 1 ? run_one<WT>(ctx, g, blocks) : run_rows<WT>(ctx, g, blocks, rows);
}

}  // namespace

extern "C" int m40llm_rglru_async(M40llmCudaContext* ctx, M40llmStateCache* state, const M40llmRgLru* c, const M40llmStepRows* r) {
    if (!ctx || !state || !c || !r || !c->packed || !c->conv_w || !c->ra || !c->ra_b || !c->ri || !c->ri_b || !c->lam || !c->out)
        return -1;
    if (c->width == 0 || c->blocks == 0 || c->width % c->blocks != 0 || c->width / c->blocks > 1024) return -2;
    if (c->ld < 2ull * c->width || r->rows == 0 || r->segments == 0 || r->max_segment_rows == 0) return -2;
    if (c->w_dtype > M40LLM_DT_BF16 || c->taps == 0 || c->taps > 32) return -3;
    if (state->dim != 0 || state->values != (uint64_t)c->width * (1u + c->taps)) return -3;
    if (r->max_segment_rows == 1 ? (!r->row_seq || !r->row_pos) : !r->seg) return -1;
    if (m40_ensure_device(ctx) != 0) return -1;
    RgArgs g = {};
    g.packed = (const float*)c->packed;
    g.conv_w = (const float*)c->conv_w;
    g.conv_b = (const float*)c->conv_b;
    g.ra = c->ra;
    g.ra_b = (const float*)c->ra_b;
    g.ri = c->ri;
    g.ri_b = (const float*)c->ri_b;
    g.lam = (const float*)c->lam;
    g.out = (float*)c->out;
    g.state = state->d_state;
    g.slot_stride = state->values;
    g.status = ctx->d_status;
    g.row_seq = r->row_seq;
    g.row_pos = r->row_pos;
    g.seg = r->seg;
    g.ld = c->ld;
    g.width = c->width;
    g.bs = c->width / c->blocks;
    g.taps = c->taps;
    g.slot_mul = r->slot_mul;
    g.slot_add = r->slot_add;
    g.slots = state->slots;
    g.rows = r->rows;
    g.step = r->max_segment_rows == 1;
    g.decay = c->decay;
    g.wide = c->w_dtype != M40LLM_DT_F32 && g.bs % 8 == 0 && (((uintptr_t)c->ra | (uintptr_t)c->ri) & 15u) == 0;
    g.tensor = c->w_dtype == M40LLM_DT_BF16 && !c->exact;
    if (c->w_dtype == M40LLM_DT_F32) return run<float>(ctx, g, c->blocks, *r);
    return c->w_dtype == M40LLM_DT_BF16 ? run<__nv_bfloat16>(ctx, g, c->blocks, *r) : run<__half>(ctx, g, c->blocks, *r);
}
