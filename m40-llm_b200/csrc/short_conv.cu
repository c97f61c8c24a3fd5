// Causal convolution over time, one filter per channel: m40llm_short_conv_async.
//
// The inputs that later tokens need live in a ring per slot, the input of position p at p % taps, so one token writes an
// entry that none of its own reads touch and nothing is ever shifted or cleared: entries of positions below zero are not read.
// A portion is cut into pieces of PIECE rows. Only the first piece reads the ring (taps - 1 <= PIECE), and the same threads
// write the portion's last inputs to it when they are done, so a channel's ring is touched by one thread per launch.
#include "short_conv.cuh"

#include <cuda_bf16.h>

namespace {

constexpr uint32_t PIECE = 32, MAX_TAPS = 32;

__device__ __forceinline__ void store_out(const M40ConvArgs& a, size_t at, float y) {
    a.out[at] = y;
    if (a.parts[0]) {
        const __nv_bfloat16 p0 = __float2bfloat16_rn(y);
        const float r1 = y - __bfloat162float(p0);
        const __nv_bfloat16 p1 = __float2bfloat16_rn(r1);
        reinterpret_cast<__nv_bfloat16*>(a.parts[0])[at] = p0;
        reinterpret_cast<__nv_bfloat16*>(a.parts[1])[at] = p1;
        reinterpret_cast<__nv_bfloat16*>(a.parts[2])[at] = __float2bfloat16_rn(r1 - __bfloat162float(p1));
    }
}

// TAPS > 0: a window of the last inputs stays in registers; 0: any number of taps, inputs read again.
template <bool DECODE, int TAPS>
__global__ void __launch_bounds__(128) short_conv_kernel(M40ConvArgs a) {
    const uint32_t taps = TAPS ? (uint32_t)TAPS : a.taps;
    const uint32_t c = blockIdx.x * 128u + threadIdx.x;
    float wv[TAPS ? TAPS : 1];
    const float* w = a.w + (size_t)min(c, a.dim - 1u) * taps;
    if (TAPS) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) wv[j] = w[j];
    }
    const float bias = a.bias ? a.bias[min(c, a.dim - 1u)] : 0.0f;
    pdl_wait();
    pdl_trigger();
    uint32_t row0, n, seq, p0;
    if (DECODE) {
        row0 = blockIdx.z, n = 1u, seq = a.row_seq[row0], p0 = a.row_pos[row0];
    } else {
        const uint32_t* sg = a.seg + 4u * blockIdx.z;
        row0 = sg[0], n = sg[1], seq = sg[2], p0 = sg[3];
    }
    const uint32_t slot = seq * a.slot_mul + a.slot_add, first = blockIdx.y * PIECE;
    if (first >= n) return;
    if (slot >= a.slots || (uint64_t)row0 + n > a.rows) {
        if (threadIdx.x == 0) atomicOr(a.status, 2u);
        return;
    }
    if (c >= a.dim) return;
    const float* x = a.x + (size_t)row0 * a.ldx + c;
    const size_t out0 = (size_t)row0 * a.dim + c;
    float* ring = a.ring ? a.ring + (size_t)slot * a.slot_stride + c : nullptr;
    const uint32_t last = min(first + PIECE, n);
    // the input `back` tokens before token t of the portion
    auto input = [&](uint32_t t, uint32_t back) {
        if (back <= t) return x[(size_t)(t - back) * a.ldx];
        if (back <= p0 + t) return ring[(size_t)((p0 + t - back) % taps) * a.dim];
        return 0.0f;
    };
    if (TAPS) {
        float win[TAPS ? TAPS : 1];  // win[j]: the input TAPS - 1 - j tokens back
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) win[j + 1] = input(first, (uint32_t)(TAPS - 1 - j));
#pragma unroll 4
        for (uint32_t t = first; t < last; ++t) {
#pragma unroll
            for (int j = 0; j + 1 < TAPS; ++j) win[j] = win[j + 1];
            win[TAPS ? TAPS - 1 : 0] = x[(size_t)t * a.ldx];
            float y = bias;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) y = fmaf(wv[j], win[j], y);
            store_out(a, out0 + (size_t)t * a.dim, a.add_input ? win[TAPS ? TAPS - 1 : 0] + y : y);
        }
    } else {
        for (uint32_t t = first; t < last; ++t) {
            float y = bias;
            for (uint32_t back = taps; back-- > 0u;) y = fmaf(w[taps - 1u - back], input(t, back), y);
            store_out(a, out0 + (size_t)t * a.dim, a.add_input ? x[(size_t)t * a.ldx] + y : y);
        }
    }
    if (first == 0u && taps > 1u) {
        const uint32_t keep = min(n, taps - 1u);
        for (uint32_t t = n - keep; t < n; ++t) ring[(size_t)((p0 + t) % taps) * a.dim] = x[(size_t)t * a.ldx];
    }
}

template <bool DECODE>
cudaError_t launch(cudaStream_t s, dim3 grid, const M40ConvArgs& a) {
    switch (a.taps) {
        case 2: return m40_launch_dependent(short_conv_kernel<DECODE, 2>, grid, dim3(128), 0, s, a);
        case 3: return m40_launch_dependent(short_conv_kernel<DECODE, 3>, grid, dim3(128), 0, s, a);
        case 4: return m40_launch_dependent(short_conv_kernel<DECODE, 4>, grid, dim3(128), 0, s, a);
        default: return m40_launch_dependent(short_conv_kernel<DECODE, 0>, grid, dim3(128), 0, s, a);
    }
}

}  // namespace

int m40_short_conv(M40llmCudaContext* ctx, cudaStream_t s, const M40ConvArgs& a, const M40llmStepRows& rows) {
    const bool decode = rows.max_segment_rows == 1;
    const dim3 grid((a.dim + 127) / 128, (rows.max_segment_rows + PIECE - 1) / PIECE, decode ? rows.rows : rows.segments);
    const cudaError_t e = decode ? launch<true>(s, grid, a) : launch<false>(s, grid, a);
    M40_COUNT_LAUNCH(ctx);
    return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? 0 : -6;
}

extern "C" int m40llm_short_conv_async(M40llmCudaContext* ctx, M40llmStateCache* ring, const M40llmShortConv* c,
                                       const M40llmStepRows* r) {
    if (!ctx || !c || !r || !c->x || !c->w || !c->out) return -1;
    if (c->dim == 0 || r->rows == 0 || r->segments == 0 || r->max_segment_rows == 0 || c->x == c->out) return -2;
    if (c->taps == 0 || c->taps > MAX_TAPS) return -3;
    if (c->taps > 1 && (!ring || ring->values != (uint64_t)c->taps * c->dim)) return -3;
    if (r->max_segment_rows == 1 ? (!r->row_seq || !r->row_pos) : !r->seg) return -1;
    if (c->ldx && c->ldx < c->dim) return -2;
    if (m40_ensure_device(ctx) != 0) return -1;
    M40ConvArgs a = {};
    a.x = (const float*)c->x;
    a.w = (const float*)c->w;
    a.bias = (const float*)c->bias;
    a.out = (float*)c->out;
    a.ring = ring ? ring->d_state : nullptr;
    a.slot_stride = ring ? ring->values : 0u;
    a.status = ctx->d_status;
    a.row_seq = r->row_seq;
    a.row_pos = r->row_pos;
    a.seg = r->seg;
    a.ldx = c->ldx ? c->ldx : c->dim;
    a.dim = c->dim;
    a.taps = c->taps;
    a.add_input = c->add_input;
    a.slot_mul = r->slot_mul;
    a.slot_add = r->slot_add;
    a.slots = ring ? ring->slots : 0xffffffffu;
    a.rows = r->rows;
    return m40_short_conv(ctx, ctx->decode_stream, a, *r);
}
