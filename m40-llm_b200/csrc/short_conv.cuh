// Causal convolution over time, one filter per channel (internal interface; see m40llm_short_conv_async).
#pragma once
#include "state_cache.cuh"

struct M40ConvArgs {
    const float* x;
    const float* w;      // [dim][taps]
    const float* bias;
    float* out;
    void* parts[3];      // optional: out cut into three bf16 parts whose sum is the f32 value, [rows][dim] each
    float* ring;         // [taps][dim] of slot 0: the input of position p at p % taps
    uint32_t* status;
    const uint32_t* row_seq;
    const uint32_t* row_pos;
    const uint32_t* seg;
    size_t slot_stride;  // floats from one slot's ring to the next
    uint32_t ldx, dim, taps, add_input, slot_mul, slot_add, slots, rows;
};
int m40_short_conv(M40llmCudaContext* ctx, cudaStream_t s, const M40ConvArgs& a, const M40llmStepRows& rows);
