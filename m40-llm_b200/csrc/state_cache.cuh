// Recurrent state kept per sequence slot (internal).
#pragma once
#include "common.cuh"

struct M40llmStateCache {
    int device_id;
    uint32_t slots, heads, dim;  // dim 0: a cache of plain values
    uint32_t values;             // f32 per slot
    float* d_state;              // matrix states: [slot][head][value][key]
};
