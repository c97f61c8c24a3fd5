// M40llmStateCache: what a recurrent layer keeps per sequence slot.
#include <stdlib.h>

#include "state_cache.cuh"

extern "C" {

M40llmStateCache* m40llm_statecache_create_values(M40llmCudaContext* ctx, uint32_t slots, uint32_t values) {
    if (!ctx || slots == 0 || values == 0) return nullptr;
    if (m40_ensure_device(ctx) != 0) return nullptr;
    M40llmStateCache* st = (M40llmStateCache*)calloc(1, sizeof(M40llmStateCache));
    if (!st) return nullptr;
    st->device_id = ctx->device_id;
    st->slots = slots;
    st->values = values;
    const size_t bytes = (size_t)slots * values * sizeof(float);
    if (cudaMalloc((void**)&st->d_state, bytes) != cudaSuccess || cudaMemset(st->d_state, 0, bytes) != cudaSuccess ||
        cudaStreamSynchronize(cudaStreamLegacy) != cudaSuccess) {
        cudaGetLastError();
        m40llm_statecache_destroy(st);
        return nullptr;
    }
    return st;
}

M40llmStateCache* m40llm_statecache_create(M40llmCudaContext* ctx, uint32_t slots, uint32_t heads, uint32_t dim) {
    if (heads == 0 || dim == 0 || dim > 256) return nullptr;
    const uint64_t values = (uint64_t)heads * dim * dim;
    if (values > 0xffffffffull) return nullptr;
    M40llmStateCache* st = m40llm_statecache_create_values(ctx, slots, (uint32_t)values);
    if (!st) return nullptr;
    st->heads = heads;
    st->dim = dim;
    return st;
}

void m40llm_statecache_destroy(M40llmStateCache* st) {
    if (!st) return;
    cudaSetDevice(st->device_id);
    if (st->d_state) cudaFree(st->d_state);
    free(st);
}

int m40llm_statecache_debug_read_values(M40llmCudaContext* ctx, M40llmStateCache* st, uint32_t slot, float* out_host) {
    if (!ctx || !st || !out_host) return -1;
    if (slot >= st->slots) return -2;
    if (m40_ensure_device(ctx) != 0) return -1;
    if (cudaMemcpyAsync(out_host, st->d_state + (size_t)slot * st->values, (size_t)st->values * sizeof(float),
                        cudaMemcpyDeviceToHost, ctx->decode_stream) != cudaSuccess ||
        cudaStreamSynchronize(ctx->decode_stream) != cudaSuccess)
        return -4;
    return 0;
}

int m40llm_statecache_debug_read(M40llmCudaContext* ctx, M40llmStateCache* st, uint32_t slot, float* out_host) {
    if (!ctx || !st || !out_host) return -1;
    if (st->dim == 0) return -3;
    float* tmp = (float*)malloc((size_t)st->values * sizeof(float));
    if (!tmp) return -5;
    const int rc = m40llm_statecache_debug_read_values(ctx, st, slot, tmp);
    for (size_t h = 0; rc == 0 && h < st->heads; ++h)
        for (size_t v = 0; v < st->dim; ++v)
            for (size_t k = 0; k < st->dim; ++k)
                out_host[(h * st->dim + k) * st->dim + v] = tmp[(h * st->dim + v) * st->dim + k];
    free(tmp);
    return rc;
}

}  // extern "C"
