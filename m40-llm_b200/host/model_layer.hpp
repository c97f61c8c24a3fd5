// The layers a DecodeModel runs. A layer enqueues its kernels for the rows of one step on the decode stream; the rows may
// be one token each of several sequences (decoding), portions of prompts, or a mixture.
//   LlamaLayer   the reference's decode layer (src/infer/forward.rs:247-667) over a flat dense cache;
//   StackLayer   norm -> mixer -> norm, norm -> feed-forward -> norm around an f32 residual (any of the norms may be absent).
//                Mixers: rotary attention, the generalised delta rule, latent attention, the real-gated linear recurrence; a
//                short convolution may stand before the mixer. Feed-forwards: gated, plain, mixture of experts;
//   JoinLayer    x <- W [x ; x0] + bias, x0 being the embedding output (what a looped block starts each pass with).
#pragma once
#include <stdint.h>

#include <string>

#include "../../include/m40llm_native.h"
#include "decode_layer.hpp"
#include "sequence_store.hpp"

namespace m40host {

// Rows of the current step. `flat_slots` is [layer][flat_stride] for layers that address a flat cache slot by slot.
struct StepBatch {
    M40llmStepRows rows;
    const uint32_t* flat_slots = nullptr;
    uint32_t flat_stride = 0;
};

// f32 work buffers of a step, all [max_rows][...]. x is the residual; a layer may leave its result in `spare` and swap.
struct StepBuffers {
    void *x = nullptr, *spare = nullptr, *x0 = nullptr;
    void *packed = nullptr, *att = nullptr, *x1 = nullptr, *hid = nullptr, *low = nullptr;
    void* conv = nullptr;  // x after a layer's input convolution
};
// Widths (values per row) a layer needs in the shared buffers.
struct BufferNeeds {
    size_t packed = 0, att = 0, hid = 0, low = 0;
    bool x0 = false, conv = false;
    void merge(const BufferNeeds& o) {
        packed = packed > o.packed ? packed : o.packed;
        att = att > o.att ? att : o.att;
        hid = hid > o.hid ? hid : o.hid;
        low = low > o.low ? low : o.low;
        x0 = x0 || o.x0;
        conv = conv || o.conv;
    }
};

class ModelLayer {
public:
    virtual ~ModelLayer() = default;
    virtual BufferNeeds needs() const = 0;
    virtual bool is_join() const { return false; }
    // 0 or the first failing ABI return code; failed_step() names it.
    virtual int enqueue(M40llmCudaContext* ctx, const StepBatch& batch, StepBuffers& b) = 0;
    const char* failed_step() const { return failed_step_; }

protected:
    int fail(int rc, const char* step) {
        failed_step_ = step;
        return rc;
    }
    const char* failed_step_ = "";
};

class LlamaLayer : public ModelLayer {
public:
    LlamaLayer(const ModelConfig& cfg, const LayerWeights& w, M40llmKVCache* kv, uint32_t index)
        : cfg_(cfg), w_(w), kv_(kv), index_(index) {}
    BufferNeeds needs() const override;
    int enqueue(M40llmCudaContext* ctx, const StepBatch& batch, StepBuffers& b) override;

private:
    ModelConfig cfg_;
    LayerWeights w_;
    M40llmKVCache* kv_;
    uint32_t index_;
};

enum class MixerKind : uint32_t { RotaryAttention = 1, DeltaRule = 2, LatentAttention = 3, RgLru = 4 };

// One layer of a stack; every pointer is device memory owned by the caller. Weights are [out][in] rows of w_dtype, norms
// and biases f32. Plain C layout: it crosses the host library's C surface as it is.
struct StackLayerDesc {
    uint32_t mixer;  // MixerKind
    uint32_t n_in;   // rows of w_in
    M40llmNorm norm1, norm1b, norm2, norm2b;
    const void* w_in;   // [n_in][width]: q | k | v | gate, or r | k | v | g | a | low-rank, or q | latent, or y | x
    const void* w_out;  // [width][mixer output]
    float eps;
    // rotary attention
    uint32_t q_heads, kv_heads, k_dim, v_dim, k_pairs, has_gate;
    float k_amp, scale;
    const void *q_norm, *k_norm, *k_turns, *v_turns;
    // delta rule
    uint32_t heads, dim, rank;
    float decay_scale, unit_eps;
    const void *w2, *w0, *a_bias, *o_norm;
    // feed-forward; ff == 0: none. Gated: down (act(gate x) * (up x)). Plain (gate null): down (mid(up x)).
    uint32_t ff, act;
    const void *gate, *up, *down;
    M40llmNorm mid;
    // mixture of experts (experts > 0): up [experts][ff][width], down [experts][width][ff], act
    uint32_t experts, identity, top, groups, keep;
    float router_scale;
    uint32_t shared_ff, n_router;  // n_router: rows of w_router
    const void *w_router;          // shared expert's up [shared_ff] | router [experts + identity] | padding, all [..][width]
    const void *shared_down, *correction;
    // input convolution: the mixer reads x + conv(x); 0: none
    uint32_t conv_taps;
    const void* conv_w;  // f32 [width][taps]
    const void* in_bias; // of w_in, f32, or null
    // latent attention (q_heads, k_dim, v_dim and scale above)
    uint32_t rank_kv;
    const void *c_norm, *uk, *uk_t, *uv, *sink;
    // real-gated linear recurrence
    uint32_t rg_width, rg_blocks, rg_taps;
    float rg_decay;
    const void *rg_conv, *rg_conv_b, *ra, *ra_b, *ri, *ri_b, *lam;
};

class StackLayer : public ModelLayer {
public:
    // Registers the layer's cache with the store; the caches are made when the store is allocated.
    StackLayer(uint32_t width, uint32_t w_dtype, bool exact, const StackLayerDesc& d, SequenceStore* store);
    BufferNeeds needs() const override;
    int enqueue(M40llmCudaContext* ctx, const StepBatch& batch, StepBuffers& b) override;

private:
    uint32_t mixer_out() const;
    MixerKind kind() const { return (MixerKind)d_.mixer; }
    int enqueue_mixer(M40llmCudaContext* ctx, const M40llmStepRows& rows, StepBuffers& b);
    int enqueue_experts(M40llmCudaContext* ctx, const M40llmLinear& proto, StepBuffers& b);
    uint32_t width_, w_dtype_;
    bool exact_;
    StackLayerDesc d_;
    SequenceStore* store_;
    size_t handle_, conv_handle_ = 0;
};

class JoinLayer : public ModelLayer {
public:
    JoinLayer(uint32_t width, uint32_t w_dtype, bool exact, const void* w, const void* bias)
        : width_(width), w_dtype_(w_dtype), exact_(exact), w_(w), bias_(bias) {}
    BufferNeeds needs() const override;
    bool is_join() const override { return true; }
    int enqueue(M40llmCudaContext* ctx, const StepBatch& batch, StepBuffers& b) override;

private:
    uint32_t width_, w_dtype_;
    bool exact_;
    const void *w_, *bias_;
};

}  // namespace m40host
