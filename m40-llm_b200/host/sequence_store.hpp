// What the live sequences of a model hold: one table of sequence slots and the caches behind it. Layers of equal shape
// share one cache object (a KV cache or a recurrent-state cache) in which slot = sequence * members + member, the
// addressing of the reference's dense cache (src/infer/kv.rs:109) applied per group of equal layers.
//
// A slot that is released needs no clearing: keys and values beyond a sequence's length are never read, and a recurrent
// state is taken as zero at position 0.
#pragma once
#include <stdint.h>

#include <string>
#include <vector>

#include "../../include/m40llm_native.h"

namespace m40host {

class SequenceStore {
public:
    // elem_dtype: element type of the KV caches (M40LLM_DT_F16 or M40LLM_DT_F32)
    SequenceStore(M40llmCudaContext* ctx, uint32_t sequences, uint32_t max_len, uint32_t elem_dtype);
    ~SequenceStore();
    SequenceStore(const SequenceStore&) = delete;
    SequenceStore& operator=(const SequenceStore&) = delete;

    // Registers one cache-bearing layer (before allocate()) and returns its handle.
    size_t add_kv(uint32_t kv_heads, uint32_t k_dim, uint32_t v_dim);
    size_t add_latent(uint32_t rank);                    // one array of `rank` values per token (kv())
    size_t add_state(uint32_t heads, uint32_t dim);
    size_t add_values(uint32_t values);                  // f32 values per sequence (state())
    int allocate();  // 0, or -1 when a cache could not be made

    M40llmKVCache* kv(size_t handle) const { return groups_[members_[handle].group].kv; }
    M40llmStateCache* state(size_t handle) const { return groups_[members_[handle].group].state; }
    uint32_t slot_mul(size_t handle) const { return groups_[members_[handle].group].members; }
    uint32_t slot_add(size_t handle) const { return members_[handle].index; }

    // Sequence table.
    uint32_t sequences() const { return (uint32_t)length_.size(); }
    uint32_t max_len() const { return max_len_; }
    long acquire();  // the lowest free slot, or -1 when all are live
    int release(uint32_t sequence);
    bool live(uint32_t sequence) const { return sequence < live_.size() && live_[sequence]; }
    uint32_t length(uint32_t sequence) const { return length_[sequence]; }
    // Marks the slot live with `length` tokens (a caller that manages positions itself).
    int set_length(uint32_t sequence, uint32_t length);

private:
    struct Group {
        bool is_state;
        uint32_t heads, a, b;  // kv: k_dim, v_dim (0: latents); state: dim, 0, or heads = 0 and the number of values
        uint32_t members;
        M40llmKVCache* kv;
        M40llmStateCache* state;
    };
    struct Member { size_t group; uint32_t index; };
    size_t add(bool is_state, uint32_t heads, uint32_t a, uint32_t b);

    M40llmCudaContext* ctx_;
    uint32_t max_len_, elem_dtype_;
    std::vector<Group> groups_;
    std::vector<Member> members_;
    std::vector<uint32_t> length_;
    std::vector<bool> live_;
};

}  // namespace m40host
