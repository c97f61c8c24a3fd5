#include "sequence_store.hpp"

namespace m40host {

SequenceStore::SequenceStore(M40llmCudaContext* ctx, uint32_t sequences, uint32_t max_len, uint32_t elem_dtype)
    : ctx_(ctx), max_len_(max_len), elem_dtype_(elem_dtype), length_(sequences, 0u), live_(sequences, false) {}

SequenceStore::~SequenceStore() {
    for (Group& g : groups_) {
        if (g.kv) m40llm_kvcache_destroy(g.kv);
        if (g.state) m40llm_statecache_destroy(g.state);
    }
}

size_t SequenceStore::add(bool is_state, uint32_t heads, uint32_t a, uint32_t b) {
    size_t g = 0;
    while (g < groups_.size() && !(groups_[g].is_state == is_state && groups_[g].heads == heads && groups_[g].a == a &&
                                   groups_[g].b == b))
        ++g;
    if (g == groups_.size()) groups_.push_back({is_state, heads, a, b, 0u, nullptr, nullptr});
    members_.push_back({g, groups_[g].members++});
    return members_.size() - 1;
}

size_t SequenceStore::add_kv(uint32_t kv_heads, uint32_t k_dim, uint32_t v_dim) { return add(false, kv_heads, k_dim, v_dim); }
size_t SequenceStore::add_latent(uint32_t rank) { return add(false, 1u, rank, 0u); }
size_t SequenceStore::add_state(uint32_t heads, uint32_t dim) { return add(true, heads, dim, 0u); }
size_t SequenceStore::add_values(uint32_t values) { return add(true, 0u, values, 0u); }

int SequenceStore::allocate() {
    for (Group& g : groups_) {
        const uint32_t slots = (uint32_t)length_.size() * g.members;
        if (g.is_state) g.state = g.heads ? m40llm_statecache_create(ctx_, slots, g.heads, g.a)
                                          : m40llm_statecache_create_values(ctx_, slots, g.a);
        else g.kv = m40llm_kvcache_create_typed(ctx_, max_len_, slots, g.heads, g.a, g.b, elem_dtype_);
        if (!g.kv && !g.state) return -1;
    }
    return 0;
}

long SequenceStore::acquire() {
    for (size_t s = 0; s < live_.size(); ++s)
        if (!live_[s]) {
            live_[s] = true;
            length_[s] = 0;
            return (long)s;
        }
    return -1;
}

int SequenceStore::release(uint32_t sequence) {
    if (!live(sequence)) return -1;
    live_[sequence] = false;
    length_[sequence] = 0;
    return 0;
}

int SequenceStore::set_length(uint32_t sequence, uint32_t length) {
    if (sequence >= live_.size() || length > max_len_) return -1;
    live_[sequence] = true;
    length_[sequence] = length;
    return 0;
}

}  // namespace m40host
