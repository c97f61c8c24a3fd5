#include "decode_model.hpp"

#include <string.h>

#include <algorithm>

namespace m40host {

namespace {
constexpr uint32_t kMaxWant = 128;  // rows per logits pass
}

DecodeModel::DecodeModel(M40llmCudaContext* ctx, const ModelConfig& cfg, const std::vector<LayerWeights>& layers,
                         const ModelHead& head, M40llmKVCache* kv, uint32_t sequences, uint32_t max_rows)
    : ctx_(ctx), cfg_(cfg), head_(head), seqs_(sequences), max_rows_(std::max(max_rows, sequences)) {
    if (!ctx || !kv || sequences == 0 || layers.empty() || !head.embeddings || !head.lm_head || head.vocab == 0) return;
    // the caller owns the cache; the store is only the table of sequences
    store_.reset(new SequenceStore(ctx, sequences, 0xffffffffu, M40LLM_DT_F16));
    for (size_t l = 0; l < layers.size(); ++l)
        layers_.emplace_back(new LlamaLayer(cfg, layers[l], kv, (uint32_t)l));
    flat_layers_ = (uint32_t)layers.size();
    ok_ = allocate() == 0;
}

DecodeModel::DecodeModel(M40llmCudaContext* ctx, uint32_t hidden, const ModelHead& head, uint32_t sequences, uint32_t max_len,
                         uint32_t max_rows, uint32_t cache_dtype)
    : ctx_(ctx), head_(head), seqs_(sequences), max_rows_(std::max(max_rows, sequences)) {
    cfg_.hidden = hidden;
    if (!ctx || hidden == 0 || sequences == 0 || max_len == 0) return;
    store_.reset(new SequenceStore(ctx, sequences, max_len, cache_dtype));
}

int DecodeModel::finish() {
    if (!store_ || layers_.empty() || !head_.embeddings || !head_.lm_head || head_.vocab == 0) return fail(-1, "incomplete_model");
    if (store_->allocate() != 0) return fail(-2, "cache_allocation");
    if (allocate() != 0) return fail(-2, "workspace_allocation");
    ok_ = true;
    return 0;
}

int DecodeModel::allocate() {
    for (const auto& l : layers_) needs_.merge(l->needs());
    const size_t r = max_rows_, h = cfg_.hidden;
    max_want_ = std::max(kMaxWant, seqs_);
    auto get = [&](size_t bytes, void** p) { return bytes == 0 || m40llm_device_malloc(ctx_, bytes, p) == 0; };
    bool good = get(r * h * 4, &buf_.x) && get(r * h * 4, &buf_.spare) && get(r * h * 4, &buf_.x1) &&
                get(r * needs_.packed * 4, &buf_.packed) && get(r * needs_.att * 4, &buf_.att) &&
                get(r * needs_.hid * 4, &buf_.hid) && get(r * needs_.low * 4, &buf_.low) &&
                get(needs_.x0 ? r * h * 4 : 0, &buf_.x0) && get(needs_.conv ? r * h * 4 : 0, &buf_.conv) && get((size_t)max_want_ * h * 4, &d_want_x_) &&
                get((size_t)max_want_ * head_.vocab * 4, &d_logits_) && get((9 * r + max_want_) * 4, &d_plan_) &&
                get((size_t)flat_layers_ * r * 4, (void**)&d_flat_) && get((size_t)kHistory * seqs_ * 4, &d_history_);
    if (!good) return -1;
    uint32_t* p = (uint32_t*)d_plan_;
    d_tokens_ = p, d_seq_ = p + r, d_pos_ = p + 2 * r, d_lens_ = p + 3 * r, d_want_ = p + 4 * r, d_seg_ = p + 5 * r;
    d_next_ = p + 9 * r;
    return 0;
}

DecodeModel::~DecodeModel() {
    if (!ctx_) return;
    m40llm_stream_synchronize(ctx_, 1);
    for (auto& g : graphs_)
        if (g.second) m40llm_cuda_graph_destroy(g.second);
    void* bufs[] = {buf_.x, buf_.spare, buf_.x0, buf_.packed, buf_.att, buf_.x1, buf_.hid, buf_.low, buf_.conv,
                    d_want_x_, d_logits_, d_plan_, d_flat_, d_history_};
    for (void* b : bufs)
        if (b) m40llm_device_free(ctx_, b);
}

int DecodeModel::fail(int rc, const std::string& step) {
    failed_step_ = step;
    return rc;
}

StepBatch DecodeModel::batch(uint32_t rows, uint32_t segments, uint32_t max_segment_rows, uint32_t max_len) const {
    StepBatch b;
    b.rows = {rows, segments, max_segment_rows, max_len, 1u, 0u, d_seq_, d_pos_, d_lens_, d_seg_, max_len ? seg_host_.data() : nullptr};
    b.flat_slots = d_flat_;
    b.flat_stride = max_rows_;
    return b;
}

int DecodeModel::upload_rows(uint32_t rows, const std::vector<uint32_t>& tokens, const std::vector<uint32_t>& seq,
                             const std::vector<uint32_t>& pos, const std::vector<uint32_t>& seg,
                             const std::vector<uint32_t>& want) {
    const size_t r = max_rows_;
    std::vector<uint32_t> host(9 * r, 0u);
    for (uint32_t i = 0; i < rows; ++i) {
        host[i] = tokens[i];
        host[r + i] = seq[i];
        host[2 * r + i] = pos[i];
        host[3 * r + i] = pos[i] + 1u;  // the new token is attended too
    }
    std::copy(want.begin(), want.end(), host.begin() + 4 * r);
    std::copy(seg.begin(), seg.end(), host.begin() + 5 * r);
    seg_host_ = seg;
    int rc = m40llm_stream_synchronize(ctx_, 1);
    if (rc != 0) return fail(rc, "stream_synchronize");
    if ((rc = m40llm_memcpy_h2d(ctx_, d_plan_, host.data(), host.size() * 4)) != 0) return fail(rc, "upload_plan");
    if (flat_layers_) {
        // slot of (sequence, layer) = sequence * layers + layer, laid out [layer][row] for the per-layer calls
        std::vector<uint32_t> flat(flat_layers_ * r, 0u);
        for (size_t l = 0; l < flat_layers_; ++l)
            for (uint32_t i = 0; i < rows; ++i) flat[l * r + i] = seq[i] * flat_layers_ + (uint32_t)l;
        if ((rc = m40llm_memcpy_h2d(ctx_, d_flat_, flat.data(), flat.size() * 4)) != 0) return fail(rc, "upload_slots");
    }
    return 0;
}

int DecodeModel::enqueue_layers(const StepBatch& b, void** x_out) {
    const uint32_t r = b.rows.rows, H = cfg_.hidden;
    StepBuffers bufs = buf_;
    int rc = m40llm_embed_tokens_async(ctx_, head_.embeddings, head_.table_dtype, d_tokens_, bufs.x, r, H, head_.vocab);
    if (rc != 0) return fail(rc, "embed_tokens");
    if (needs_.x0 && (rc = m40llm_memcpy_d2d_async(ctx_, bufs.x0, bufs.x, (size_t)r * H * 4, 1u)) != 0)
        return fail(rc, "keep_embedding");
    size_t traced = 0;
    for (size_t l = 0; l < layers_.size(); ++l) {
        if ((rc = layers_[l]->enqueue(ctx_, b, bufs)) != 0)
            return fail(rc, "layer " + std::to_string(l) + " " + layers_[l]->failed_step());
        if (layer_trace_ && !layers_[l]->is_join()) {
            if ((rc = m40llm_stream_synchronize(ctx_, 1)) != 0) return fail(rc, "trace_synchronize");
            if ((rc = m40llm_memcpy_d2h(ctx_, layer_trace_ + traced * r * H, bufs.x, (size_t)r * H * 4)) != 0)
                return fail(rc, "trace_copy");
            ++traced;
        }
    }
    *x_out = bufs.x;
    return 0;
}

int DecodeModel::enqueue_head(const void* x, uint32_t rows) {
    int rc;
    if (!head_.generic) {
        rc = m40llm_logits_head_f32_async(ctx_, x, head_.output_norm, 1u, cfg_.rms_eps, head_.lm_head, d_logits_, rows, cfg_.hidden,
                                          head_.vocab);
        return rc == 0 ? 0 : fail(rc, "logits_head");
    }
    M40llmLinear c = {};
    c.x = x;
    c.w = head_.lm_head;
    c.out = d_logits_;
    c.pre = head_.norm;
    c.rows = rows;
    c.K = cfg_.hidden;
    c.N = head_.vocab;
    c.w_dtype = head_.table_dtype;
    c.exact = head_.exact ? 1u : 0u;
    c.soft_cap = head_.soft_cap;
    rc = m40llm_linear_async(ctx_, &c, 1u);
    return rc == 0 ? 0 : fail(rc, "logits_head");
}

int DecodeModel::step(const std::vector<StepEntry>& entries, const uint32_t* tokens, const std::vector<uint32_t>& want,
                      float* out_logits, uint32_t* out_next) {
    if (!ok_) return fail(-1, "not_initialised");
    uint64_t total = 0;
    std::vector<bool> seen(seqs_, false);
    for (const StepEntry& e : entries) {
        if (e.count == 0 || !store_->live(e.sequence) || seen[e.sequence]) return fail(-2, "step_entry");
        if ((uint64_t)store_->length(e.sequence) + e.count > store_->max_len()) return fail(-3, "sequence_too_long");
        seen[e.sequence] = true;
        total += e.count;
    }
    if (total == 0 || total > 0x7fffffffu) return fail(-2, "step_entry");
    for (size_t i = 0; i < want.size(); ++i)
        if (want[i] >= total || (i && want[i] <= want[i - 1])) return fail(-2, "wanted_rows");
    for (uint64_t i = 0; i < total; ++i)
        if (tokens[i] >= head_.vocab) return fail(-2, "token_id");

    size_t entry = 0, next_want = 0;
    uint32_t done_in_entry = 0;
    uint64_t base = 0;  // rows of earlier passes
    while (base < total) {
        std::vector<uint32_t> tok, seq, pos, seg, local;
        uint32_t max_seg = 0, max_len = 0;
        std::vector<StepEntry> advanced;
        while (entry < entries.size() && tok.size() < max_rows_) {
            const StepEntry& e = entries[entry];
            const uint32_t room = max_rows_ - (uint32_t)tok.size(), left = e.count - done_in_entry;
            const uint32_t n = std::min(room, left), p0 = store_->length(e.sequence);
            seg.insert(seg.end(), {(uint32_t)tok.size(), n, e.sequence, p0});
            for (uint32_t i = 0; i < n; ++i) {
                tok.push_back(tokens[base + tok.size()]);
                seq.push_back(e.sequence);
                pos.push_back(p0 + i);
            }
            max_seg = std::max(max_seg, n);
            max_len = std::max(max_len, p0 + n);
            advanced.push_back({e.sequence, n});
            done_in_entry += n;
            if (done_in_entry == e.count) ++entry, done_in_entry = 0;
            else break;  // one portion of a sequence per pass
        }
        const uint32_t rows = (uint32_t)tok.size();
        size_t want_end = next_want;
        while (want_end < want.size() && want[want_end] < base + rows) local.push_back((uint32_t)(want[want_end++] - base));
        int rc = upload_rows(rows, tok, seq, pos, seg, local);
        if (rc != 0) return rc;
        void* x = nullptr;
        if ((rc = enqueue_layers(batch(rows, (uint32_t)(seg.size() / 4), max_seg, max_len), &x)) != 0) return rc;
        for (size_t w = 0; w < local.size(); w += max_want_) {
            const uint32_t n = (uint32_t)std::min<size_t>(max_want_, local.size() - w);
            rc = m40llm_gather_rows_async(ctx_, x, d_want_ + w, d_want_x_, n, cfg_.hidden, rows);
            if (rc != 0) return fail(rc, "gather_wanted");
            if ((rc = enqueue_head(d_want_x_, n)) != 0) return rc;
            if (out_next && (rc = m40llm_argmax_f32_async(ctx_, d_logits_, n, head_.vocab, d_next_)) != 0)
                return fail(rc, "argmax");
            if ((rc = m40llm_stream_synchronize(ctx_, 1)) != 0) return fail(rc, "stream_synchronize");
            if (out_logits && (rc = m40llm_memcpy_d2h(ctx_, out_logits + (next_want + w) * head_.vocab, d_logits_,
                                                      (size_t)n * head_.vocab * 4)) != 0)
                return fail(rc, "read_logits");
            if (out_next && (rc = m40llm_memcpy_d2h(ctx_, out_next + next_want + w, d_next_, (size_t)n * 4)) != 0)
                return fail(rc, "read_ids");
        }
        if ((rc = m40llm_stream_synchronize(ctx_, 1)) != 0) return fail(rc, "stream_synchronize");
        for (const StepEntry& e : advanced) store_->set_length(e.sequence, store_->length(e.sequence) + e.count);
        next_want = want_end;
        base += rows;
    }
    uint32_t status = 0;
    if (m40llm_context_take_device_status(ctx_, &status) == 0 && status != 0) return fail(-(int)(1000 + status), "device_status");
    return 0;
}

int DecodeModel::begin(const uint32_t* token_ids, const uint32_t* positions) {
    if (!ok_) return fail(-1, "not_initialised");
    std::vector<uint32_t> sequences(seqs_);
    for (uint32_t s = 0; s < seqs_; ++s) {
        sequences[s] = s;
        if (store_->set_length(s, positions[s]) != 0) return fail(-3, "position");
    }
    return begin_sequences(seqs_, sequences.data(), token_ids);
}

int DecodeModel::begin_sequences(uint32_t n, const uint32_t* sequences, const uint32_t* token_ids) {
    if (!ok_) return fail(-1, "not_initialised");
    if (n == 0 || n > seqs_) return fail(-2, "begin_rows");
    std::vector<uint32_t> tok(token_ids, token_ids + n), seq(sequences, sequences + n), pos(n), seg;
    std::vector<bool> seen(seqs_, false);
    for (uint32_t i = 0; i < n; ++i) {
        if (!store_->live(seq[i]) || seen[seq[i]]) return fail(-2, "begin_sequence");
        seen[seq[i]] = true;
        pos[i] = store_->length(seq[i]);
        seg.insert(seg.end(), {i, 1u, seq[i], pos[i]});
    }
    const int rc = upload_rows(n, tok, seq, pos, seg, {});
    if (rc != 0) return rc;
    rows_ = n;
    row_sequences_ = seq;
    return 0;
}

// One token for every row: embed -> layers -> logits -> arg-max into the token array (the next step's input) -> positions
// and lengths advance. The chosen ids are also appended to the history ring by a device-to-device copy so that a replayed
// graph leaves a trace per step.
int DecodeModel::enqueue_token_step() {
    void* x = nullptr;
    int rc = enqueue_layers(batch(rows_, rows_, 1u, 0u), &x);
    if (rc != 0) return rc;
    if ((rc = enqueue_head(x, rows_)) != 0) return rc;
    rc = m40llm_argmax_f32_async(ctx_, d_logits_, rows_, head_.vocab, d_tokens_);
    if (rc != 0) return fail(rc, "argmax");
    rc = m40llm_advance_positions_async(ctx_, d_pos_, d_lens_, rows_);
    if (rc != 0) return fail(rc, "advance_positions");
    return 0;
}

int DecodeModel::generate(uint32_t steps, bool use_graph, uint32_t* out_ids, float* out_logits) {
    if (!ok_) return fail(-1, "not_initialised");
    if (steps == 0) return 0;
    if (rows_ == 0) return fail(-2, "generate_before_begin");
    if (out_ids && steps > kHistory) return fail(-2, "too_many_steps_for_history");
    for (uint32_t s : row_sequences_)
        if ((uint64_t)store_->length(s) + steps > store_->max_len()) return fail(-3, "sequence_too_long");
    int rc;
    for (uint32_t t = 0; t < steps; ++t) {
        M40llmCudaGraphExec* graph = use_graph ? graphs_[rows_] : nullptr;
        if (graph) {
            if ((rc = m40llm_cuda_graph_launch(ctx_, graph, 1u)) != 0) return fail(rc, "graph_launch");
            ++graph_replays_;
        } else {
            uint64_t n0 = 0, n1 = 0;
            m40llm_context_launch_count(ctx_, &n0);
            if ((rc = enqueue_token_step()) != 0) return rc;
            m40llm_context_launch_count(ctx_, &n1);
            launches_per_step_ = n1 - n0;
        }
        // the ids chosen by this step, kept per step so that back-to-back replays leave a trace
        if (out_ids && (rc = m40llm_memcpy_d2d_async(ctx_, (char*)d_history_ + (size_t)t * rows_ * 4, d_tokens_,
                                                     (size_t)rows_ * 4, 1u)) != 0)
            return fail(rc, "history_copy");
        if (!graph && use_graph && !capture_tried_[rows_] && t + 1 < steps) {
            // the eager step sized every scratch arena; capture the same sequence once for all later tokens
            capture_tried_[rows_] = true;
            if ((rc = m40llm_stream_synchronize(ctx_, 1u)) != 0) return fail(rc, "sync_before_capture");
            if (m40llm_cuda_graph_begin_capture(ctx_, 1u) == 0) {
                rc = enqueue_token_step();
                if (rc != 0) {
                    m40llm_cuda_graph_cancel_capture(ctx_, 1u);
                    return rc;
                }
                M40llmCudaGraphExec* exec = nullptr;
                if (m40llm_cuda_graph_end_capture(ctx_, 1u, &exec) == 0 && exec) graphs_[rows_] = exec;
            }
        }
    }
    if ((rc = m40llm_stream_synchronize(ctx_, 1u)) != 0) return fail(rc, "stream_synchronize");
    for (uint32_t s : row_sequences_) store_->set_length(s, store_->length(s) + steps);
    if (out_ids && (rc = m40llm_memcpy_d2h(ctx_, out_ids, d_history_, (size_t)steps * rows_ * 4)) != 0)
        return fail(rc, "read_ids");
    if (out_logits && (rc = m40llm_memcpy_d2h(ctx_, out_logits, d_logits_, (size_t)rows_ * head_.vocab * 4)) != 0)
        return fail(rc, "read_logits");
    uint32_t status = 0;
    if (m40llm_context_take_device_status(ctx_, &status) == 0 && status != 0) return fail(-(int)(1000 + status), "device_status");
    return 0;
}

}  // namespace m40host
