// Whole-model execution over the m40llm C ABI: token embedding -> layers -> logits head -> arg-max, for a batch of
// independent sequences. Host-side mirror of the reference's session loop
// (DecodeSession::logits_for_token / forward_with_optional_graph, src/decode_session.rs:637-954;
// forward_one_token_all_layers_for_sequence, src/infer/forward.rs:1659-1716; logits_from_hidden_into,
// src/infer/logits.rs:57-116; Sampler::sample_greedy, src/sampling.rs:95-108).
//
// The layers are ModelLayer objects (model_layer.hpp): the reference's decode layer over a dense FP16 cache addressed as
// the reference does, slot = sequence * layers + layer (src/infer/kv.rs:109), or the layers of a stack whose caches and
// recurrent states live in the model's SequenceStore. Two ways to run them:
//   step()      any portions of any live sequences, host tokens in, logits of chosen rows (and greedy ids) out;
//   generate()  greedy tokens for a fixed set of sequences: token ids, positions and lengths live in device arrays that
//               the step itself advances, and the arg-max runs on the device, so one captured CUDA graph is replayed per
//               token with no host work between tokens; the host reads the generated ids when it wants them.
#pragma once
#include <stdint.h>

#include <map>
#include <memory>
#include <string>
#include <vector>

#include "decode_layer.hpp"
#include "model_layer.hpp"
#include "sequence_store.hpp"

namespace m40host {

struct ModelHead {
    const void* embeddings = nullptr;   // [vocab][hidden] of table_dtype
    const void* output_norm = nullptr;  // f32 [hidden] or null
    const void* lm_head = nullptr;      // [vocab][hidden] of table_dtype
    uint32_t vocab = 0;
    uint32_t table_dtype = M40LLM_DT_F16;
    // Heads beyond an f16 projection with an RMS norm: `generic` selects norm (instead of output_norm / rms_eps), soft cap
    // and the exact mode of m40llm_linear_async.
    bool generic = false;
    M40llmNorm norm = {};
    float soft_cap = 0.0f;
    bool exact = false;
};

// The next `count` tokens of a live sequence.
struct StepEntry {
    uint32_t sequence, count;
};

class DecodeModel {
public:
    // The reference's layer stack. `kv` must be a dense cache with at least sequences * layers slots.
    DecodeModel(M40llmCudaContext* ctx, const ModelConfig& cfg, const std::vector<LayerWeights>& layers,
                const ModelHead& head, M40llmKVCache* kv, uint32_t sequences, uint32_t max_rows = 0);
    // Any stack: add layers (their caches register with store()), then finish().
    DecodeModel(M40llmCudaContext* ctx, uint32_t hidden, const ModelHead& head, uint32_t sequences, uint32_t max_len,
                uint32_t max_rows, uint32_t cache_dtype);
    ~DecodeModel();
    DecodeModel(const DecodeModel&) = delete;
    DecodeModel& operator=(const DecodeModel&) = delete;
    bool ok() const { return ok_; }
    void add_layer(std::unique_ptr<ModelLayer> layer) { layers_.push_back(std::move(layer)); }
    int finish();  // allocates caches and work buffers; ok() afterwards
    SequenceStore& store() { return *store_; }
    uint32_t hidden() const { return cfg_.hidden; }

    // Runs the next tokens of the entries (each sequence at most once) on top of what its slot holds. `want` are row
    // indexes into the concatenated tokens whose logits are copied to out_logits [n_want][vocab] (ascending); out_next,
    // when given, receives the greedy choice after every wanted row. More rows than max_rows run as several passes.
    int step(const std::vector<StepEntry>& entries, const uint32_t* tokens, const std::vector<uint32_t>& want,
             float* out_logits, uint32_t* out_next);

    // Sets the next input token and its position (= tokens already in the cache) of sequences 0 .. n-1 (n = all), or of
    // the given live sequences at their stored lengths.
    int begin(const uint32_t* token_ids, const uint32_t* positions);
    int begin_sequences(uint32_t n, const uint32_t* sequences, const uint32_t* token_ids);
    // Runs `steps` greedy tokens back to back (graph replay after the first step when use_graph). When out_ids is
    // given it receives [steps][rows] generated ids (read back once, at the end); when out_logits is given it
    // receives the logits of the LAST step, [rows][vocab]. rows = the sequences of the last begin call.
    int generate(uint32_t steps, bool use_graph, uint32_t* out_ids, float* out_logits);
    uint32_t rows() const { return rows_; }

    // While set, step() copies the residual after every layer (joins excluded) to [layer][rows][hidden]; the steps must
    // fit in one pass.
    void trace_layers(float* out) { layer_trace_ = out; }

    const std::string& failed_step() const { return failed_step_; }
    uint64_t graph_replays() const { return graph_replays_; }
    uint64_t launches_per_step() const { return launches_per_step_; }

private:
    int allocate();
    int upload_rows(uint32_t rows, const std::vector<uint32_t>& tokens, const std::vector<uint32_t>& seq,
                    const std::vector<uint32_t>& pos, const std::vector<uint32_t>& seg, const std::vector<uint32_t>& want);
    StepBatch batch(uint32_t rows, uint32_t segments, uint32_t max_segment_rows, uint32_t max_len) const;
    int enqueue_layers(const StepBatch& batch, void** x_out);
    int enqueue_head(const void* x, uint32_t rows);
    int enqueue_token_step();
    int fail(int rc, const std::string& step);

    M40llmCudaContext* ctx_;
    ModelConfig cfg_;
    std::vector<std::unique_ptr<ModelLayer>> layers_;
    ModelHead head_;
    std::unique_ptr<SequenceStore> store_;
    uint32_t seqs_, max_rows_, max_want_ = 0, flat_layers_ = 0;
    bool ok_ = false;
    BufferNeeds needs_;
    StepBuffers buf_;
    void *d_want_x_ = nullptr, *d_logits_ = nullptr;
    // u32 arrays [max_rows] in one block: tokens | sequence | position | length | wanted rows, then segments [max_rows][4]
    void* d_plan_ = nullptr;
    uint32_t *d_tokens_ = nullptr, *d_seq_ = nullptr, *d_pos_ = nullptr, *d_lens_ = nullptr, *d_want_ = nullptr,
             *d_seg_ = nullptr, *d_next_ = nullptr;
    uint32_t* d_flat_ = nullptr;  // [flat layers][max_rows] cache slots
    void* d_history_ = nullptr;   // u32 [kHistory][sequences]: ids generated by the steps of one generate() call
    uint32_t rows_ = 0;           // rows of the current token step
    std::vector<uint32_t> row_sequences_;
    std::vector<uint32_t> seg_host_;  // segments of the last upload
    std::map<uint32_t, M40llmCudaGraphExec*> graphs_;  // by rows
    std::map<uint32_t, bool> capture_tried_;
    float* layer_trace_ = nullptr;
    std::string failed_step_;
    uint64_t graph_replays_ = 0, launches_per_step_ = 0;
    static constexpr uint32_t kHistory = 4096;
};

}  // namespace m40host
