#include "model_layer.hpp"

#include <utility>

namespace m40host {

namespace {
// Portions from this many rows on compute the delta rule's low-rank decay as a projection of its own; below (and when
// every row is a token of its own sequence) the mixer kernel does it.
constexpr uint32_t LOW_RANK_ROWS = 2;
}  // namespace

BufferNeeds LlamaLayer::needs() const {
    BufferNeeds n;
    n.packed = n.att = (size_t)cfg_.q_heads * cfg_.head_dim;
    n.hid = cfg_.ffn;
    return n;
}

int LlamaLayer::enqueue(M40llmCudaContext* ctx, const StepBatch& batch, StepBuffers& b) {
    const uint32_t H = cfg_.hidden, QD = cfg_.q_heads * cfg_.head_dim, r = batch.rows.rows;
    const uint32_t* slots = batch.flat_slots + (size_t)index_ * batch.flat_stride;
    int rc = m40llm_qkv_rope_append_attention_async(ctx, kv_, b.x, w_.attn_norm, 1u, cfg_.rms_eps, w_.wq, w_.wk, w_.wv, w_.bq,
                                                    w_.bk, w_.bv, slots, batch.rows.row_pos, batch.rows.row_len, r, H,
                                                    cfg_.q_heads, cfg_.rope_base, cfg_.rope_scale, cfg_.rope_layout, b.packed,
                                                    b.att);
    if (rc != 0) return fail(rc, "qkv_rope_append_attention");
    rc = m40llm_attn_out_ffn_async(ctx, b.att, w_.wo, b.x, w_.ffn_norm, 1u, cfg_.rms_eps, w_.wg, w_.wu, w_.wd,
                                   w_.ffn_q80 ? 1u : 0u, b.x1, b.hid, b.spare, r, H, QD, cfg_.ffn);
    if (rc != 0) return fail(rc, "attn_out_ffn");
    std::swap(b.x, b.spare);
    return 0;
}

StackLayer::StackLayer(uint32_t width, uint32_t w_dtype, bool exact, const StackLayerDesc& d, SequenceStore* store)
    : width_(width), w_dtype_(w_dtype), exact_(exact), d_(d), store_(store) {
    handle_ = d.mixer == (uint32_t)MixerKind::DeltaRule ? store->add_state(d.heads, d.dim)
                                                        : store->add_kv(d.kv_heads, d.k_dim, d.v_dim);
}

uint32_t StackLayer::mixer_out() const {
    return d_.mixer == (uint32_t)MixerKind::DeltaRule ? d_.heads * d_.dim : d_.q_heads * d_.v_dim;
}

BufferNeeds StackLayer::needs() const {
    BufferNeeds n;
    n.packed = d_.n_in;
    n.att = mixer_out();
    n.hid = d_.ff;
    if (d_.mixer == (uint32_t)MixerKind::DeltaRule) n.low = mixer_out();
    return n;
}

int StackLayer::enqueue(M40llmCudaContext* ctx, const StepBatch& batch, StepBuffers& b) {
    M40llmStepRows rows = batch.rows;
    rows.slot_mul = store_->slot_mul(handle_);
    rows.slot_add = store_->slot_add(handle_);
    M40llmLinear in = {};
    in.x = b.x;
    in.w = d_.w_in;
    in.out = b.packed;
    in.pre = d_.norm1;
    in.rows = rows.rows;
    in.K = width_;
    in.N = d_.n_in;
    in.w_dtype = w_dtype_;
    in.exact = exact_ ? 1u : 0u;
    int rc = m40llm_linear_async(ctx, &in, 1u);
    if (rc != 0) return fail(rc, "mixer_in");

    if (d_.mixer == (uint32_t)MixerKind::DeltaRule) {
        const uint32_t HD = d_.heads * d_.dim;
        M40llmDeltaRule m = {};
        m.packed = b.packed;
        m.ld = d_.n_in;
        if (rows.max_segment_rows >= LOW_RANK_ROWS) {
            M40llmLinear low = {};
            low.x = (const float*)b.packed + (size_t)5 * HD;
            low.ldx = d_.n_in;
            low.w = d_.w2;
            low.out = b.low;
            low.pre.kind = M40LLM_NORM_DYT;  // a bare tanh
            low.pre.alpha = 1.0f;
            low.rows = rows.rows;
            low.K = d_.rank;
            low.N = HD;
            low.w_dtype = w_dtype_;
            low.exact = in.exact;
            if ((rc = m40llm_linear_async(ctx, &low, 1u)) != 0) return fail(rc, "delta_low_rank");
            m.decay_in = b.low;
        }
        m.w2 = d_.w2;
        m.rank = d_.rank;
        m.w_dtype = w_dtype_;
        m.w0 = d_.w0;
        m.a_bias = d_.a_bias;
        m.norm = d_.o_norm;
        m.out = b.att;
        m.decay_scale = d_.decay_scale;
        m.unit_eps = d_.unit_eps;
        m.eps = d_.eps;
        if ((rc = m40llm_delta_rule_async(ctx, store_->state(handle_), &m, &rows)) != 0) return fail(rc, "delta_rule");
    } else {
        M40llmRotaryAttention m = {};
        m.packed = b.packed;
        m.ld = d_.n_in;
        m.q_norm = d_.q_norm;
        m.k_norm = d_.k_norm;
        m.k_turns = d_.k_turns;
        m.v_turns = d_.v_turns;
        m.out = b.att;
        m.q_heads = d_.q_heads;
        m.k_pairs = d_.k_pairs;
        m.has_gate = d_.has_gate;
        m.eps = d_.eps;
        m.k_amp = d_.k_amp;
        m.scale = d_.scale;
        if ((rc = m40llm_attention_rotary_async(ctx, store_->kv(handle_), &m, &rows)) != 0) return fail(rc, "attention_rotary");
    }

    M40llmLinear out = in;
    out.x = b.att;
    out.w = d_.w_out;
    out.out = b.x;
    out.residual = b.x;
    out.pre = M40llmNorm{};
    out.post = d_.norm1b;
    out.K = mixer_out();
    out.N = width_;
    if ((rc = m40llm_linear_async(ctx, &out, 1u)) != 0) return fail(rc, "mixer_out");
    if (d_.ff == 0) return 0;

    M40llmLinear up = in;
    up.w = d_.gate;
    up.w2 = d_.up;
    up.act = d_.act;
    up.out = b.hid;
    up.pre = d_.norm2;
    up.N = d_.ff;
    if ((rc = m40llm_linear_async(ctx, &up, 1u)) != 0) return fail(rc, "mlp_up");
    M40llmLinear down = out;
    down.x = b.hid;
    down.w = d_.down;
    down.post = d_.norm2b;
    down.K = d_.ff;
    if ((rc = m40llm_linear_async(ctx, &down, 1u)) != 0) return fail(rc, "mlp_down");
    return 0;
}

BufferNeeds JoinLayer::needs() const {
    BufferNeeds n;
    n.packed = 2 * (size_t)width_;
    n.x0 = true;
    return n;
}

int JoinLayer::enqueue(M40llmCudaContext* ctx, const StepBatch& batch, StepBuffers& b) {
    int rc = m40llm_concat_rows_async(ctx, b.x, b.x0, b.packed, batch.rows.rows, width_);
    if (rc != 0) return fail(rc, "join_concat");
    M40llmLinear c = {};
    c.x = b.packed;
    c.w = w_;
    c.out = b.x;
    c.bias = bias_;
    c.rows = batch.rows.rows;
    c.K = 2 * width_;
    c.N = width_;
    c.w_dtype = w_dtype_;
    c.exact = exact_ ? 1u : 0u;
    if ((rc = m40llm_linear_async(ctx, &c, 1u)) != 0) return fail(rc, "join_projection");
    return 0;
}

}  // namespace m40host
