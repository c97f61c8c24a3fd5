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
    switch (kind()) {
        case MixerKind::DeltaRule: handle_ = store->add_state(d.heads, d.dim); break;
        case MixerKind::LatentAttention: handle_ = store->add_latent(d.rank_kv); break;
        case MixerKind::RgLru: handle_ = store->add_values(d.rg_width * (1u + d.rg_taps)); break;
        default: handle_ = store->add_kv(d.kv_heads, d.k_dim, d.v_dim);
    }
    if (d.conv_taps > 1) conv_handle_ = store->add_values(d.conv_taps * width);
}

uint32_t StackLayer::mixer_out() const {
    switch (kind()) {
        case MixerKind::DeltaRule: return d_.heads * d_.dim;
        case MixerKind::RgLru: return d_.rg_width;
        default: return d_.q_heads * d_.v_dim;
    }
}

BufferNeeds StackLayer::needs() const {
    BufferNeeds n;
    n.packed = d_.n_in;
    n.att = mixer_out();
    n.hid = d_.experts ? d_.n_router : d_.ff;
    n.conv = d_.conv_taps > 0;
    if (kind() == MixerKind::DeltaRule) n.low = mixer_out();
    if (d_.experts && d_.shared_ff) n.low = width_;  // the shared expert's output
    return n;
}

int StackLayer::enqueue(M40llmCudaContext* ctx, const StepBatch& batch, StepBuffers& b) {
    M40llmStepRows rows = batch.rows;
    const void* x_in = b.x;
    int rc;
    if (d_.conv_taps) {
        if (d_.conv_taps > 1) rows.slot_mul = store_->slot_mul(conv_handle_), rows.slot_add = store_->slot_add(conv_handle_);
        const M40llmShortConv c = {b.x, d_.conv_w, nullptr, b.conv, 0, width_, d_.conv_taps, 1u};
        rc = m40llm_short_conv_async(ctx, d_.conv_taps > 1 ? store_->state(conv_handle_) : nullptr, &c, &rows);
        if (rc != 0) return fail(rc, "input_convolution");
        x_in = b.conv;
    }
    rows.slot_mul = store_->slot_mul(handle_);
    rows.slot_add = store_->slot_add(handle_);
    M40llmLinear in = {};
    in.x = x_in;
    in.w = d_.w_in;
    in.out = b.packed;
    in.bias = d_.in_bias;
    in.pre = d_.norm1;
    in.rows = rows.rows;
    in.K = width_;
    in.N = d_.n_in;
    in.w_dtype = w_dtype_;
    in.exact = exact_ ? 1u : 0u;
    if ((rc = m40llm_linear_async(ctx, &in, 1u)) != 0) return fail(rc, "mixer_in");
    if ((rc = enqueue_mixer(ctx, rows, b)) != 0) return rc;

    M40llmLinear out = in;
    out.x = b.att;
    out.w = d_.w_out;
    out.out = b.x;
    out.bias = nullptr;
    out.residual = b.x;
    out.pre = M40llmNorm{};
    out.post = d_.norm1b;
    out.K = mixer_out();
    out.N = width_;
    if ((rc = m40llm_linear_async(ctx, &out, 1u)) != 0) return fail(rc, "mixer_out");
    if (d_.ff == 0) return 0;

    M40llmLinear up = in;
    up.x = b.x;
    up.bias = nullptr;
    up.pre = d_.norm2;
    if (d_.experts) return enqueue_experts(ctx, up, b);
    up.w = d_.gate ? d_.gate : d_.up;
    up.w2 = d_.gate ? d_.up : nullptr;
    up.act = d_.act;
    up.out = b.hid;
    up.N = d_.ff;
    if ((rc = m40llm_linear_async(ctx, &up, 1u)) != 0) return fail(rc, "mlp_up");
    M40llmLinear down = out;
    down.x = b.hid;
    down.w = d_.down;
    down.pre = d_.mid;
    down.post = d_.norm2b;
    down.K = d_.ff;
    if ((rc = m40llm_linear_async(ctx, &down, 1u)) != 0) return fail(rc, "mlp_down");
    return 0;
}

int StackLayer::enqueue_mixer(M40llmCudaContext* ctx, const M40llmStepRows& rows, StepBuffers& b) {
    int rc;
    if (kind() == MixerKind::DeltaRule) {
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
            low.exact = exact_ ? 1u : 0u;
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
        return 0;
    }
    if (kind() == MixerKind::LatentAttention) {
        M40llmLatentAttention m = {};
        m.packed = b.packed;
        m.ld = d_.n_in;
        m.c_norm = d_.c_norm;
        m.uk = d_.uk;
        m.uk_t = d_.uk_t;
        m.uv = d_.uv;
        m.sink = d_.sink;
        m.out = b.att;
        m.heads = d_.q_heads;
        m.dim = d_.k_dim;
        m.vdim = d_.v_dim;
        m.w_dtype = w_dtype_;
        m.eps = d_.eps;
        m.scale = d_.scale;
        if ((rc = m40llm_attention_latent_async(ctx, store_->kv(handle_), &m, &rows)) != 0) return fail(rc, "attention_latent");
        return 0;
    }
    if (kind() == MixerKind::RgLru) {
        M40llmRgLru m = {};
        m.packed = b.packed;
        m.ld = d_.n_in;
        m.conv_w = d_.rg_conv;
        m.conv_b = d_.rg_conv_b;
        m.ra = d_.ra;
        m.ra_b = d_.ra_b;
        m.ri = d_.ri;
        m.ri_b = d_.ri_b;
        m.lam = d_.lam;
        m.out = b.att;
        m.width = d_.rg_width;
        m.blocks = d_.rg_blocks;
        m.taps = d_.rg_taps;
        m.w_dtype = w_dtype_;
        m.exact = exact_ ? 1u : 0u;
        m.decay = d_.rg_decay;
        if ((rc = m40llm_rglru_async(ctx, store_->state(handle_), &m, &rows)) != 0) return fail(rc, "rglru");
        return 0;
    }
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
    return 0;
}

// `proto`: a projection of the layer's rows of x. The router and the shared expert's first matrix are one projection.
int StackLayer::enqueue_experts(M40llmCudaContext* ctx, const M40llmLinear& proto, StepBuffers& b) {
    int rc;
    M40llmLinear first = proto;
    first.w = d_.w_router;
    first.out = b.hid;
    first.N = d_.n_router;
    if ((rc = m40llm_linear_async(ctx, &first, 1u)) != 0) return fail(rc, "router");
    if (d_.shared_ff) {
        M40llmLinear down = proto;
        down.x = b.hid;
        down.ldx = d_.n_router;
        down.w = d_.shared_down;
        down.out = b.low;
        down.pre = M40llmNorm{};
        down.pre.kind = M40LLM_NORM_ACT;
        down.pre.act = d_.act;
        down.K = d_.shared_ff;
        down.N = width_;
        if ((rc = m40llm_linear_async(ctx, &down, 1u)) != 0) return fail(rc, "shared_expert");
    }
    M40llmMoe m = {};
    m.x = b.x;
    m.logits = (const float*)b.hid + d_.shared_ff;
    m.ld_logits = d_.n_router;
    m.correction = d_.correction;
    m.up = d_.up;
    m.down = d_.down;
    m.add = d_.shared_ff ? b.low : nullptr;
    m.residual = b.x;
    m.out = b.x;
    m.post = d_.norm2b;
    m.rows = proto.rows;
    m.K = width_;
    m.ff = d_.ff;
    m.experts = d_.experts;
    m.identity = d_.identity;
    m.top = d_.top;
    m.groups = d_.groups;
    m.keep = d_.keep;
    m.w_dtype = w_dtype_;
    m.act = d_.act;
    m.exact = exact_ ? 1u : 0u;
    m.scale = d_.router_scale;
    if ((rc = m40llm_moe_async(ctx, &m, 1u)) != 0) return fail(rc, "experts");
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
