// Parts for designs with several residual streams and memories with a decay per channel: the norm without statistics
// (`dynamic_tanh`), the way a sublayer reads and joins the streams (`hyper`, hyper-connections with a layer scale), the
// arrangement around them (`streams`), and the mixer `channel_memory` (gated linear attention, or the gated delta rule with
// short convolutions).  Every size and constant is an option of the part's spec; none knows the model it is in.
#pragma once

#include "gated_parts.h"

namespace liyab::builtin {

// ---- a norm without statistics: y = tanh(alpha x) * weight + bias, alpha one number -------------------------------

class TanhNorm final : public Norm {
public:
    TanhNorm(const PartSpec& s, const Params& p) : size(need_int(s, "size")) {
        recipe_.alpha = f32_or_null(&p.at("alpha"));
        recipe_.gain = f32_or_null(&p.at("weight"));
        recipe_.offset = f32_or_null(&p.at("bias"));
    }
    static std::vector<ParamDecl> parameters(const PartSpec& s) {
        const int64_t size = need_int(s, "size");
        return {{"alpha", {1}, ParamKind::Vector}, {"weight", {size}, ParamKind::Vector}, {"bias", {size}, ParamKind::Vector}};
    }
    bool capturable() const override { return true; }
    void forward(StepContext& ctx, const Rows& x, const Rows& out, int n_rows, const int32_t* rows) override {
        kernels::streams_read(ctx.stream(), out.dtype, x, 1, rows, n_rows, recipe_, out);
    }
    std::optional<StreamReader> tanh_recipe() const override { return recipe_; }
    int64_t size;

private:
    StreamReader recipe_;
};

// ---- hyper-connections: how a sublayer reads the streams and joins them ----------------------------------------------
// Options: streams, size, layer_scale (a learned factor for every value of the sublayer's output).

class HyperJoin final : public Join {
public:
    HyperJoin(const PartSpec& s, const Params& p) : n(static_cast<int>(need_int(s, "streams"))) {
        in_ = f32_or_null(&p.at("in"));
        out_ = f32_or_null(&p.at("out"));
        mix_ = f32_or_null(&p.at("mix"));
        if (s.options.get_bool("layer_scale", false)) scale_ = f32_or_null(&p.at("scale"));
    }
    static std::vector<ParamDecl> parameters(const PartSpec& s) {
        const int64_t n = need_int(s, "streams");
        std::vector<ParamDecl> out{{"in", {n}, ParamKind::Vector}, {"out", {n}, ParamKind::Vector}, {"mix", {n, n}, ParamKind::Vector}};
        if (s.options.get_bool("layer_scale", false)) out.push_back({"scale", {need_int(s, "size")}, ParamKind::Vector});
        return out;
    }
    bool capturable() const override { return true; }
    int streams() const override { return n; }
    const float* in() const override { return in_; }
    const float* out() const override { return out_; }
    const float* mix() const override { return mix_; }
    const float* scale() const override { return scale_; }
    int n;

private:
    const float* in_ = nullptr;
    const float* out_ = nullptr;
    const float* mix_ = nullptr;
    const float* scale_ = nullptr;
};

// ---- the arrangement over several streams ----------------------------------------------------------------------------
// For each sublayer: u = sum_s in[s] x_s; y = sublayer(norm(u)); x_t <- sum_s mix[s, t] x_s + out[t] scale y.  Slots: mixer_join (join), mixer_norm
// (norm), mixer, and, unless the block has no feed-forward, ff_join, ff_norm and feed_forward.  The streams lie one after the other in a row of x
// (float32).  Between two sublayers there is one launch: it adds up the sublayer's output from its terms, moves the streams and, where the
// next norm acts on every value by itself, makes the next sublayer's input (also the next block's), and routes its rows where that
// sublayer is a set of routed experts.

class StreamsBlock final : public Arrangement {
public:
    StreamsBlock(const LayerSpec& spec, const LayerParts& parts)
        : mixer_join(parts.get<Join>("mixer_join")), mixer_norm(parts.get<Norm>("mixer_norm")), mixer(parts.get<Mixer>("mixer")), keep_(parts) {
        const bool with_ff = spec.find("feed_forward") != nullptr;
        if (with_ff) {
            ff_join = &parts.get<Join>("ff_join");
            ff_norm = &parts.get<Norm>("ff_norm");
            feed_forward = &parts.get<FeedForward>("feed_forward");
            if (ff_join->streams() != mixer_join.streams()) throw invalid_model("arrangement 'streams': a block's sublayers work on equally many streams");
        }
        if (spec.slots.size() != (with_ff ? 6u : 3u))
            throw invalid_model("arrangement 'streams' takes the slots mixer_join, mixer_norm and mixer, and ff_join and ff_norm with feed_forward, only");
    }
    bool capturable() const override {
        return mixer_norm.capturable() && mixer.capturable() && (feed_forward == nullptr || (ff_norm->capturable() && feed_forward->capturable()));
    }
    std::vector<Mixer*> mixers() const override { return {&mixer}; }
    int streams() const override { return mixer_join.streams(); }
    std::optional<StreamReader> reader() const override { return reader_of(mixer_join, mixer_norm); }
    void forward(StepContext& ctx, const Rows& x, CacheUnit unit) override {
        const int T = ctx.n_tokens;
        const int64_t width = x.cols / streams();
        const DType dt = ctx.runtime.dtype;
        cudaStream_t s = ctx.stream();
        const Rows h = ctx.workspace->get("block.normed", T, width, dt), y = ctx.workspace->get("block.sublayer", T, width, DType::F32);
        ctx.phase(Phase::Mixer);
        if (ctx.next_input_entry != unit.entry || ctx.next_input.data != h.data) make_input(ctx, x, mixer_join, mixer_norm, h);
        ctx.tap("mixer_norm", h);
        OutputTerms terms = mixer.forward_terms(ctx, h, y, unit);
        show_terms(ctx, "mixer.out", terms, width);
        if (feed_forward != nullptr) {
            const std::optional<StreamReader> next = reader_of(*ff_join, *ff_norm);
            const std::optional<RowRouter> router = next ? feed_forward->row_router(ctx) : std::nullopt;
            kernels::streams_join(s, dt, x, mixer_join, terms, T, next ? &*next : nullptr, next ? &h : nullptr, router ? &*router : nullptr);
            ctx.tap("mixer", x);
            ctx.phase(Phase::FeedForward);
            if (!next) make_input(ctx, x, *ff_join, *ff_norm, h);
            ctx.tap("ff_norm", h);
            terms = feed_forward->forward_terms(ctx, h, y, router.has_value());
            show_terms(ctx, "feed_forward.out", terms, width);
        }
        // The last launch of the block makes the next block's input as well.
        kernels::streams_join(s, dt, x, feed_forward != nullptr ? *ff_join : mixer_join, terms, T, ctx.next_reader, ctx.next_reader != nullptr ? &h : nullptr, nullptr);
        ctx.next_input = h;
        ctx.next_input_entry = ctx.next_reader != nullptr ? unit.entry + 1 : -1;
        ctx.tap(feed_forward != nullptr ? "feed_forward" : "mixer", x);
    }
    Join& mixer_join;
    Norm& mixer_norm;
    Mixer& mixer;
    Join* ff_join = nullptr;
    Norm* ff_norm = nullptr;
    FeedForward* feed_forward = nullptr;

private:
    static std::optional<StreamReader> reader_of(const Join& j, const Norm& n) {
        std::optional<StreamReader> r = n.tanh_recipe();
        if (r) r->in = j.in();
        return r;
    }
    // A sublayer's input in launches of its own: one, or two where the norm needs the whole row.
    static void make_input(StepContext& ctx, const Rows& x, const Join& j, Norm& n, const Rows& h) {
        if (const auto r = reader_of(j, n)) {
            kernels::streams_read(ctx.stream(), h.dtype, x, j.streams(), nullptr, ctx.n_tokens, *r, h);
            return;
        }
        const Rows u = ctx.workspace->get("block.read", ctx.n_tokens, h.cols, DType::F32);
        StreamReader plain;
        plain.in = j.in();
        kernels::streams_read(ctx.stream(), DType::F32, x, j.streams(), nullptr, ctx.n_tokens, plain, u);
        n.forward(ctx, u, h, ctx.n_tokens, nullptr);
    }
    LayerParts keep_;
};

// ---- a matrix memory per head with a decay per key channel -----------------------------------------------------------
// S_t = diag(a_t) S_{t-1} + k_t u_t^T, o_t = S_t^T q_t per head (32-bit, carried in the request's state slot, zero at a sequence's start).
// `rule` "linear": u_t = v_t; "delta": u_t = beta_t (v_t - (diag(a_t) S_{t-1})^T k_t), beta = sigmoid of one more number a head of the projection.
// The decays come through a map of low rank (`rank`): z = W_a2 (W_a1 h) + bias (`decay_bias`); `decay` "sigmoid": a = sigmoid(z)^(1 / tau); "softplus":
// a = exp(-exp(a_log[head]) softplus(z)).  `taps` > 0: queries, keys and values pass a causal convolution per channel over so many inputs and SiLU.
// `unit`: queries and keys over sqrt(sum of squares + unit_eps), per head.  `q_scale` on the queries.  n_head / n_kv_head heads in a row read one query
// and key row.  Every head's o over its root mean square, times the gain `norm.weight` [vdim], times `gate` (silu, sigmoid) of W_g h, or, with
// `gate_rank` > 0, of W_g2 (W_g1 h); then the output projection.
// One projection makes [q | k | v | W_a1 h | W_g h or W_g1 h | beta's] in 32-bit.  Steps of single tokens and short portions go from there to the
// gated heads in one launch.

class ChannelMemory final : public Mixer {
public:
    ChannelMemory(const PartSpec& s, const Params& p) {
        hidden = need_int(s, "hidden");
        m.n_head = static_cast<int>(need_int(s, "n_head"));
        m.kv_head = static_cast<int>(s.options.get_int("n_kv_head", m.n_head));
        m.dim = static_cast<int>(need_int(s, "dim"));
        m.vdim = static_cast<int>(need_int(s, "vdim"));
        if (m.kv_head < 1 || m.n_head % m.kv_head != 0) throw invalid_model("channel_memory: {} heads do not share {} query and key heads", m.n_head, m.kv_head);
        if (m.dim > 256 || m.vdim > 256) throw unsupported("channel_memory: heads of {} and {} values are more than the kernels take (256)", m.dim, m.vdim);
        const std::string rule = s.options.get_string("rule", "linear");
        if (rule != "linear" && rule != "delta") throw unsupported("channel_memory: rule '{}' is not supported; supported: linear, delta", rule);
        m.delta = rule == "delta";
        m.rank = static_cast<int>(need_int(s, "rank"));
        m.gate_rank = static_cast<int>(s.options.get_int("gate_rank", 0));
        m.taps = static_cast<int>(s.options.get_int("taps", 0));
        if (m.taps < 0 || m.taps > 64) throw invalid_model("channel_memory: a convolution over {} inputs is outside [0, 64]", m.taps);
        m.unit = s.options.get_bool("unit", false);
        m.unit_eps = static_cast<float>(s.options.get_number("unit_eps", 1e-6));
        m.q_scale = static_cast<float>(s.options.get_number("q_scale", 1.0));
        m.eps = static_cast<float>(s.options.get_number("eps", 1e-6));
        m.gate = kernels::gate_from_name(s.options.get_string("gate", "silu"));
        if (m.gate != kernels::kSilu && m.gate != kernels::kSigmoid) throw unsupported("channel_memory: the gate is silu or sigmoid");
        const std::string decay = decay_of(s);
        if (decay == "softplus") {
            m.a_log = f32_or_null(&p.at("a_log"));
        } else {
            m.tau = static_cast<float>(s.options.get_number("tau", 1.0));
            if (!(m.tau > 0.0f)) throw invalid_model("channel_memory: tau {} is not positive", m.tau);
        }
        proj = Linear(p, "proj.", "channel_memory.proj");
        out = Linear(p, "out.", "channel_memory.out");
        m.a2 = p.at("decay.weight");
        if (s.options.get_bool("decay_bias", true)) m.z_bias = f32_or_null(&p.at("decay.bias"));
        if (m.gate_rank > 0) m.g2 = p.at("gate.weight");
        if (m.taps > 0) m.conv = f32_or_null(&p.at("conv.weight"));
        m.norm = f32_or_null(&p.at("norm.weight"));
    }
    static std::string decay_of(const PartSpec& s) {
        const std::string decay = s.options.get_string("decay", "sigmoid");
        if (decay != "sigmoid" && decay != "softplus") throw unsupported("channel_memory: decay '{}' is not supported; supported: sigmoid, softplus", decay);
        return decay;
    }
    static std::vector<ParamDecl> parameters(const PartSpec& s) {
        const int64_t hidden = need_int(s, "hidden"), H = need_int(s, "n_head"), G = s.options.get_int("n_kv_head", H), D = need_int(s, "dim"), E = need_int(s, "vdim");
        const int64_t rank = need_int(s, "rank"), gate_rank = s.options.get_int("gate_rank", 0), taps = s.options.get_int("taps", 0);
        const bool delta = s.options.get_string("rule", "linear") == "delta";
        std::vector<ParamDecl> out;
        Linear::declare(out, "proj.", 2 * G * D + H * E + rank + (gate_rank > 0 ? gate_rank : H * E) + (delta ? H : 0), hidden, false);
        out.push_back({"decay.weight", {H * D, rank}, ParamKind::Matrix});
        if (s.options.get_bool("decay_bias", true)) out.push_back({"decay.bias", {H * D}, ParamKind::Vector});
        if (decay_of(s) == "softplus") out.push_back({"a_log", {H}, ParamKind::Vector});
        if (gate_rank > 0) out.push_back({"gate.weight", {H * E, gate_rank}, ParamKind::Matrix});
        if (taps > 0) out.push_back({"conv.weight", {2 * G * D + H * E, taps}, ParamKind::Vector});
        out.push_back({"norm.weight", {E}, ParamKind::Vector});
        Linear::declare(out, "out.", hidden, H * E, false);
        return out;
    }
    bool capturable() const override { return true; }
    std::optional<StateNeed> state_need() const override { return StateNeed{{m.slot_floats()}, DType::F32}; }
    void forward(StepContext& ctx, const Rows& h, const Rows& x, CacheUnit unit) override { run(ctx, h, x, &x, unit); }
    void forward_into(StepContext& ctx, const Rows& h, const Rows& y, CacheUnit unit) override { run(ctx, h, y, nullptr, unit); }

    // Steps whose longest portion has this many rows or more work in pieces.
    static constexpr int kPiecesFrom = 16;
    kernels::ChannelMemoryShape m;
    int64_t hidden = 0;
    Linear proj, out;

private:
    void run(StepContext& ctx, const Rows& h, const Rows& y, const Rows* residual, CacheUnit unit) {
        if (!unit.write) throw invalid_model("channel_memory: a memory is carried by the run that owns it; the run order lets another read it");
        const int T = ctx.n_tokens;
        const int64_t HE = static_cast<int64_t>(m.n_head) * m.vdim;
        Workspace& ws = *ctx.workspace;
        cudaStream_t s = ctx.stream();
        // Rows on 16-byte borders whatever the number of columns, so that the product may store them in large pieces.
        const Rows pr = ws.get("channel_memory.proj", T, (m.cols() + 7) / 8 * 8, DType::F32).columns(0, m.cols());
        kernels::linear(ctx.runtime, &ws, h, proj.weight, nullptr, pr, T, kernels::kNone, nullptr);
        const Rows heads = ws.get("channel_memory.heads", T, HE, ctx.runtime.dtype);
        Rows o;
        if (ctx.tap_fn != nullptr) o = ws.get("channel_memory.o", T, HE, DType::F32);
        const kernels::ChannelStep step{ctx.positions, ctx.tok_seq, ctx.q_start, ctx.state_slots, static_cast<float*>(ctx.state(unit.read)), T, ctx.n_seq, ctx.decode_only};
        if (ctx.max_q_len >= kPiecesFrom) kernels::channel_memory_pieces(s, &ws, m, step, pr, o, heads);
        else kernels::channel_memory_rows(s, m, step, pr, o, heads);
        if (ctx.tap_fn != nullptr) ctx.tap("memory", o);
        ctx.tap("memory.heads", heads);
        kernels::linear(ctx.runtime, &ws, heads, out.weight, nullptr, y, T, kernels::kNone, residual);
    }
};

}  // namespace liyab::builtin
