#include "gekitar.h"

#include <cmath>

#include "config_keys.h"

namespace liyab {
namespace {

void read_rotation(const Json& m, const std::string& mw, int64_t most, bool may_stretch, GekitarConfig::Layer* l) {
    const Json* r = optional_in(m, "rot");
    if (r == nullptr) return;
    const std::string rw = mw + "rot.";
    l->rot_dims = int_in(*r, "dims", rw, 0, most);
    if (l->rot_dims % 2 != 0) throw invalid_model("invalid {}dims in config.json: {} values cannot be rotated in pairs", rw, l->rot_dims);
    l->rot_base = number_in(*r, "base", rw);
    if (!(l->rot_base > 0)) throw invalid_model("invalid {}base in config.json (need a positive number)", rw);
    const Json* s = optional_in(*r, "scaling");
    if (s == nullptr) return;
    if (!may_stretch) throw unsupported("{}scaling is not supported on a layer of this type", rw);
    l->rot_scaled = true;
    for (const auto& [key, value] : std::initializer_list<std::pair<const char*, double*>>{
             {"factor", &l->factor}, {"original", &l->original}, {"fast", &l->fast}, {"slow", &l->slow}}) {
        *value = number_in(*s, key, rw + "scaling.");
        if (!(*value > 0)) throw invalid_model("invalid {}scaling.{} in config.json (need a positive number)", rw, key);
    }
    if (l->rot_base == 1.0) throw invalid_model("invalid {}base in config.json: a stretched rotation needs a base other than 1", rw);
}

}  // namespace

std::unique_ptr<GekitarConfig> GekitarConfig::parse(const Json& raw) {
    auto c = std::make_unique<GekitarConfig>();
    c->raw = raw;
    c->vocab = int_in(raw, "vocab", "", 1);
    c->width = int_in(raw, "width", "", 1);
    c->norm_eps = number_in(object_in(raw, "norm", ""), "eps", "norm.");
    if (c->norm_eps < 0) throw invalid_model("invalid norm.eps {} in config.json", c->norm_eps);
    if (const Json* e = optional_in(raw, "embedding")) c->embedding_scale = number_in(*e, "scale", "embedding.");
    if (optional_in(raw, "max_positions") != nullptr) c->max_positions = int_in(raw, "max_positions", "", 1);
    const Json* layers = raw.find("layers");
    if (layers == nullptr || !layers->is_array() || layers->size() == 0) throw invalid_model("missing or invalid layers in config.json (need a list of layers)");
    for (size_t i = 0; i < layers->size(); ++i) {
        const Json& lj = (*layers)[i];
        const std::string where = std::format("layers[{}].", i);
        if (!lj.is_object()) throw invalid_model("invalid {} in config.json (need an object)", where);
        Layer l;
        const std::string type = lj.get_string("type", "");
        const Json& m = object_in(lj, "mixer", where);
        const std::string mw = where + "mixer.";
        l.heads = int_in(m, "heads", mw, 1, 65535);
        l.dim = int_in(m, "dim", mw, 1);
        l.vdim = m.contains("vdim") ? int_in(m, "vdim", mw, 1) : l.dim;
        if (const Json* mask = optional_in(m, "mask")) l.window = int_in(*mask, "size", mw + "mask.", 1);
        if (type == "attention") {
            l.mixer = Mixer::Attention;
            l.kv_heads = m.contains("kv_heads") ? int_in(m, "kv_heads", mw, 1, l.heads) : l.heads;
            if (l.heads % l.kv_heads != 0) throw invalid_model("invalid {}kv_heads in config.json: {} heads do not split over {}", mw, l.heads, l.kv_heads);
            l.scale = m.contains("scale") ? number_in(m, "scale", mw) : 1.0 / std::sqrt(static_cast<double>(l.dim));
            if (optional_in(m, "softcap") != nullptr) {
                l.soft_cap = number_in(m, "softcap", mw);
                if (!(l.soft_cap > 0)) throw invalid_model("invalid {}softcap in config.json (need a positive number)", mw);
            }
            read_rotation(m, mw, l.dim, true, &l);
        } else if (type == "latent_attention" || type == "latent_attention_2") {
            l.mixer = Mixer::Latent;
            l.gated = type == "latent_attention";
            l.rot_dim = int_in(m, "rot_dim", mw, 0);
            l.kv_rank = int_in(m, "kv_rank", mw, 1);
            l.q_rank = int_in(m, "q_rank", mw, 1);
            l.scale = m.contains("scale") ? number_in(m, "scale", mw) : 1.0 / std::sqrt(static_cast<double>(l.dim + l.rot_dim));
            l.rot_dims = l.rot_dim - l.rot_dim % 2;          // the whole rotated part unless `rot.dims` says less
            read_rotation(m, mw, l.rot_dim, false, &l);
            if (optional_in(m, "kv_from") != nullptr) {
                l.kv_from = int_in(m, "kv_from", mw, 0);
                if (l.kv_from >= static_cast<int64_t>(i)) throw invalid_model("invalid {}kv_from in config.json: layer {} does not come before this one", mw, l.kv_from);
                const Layer& from = c->layers[static_cast<size_t>(l.kv_from)];
                if (from.mixer != Mixer::Latent || from.kv_from >= 0 || from.kv_rank != l.kv_rank || from.rot_dim != l.rot_dim || from.rot_dims != l.rot_dims ||
                    from.rot_base != l.rot_base)
                    throw invalid_model("invalid {}kv_from in config.json: layer {} makes no latent rows of this layer's shape and rotation", mw, l.kv_from);
            }
        } else {
            throw unsupported("{}type '{}' is not supported; supported: attention, latent_attention, latent_attention_2", where, type);
        }
        if (const Json* mlp = optional_in(lj, "mlp")) {
            const std::string kind = mlp->get_string("kind", ""), fw = where + "mlp.";
            if (kind == "dense") {
                l.ff = int_in(*mlp, "ff", fw, 1);
                l.limit = number_in(*mlp, "limit", fw);
            } else if (kind == "moe") {
                const Json& router = object_in(*mlp, "router", fw);
                l.experts = int_in(router, "experts", fw + "router.", 1, 4096);
                l.top = int_in(router, "top", fw + "router.", 1, l.experts);
                l.expert_ff = int_in(object_in(*mlp, "expert", fw), "ff", fw + "expert.", 1);
                if (const Json* s = optional_in(*mlp, "shared")) l.shared_ff = int_in(*s, "ff", fw + "shared.", 1);
            } else {
                throw unsupported("{}kind '{}' is not supported; supported: dense, moe", fw, kind);
            }
        }
        c->layers.push_back(std::move(l));
    }
    return c;
}

ModelSpec GekitarConfig::model_spec() const {
    ModelSpec m;
    m.architecture = "gekitar";
    m.embedding = {vocab, width, embedding_scale};
    m.position = {"none", Json::object().set("max_positions", max_positions)};
    const PartSpec norm{"rms_norm", Json::object().set("size", width).set("groups", 1).set("eps", norm_eps).set("gain_offset", 1.0)};
    for (size_t i = 0; i < layers.size(); ++i) {
        const Layer& c = layers[i];
        LayerSpec l;
        l.arrangement = "sandwich_norm";
        PartSpec mixer;
        if (c.mixer == Mixer::Attention) {
            mixer = {"gated_attention", Json::object().set("hidden", width).set("n_head", c.heads).set("n_kv_head", c.kv_heads).set("dim", c.dim).set("vdim", c.vdim)
                                            .set("scale", c.scale).set("window", c.window).set("bias", true).set("out_bias", true).set("gate", "none")
                                            .set("eps", norm_eps).set("qk_norm", true).set("qk_gain", false).set("qk_norm_at", "rotated")
                                            .set("rot_dims", c.rot_dims).set("rot_base", c.rot_base).set("rot_layout", "interleaved").set("soft_cap", c.soft_cap)
                                            .set("unit_sink", true)};
            if (c.rot_scaled)
                mixer.options.set("rot_scaling", Json::object().set("factor", c.factor).set("original", c.original).set("fast", c.fast).set("slow", c.slow));
        } else {
            mixer = {"latent_attention", Json::object().set("hidden", width).set("n_head", c.heads).set("dim", c.dim).set("rot_dim", c.rot_dim)
                                             .set("rot_dims", c.rot_dims).set("rot_base", c.rot_base).set("rot_layout", "interleaved").set("vdim", c.vdim)
                                             .set("kv_rank", c.kv_rank).set("q_rank", c.q_rank).set("window", c.window).set("scale", c.scale).set("eps", norm_eps)
                                             .set("own_latent", c.kv_from < 0).set("value_gate", c.gated)};
        }
        l.slots.push_back({"mixer_norm", Role::Norm, norm});
        l.slots.push_back({"mixer", Role::Mixer, mixer});
        l.slots.push_back({"mixer_out_norm", Role::Norm, norm});
        if (c.has_ff()) {
            PartSpec ff;
            if (c.ff > 0)
                ff = {"gated", Json::object().set("hidden", width).set("inner", c.ff).set("activation", "capped").set("gate_alpha", 1.702).set("gate_limit", c.limit)};
            else
                ff = {"routed", Json::object().set("hidden", width).set("experts", c.experts).set("top", c.top).set("inner", c.expert_ff).set("expert", "plain")
                                    .set("activation", "relu2").set("score", "softmax").set("renormalise", true).set("weight_on", "output")
                                    .set("shared_inner", c.shared_ff).set("shared_gate", c.shared_ff > 0)};
            l.slots.push_back({"ff_norm", Role::Norm, norm});
            l.slots.push_back({"feed_forward", Role::FeedForward, ff});
            l.slots.push_back({"ff_out_norm", Role::Norm, norm});
        }
        m.layers.push_back(std::move(l));
        m.run_order.push_back({static_cast<int>(i), static_cast<int>(c.kv_from >= 0 ? c.kv_from : static_cast<int64_t>(i)), -1});
    }
    m.final_norm = norm;
    m.head = {vocab, width, false, false, 1.0, 0.0};
    m.max_positions = max_positions;
    return m;
}

CheckpointMap GekitarConfig::checkpoint_map() const {
    using K = ParamKind;
    CheckpointMap m;
    auto inv_sqrt = [](int64_t n) { return 1.0 / std::sqrt(static_cast<double>(n)); };
    const double w_std = inv_sqrt(width);
    auto matrix = [&](const std::string& path, const std::string& name, int64_t rows, int64_t cols) {
        m.push_back({path, CheckpointTensor::one(name, {rows, cols}, K::Matrix, "none", 0.0, inv_sqrt(cols))});
    };
    auto vector = [&](const std::string& path, const std::string& name, int64_t n, double mean, double std_dev) {
        m.push_back({path, CheckpointTensor::one(name, {n}, K::Vector, "none", mean, std_dev)});
    };
    auto norm = [&](const std::string& path, const std::string& name) { vector(path + ".weight", name, width, 0.0, 0.1); };
    m.push_back({"embedding.weight", CheckpointTensor::one("embed", {vocab, width}, K::Table, "none", 0.0, 1.0)});
    matrix("head.weight", "head", vocab, width);
    norm("final_norm", "final.norm");
    for (size_t i = 0; i < layers.size(); ++i) {
        const Layer& c = layers[i];
        const std::string p = std::format("layers.{}.", i), f = std::format("l{}.", i);
        norm(p + "mixer_norm", f + "norm1");
        norm(p + "mixer_out_norm", f + "norm1b");
        const int64_t OD = c.heads * c.vdim;
        if (c.mixer == Mixer::Attention) {
            const int64_t QD = c.heads * c.dim, KD = c.kv_heads * c.dim, VD = c.kv_heads * c.vdim;
            m.push_back({p + "mixer.proj.weight", joined({{f + "mix.q", {QD, width}}, {f + "mix.k", {KD, width}}, {f + "mix.v", {VD, width}}}, K::Matrix, w_std)});
            m.push_back({p + "mixer.qkv_bias", joined({{f + "mix.q.b", {QD}}, {f + "mix.k.b", {KD}}, {f + "mix.v.b", {VD}}}, K::Vector, 0.1)});
            vector(p + "mixer.out.bias", f + "mix.o.b", width, 0.0, 0.1);
        } else {
            const bool own = c.kv_from < 0;
            std::vector<CheckpointSource> rows{{f + "mix.dq", {c.q_rank, width}}};
            if (own) rows.push_back({f + "mix.dkv", {c.kv_rank + c.rot_dim, width}});
            if (c.gated) rows.push_back({f + "mix.g", {OD, width}});
            m.push_back({p + "mixer.proj.weight", joined(std::move(rows), K::Matrix, w_std)});
            vector(p + "mixer.q_norm.weight", f + "mix.dq.norm", c.q_rank, 1.0, 0.1);
            matrix(p + "mixer.q_up.weight", f + "mix.uq", c.heads * (c.dim + c.rot_dim), c.q_rank);
            if (own) vector(p + "mixer.latent_norm.weight", f + "mix.dkv.norm", c.kv_rank, 1.0, 0.1);
            matrix(p + "mixer.uk.weight", f + "mix.uk", c.heads * c.dim, c.kv_rank);
            matrix(p + "mixer.uv.weight", f + "mix.uv", OD, c.kv_rank);
        }
        matrix(p + "mixer.out.weight", f + "mix.o", width, OD);
        if (!c.has_ff()) continue;
        norm(p + "ff_norm", f + "norm2");
        norm(p + "ff_out_norm", f + "norm2b");
        if (c.ff > 0) {
            m.push_back({p + "feed_forward.gate_up.weight", joined({{f + "mlp.gate", {c.ff, width}}, {f + "mlp.up", {c.ff, width}}}, K::Matrix, w_std)});
            matrix(p + "feed_forward.down.weight", f + "mlp.down", width, c.ff);
            continue;
        }
        // The shared expert's gate is the last row of the router's matrix.
        std::vector<CheckpointSource> router{{f + "mlp.router", {c.experts, width}}}, up, down;
        if (c.shared_ff > 0) {
            router.push_back({f + "mlp.shared.sg", {1, width}});
            matrix(p + "feed_forward.shared.up.weight", f + "mlp.shared.up", c.shared_ff, width);
            matrix(p + "feed_forward.shared.down.weight", f + "mlp.shared.down", width, c.shared_ff);
        }
        m.push_back({p + "feed_forward.router.weight", joined(std::move(router), K::Matrix, w_std)});
        for (int64_t e = 0; e < c.experts; ++e) {
            up.push_back({std::format("{}mlp.e{}.up", f, e), {c.expert_ff, width}});
            down.push_back({std::format("{}mlp.e{}.down", f, e), {width, c.expert_ff}});
        }
        m.push_back({p + "feed_forward.experts.up.weight", joined(std::move(up), K::Matrix, w_std)});
        m.push_back({p + "feed_forward.experts.down.weight", joined(std::move(down), K::Matrix, inv_sqrt(c.expert_ff))});
    }
    return m;
}

// A block without a feed-forward may still carry that sublayer's norms.
std::vector<std::string> GekitarConfig::ignored_tensors() const {
    std::vector<std::string> out;
    for (size_t i = 0; i < layers.size(); ++i)
        if (!layers[i].has_ff()) out.push_back(std::format("l{}\\.norm2b?", i));
    return out;
}

void register_gekitar() {
    register_architecture({"gekitar", {"Gekitar", "GekitarForCausalLM"}, [](const Json& raw) -> std::unique_ptr<ArchitectureConfig> {
                               return GekitarConfig::parse(raw);
                           }});
}

}  // namespace liyab
