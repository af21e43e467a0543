#include "mokisun.h"

#include <cmath>

#include "config_keys.h"

namespace liyab {
namespace {

MokisunConfig::Attention attention_from(const Json& m, const std::string& mw) {
    MokisunConfig::Attention a;
    a.heads = int_in(m, "heads", mw, 1, 65535);
    a.kv_heads = m.contains("kv_heads") ? int_in(m, "kv_heads", mw, 1, a.heads) : a.heads;
    if (a.heads % a.kv_heads != 0) throw invalid_model("invalid {}kv_heads in config.json: {} heads do not split over {}", mw, a.heads, a.kv_heads);
    a.dim = int_in(m, "dim", mw, 1);
    a.vdim = m.contains("vdim") ? int_in(m, "vdim", mw, 1) : a.dim;
    a.scale = m.contains("scale") ? number_in(m, "scale", mw) : 1.0 / std::sqrt(static_cast<double>(a.dim));
    if (const Json* mask = optional_in(m, "mask")) a.window = int_in(*mask, "size", mw + "mask.", 1);
    if (const Json* r = optional_in(m, "rot")) {
        a.rot_dims = int_in(*r, "dims", mw + "rot.", 0, a.dim);
        if (a.rot_dims % 2 != 0) throw invalid_model("invalid {}rot.dims in config.json: {} values cannot be rotated in pairs", mw, a.rot_dims);
        a.rot_base = number_in(*r, "base", mw + "rot.");
        if (!(a.rot_base > 0)) throw invalid_model("invalid {}rot.base in config.json (need a positive number)", mw);
    }
    return a;
}

MokisunConfig::Memory memory_from(const Json& m, const std::string& mw) {
    MokisunConfig::Memory c;
    c.heads = int_in(m, "heads", mw, 1, 65535);
    c.kv_heads = m.contains("kv_heads") ? int_in(m, "kv_heads", mw, 1, c.heads) : c.heads;
    if (c.heads % c.kv_heads != 0) throw invalid_model("invalid {}kv_heads in config.json: {} heads do not split over {}", mw, c.heads, c.kv_heads);
    c.dim = int_in(m, "dim", mw, 1);
    c.vdim = m.contains("vdim") ? int_in(m, "vdim", mw, 1) : c.dim;
    if (m.contains("a_rank")) c.a_rank = int_in(m, "a_rank", mw, 1);
    if (m.contains("g_rank")) c.g_rank = int_in(m, "g_rank", mw, 1);
    return c;
}

}  // namespace

std::unique_ptr<MokisunConfig> MokisunConfig::parse(const Json& raw) {
    auto c = std::make_unique<MokisunConfig>();
    c->raw = raw;
    c->vocab = int_in(raw, "vocab", "", 1);
    c->width = int_in(raw, "width", "", 1);
    c->streams = int_in(raw, "streams", "", 1, 16);
    c->norm_eps = number_in(object_in(raw, "norm", ""), "eps", "norm.");
    if (c->norm_eps < 0) throw invalid_model("invalid norm.eps {} in config.json", c->norm_eps);
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
        if (type == "attention") {
            l.mixer = Mixer::Attention;
            l.attention = attention_from(m, mw);
        } else if (type == "gla") {
            l.mixer = Mixer::Gla;
            l.memory = memory_from(m, mw);
            if (l.memory.kv_heads != l.memory.heads) throw invalid_model("invalid {}kv_heads in config.json: every head has queries and keys of its own", mw);
            l.memory.tau = number_in(m, "tau", mw);
            if (!(l.memory.tau > 0)) throw invalid_model("invalid {}tau in config.json (need a positive number)", mw);
        } else if (type == "parallel") {
            l.mixer = Mixer::Parallel;
            l.attention = attention_from(object_in(m, "left", mw), mw + "left.");
            if (l.attention.vdim != l.attention.dim)
                throw invalid_model("invalid {}left.vdim in config.json: the values are the keys, {} values a head, not {}", mw, l.attention.dim, l.attention.vdim);
            if (l.attention.rot_dims != 0) throw invalid_model("invalid {}left.rot in config.json: this side rotates nothing", mw);
            const Json& r = object_in(m, "right", mw);
            l.memory = memory_from(r, mw + "right.");
            l.memory.taps = int_in(r, "conv", mw + "right.", 1, 64);
            l.left_scale = m.contains("left_scale") ? number_in(m, "left_scale", mw) : 1.0;
            l.right_scale = m.contains("right_scale") ? number_in(m, "right_scale", mw) : 1.0;
        } else {
            throw unsupported("{}type '{}' is not supported; supported: attention, gla, parallel", where, type);
        }
        if (const Json* mlp = optional_in(lj, "mlp")) {
            const std::string kind = mlp->get_string("kind", ""), fw = where + "mlp.", rw = fw + "router.";
            if (kind != "moe") throw unsupported("{}kind '{}' is not supported; supported: moe", fw, kind);
            const Json& router = object_in(*mlp, "router", fw);
            l.experts = int_in(router, "experts", rw, 1, 4096);
            l.identity = router.contains("identity") ? int_in(router, "identity", rw, 0, 4096 - l.experts) : 0;
            l.top = int_in(router, "top", rw, 1, l.experts + l.identity);
            l.route_scale = router.contains("scale") ? number_in(router, "scale", rw) : 1.0;
            if (const Json* g = optional_in(router, "groups")) {
                l.groups = int_in(*g, "count", rw + "groups.", 1, l.experts + l.identity);
                l.keep = int_in(*g, "keep", rw + "groups.", 1, l.groups);
            }
            if ((l.experts + l.identity) % l.groups != 0)
                throw invalid_model("invalid {}groups.count in config.json: {} experts and {} identities do not form {} equal groups", rw, l.experts, l.identity, l.groups);
            if (l.top > (l.experts + l.identity) / l.groups * l.keep)
                throw invalid_model("invalid {}top in config.json: {} groups of {} hold fewer than {}", rw, l.keep, (l.experts + l.identity) / l.groups, l.top);
            l.expert_ff = int_in(object_in(*mlp, "expert", fw), "ff", fw + "expert.", 1);
        }
        c->layers.push_back(std::move(l));
    }
    return c;
}

// Only the file's tensors tell the ranks of the low-rank maps.
void MokisunConfig::read_shapes(const ShapeOf& shape_of) {
    auto rows_of = [&](const std::string& name, int64_t* rank) {
        const std::vector<int64_t>* s = shape_of(name);
        if (s != nullptr && s->size() == 2 && (*s)[0] > 0) *rank = (*s)[0];
    };
    for (size_t i = 0; i < layers.size(); ++i) {
        const std::string p = std::format("l{}.mix.{}", i, layers[i].mixer == Mixer::Parallel ? "right." : "");
        rows_of(p + "a1", &layers[i].memory.a_rank);
        rows_of(p + "g1", &layers[i].memory.g_rank);
    }
}

ModelSpec MokisunConfig::model_spec() const {
    ModelSpec m;
    m.architecture = "mokisun";
    m.embedding = {vocab, width, 1.0};
    m.streams = streams;
    m.position = {"none", Json::object().set("max_positions", max_positions)};
    const PartSpec norm{"dynamic_tanh", Json::object().set("size", width)};
    const PartSpec join{"hyper", Json::object().set("streams", streams).set("size", width).set("layer_scale", true)};
    auto attention = [&](const Attention& a) {
        return Json::object().set("hidden", width).set("n_head", a.heads).set("n_kv_head", a.kv_heads).set("dim", a.dim).set("vdim", a.vdim).set("scale", a.scale)
            .set("window", a.window).set("qk_norm", false).set("bias", false).set("gate", "none").set("eps", norm_eps);
    };
    auto memory = [&](const Memory& c) {
        return Json::object().set("hidden", width).set("n_head", c.heads).set("n_kv_head", c.kv_heads).set("dim", c.dim).set("vdim", c.vdim).set("rank", c.a_rank)
            .set("q_scale", 1.0 / std::sqrt(static_cast<double>(c.dim))).set("eps", norm_eps);
    };
    for (size_t i = 0; i < layers.size(); ++i) {
        const Layer& c = layers[i];
        LayerSpec l;
        l.arrangement = "streams";
        PartSpec mixer;
        if (c.mixer == Mixer::Attention) {
            mixer = {"gated_attention", attention(c.attention).set("rot_dims", c.attention.rot_dims).set("rot_base", c.attention.rot_base).set("rot_layout", "interleaved")
                                            .set("sink", true)};
        } else if (c.mixer == Mixer::Gla) {
            mixer = {"channel_memory", memory(c.memory).set("rule", "linear").set("decay", "sigmoid").set("tau", c.memory.tau).set("gate", "silu")};
        } else {
            const PartSpec left{"gated_attention", attention(c.attention).set("values", "keys").set("slopes", true).set("unit_sink", true)};
            const PartSpec right{"channel_memory", memory(c.memory).set("rule", "delta").set("decay", "softplus").set("taps", c.memory.taps).set("unit", true)
                                                       .set("unit_eps", 1e-6).set("gate", "sigmoid").set("gate_rank", c.memory.g_rank)};
            Json branches = Json::array();
            branches.push(Json::object().set("name", "left").set("part", left.to_json()).set("scale", c.left_scale));
            branches.push(Json::object().set("name", "right").set("part", right.to_json()).set("scale", c.right_scale));
            mixer = {"branch_sum", Json::object().set("size", width).set("norm", false).set("branches", branches)};
        }
        l.slots.push_back({"mixer_join", Role::Join, join});
        l.slots.push_back({"mixer_norm", Role::Norm, norm});
        l.slots.push_back({"mixer", Role::Mixer, mixer});
        if (c.routed()) {
            l.slots.push_back({"ff_join", Role::Join, join});
            l.slots.push_back({"ff_norm", Role::Norm, norm});
            l.slots.push_back({"feed_forward", Role::FeedForward,
                               {"routed", Json::object().set("hidden", width).set("experts", c.experts).set("identity", c.identity).set("top", c.top)
                                              .set("inner", c.expert_ff).set("activation", "silu").set("score", "softmax").set("renormalise", false)
                                              .set("weight_on", "output").set("correction", true).set("groups", c.groups).set("keep_groups", c.keep)
                                              .set("route_scale", c.route_scale).set("shared_inner", 0)}});
        }
        m.layers.push_back(std::move(l));
        m.run_order.push_back({static_cast<int>(i), static_cast<int>(i), -1});
    }
    m.final_norm = norm;
    m.head = {vocab, width, false, false, 1.0, 0.0};
    m.max_positions = max_positions;
    return m;
}

CheckpointMap MokisunConfig::checkpoint_map() const {
    using K = ParamKind;
    CheckpointMap m;
    auto inv_sqrt = [](int64_t n) { return 1.0 / std::sqrt(static_cast<double>(n)); };
    const double w_std = inv_sqrt(width);
    auto matrix = [&](const std::string& path, const std::string& name, int64_t rows, int64_t cols) {
        m.push_back({path, CheckpointTensor::one(name, {rows, cols}, K::Matrix, "none", 0.0, inv_sqrt(cols))});
    };
    auto vector = [&](const std::string& path, const std::string& name, std::vector<int64_t> shape, double mean, double std_dev) {
        m.push_back({path, CheckpointTensor::one(name, std::move(shape), K::Vector, "none", mean, std_dev)});
    };
    auto norm = [&](const std::string& path, const std::string& name) {
        m.push_back({path + ".alpha", CheckpointTensor::repeated(name + ".alpha", 1, K::Vector, 0.5, 0.05)});
        vector(path + ".weight", name, {width}, 1.0, 0.1);
        vector(path + ".bias", name + ".b", {width}, 0.0, 0.1);
    };
    auto join = [&](const std::string& path, const std::string& layer, int q) {
        const std::string hc = std::format("{}hc{}.", layer, q);
        vector(path + ".in", hc + "in", {streams}, 1.0 / static_cast<double>(streams), 0.1);
        vector(path + ".out", hc + "out", {streams}, 1.0, 0.2);
        vector(path + ".mix", hc + "mix", {streams, streams}, 1.0 / static_cast<double>(streams), 0.1);
        vector(path + ".scale", std::format("{}ls{}", layer, q), {width}, 0.5, 0.1);
    };
    m.push_back({"embedding.weight", CheckpointTensor::one("embed", {vocab, width}, K::Table, "none", 0.0, 1.0)});
    matrix("head.weight", "head", vocab, width);
    norm("final_norm", "final.norm");
    for (size_t i = 0; i < layers.size(); ++i) {
        const Layer& c = layers[i];
        const std::string p = std::format("layers.{}.", i), f = std::format("l{}.", i);
        join(p + "mixer_join", f, 1);
        norm(p + "mixer_norm", f + "norm1");
        auto attention = [&](const std::string& to, const std::string& from, const Attention& a, bool own_values) {
            std::vector<CheckpointSource> rows{{from + "q", {a.heads * a.dim, width}}, {from + "k", {a.kv_heads * a.dim, width}}};
            if (own_values) rows.push_back({from + "v", {a.kv_heads * a.vdim, width}});
            m.push_back({to + "proj.weight", joined(std::move(rows), K::Matrix, w_std)});
            if (own_values) vector(to + "sink", from + "sink", {a.heads}, 0.0, 1.0);
            matrix(to + "out.weight", from + "o", width, a.heads * a.vdim);
        };
        auto memory = [&](const std::string& to, const std::string& from, const Memory& a, bool delta) {
            const int64_t QD = a.kv_heads * a.dim, HD = a.heads * a.dim, HE = a.heads * a.vdim;
            std::vector<CheckpointSource> rows{{from + "q", {QD, width}}, {from + "k", {QD, width}}, {from + "v", {HE, width}}, {from + "a1", {a.a_rank, width}}};
            if (delta) {
                rows.push_back({from + "g1", {a.g_rank, width}});
                rows.push_back({from + "b", {a.heads, width}});
            } else {
                rows.push_back({from + "g", {HE, width}});
            }
            m.push_back({to + "proj.weight", joined(std::move(rows), K::Matrix, w_std)});
            matrix(to + "decay.weight", from + "a2", HD, a.a_rank);
            if (delta) {
                vector(to + "decay.bias", from + "dt_bias", {HD}, -2.0, 1.0);
                vector(to + "a_log", from + "A_log", {a.heads}, -1.0, 1.0);
                matrix(to + "gate.weight", from + "g2", HE, a.g_rank);
                m.push_back({to + "conv.weight", joined({{from + "q.conv", {QD, a.taps}}, {from + "k.conv", {QD, a.taps}}, {from + "v.conv", {HE, a.taps}}}, K::Vector,
                                                        inv_sqrt(a.taps))});
            } else {
                vector(to + "decay.bias", from + "a2.b", {HD}, 2.0, 1.0);
            }
            vector(to + "norm.weight", from + "norm", {a.vdim}, 1.0, 0.1);
            matrix(to + "out.weight", from + "o", width, HE);
        };
        if (c.mixer == Mixer::Attention) {
            attention(p + "mixer.", f + "mix.", c.attention, true);
        } else if (c.mixer == Mixer::Gla) {
            memory(p + "mixer.", f + "mix.", c.memory, false);
        } else {
            attention(p + "mixer.left.", f + "mix.left.", c.attention, false);
            memory(p + "mixer.right.", f + "mix.right.", c.memory, true);
        }
        if (!c.routed()) continue;
        join(p + "ff_join", f, 2);
        norm(p + "ff_norm", f + "norm2");
        matrix(p + "feed_forward.router.weight", f + "mlp.router", c.experts + c.identity, width);
        vector(p + "feed_forward.router.correction", f + "mlp.correction", {c.experts + c.identity}, 0.0, 0.05);
        std::vector<CheckpointSource> gate_up, down;
        for (int64_t e = 0; e < c.experts; ++e) {
            const std::string ef = std::format("{}mlp.e{}.", f, e);
            gate_up.push_back({ef + "gate", {c.expert_ff, width}});
            gate_up.push_back({ef + "up", {c.expert_ff, width}});
            down.push_back({ef + "down", {width, c.expert_ff}});
        }
        m.push_back({p + "feed_forward.experts.gate_up.weight", joined(std::move(gate_up), K::Matrix, w_std)});
        m.push_back({p + "feed_forward.experts.down.weight", joined(std::move(down), K::Matrix, inv_sqrt(c.expert_ff))});
    }
    return m;
}

// A block without a feed-forward may still carry that sublayer's norm, scale and connections.
std::vector<std::string> MokisunConfig::ignored_tensors() const {
    std::vector<std::string> out;
    for (size_t i = 0; i < layers.size(); ++i)
        if (!layers[i].routed()) out.push_back(std::format("l{}\\.(norm2(\\.b|\\.alpha)?|ls2|hc2\\.(in|out|mix))", i));
    return out;
}

void register_mokisun() {
    register_architecture({"mokisun", {"Mokisun", "MokisunForCausalLM"}, [](const Json& raw) -> std::unique_ptr<ArchitectureConfig> {
                               return MokisunConfig::parse(raw);
                           }});
}

}  // namespace liyab
