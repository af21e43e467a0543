// Gekitar: a decoder whose sublayers lie between two norms, x += norm_b(sublayer(norm_a(x))), RMS norms with gains stored around zero.  A layer's mixer
// is one of three: softmax attention with capped scores (grouped key/value heads, biases, pairs of neighbouring values rotated at frequencies that may
// be stretched over more positions, every query and key head over its root mean square after the rotation, one added to the softmax's divisor);
// attention over latent rows (queries through a latent of their own, a gate for every value of every head); or attention over latent rows under
// a sliding window, whose rows may be another layer's.  The feed-forward is dense with a capped gate, or a set of small experts without gates
// chosen by their softmax scores, beside a shared one with a gate of its own; or absent.  No position table; the head is a matrix of its own.
//
// config.json: {"architecture": "Gekitar", "vocab", "width", "norm": {"eps"}, "embedding": {"scale"}, "layers": [
//   {"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap",
//                                   "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}}} |
//   {"type": "latent_attention" | "latent_attention_2", "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot": {"base", "dims"},
//                                                                 "mask": {"size"}, "kv_from"}},
//   each with "mlp": {"kind": "dense", "ff", "limit"} | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}, "shared": {"ff"}} | null]}.
// Tensors: embed, head, final.norm, and per layer l<i>.norm1, norm1b, norm2, norm2b, mix.*, mlp.*.
#pragma once

#include "arch.h"

namespace liyab {

struct GekitarConfig final : public ArchitectureConfig {
    enum class Mixer { Attention, Latent };
    struct Layer {
        Mixer mixer = Mixer::Attention;
        int64_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, rot_dims = 0, window = 0;
        double scale = 1.0, rot_base = 10000.0, soft_cap = 0.0;
        bool rot_scaled = false;                 // a stretched rotation: the four numbers below
        double factor = 1.0, original = 0.0, fast = 0.0, slow = 0.0;
        int64_t rot_dim = 0, kv_rank = 0, q_rank = 0;
        int64_t kv_from = -1;                    // the layer whose latent rows this one reads; -1: its own
        bool gated = false;                      // a gate for every value
        // feed-forward: dense (ff > 0), routed (experts > 0) or none
        int64_t ff = 0, experts = 0, top = 0, expert_ff = 0, shared_ff = 0;
        double limit = 0.0;
        bool has_ff() const { return ff > 0 || experts > 0; }
    };
    int64_t vocab = 0, width = 0;
    double norm_eps = 1e-6, embedding_scale = 1.0;
    int64_t max_positions = int64_t{1} << 17;    // the design has no limit of its own; the engine's tables need one
    std::vector<Layer> layers;
    Json raw;

    static std::unique_ptr<GekitarConfig> parse(const Json& raw);
    Json to_json() const override { return raw; }
    ModelSpec model_spec() const override;
    CheckpointMap checkpoint_map() const override;
    std::vector<std::string> ignored_tensors() const override;
};

}  // namespace liyab
