// Mokisun: a decoder over several residual streams.  The streams start as the embedded row; every sublayer reads a weighted sum of them
// through a norm without statistics (tanh of the scaled value, gain, offset) and its output, scaled value by value, joins all streams while a
// matrix mixes them; at the end the streams are summed.  A layer's mixer is one of three: softmax attention under a sliding window (grouped
// key/value heads, pairs of neighbouring values rotated in part of a head, a sink a head in the softmax's divisor); gated linear attention (a
// matrix memory per head with a decay per key channel); or two mixers side by side on the same input, attention whose values are its keys
// (a slope a head off the scores, one added to the divisor, a window) and a gated delta rule (short convolutions, unit queries and keys, a
// decay per head and key channel).  The feed-forward is a set of small gated experts, some of which pass the input on as it is, chosen by
// corrected softmax scores inside the best groups; or absent.  No position table; the head is a matrix of its own.
//
// config.json: {"architecture": "Mokisun", "vocab", "width", "streams", "norm": {"eps"}, "layers": [
//   {"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}, "rot": {"base", "dims"}}} |
//   {"type": "gla", "mixer": {"heads", "dim", "vdim", "tau"}} |
//   {"type": "parallel", "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}}, "left_scale",
//                                  "right": {"heads", "kv_heads", "dim", "vdim", "conv"}, "right_scale"}},
//   each with "mlp": {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "identity", "scale", "groups": {"count", "keep"}}} | null]}.
// The ranks of the low-rank maps are the file's tensors' shapes; where there is no file yet they may be given as "a_rank" and "g_rank" of a mixer.
// Tensors: embed, head, final.norm(.b, .alpha), and per layer l<i>.norm1, norm2 (.b, .alpha), ls1, ls2, hc1.*, hc2.*, mix.*, mlp.*.
#pragma once

#include "arch.h"

namespace liyab {

struct MokisunConfig final : public ArchitectureConfig {
    enum class Mixer { Attention, Gla, Parallel };
    struct Attention {
        int64_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, window = 0, rot_dims = 0;
        double scale = 1.0, rot_base = 10000.0;
    };
    struct Memory {
        int64_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, a_rank = 16, g_rank = 16, taps = 0;
        double tau = 1.0;
    };
    struct Layer {
        Mixer mixer = Mixer::Attention;
        Attention attention;         // attention, and the left side of a pair
        Memory memory;               // gated linear attention, and the right side of a pair
        double left_scale = 1.0, right_scale = 1.0;
        // feed-forward: experts + identity > 0, or none
        int64_t experts = 0, identity = 0, top = 0, groups = 1, keep = 1, expert_ff = 0;
        double route_scale = 1.0;
        bool routed() const { return experts > 0; }
    };
    int64_t vocab = 0, width = 0, streams = 1;
    double norm_eps = 1e-6;
    int64_t max_positions = int64_t{1} << 17;        // the design has no limit of its own; the engine's tables need one
    std::vector<Layer> layers;
    Json raw;

    static std::unique_ptr<MokisunConfig> parse(const Json& raw);
    Json to_json() const override { return raw; }
    ModelSpec model_spec() const override;
    CheckpointMap checkpoint_map() const override;
    std::vector<std::string> ignored_tensors() const override;
    void read_shapes(const ShapeOf& shape_of) override;
};

}  // namespace liyab
