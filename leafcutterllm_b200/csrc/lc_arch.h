// Model designs that arrive as a checkpoint directory (config.json + model.safetensors): the description that a config is
// parsed into, and the registry that finds the parser by the config's "architecture".
#pragma once
#include <string>
#include <vector>
#include "lc_common.cuh"

namespace lc {

enum class MixerKind { ChannelDelta, LatentAttention, Attention };
// Relu2: down(relu(up x)^2).  GatedSilu: down(silu(gate x) * (up x)).  Moe: a mixture of Relu2 experts (MoeSpec).
enum class FfnKind { None, Relu2, GatedSilu, Moe };
const char* mixer_name(MixerKind k);

// Rotary embedding, optionally with YaRN's interpolation of the frequencies.  Which dimensions form a pair is the mixer's:
// neighbours in LatentAttention, halves (i with i + dims / 2) in Attention.
struct RotarySpec {
    int dims = 0;
    double base = 10000.0;
    bool yarn = false;
    double factor = 1.0, original = 0.0, fast = 0.0, slow = 0.0;
    bool operator==(const RotarySpec& o) const {
        return dims == o.dims && base == o.base && yarn == o.yarn && factor == o.factor && original == o.original && fast == o.fast && slow == o.slow;
    }
};
// Angular frequency of every pair and the factor on cos and sin.
void rotary_frequencies(const RotarySpec& r, std::vector<double>* freq, double* magnitude);

// Which keys a position sees besides causality: those nearer than `size` (0: all) and the sequence's first `keep_first`.
struct MaskSpec { int size = 0, keep_first = 0; };

constexpr int kMaxRouterOutputs = 1024, kMaxChoices = 32;
// Router over `experts` feed-forwards and `identity` experts that return their input: softmax scores over all; the `top` largest
// of score + correction among the best `keep` of `groups` equal groups are chosen and weighted with their scores.
struct MoeSpec {
    int experts = 0, identity = 0, top = 0, groups = 1, keep = 1, ff = 0;
    int shared_ff = 0;  // 0: no shared expert; otherwise one that runs for every token, times a sigmoid gate
    int outputs() const { return experts + identity; }
};

struct LayerSpec {
    MixerKind mixer = MixerKind::ChannelDelta;
    int heads = 0, dim = 0, vdim = 0;
    int kv_heads = 0;                             // ChannelDelta, Attention
    int conv_taps = 0;                            // ChannelDelta
    float unit_eps = 1e-6f;                       // ChannelDelta: inside the root that makes q and k unit vectors
    int q_rank = 0, kv_rank = 0, rot_dim = 0;     // LatentAttention (q_rank 0: the tensor's shape gives it)
    float scale = 1.0f;
    RotarySpec rot;
    MaskSpec mask;                                // Attention
    int kv_from = -1;                             // Attention: the layer whose keys and values are read (-1: its own)
    FfnKind ffn = FfnKind::None;
    int ff = 0;
    MoeSpec moe;
};

// A stack of layers with norms on the sublayers' outputs, x += norm1(mixer(x)), x += norm2(ffn(x)); norm_inputs: on their
// inputs too, x += norm1b(mixer(norm1(x))), x += norm2b(ffn(norm2(x))).
struct ArchSpec {
    std::string name;
    std::vector<LayerSpec> layers;
    int width = 0, vocab = 0;
    float eps = 1e-6f;
    bool norm_inputs = false;
    float embed_scale = 1.0f;
    float logit_scale = 1.0f, logit_softcap = 0.0f;  // softcap 0: none
};

// Parses a config.json; the design is looked up by its "architecture".
int32_t arch_from_json(const char* text, size_t len, ArchSpec* out);

}  // namespace lc
