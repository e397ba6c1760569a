// Model designs that arrive as a checkpoint directory (config.json + model.safetensors): the description that a config is
// parsed into, and the registry that finds the parser by the config's "architecture".
#pragma once
#include <string>
#include <vector>
#include "lc_common.cuh"

namespace lc {

enum class MixerKind { ChannelDelta, LatentAttention };
enum class FfnKind { None, Relu2 };  // Relu2: down(relu(up x)^2)

// Rotary embedding of interleaved pairs, optionally with YaRN's interpolation of the frequencies.
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

struct LayerSpec {
    MixerKind mixer = MixerKind::ChannelDelta;
    int heads = 0, dim = 0, vdim = 0;
    int kv_heads = 0, conv_taps = 0;              // ChannelDelta
    float unit_eps = 1e-6f;                       // ChannelDelta: inside the root that makes q and k unit vectors
    int q_rank = 0, kv_rank = 0, rot_dim = 0;     // LatentAttention (q_rank 0: the tensor's shape gives it)
    float scale = 1.0f;
    RotarySpec rot;
    FfnKind ffn = FfnKind::None;
    int ff = 0;
};

// A stack of layers whose norms sit on the sublayers' outputs: x += norm1(mixer(x)), x += norm2(ffn(x)).
struct ArchSpec {
    std::string name;
    std::vector<LayerSpec> layers;
    int width = 0, vocab = 0;
    float eps = 1e-6f;
    float logit_scale = 1.0f, logit_softcap = 0.0f;  // softcap 0: none
};

// Parses a config.json; the design is looked up by its "architecture".
int32_t arch_from_json(const char* text, size_t len, ArchSpec* out);

}  // namespace lc
