// Model designs that arrive as a checkpoint directory (config.json + model.safetensors): the description that a config is
// parsed into, and the registry that finds the parser by the config's "architecture".
#pragma once
#include <string>
#include <vector>
#include "lc_common.cuh"

namespace lc {

enum class MixerKind { ChannelDelta, LatentAttention, Attention, LinearState, GeneralDelta };
// Relu2: down(relu(up x)^2).  GatedSilu, GatedGelu: down(act(gate x) * (up x)), gelu in its tanh form.  Moe: a mixture of such (MoeSpec).
enum class FfnKind { None, Relu2, GatedSilu, GatedGelu, Moe };
const char* mixer_name(MixerKind k);

// Rotary embedding, optionally with scaled frequencies: YaRN's interpolation over pairs, or by wavelength (pairs that turn more
// than `high` times over the original context keep their frequency, those that turn less than `low` times are slowed by
// `factor`, linear in the turns between).  Which dimensions form a pair is the mixer's (AttnPairs; neighbours in LatentAttention).
enum class RotaryScaling { None, Yarn, Wavelength };
struct RotarySpec {
    int dims = 0;
    double base = 10000.0;
    RotaryScaling scaling = RotaryScaling::None;
    double factor = 1.0, original = 0.0, fast = 0.0, slow = 0.0;  // Wavelength: fast, slow = high, low
    bool operator==(const RotarySpec& o) const {
        return dims == o.dims && base == o.base && scaling == o.scaling && factor == o.factor && original == o.original && fast == o.fast && slow == o.slow;
    }
};
// Angular frequency of every pair and the factor on cos and sin.
void rotary_frequencies(const RotarySpec& r, std::vector<double>* freq, double* magnitude);

// Which keys a position sees besides causality: those nearer than `size` (0: all) and the sequence's first `keep_first`.
struct MaskSpec { int size = 0, keep_first = 0; };

constexpr int kMaxRouterOutputs = 1024, kMaxChoices = 32;
// Router over `experts` feed-forwards and `identity` experts that return their input.  Scores: softmax over all outputs, or a
// sigmoid of each.  The `top` largest of score + correction among the best `keep` of `groups` equal groups are chosen and weighted
// with their scores; a group counts with the sum of its `group_top` (1 or 2) largest.
enum class RouterScore { Softmax, Sigmoid };
struct MoeSpec {
    int experts = 0, identity = 0, top = 0, groups = 1, keep = 1, ff = 0;
    int shared_ff = 0;  // 0: no shared expert; otherwise one that runs for every token, times a sigmoid gate
    RouterScore score = RouterScore::Softmax;
    int group_top = 1;
    bool gated = false; // experts are GatedSilu instead of Relu2 (then without a shared one)
    int outputs() const { return experts + identity; }
};

// Norms of attention's queries and keys: over all heads together ahead of the rotation (weights of all heads), per head ahead of it
// (one weight of `dim`), per head behind it (no weight), none.
enum class QkNorm { AllHeads, PerHead, PerHeadAfter, None };
// Factor 1 + coef ln(floor((position + 1) / every) + 1) on attention's queries (coef 0: none).
struct QueryTemperature {
    double coef = 0.0, every = 1.0;
    bool operator==(const QueryTemperature& o) const { return coef == o.coef && every == o.every; }
};
// The two dimensions of a rotation pair: i and i + dims / 2, or 2i and 2i + 1.
enum class AttnPairs { Halves, Neighbours };
// LinearState: S = decay S + step k v^T, read with q, per head.  Constant: decays from the config, q, k and v through silu, the heads
// normed together, a sigmoid gate on the result.  StateSpace: decay and step from the token, q and k shared by the heads of a
// group, a convolution with bias ahead of the silu, a skip term, a silu gate ahead of the norm in parts.
enum class LinearKind { Constant, StateSpace };

struct MixerSpec {
    MixerKind kind = MixerKind::ChannelDelta;
    int heads = 0, dim = 0, vdim = 0;
    int kv_heads = 0;                             // ChannelDelta, Attention; LinearState: groups that share q and k
    int conv_taps = 0;                            // ChannelDelta, Attention, LinearState (0: none)
    float unit_eps = 1e-6f;                       // ChannelDelta: inside the root that makes q and k unit vectors
    int q_rank = 0, kv_rank = 0, rot_dim = 0;     // LatentAttention (q_rank 0: the tensor's shape gives it)
    float scale = 1.0f;
    RotarySpec rot;
    // Attention
    MaskSpec mask;
    int kv_from = -1;                             // the layer whose keys and values are read (-1: its own)
    QkNorm qk_norm = QkNorm::AllHeads;
    AttnPairs pairs = AttnPairs::Halves;
    float softcap = 0.0f;                         // scores through cap * tanh(. / cap); 0: none
    bool out_gate = false;                        // a sigmoid gate per output element
    bool head_gate = false;                       // a sigmoid gate per head
    bool qkv_bias = false, out_bias = false;
    QueryTemperature q_temp;
    // GeneralDelta: S = diag(w) S - (a u) (u^T S) + k v^T over the old S, u the unit key; w = exp(-decay_scale * sigmoid(.)) and a =
    // sigmoid(.) per key channel
    double decay_scale = 0.0;
    // LinearState
    LinearKind linear = LinearKind::Constant;
    int norm_parts = 1;
    std::vector<double> decay;                    // Constant: per head
};

// Two mixers over one input.  Scaled: scale[0] left + scale[1] right.  Normed: half the sum of the two, each through an RMS norm.
enum class Combine { Single, Scaled, Normed };
struct LayerSpec {
    MixerSpec mix[2];                             // the second one: side by side with the first
    Combine combine = Combine::Single;
    float mix_scale[2] = {1.0f, 1.0f};
    int mixers() const { return combine == Combine::Single ? 1 : 2; }
    FfnKind ffn = FfnKind::None;
    int ff = 0;
    MoeSpec moe;
};

// A second embedding by (previous token, token): row (previous * mul_prev + token * mul_cur) mod buckets, for a sequence's first
// token row `buckets` (0 buckets: none).  The factors are kept modulo buckets.
struct BigramSpec { int64_t buckets = 0, mul_prev = 0, mul_cur = 0; };

// A stack of layers with norms on the sublayers' outputs, x += norm1(mixer(x)), x += norm2(ffn(x)); norm_inputs: on their
// inputs too, x += norm1b(mixer(norm1(x))), x += norm2b(ffn(norm2(x))), or (norm_outputs false) there alone, x += mixer(norm1(x)),
// x += ffn(norm2(x)).  side_dim: every layer ends with x += norm(proj(gelu(gate x) * e)), e the layer's part of the token's row in
// a table of [vocab, layers * side_dim].  depth_average: what leaves layer i is sum_j dwa[j] X_j over the embedding X_0 and the
// results X_1 .. X_(i + 1) of the layers so far, before their averaging.
struct ArchSpec {
    std::string name;
    std::vector<LayerSpec> layers;
    int width = 0, vocab = 0;
    float eps = 1e-6f;
    bool norm_inputs = false, norm_outputs = true;
    bool norm_one_plus = false;  // norm weights stored around zero: 1 + w
    bool norm_scalar = false;    // one number for all elements
    bool depth_average = false;
    BigramSpec bigram;
    int side_dim = 0;
    float embed_scale = 1.0f;
    float logit_scale = 1.0f, logit_softcap = 0.0f;  // softcap 0: none
};

// Parses a config.json; the design is looked up by its "architecture".
int32_t arch_from_json(const char* text, size_t len, ArchSpec* out);

}  // namespace lc
