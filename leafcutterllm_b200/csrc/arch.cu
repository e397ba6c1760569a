// Registry of the checkpoint-directory designs and the loader of such directories: config.json names the design and gives
// every size and constant, model.safetensors holds the weights (an 8-byte little-endian header length, a JSON header of
// name -> dtype, shape, data_offsets, then the data).
#include <cmath>
#include <cstring>
#include <initializer_list>
#include "lc_arch.h"
#include "lc_json.h"
#include "lc_model.h"

namespace lc {

const char* mixer_name(MixerKind k) {
    return k == MixerKind::ChannelDelta ? "channel_delta" : k == MixerKind::LatentAttention ? "latent_attention" : k == MixerKind::Attention ? "attention" : k == MixerKind::GeneralDelta ? "general_delta" : "linear_state";
}

void rotary_frequencies(const RotarySpec& r, std::vector<double>* freq, double* magnitude) {
    const int n = r.dims / 2;
    freq->assign((size_t)n, 0.0);
    *magnitude = 1.0;
    for (int i = 0; i < n; i++) (*freq)[i] = std::pow(r.base, -2.0 * i / r.dims);
    const double pi = 3.14159265358979323846;
    if (r.scaling == RotaryScaling::None) return;
    if (r.scaling == RotaryScaling::Wavelength) {
        for (double& f : *freq) {
            const double turns = r.original * f / (2.0 * pi);
            const double keep = turns > r.fast ? 1.0 : turns < r.slow ? 0.0 : (turns - r.slow) / (r.fast - r.slow);
            f = (1.0 - keep) * f / r.factor + keep * f;
        }
        return;
    }
    auto pair_at = [&](double turns) { return r.dims * std::log(r.original / (2.0 * pi * turns)) / (2.0 * std::log(r.base)); };
    const double lo = std::fmax(std::floor(pair_at(r.fast)), 0.0), hi = std::fmin(std::ceil(pair_at(r.slow)), r.dims - 1.0);
    for (int i = 0; i < n; i++) {
        const double ramp = std::fmin(std::fmax((i - lo) / std::fmax(hi - lo, 0.001), 0.0), 1.0);
        (*freq)[i] = (*freq)[i] / r.factor * ramp + (*freq)[i] * (1.0 - ramp);
    }
    *magnitude = 0.1 * std::log(r.factor) + 1.0;
}

namespace {

// Typed access to one JSON object; the first problem is kept as the error text.
struct Fields {
    const JValue* o = nullptr;
    std::string where;
    const JValue* need(const char* key, JValue::Kind kind) const {
        const JValue* v = o ? o->get(key) : nullptr;
        if (!v || v->kind != kind) { set_error("config: %s lacks '%s' or it has the wrong type", where.c_str(), key); return nullptr; }
        return v;
    }
    int32_t integer(const char* key, int* out, int lo) const {
        const JValue* v = need(key, JValue::NUM);
        if (!v) return LC_ERR_INVALID;
        LC_CHECK(v->num == std::floor(v->num) && v->num >= lo && v->num < 2147483648.0, LC_ERR_INVALID, "config: %s: '%s' = %g is out of range", where.c_str(), key, v->num);
        *out = (int)v->num;
        return LC_OK;
    }
    int32_t real(const char* key, double* out) const {
        const JValue* v = need(key, JValue::NUM);
        if (!v) return LC_ERR_INVALID;
        *out = v->num;
        return LC_OK;
    }
    int32_t real(const char* key, float* out) const {
        double d = 0;
        LC_TRY(real(key, &d));
        *out = (float)d;
        return LC_OK;
    }
    int32_t child(const char* key, Fields* out) const {
        out->o = need(key, JValue::OBJ);
        out->where = where + "." + key;
        return out->o ? LC_OK : LC_ERR_INVALID;
    }
    bool has(const char* key) const { const JValue* v = o->get(key); return v && v->kind != JValue::NUL; }
};

// scaling: what "scaling" means in the design
int32_t parse_rotary(const JValue& v, const std::string& where, RotaryScaling scaling, RotarySpec* out) {
    Fields f{&v, where + ".rot"};
    LC_TRY(f.integer("dims", &out->dims, 2));
    LC_CHECK(out->dims % 2 == 0, LC_ERR_INVALID, "config: %s: an odd number of rotated dimensions", f.where.c_str());
    LC_TRY(f.real("base", &out->base));
    if (f.has("scaling")) {
        const JValue* sv = f.need("scaling", JValue::OBJ);
        if (!sv) return LC_ERR_INVALID;
        Fields s{sv, f.where + ".scaling"};
        out->scaling = scaling;
        const bool yarn = scaling == RotaryScaling::Yarn;
        LC_TRY(s.real("factor", &out->factor));
        LC_TRY(s.real("original", &out->original));
        LC_TRY(s.real(yarn ? "fast" : "high", &out->fast));
        LC_TRY(s.real(yarn ? "slow" : "low", &out->slow));
    }
    return LC_OK;
}

// The sizes that every mixer has.
int32_t parse_heads(const Fields& m, MixerSpec* out) {
    LC_TRY(m.integer("heads", &out->heads, 1));
    LC_TRY(m.integer("vdim", &out->vdim, 1));
    return LC_OK;
}
int32_t parse_sharing(const Fields& m, const char* key, MixerSpec* out) {
    LC_TRY(m.integer(key, &out->kv_heads, 1));
    LC_CHECK(out->heads % out->kv_heads == 0, LC_ERR_INVALID, "config: %s: %d heads over %d key heads", m.where.c_str(), out->heads, out->kv_heads);
    return LC_OK;
}

// The constants of attention: heads over shared key/value heads, rotation, window, the layer whose cache it reads.
int32_t parse_attention(const Fields& m, int index, RotaryScaling scaling, MixerSpec* out) {
    out->kind = MixerKind::Attention;
    LC_TRY(parse_heads(m, out));
    LC_TRY(m.integer("dim", &out->dim, 1));
    LC_TRY(parse_sharing(m, "kv_heads", out));
    LC_TRY(m.real("scale", &out->scale));
    if (m.has("softcap")) {
        LC_TRY(m.real("softcap", &out->softcap));
        LC_CHECK(out->softcap > 0.0f, LC_ERR_INVALID, "config: %s: 'softcap' = %g", m.where.c_str(), out->softcap);
    }
    if (m.has("rot")) {
        const JValue* rot = m.need("rot", JValue::OBJ);
        if (!rot) return LC_ERR_INVALID;
        LC_TRY(parse_rotary(*rot, m.where, scaling, &out->rot));
        LC_CHECK(out->rot.dims <= out->dim, LC_ERR_INVALID, "config: %s: %d of %d dimensions rotated", m.where.c_str(), out->rot.dims, out->dim);
    }
    if (m.has("mask")) {
        Fields k;
        LC_TRY(m.child("mask", &k));
        LC_TRY(k.integer("size", &out->mask.size, 1));
        if (k.has("keep_first")) LC_TRY(k.integer("keep_first", &out->mask.keep_first, 0));
    }
    if (m.has("kv_from")) {
        LC_TRY(m.integer("kv_from", &out->kv_from, 0));
        LC_CHECK(out->kv_from < index, LC_ERR_INVALID, "config: %s: 'kv_from' %d is not an earlier layer", m.where.c_str(), out->kv_from);
    }
    return LC_OK;
}

int32_t parse_delta(const Fields& m, MixerSpec* out) {
    out->kind = MixerKind::ChannelDelta;
    LC_TRY(parse_heads(m, out));
    LC_TRY(m.integer("dim", &out->dim, 1));
    LC_TRY(parse_sharing(m, "kv_heads", out));
    return m.integer("conv", &out->conv_taps, 1);
}

int32_t parse_latent(const Fields& m, MixerSpec* out) {
    out->kind = MixerKind::LatentAttention;
    LC_TRY(parse_heads(m, out));
    LC_TRY(m.integer("dim", &out->dim, 1));
    LC_TRY(m.integer("kv_rank", &out->kv_rank, 1));
    LC_TRY(m.integer("rot_dim", &out->rot_dim, 2));
    if (m.has("q_rank")) LC_TRY(m.integer("q_rank", &out->q_rank, 1));
    LC_TRY(m.real("scale", &out->scale));
    const JValue* rot = m.need("rot", JValue::OBJ);
    if (!rot) return LC_ERR_INVALID;
    LC_TRY(parse_rotary(*rot, m.where, RotaryScaling::Yarn, &out->rot));
    LC_CHECK(out->rot.dims <= out->rot_dim, LC_ERR_INVALID, "config: %s: %d of %d dimensions rotated", m.where.c_str(), out->rot.dims, out->rot_dim);
    return LC_OK;
}

int32_t parse_state_space(const Fields& m, MixerSpec* out) {
    out->kind = MixerKind::LinearState;
    out->linear = LinearKind::StateSpace;
    LC_TRY(parse_heads(m, out));
    LC_TRY(m.integer("state", &out->dim, 1));
    LC_TRY(parse_sharing(m, "groups", out));
    LC_TRY(m.integer("conv", &out->conv_taps, 1));
    LC_TRY(m.integer("norm_groups", &out->norm_parts, 1));
    LC_CHECK(out->heads * out->vdim % out->norm_parts == 0, LC_ERR_INVALID, "config: %s: %d channels in %d 'norm_groups'", m.where.c_str(), out->heads * out->vdim, out->norm_parts);
    return LC_OK;
}

int32_t parse_lightning(const Fields& m, MixerSpec* out) {
    out->kind = MixerKind::LinearState;
    out->linear = LinearKind::Constant;
    LC_TRY(parse_heads(m, out));
    LC_TRY(m.integer("dim", &out->dim, 1));
    out->kv_heads = out->heads;
    const JValue* d = m.need("decay", JValue::ARR);
    if (!d) return LC_ERR_INVALID;
    LC_CHECK((int)d->arr.size() == out->heads, LC_ERR_INVALID, "config: %s: %zu values of 'decay' for %d heads", m.where.c_str(), d->arr.size(), out->heads);
    for (const JValue& v : d->arr) {
        LC_CHECK(v.kind == JValue::NUM && v.num >= 0.0 && v.num <= 1.0, LC_ERR_INVALID, "config: %s: 'decay' is not in 0 .. 1", m.where.c_str());
        out->decay.push_back(v.num);
    }
    return LC_OK;
}

// Two mixers side by side; `type` tells which, and how their outputs meet.
int32_t parse_parallel(const Fields& m, const std::string& type, int index, LayerSpec* out) {
    Fields left, right;
    LC_TRY(m.child("left", &left));
    LC_TRY(m.child("right", &right));
    MixerSpec& a = out->mix[0];
    LC_CHECK(!left.has("kv_from"), LC_ERR_UNSUPPORTED, "config: %s: 'kv_from' beside another mixer", left.where.c_str());
    LC_TRY(parse_attention(left, index, RotaryScaling::Wavelength, &a));
    a.pairs = AttnPairs::Neighbours;
    if (type == "parallel") {
        a.qk_norm = QkNorm::PerHead;
        a.out_gate = true;
        LC_TRY(parse_state_space(right, &out->mix[1]));
        out->combine = Combine::Scaled;
        LC_TRY(m.real("left_scale", &out->mix_scale[0]));
        return m.real("right_scale", &out->mix_scale[1]);
    }
    a.qk_norm = QkNorm::PerHeadAfter;
    LC_TRY(left.integer("conv", &a.conv_taps, 1));
    out->combine = Combine::Normed;
    return parse_lightning(right, &out->mix[1]);
}

// One mixer per layer, by its parser.
template <int32_t (*PARSE)(const Fields&, MixerSpec*)>
int32_t single(const Fields& m, const std::string&, int, LayerSpec* out) { return PARSE(m, &out->mix[0]); }

int32_t parse_sunk_attention(const Fields& m, const std::string&, int index, LayerSpec* out) { return parse_attention(m, index, RotaryScaling::Yarn, &out->mix[0]); }

// Attention with biases and a gate per head; the first kind bounds its scores and warms its queries, the second has norms per head.
int32_t parse_head_gated(const Fields& m, const std::string& type, int index, LayerSpec* out) {
    MixerSpec& a = out->mix[0];
    LC_TRY(parse_attention(m, index, RotaryScaling::Yarn, &a));
    const bool second = type == "attention_2";
    a.qk_norm = second ? QkNorm::PerHead : QkNorm::None;
    a.head_gate = a.qkv_bias = true;
    a.out_bias = !second;
    if (m.has("q_temp")) {
        Fields t;
        LC_TRY(m.child("q_temp", &t));
        LC_TRY(t.real("coef", &a.q_temp.coef));
        LC_TRY(t.real("every", &a.q_temp.every));
        LC_CHECK(a.q_temp.every > 0.0, LC_ERR_INVALID, "config: %s: 'every' = %g", t.where.c_str(), a.q_temp.every);
    }
    return LC_OK;
}

int32_t parse_general_delta(const Fields& m, MixerSpec* out) {
    out->kind = MixerKind::GeneralDelta;
    LC_TRY(m.integer("heads", &out->heads, 1));
    LC_TRY(m.integer("dim", &out->dim, 1));
    out->kv_heads = out->heads;
    out->vdim = out->dim;
    out->decay_scale = std::exp(-0.5);
    return LC_OK;
}

// What the designs do not share: the types of layers and what they hold, the kind of feed-forward that "dense" means, how routers work.
struct LayerType { const char* name; int32_t (*parse)(const Fields& mixer, const std::string& type, int index, LayerSpec* out); };
struct Rules {
    std::initializer_list<LayerType> types;
    FfnKind dense;
    bool mixtures = false;
    MoeSpec moe;
};

int32_t parse_moe(const Fields& p, MoeSpec* out) {
    Fields expert, router;
    LC_TRY(p.child("expert", &expert));
    LC_TRY(expert.integer("ff", &out->ff, 1));
    LC_TRY(p.child("router", &router));
    LC_TRY(router.integer("experts", &out->experts, 1));
    LC_TRY(router.integer("top", &out->top, 1));
    if (router.has("identity")) LC_TRY(router.integer("identity", &out->identity, 0));
    if (router.has("groups")) {
        Fields g;
        LC_TRY(router.child("groups", &g));
        LC_TRY(g.integer("count", &out->groups, 1));
        LC_TRY(g.integer("keep", &out->keep, 1));
    }
    if (p.has("shared")) {
        LC_CHECK(!out->gated, LC_ERR_UNSUPPORTED, "config: %s: a shared expert beside gated experts", p.where.c_str());
        Fields sh;
        LC_TRY(p.child("shared", &sh));
        LC_TRY(sh.integer("ff", &out->shared_ff, 1));
    }
    const int n = out->outputs();
    LC_CHECK(n % out->groups == 0 && out->keep <= out->groups, LC_ERR_INVALID, "config: %s: %d router outputs in %d groups, %d kept", router.where.c_str(), n, out->groups, out->keep);
    LC_CHECK(out->top <= n / out->groups * out->keep, LC_ERR_INVALID, "config: %s: 'top' %d of at most %d", router.where.c_str(), out->top, n / out->groups * out->keep);
    LC_CHECK(n <= kMaxRouterOutputs && out->top <= kMaxChoices, LC_ERR_UNSUPPORTED, "config: %s: %d router outputs, top %d (at most %d, %d)", router.where.c_str(), n, out->top,
             kMaxRouterOutputs, kMaxChoices);
    return LC_OK;
}

int32_t parse_layer(const JValue& v, int index, const Rules& rules, LayerSpec* out) {
    Fields f{&v, "layer " + std::to_string(index)};
    const JValue *type = f.need("type", JValue::STR), *mixer = f.need("mixer", JValue::OBJ);
    if (!type || !mixer) return LC_ERR_INVALID;
    const Fields m{mixer, f.where + ".mixer"};
    const LayerType* known = nullptr;
    for (const LayerType& t : rules.types)
        if (type->str == t.name) known = &t;
    LC_CHECK(known, LC_ERR_UNSUPPORTED, "config: %s: unknown mixer type '%s'", f.where.c_str(), type->str.c_str());
    LC_TRY(known->parse(m, type->str, index, out));
    if (f.has("mlp")) {
        Fields p;
        LC_TRY(f.child("mlp", &p));
        const JValue* kind = p.need("kind", JValue::STR);
        if (!kind) return LC_ERR_INVALID;
        if (kind->str == "dense") {
            out->ffn = rules.dense;
            LC_TRY(p.integer("ff", &out->ff, 1));
        } else if (kind->str == "moe" && rules.mixtures) {
            out->ffn = FfnKind::Moe;
            out->moe = rules.moe;
            LC_TRY(parse_moe(p, &out->moe));
        } else {
            set_error("config: %s: unknown kind '%s'", p.where.c_str(), kind->str.c_str());
            return LC_ERR_UNSUPPORTED;
        }
    }
    return LC_OK;
}

int32_t parse_stack(const Fields& f, const Rules& rules, ArchSpec* out) {
    LC_TRY(f.integer("width", &out->width, 1));
    LC_TRY(f.integer("vocab", &out->vocab, 1));
    const JValue* norm = f.need("norm", JValue::OBJ);
    if (!norm) return LC_ERR_INVALID;
    LC_TRY((Fields{norm, "norm"}.real("eps", &out->eps)));
    const JValue* layers = f.need("layers", JValue::ARR);
    if (!layers) return LC_ERR_INVALID;
    LC_CHECK(!layers->arr.empty(), LC_ERR_INVALID, "config: no layers");
    for (size_t i = 0; i < layers->arr.size(); i++) {
        LayerSpec ly;
        LC_TRY(parse_layer(layers->arr[i], (int)i, rules, &ly));
        const MixerSpec& own = ly.mix[0];
        if (own.kv_from >= 0) {
            const MixerSpec& src = out->layers[(size_t)own.kv_from].mix[0];
            LC_CHECK(src.kind == MixerKind::Attention && src.kv_from < 0 && src.kv_heads == own.kv_heads && src.dim == own.dim && src.vdim == own.vdim, LC_ERR_INVALID,
                     "config: layer %d cannot read the keys and values of layer %d", (int)i, own.kv_from);
        }
        out->layers.push_back(ly);
    }
    return LC_OK;
}

// Varasun: a free mix of gated-delta-rule layers and latent-attention layers, listed one by one.
int32_t parse_varasun(const JValue& cfg, ArchSpec* out) {
    Fields f{&cfg, "the model"};
    LC_TRY(f.real("logit_scale", &out->logit_scale));
    LC_TRY(f.real("logit_softcap", &out->logit_softcap));
    return parse_stack(f, Rules{{{"channel_delta", single<parse_delta>}, {"latent_attention", single<parse_latent>}}, FfnKind::Relu2}, out);
}

// Tenetar: windowed attention layers, some of which read an earlier layer's keys and values, with gated or mixture
// feed-forwards; norms on both sides of every sublayer.
int32_t parse_tenetar(const JValue& cfg, ArchSpec* out) {
    Fields f{&cfg, "the model"}, e;
    LC_TRY(f.child("embedding", &e));
    LC_TRY(e.real("scale", &out->embed_scale));
    out->norm_inputs = true;
    return parse_stack(f, Rules{{{"attention", parse_sunk_attention}}, FfnKind::GatedSilu, true}, out);
}

// Munisun: attention and a linear recurrence side by side in every layer, gated or mixture feed-forwards, norms (stored around
// zero) on both sides of every sublayer, a per-layer input from the token.
int32_t parse_munisun(const JValue& cfg, ArchSpec* out) {
    Fields f{&cfg, "the model"}, e, side;
    LC_TRY(f.child("embedding", &e));
    LC_TRY(e.real("scale", &out->embed_scale));
    LC_TRY(f.child("token_side", &side));
    LC_TRY(side.integer("dim", &out->side_dim, 1));
    out->norm_inputs = out->norm_one_plus = true;
    Rules r{{{"parallel", parse_parallel}, {"parallel_2", parse_parallel}}, FfnKind::GatedSilu, true};
    r.moe.score = RouterScore::Sigmoid;
    r.moe.group_top = 2;
    r.moe.gated = true;
    return parse_stack(f, r, out);
}

// Nepudra: attention of two kinds and a delta rule with separate removal, norms on the sublayers' inputs, an embedding per pair of
// tokens, averages over depth.
int32_t parse_nepudra(const JValue& cfg, ArchSpec* out) {
    Fields f{&cfg, "the model"}, e, b;
    LC_TRY(f.child("embedding", &e));
    LC_TRY(e.child("bigram", &b));
    int buckets = 0;
    double mul[2];
    LC_TRY(b.integer("buckets", &buckets, 1));
    LC_TRY(b.real("mul_prev", &mul[0]));
    LC_TRY(b.real("mul_cur", &mul[1]));
    for (double v : mul) LC_CHECK(v == std::floor(v) && v >= 0.0 && v < 9007199254740992.0, LC_ERR_INVALID, "config: %s: a factor of %g", b.where.c_str(), v);
    out->bigram = BigramSpec{buckets, (int64_t)mul[0] % buckets, (int64_t)mul[1] % buckets};
    out->norm_inputs = out->norm_scalar = out->depth_average = true;
    out->norm_outputs = false;
    return parse_stack(f, Rules{{{"attention", parse_head_gated}, {"attention_2", parse_head_gated}, {"general_delta", single<parse_general_delta>}}, FfnKind::GatedGelu}, out);
}

struct ArchEntry { const char* name; int32_t (*parse)(const JValue&, ArchSpec*); };
const ArchEntry kRegistry[] = {{"Varasun", parse_varasun}, {"Tenetar", parse_tenetar}, {"Munisun", parse_munisun}, {"Nepudra", parse_nepudra}};

uint32_t safetensors_type(const std::string& dtype) {
    if (dtype == "BF16") return LC_TYPE_BF16;
    if (dtype == "F16") return LC_TYPE_F16;
    if (dtype == "F32") return LC_TYPE_F32;
    return ~0u;
}

int32_t load_safetensors(lc_model* m, const std::string& path) {
    Mapping file;
    LC_TRY(file.open_file(path));
    const uint8_t* base = (const uint8_t*)file.base;
    LC_CHECK(file.size >= 8, LC_ERR_INVALID, "%s: too short", path.c_str());
    uint64_t hlen = 0;
    for (int i = 0; i < 8; i++) hlen |= (uint64_t)base[i] << (8 * i);
    LC_CHECK(hlen <= file.size - 8, LC_ERR_INVALID, "%s: the header reaches past the end of the file", path.c_str());
    const std::string text((const char*)base + 8, (size_t)hlen);  // a copy that ends in 0: the reader's number parsing may look one character ahead
    JReader jr{text.c_str(), text.c_str() + text.size()};
    const JValue head = jr.value();
    LC_CHECK(jr.ok && head.kind == JValue::OBJ, LC_ERR_INVALID, "%s: the header is not a JSON object", path.c_str());
    const uint8_t* data = base + 8 + hlen;
    const size_t room = file.size - 8 - (size_t)hlen;
    for (auto& kv : head.obj) {
        if (kv.first == "__metadata__") continue;
        const JValue *dtype = kv.second.get("dtype"), *shape = kv.second.get("shape"), *off = kv.second.get("data_offsets");
        LC_CHECK(dtype && shape && off && shape->kind == JValue::ARR && off->kind == JValue::ARR && off->arr.size() == 2, LC_ERR_INVALID,
                 "%s: tensor %s has a malformed entry", path.c_str(), kv.first.c_str());
        const uint32_t typ = safetensors_type(dtype->str);
        LC_CHECK(typ != ~0u, LC_ERR_UNSUPPORTED, "%s: tensor %s has dtype %s", path.c_str(), kv.first.c_str(), dtype->str.c_str());
        std::vector<uint64_t> dims;  // fastest first
        uint64_t count = 1;
        for (size_t i = shape->arr.size(); i > 0; i--) { dims.push_back((uint64_t)shape->arr[i - 1].num); count *= dims.back(); }
        if (dims.empty()) dims.push_back(1);
        LC_CHECK(dims.size() <= 4 && count > 0, LC_ERR_UNSUPPORTED, "%s: tensor %s has an unsupported shape", path.c_str(), kv.first.c_str());
        const double b = off->arr[0].num, e = off->arr[1].num;
        LC_CHECK(b >= 0 && e >= b && e <= (double)room && (uint64_t)(e - b) == lc_tensor_bytes(typ, count), LC_ERR_INVALID,
                 "%s: tensor %s: its offsets do not match its shape or the file", path.c_str(), kv.first.c_str());
        LC_TRY(lc_model_set_tensor(m, kv.first.c_str(), typ, dims.data(), (int32_t)dims.size(), data + (size_t)b, (size_t)(e - b)));
    }
    return LC_OK;
}

}  // namespace

int32_t arch_from_json(const char* text, size_t len, ArchSpec* out) {
    const std::string copy(text, len);
    JReader jr{copy.c_str(), copy.c_str() + copy.size()};
    const JValue cfg = jr.value();
    LC_CHECK(jr.ok && cfg.kind == JValue::OBJ, LC_ERR_INVALID, "config: not a JSON object");
    const JValue* name = cfg.get("architecture");
    LC_CHECK(name && name->kind == JValue::STR, LC_ERR_INVALID, "config: no 'architecture'");
    for (const ArchEntry& a : kRegistry)
        if (name->str == a.name) {
            out->name = a.name;
            return a.parse(cfg, out);
        }
    set_error("config: architecture '%s' is not known to this library", name->str.c_str());
    return LC_ERR_UNSUPPORTED;
}

}  // namespace lc

extern "C" int32_t lc_model_load_dir(const char* dir, const lc_model_config* overrides, lc_model** out) {
    LC_CHECK(dir && out, LC_ERR_INVALID, "lc_model_load_dir: null argument");
    *out = nullptr;
    std::string text;
    {
        Mapping cfg;
        LC_TRY(cfg.open_file(std::string(dir) + "/config.json"));
        text.assign((const char*)cfg.base, cfg.size);
    }
    lc_model* m = nullptr;
    LC_TRY(lc_model_create_json(text.c_str(), overrides, &m));
    int32_t st = load_safetensors(m, std::string(dir) + "/model.safetensors");
    if (st == LC_OK) st = lc_model_finalize(m);
    if (st != LC_OK) {
        const std::string keep = get_error();
        lc_model_destroy(m);
        set_error("%s", keep.c_str());
        return st;
    }
    *out = m;
    return LC_OK;
}
