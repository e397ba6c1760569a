// The layers of a checkpoint-directory design on the device: binding of the weights, the cache and state they keep, and the
// launches of one pass over T tokens.  Per layer:
//   ChannelDelta     in = q | k | v | a1 | g1 | b (one product)  ->  a2 (log decay in its epilogue), g2  ->  convolutions + unit
//                    vectors -> recurrence -> per-head norm and gate -> out
//   LatentAttention  in = dq | dkv (one product)  ->  latent norms, key rotation, cache append  ->  uq -> (per head) uk^T
//                    -> attention over the latents -> (per head) uv -> out
//   Attention        in = q | k | v | gates per head (one product, biases in its epilogue)  ->  norms over all heads or per head,
//                    rotation, factors on queries, cache append  ->  attention (gated) -> out
//   GeneralDelta     in = r | k | v | a (32-bit) | w1 (through tanh) | g (one product)  ->  w2 (log decay in its epilogue)  ->
//                    recurrence -> per-head norm and gate -> out
//   Attention and    in = both mixers' projections (one product, silu where a mixer wants it)  ->  convolutions, norms, rotation, cache
//   LinearState      append -> attention (gated) | convolutions -> recurrence -> norm and gate  ->  out: one product over both outputs side
//   side by side     by side, or one each where they are normed before they meet
//   Relu2            up (squared relu in its epilogue) -> down
//   GatedSilu, GatedGelu  gate and up rows in turn (one product, act(gate) * up in its epilogue) -> down
//   Moe              router | shared gate | shared up (one product) -> choice, token lists -> experts' up, experts' down
//                    (grouped products), shared down
//   token input      gate (gelu times the token's row of a table in its epilogue) -> proj
// each followed by x += rms_norm(y) w (for Moe on the weighted sum of the experts' rows) or, without norms on outputs, x += y, which
// also takes the sum over depth at a layer's end and writes the activations the next product reads: the sum, or its norm where the
// design has norms on inputs and no token input follows.
#include <cmath>
#include <cstring>
#include "lc_model.h"

namespace lc {

namespace {

typedef __nv_bfloat16 bf16;
constexpr int kGatheredRows = 32;    // experts with larger tiles of rows read a copy in expert order (a gather brings about a row per 14 cycles)
constexpr int kContextRows = 16384;  // rows of projected keys and values at a time (one longer context is taken whole)

int32_t zalloc(LayerStack& st, void** p, size_t bytes) {
    uint8_t* q = nullptr;
    LC_TRY(dalloc(&q, bytes));
    st.owned.push_back(q);
    LC_CUDA(cudaMemsetAsync(q, 0, std::max<size_t>(bytes, 16), stream()));
    *p = q;
    return LC_OK;
}

int32_t upload(LayerStack& st, const std::vector<float>& h, const float** out, cudaStream_t s) {
    void* d = nullptr;
    LC_TRY(zalloc(st, &d, h.size() * 4));
    LC_CUDA(cudaMemcpyAsync(d, h.data(), h.size() * 4, cudaMemcpyHostToDevice, s));
    LC_CUDA(cudaStreamSynchronize(s));
    *out = (const float*)d;
    return LC_OK;
}

// The same for a plain copy of a weight.
int32_t talloc(LayerStack& st, void** p, size_t bytes) {
    LC_TRY(zalloc(st, p, bytes));
    st.temps.push_back(st.owned.back());
    st.owned.pop_back();
    return LC_OK;
}

// bf16 products read weights in blocks: builds them for `ws`, then drops the plain copies and the checkpoint's tensors they
// came from.  A model in true 32-bit keeps the plain forms.
int32_t block_weights(lc_model* m, std::vector<DenseWeight*> ws) {
    LayerStack& st = *m->stack;
    if (st.f32) {
        st.owned.insert(st.owned.end(), st.temps.begin(), st.temps.end());
        st.temps.clear();
        return LC_OK;
    }
    for (DenseWeight* w : ws) {
        if (!w->data) continue;
        uint8_t* p = nullptr;
        LC_TRY(dalloc(&p, dense_tile_bytes(*w)));
        st.owned.push_back(p);
        LC_TRY(dense_weight_tile(w, p, m->stream));
    }
    LC_CUDA(cudaStreamSynchronize(m->stream));
    for (void* p : st.temps) cudaFree(p);
    st.temps.clear();
    for (const std::string& name : st.packed) {
        DevTensor& t = m->tensors[name];
        if (t.dev) cudaFree(t.dev);
        t.dev = t.view = nullptr;
    }
    st.packed.clear();
    return LC_OK;
}

// A bf16 matrix [rows, cols] by name; rows / cols = 0: whatever the tensor has.
int32_t matrix(lc_model* m, const std::string& name, int rows, int cols, DevTensor** out) {
    auto it = m->tensors.find(name);
    LC_CHECK(it != m->tensors.end(), LC_ERR_MISSING, "missing tensor %s", name.c_str());
    DevTensor& t = it->second;
    LC_CHECK(t.typ == LC_TYPE_BF16, LC_ERR_UNSUPPORTED, "tensor %s: bf16 expected", name.c_str());
    LC_CHECK((rows == 0 || (int)t.rows == rows) && (cols == 0 || (int)t.cols == cols), LC_ERR_INVALID, "tensor %s is [%zu x %zu], expected [%d x %d]", name.c_str(),
             t.rows, t.cols, rows, cols);
    *out = &t;
    m->stack->packed.push_back(name);
    return LC_OK;
}

// A plain [n, k] weight: in place when its rows keep 16-byte alignment, else a copy with padded rows.  `col` pads groups of
// columns (to k_out columns in all).
int32_t plain_weight(lc_model* m, const std::string& name, int n, int k, DenseWeight* w, PackMap col = PackMap(), int k_out = 0) {
    DevTensor* t = nullptr;
    LC_TRY(matrix(m, name, n, k, &t));
    if (k_out == 0) k_out = k;
    if (k_out == k && k % 8 == 0) return dense_weight_init(w, (const bf16*)t->view, n, k, k);
    void* p = nullptr;
    const int ld = round8(k_out);
    LC_TRY(talloc(*m->stack, &p, (size_t)n * ld * 2));
    LC_TRY(launch_pack((const bf16*)t->view, n, k, (bf16*)p, ld, PackMap(), col, false, m->stream));
    return dense_weight_init(w, (const bf16*)p, n, k_out, ld);
}

// Several matrices over the same input as one, each part's rows starting at a multiple of eight; `offs` receives the starts.
// The last part starts at a multiple of `last_align`.
int32_t fused_weight(lc_model* m, const std::vector<std::string>& names, const std::vector<int>& rows, int k, DenseWeight* w, std::vector<int>* offs, int last_align = 8) {
    int total = 0;
    for (size_t i = 0; i < rows.size(); i++) {
        if (i + 1 == rows.size()) total = (total + last_align - 1) / last_align * last_align;
        offs->push_back(total);
        total += round8(rows[i]);
    }
    const int ld = round8(k);
    void* p = nullptr;
    LC_TRY(talloc(*m->stack, &p, (size_t)total * ld * 2));
    for (size_t i = 0; i < names.size(); i++) {
        DevTensor* t = nullptr;
        LC_TRY(matrix(m, names[i], rows[i], k, &t));
        bf16* dst = (bf16*)p + (size_t)(*offs)[i] * ld;
        LC_TRY(launch_pack((const bf16*)t->view, rows[i], k, dst, ld, PackMap(), PackMap(), false, m->stream));
    }
    return dense_weight_init(w, (const bf16*)p, total, k, ld);
}

int rows_of(lc_model* m, const std::string& name) {
    auto it = m->tensors.find(name);
    return it == m->tensors.end() ? 0 : (int)it->second.rows;
}

// A vector put through `f`, on the host.
template <typename F>
int32_t changed_gain(lc_model* m, const std::string& name, int n, F f, const float** out) {
    const float* g = nullptr;
    LC_TRY(model_gain_f32(m, name, n, &g));
    std::vector<float> h((size_t)n);
    LC_CUDA(cudaMemcpyAsync(h.data(), g, h.size() * 4, cudaMemcpyDeviceToHost, m->stream));
    LC_CUDA(cudaStreamSynchronize(m->stream));
    for (float& v : h) v = f(v);
    return upload(*m->stack, h, out, m->stream);
}

// The weight of one of the model's norms.
int32_t norm_gain(lc_model* m, const std::string& name, const float** out) {
    LayerStack& st = *m->stack;
    const ArchSpec& sp = st.spec;
    if (sp.norm_scalar) {  // one number, for every element
        const float* g = nullptr;
        float v = 0.0f;
        LC_TRY(model_gain_f32(m, name, 1, &g));
        LC_CUDA(cudaMemcpyAsync(&v, g, 4, cudaMemcpyDeviceToHost, m->stream));
        LC_CUDA(cudaStreamSynchronize(m->stream));
        return upload(st, std::vector<float>((size_t)sp.width, v), out, m->stream);
    }
    return sp.norm_one_plus ? changed_gain(m, name, sp.width, [](float v) { return 1.0f + v; }, out) : model_gain_f32(m, name, sp.width, out);
}

// The taps of the convolutions on q, k and v as one f32 table.
int32_t conv_table(lc_model* m, const std::string& p, const std::vector<int>& channels, int taps, const float** out) {
    const char* names[3] = {"q.conv", "k.conv", "v.conv"};
    void* d = nullptr;
    LC_TRY(zalloc(*m->stack, &d, (size_t)(channels[0] + channels[1] + channels[2]) * taps * 4));
    float* at = (float*)d;
    for (int i = 0; i < 3; i++) {
        const float* g = nullptr;
        LC_TRY(model_gain_f32(m, p + names[i], channels[i] * taps, &g));
        LC_CUDA(cudaMemcpyAsync(at, g, (size_t)channels[i] * taps * 4, cudaMemcpyDeviceToDevice, m->stream));
        at += (size_t)channels[i] * taps;
    }
    *out = (const float*)d;
    return LC_OK;
}

int32_t bind_delta(lc_model* m, MixerUnit& L, const std::string& p) {
    LayerStack& st = *m->stack;
    const MixerSpec& s = L.s;
    const int W = st.spec.width, nk = s.kv_heads * s.dim, nv = s.heads * s.vdim, nd = s.heads * s.dim;
    const int ra = rows_of(m, p + "a1"), rg = rows_of(m, p + "g1");
    LC_CHECK(ra > 0 && rg > 0, LC_ERR_MISSING, "missing tensor %sa1 or %sg1", p.c_str(), p.c_str());
    LC_CHECK(s.dim <= 256, LC_ERR_UNSUPPORTED, "%s: %d key dimensions per head (at most 256)", p.c_str(), s.dim);
    std::vector<int> offs;
    LC_TRY(fused_weight(m, {p + "q", p + "k", p + "v", p + "a1", p + "g1", p + "b"}, {nk, nk, nv, ra, rg, s.heads}, W, &L.in, &offs));
    L.off_a = offs[3]; L.off_g = offs[4];
    L.dg = DeltaShape{s.heads, s.kv_heads, s.dim, s.vdim, s.conv_taps, L.in.n, offs[1], offs[2], offs[5], 2 * nk + nv, s.unit_eps, st.spec.eps};
    LC_TRY(plain_weight(m, p + "a2", nd, ra, &L.a2));
    LC_TRY(plain_weight(m, p + "g2", nv, rg, &L.g2));
    LC_TRY(plain_weight(m, p + "o", W, nv, &L.out));
    LC_TRY(conv_table(m, p, {nk, nk, nv}, s.conv_taps, &L.conv));
    LC_TRY(changed_gain(m, p + "A_log", s.heads, [](float v) { return std::exp(v); }, &L.a_exp));
    LC_TRY(model_gain_f32(m, p + "dt_bias", nd, &L.dt_bias));
    LC_TRY(model_gain_f32(m, p + "norm", s.vdim, &L.o_norm));
    return LC_OK;
}

int32_t rot_table(lc_model* m, const RotarySpec& r, const float2** out) {
    LayerStack& st = *m->stack;
    for (auto& t : st.rot_tables)
        if (t.first == r) { *out = t.second; return LC_OK; }
    std::vector<double> freq;
    double mag = 1.0;
    rotary_frequencies(r, &freq, &mag);
    void *d = nullptr, *tab = nullptr;
    LC_TRY(zalloc(st, &d, freq.size() * 8));
    LC_CUDA(cudaMemcpyAsync(d, freq.data(), freq.size() * 8, cudaMemcpyHostToDevice, m->stream));
    LC_TRY(zalloc(st, &tab, freq.size() * (size_t)m->cfg.max_seq_len * sizeof(float2)));
    LC_TRY(launch_rot_table((const double*)d, (int)freq.size(), mag, m->cfg.max_seq_len, (float2*)tab, m->stream));
    LC_CUDA(cudaStreamSynchronize(m->stream));
    st.rot_tables.push_back({r, (const float2*)tab});
    *out = (const float2*)tab;
    return LC_OK;
}

int32_t bind_latent(lc_model* m, MixerUnit& L, const std::string& p) {
    LayerStack& st = *m->stack;
    MixerSpec& s = L.s;
    const int W = st.spec.width, qr = rows_of(m, p + "dq");
    LC_CHECK(qr > 0, LC_ERR_MISSING, "missing tensor %sdq", p.c_str());
    LC_CHECK(s.q_rank == 0 || s.q_rank == qr, LC_ERR_INVALID, "%sdq has %d rows, the config says %d", p.c_str(), qr, s.q_rank);
    s.q_rank = qr;
    std::vector<int> offs;
    LC_TRY(fused_weight(m, {p + "dq", p + "dkv"}, {qr, s.kv_rank + s.rot_dim}, W, &L.in, &offs));
    L.off_c = offs[1];
    L.off_r = offs[1] + s.kv_rank;
    LatentShape& g = L.lg;
    g.heads = s.heads; g.dim = s.dim; g.rot = s.rot_dim; g.rank = s.kv_rank;
    g.dp = round8(s.dim); g.cp = round8(s.kv_rank); g.rp = round8(s.rot_dim); g.ld_q = g.dp + g.rp;
    g.rot_pairs = s.rot.dims / 2;
    g.scale = s.scale;
    DevTensor* t = nullptr;
    // queries head by head, both parts padded to eight rows
    LC_TRY(matrix(m, p + "uq", s.heads * (s.dim + s.rot_dim), qr, &t));
    if (g.dp == s.dim && g.rp == s.rot_dim && qr % 8 == 0) {
        LC_TRY(dense_weight_init(&L.uq, (const bf16*)t->view, s.heads * g.ld_q, qr, qr));
    } else {
        void* u = nullptr;
        const int ld = round8(qr);
        LC_TRY(talloc(st, &u, (size_t)s.heads * g.ld_q * ld * 2));
        LC_TRY(launch_pack((const bf16*)t->view, s.heads * (s.dim + s.rot_dim), qr, (bf16*)u, ld, PackMap{s.dim + s.rot_dim, g.ld_q, s.dim, g.dp - s.dim}, PackMap(),
                           false, m->stream));
        LC_TRY(dense_weight_init(&L.uq, (const bf16*)u, s.heads * g.ld_q, qr, ld));
    }
    // key projection, transposed per head: [heads][rank][dim]
    LC_TRY(matrix(m, p + "uk", s.heads * s.dim, s.kv_rank, &t));
    void* kt = nullptr;
    LC_TRY(talloc(st, &kt, (size_t)s.heads * s.kv_rank * g.dp * 2));
    LC_TRY(launch_pack((const bf16*)t->view, s.heads * s.dim, s.kv_rank, (bf16*)kt, g.dp, PackMap{s.dim, s.kv_rank, 0, 0}, PackMap(), true, m->stream));
    LC_TRY(dense_weight_init(&L.uk_t, (const bf16*)kt, s.kv_rank, s.dim, g.dp, s.heads, (size_t)s.kv_rank * g.dp));
    LC_TRY(matrix(m, p + "uv", s.heads * s.vdim, s.kv_rank, &t));
    const bf16* uv = (const bf16*)t->view;
    if (g.cp != s.kv_rank) {
        void* v = nullptr;
        LC_TRY(talloc(st, &v, (size_t)s.heads * s.vdim * g.cp * 2));
        LC_TRY(launch_pack(uv, s.heads * s.vdim, s.kv_rank, (bf16*)v, g.cp, PackMap(), PackMap(), false, m->stream));
        uv = (const bf16*)v;
    }
    LC_TRY(dense_weight_init(&L.uv, uv, s.vdim, s.kv_rank, g.cp, s.heads, (size_t)s.vdim * g.cp));
    L.ep = round8(s.vdim);
    // the same two projections for whole contexts
    if (latent_prefill_applies(g, L.ep, st.f32)) {
        auto all_heads = [&](const char* name, int per, int per_p, DenseWeight* w) -> int32_t {
            DevTensor* wt = nullptr;
            LC_TRY(matrix(m, p + name, s.heads * per, s.kv_rank, &wt));
            if (per == per_p && g.cp == s.kv_rank) return dense_weight_init(w, (const bf16*)wt->view, s.heads * per, s.kv_rank, s.kv_rank);
            void* q = nullptr;
            LC_TRY(talloc(st, &q, (size_t)s.heads * per_p * g.cp * 2));
            LC_TRY(launch_pack((const bf16*)wt->view, s.heads * per, s.kv_rank, (bf16*)q, g.cp, PackMap{per, per_p, 0, 0}, PackMap(), false, m->stream));
            return dense_weight_init(w, (const bf16*)q, s.heads * per_p, s.kv_rank, g.cp);
        };
        LC_TRY(all_heads("uk", s.dim, g.dp, &L.uk_all));
        LC_TRY(all_heads("uv", s.vdim, L.ep, &L.uv_all));
    }
    LC_TRY(plain_weight(m, p + "o", W, s.heads * s.vdim, &L.out, PackMap{s.vdim, L.ep, 0, 0}, s.heads * L.ep));
    LC_TRY(model_gain_f32(m, p + "dq.norm", qr, &L.q_norm));
    LC_TRY(model_gain_f32(m, p + "dkv.norm", s.kv_rank, &L.c_norm));
    return rot_table(m, s.rot, &L.rot);
}

void attention_shape(const LayerStack& st, MixerUnit& L) {
    const MixerSpec& s = L.s;
    AttnShape& g = L.ag;
    g.heads = s.heads; g.kv_heads = s.kv_heads; g.dim = s.dim; g.vdim = s.vdim; g.dp = round8(s.dim); g.ep = round8(s.vdim); g.rot_dims = s.rot.dims;
    g.scale = s.scale; g.cap = s.softcap; g.window = s.mask.size; g.keep_first = s.mask.keep_first; g.norm = s.qk_norm; g.pairs = s.pairs; g.taps = s.conv_taps;
    attn_cache_layout(&g, st.f32);
    L.ep = g.ep;
}

// The factors on queries of every position.
int32_t q_factor_table(lc_model* m, const QueryTemperature& t, const float** out) {
    LayerStack& st = *m->stack;
    for (auto& f : st.q_factors)
        if (f.first == t) { *out = f.second; return LC_OK; }
    std::vector<float> h((size_t)m->cfg.max_seq_len);
    for (size_t p = 0; p < h.size(); p++) h[p] = (float)(1.0 + t.coef * std::log(std::floor((double)(p + 1) / t.every) + 1.0));
    LC_TRY(upload(st, h, out, m->stream));
    st.q_factors.push_back({t, *out});
    return LC_OK;
}

int32_t bind_attention(lc_model* m, MixerUnit& L, const std::string& p) {
    LayerStack& st = *m->stack;
    const MixerSpec& s = L.s;
    const bool own = s.kv_from < 0;
    const int W = st.spec.width, nq = s.heads * s.dim, nk = s.kv_heads * s.dim, nv = s.kv_heads * s.vdim;
    LC_CHECK(s.qk_norm == QkNorm::AllHeads || std::max(s.dim, s.vdim) <= 512, LC_ERR_UNSUPPORTED, "%s: heads of %d and %d dimensions (at most 512)", p.c_str(), s.dim, s.vdim);
    attention_shape(st, L);
    std::vector<std::string> names = {p + "q"};
    std::vector<int> rows = {nq}, offs;
    if (own) { names.insert(names.end(), {p + "k", p + "v"}); rows.insert(rows.end(), {nk, nv}); }
    const size_t biased = names.size();
    if (s.head_gate) { names.push_back(p + "g"); rows.push_back(s.heads); }
    if (names.size() == 1) { LC_TRY(plain_weight(m, p + "q", nq, W, &L.in)); offs = {0}; }
    else LC_TRY(fused_weight(m, names, rows, W, &L.in, &offs));
    if (own) { L.off_k = offs[1]; L.off_v = offs[2]; }
    if (s.head_gate) L.off_hg = offs[biased];
    if (s.qkv_bias) {
        void* d = nullptr;
        LC_TRY(zalloc(st, &d, (size_t)L.in.n * 4));
        L.in_bias = (const float*)d;
        for (size_t i = 0; i < biased; i++) {
            const float* b = nullptr;
            LC_TRY(model_gain_f32(m, names[i] + ".b", rows[i], &b));
            LC_CUDA(cudaMemcpyAsync((float*)d + offs[i], b, (size_t)rows[i] * 4, cudaMemcpyDeviceToDevice, m->stream));
        }
    }
    if (s.out_bias) LC_TRY(model_gain_f32(m, p + "o.b", W, &L.out_bias));
    if (s.q_temp.coef != 0.0) LC_TRY(q_factor_table(m, s.q_temp, &L.q_factor));
    if (s.qk_norm == QkNorm::AllHeads || s.qk_norm == QkNorm::PerHead) {
        const bool all = s.qk_norm == QkNorm::AllHeads;
        LC_TRY(model_gain_f32(m, p + "q.norm", all ? nq : s.dim, &L.q_norm));
        if (own) LC_TRY(model_gain_f32(m, p + "k.norm", all ? nk : s.dim, &L.k_norm));
    }
    if (m->tensors.count(p + "sink")) LC_TRY(model_gain_f32(m, p + "sink", s.heads, &L.sink));
    LC_TRY(plain_weight(m, p + "o", W, s.heads * s.vdim, &L.out, PackMap{s.vdim, L.ep, 0, 0}, s.heads * L.ep));
    return s.rot.dims ? rot_table(m, s.rot, &L.rot) : LC_OK;
}

int32_t bind_general_delta(lc_model* m, MixerUnit& L, const std::string& p) {
    LayerStack& st = *m->stack;
    const MixerSpec& s = L.s;
    const int W = st.spec.width, n = s.heads * s.dim, n8 = round8(n), rank = rows_of(m, p + "w1"), ld = round8(W);
    LC_CHECK(rank > 0, LC_ERR_MISSING, "missing tensor %sw1", p.c_str());
    LC_CHECK(s.dim <= 256, LC_ERR_UNSUPPORTED, "%s: %d dimensions per head (at most 256)", p.c_str(), s.dim);
    L.in_split = (4 * n8 + 31) / 32 * 32;
    L.act_end = L.in_split + round8(rank);
    const struct { const char* name; int rows, at; } parts[] = {{"r", n, 0}, {"k", n, n8}, {"v", n, 2 * n8}, {"a", n, 3 * n8}, {"w1", rank, L.in_split}, {"g", n, L.act_end}};
    const int total = L.act_end + n8;
    void* d = nullptr;
    LC_TRY(talloc(st, &d, (size_t)total * ld * 2));
    for (const auto& q : parts) {
        DevTensor* t = nullptr;
        LC_TRY(matrix(m, p + q.name, q.rows, W, &t));
        LC_TRY(launch_pack((const bf16*)t->view, q.rows, W, (bf16*)d + (size_t)q.at * ld, ld, PackMap(), PackMap(), false, m->stream));
    }
    LC_TRY(dense_weight_init(&L.in, (const bf16*)d, total, W, ld));
    L.off_g = L.act_end - L.in_split;
    L.gg = GeneralShape{s.heads, s.dim, L.in_split, n8, 2 * n8, 3 * n8, s.unit_eps, st.spec.eps};
    LC_TRY(plain_weight(m, p + "w2", n, rank, &L.a2));
    LC_TRY(model_gain_f32(m, p + "w0", n, &L.dt_bias));
    LC_TRY(model_gain_f32(m, p + "a.b", n, &L.a_bias));
    LC_TRY(model_gain_f32(m, p + "norm", n, &L.o_norm));
    return plain_weight(m, p + "o", W, n, &L.out);
}

// Attention and a linear recurrence side by side.
int32_t bind_pair(lc_model* m, StackLayer& L, const std::string& p) {
    LayerStack& st = *m->stack;
    MixerUnit &a = L.mix[0], &b = L.mix[1];
    const MixerSpec &sa = a.s, &sb = b.s;
    const std::string pl = p + "left.", pr = p + "right.";
    const int W = st.spec.width, nq = sa.heads * sa.dim, nk = sa.kv_heads * sa.dim, nv = sa.kv_heads * sa.vdim, inner = sb.heads * sb.vdim;
    const bool space = sb.linear == LinearKind::StateSpace;
    LC_CHECK(sb.dim <= 256 && std::max(sa.dim, sa.vdim) <= 512, LC_ERR_UNSUPPORTED, "%s: %d state dimensions (at most 256), heads of %d and %d dimensions (at most 512)", p.c_str(),
             sb.dim, sa.dim, sa.vdim);
    attention_shape(st, a);
    LinearShape& g = b.ng;
    g.kind = sb.linear; g.heads = sb.heads; g.groups = sb.kv_heads; g.dim = sb.dim; g.vdim = sb.vdim; g.taps = sb.conv_taps; g.norm_parts = sb.norm_parts; g.eps = st.spec.eps;
    g.channels = space ? inner + 2 * sb.kv_heads * sb.dim : 0;
    g.ld_in = round8(g.channels);
    // rows [row0, row0 + rows) of a tensor of `all` rows; off: where they start
    struct Part { std::string name; int all, row0, rows; int* off; };
    std::vector<Part> wide = {{pl + "q", nq, 0, nq, nullptr}, {pl + "k", nk, 0, nk, &a.off_k}, {pl + "v", nv, 0, nv, &a.off_v}}, silu, plain;
    if (sa.out_gate) plain.push_back({pl + "g", sa.heads * sa.vdim, 0, sa.heads * sa.vdim, &a.off_g});
    if (space) {
        const int all = inner + g.channels + sb.heads;
        wide.push_back({pr + "in", all, inner + g.channels, sb.heads, &g.off_dt});
        plain.push_back({pr + "in", all, 0, inner, &g.off_g});
        plain.push_back({pr + "in", all, inner, g.channels, &g.off_v});
    } else {
        silu = {{pr + "q", sb.heads * sb.dim, 0, sb.heads * sb.dim, &g.off_q}, {pr + "k", sb.heads * sb.dim, 0, sb.heads * sb.dim, &g.off_k}, {pr + "v", inner, 0, inner, &g.off_v}};
        plain.push_back({pr + "g", inner, 0, inner, &g.off_g});
    }
    auto rows_of_parts = [](const std::vector<Part>& ps) { int n = 0; for (const Part& q : ps) n += round8(q.rows); return n; };
    L.in_split = (rows_of_parts(wide) + 31) / 32 * 32;
    L.act_end = L.in_split + rows_of_parts(silu);
    const int total = L.act_end + rows_of_parts(plain), ld = round8(W);
    void* d = nullptr;
    LC_TRY(talloc(st, &d, (size_t)total * ld * 2));
    auto place = [&](const std::vector<Part>& ps, int at, int base) -> int32_t {
        for (const Part& q : ps) {
            DevTensor* t = nullptr;
            LC_TRY(matrix(m, q.name, q.all, W, &t));
            LC_TRY(launch_pack((const bf16*)t->view + (size_t)q.row0 * W, q.rows, W, (bf16*)d + (size_t)at * ld, ld, PackMap(), PackMap(), false, m->stream));
            if (q.off) *q.off = at - base;
            at += round8(q.rows);
        }
        return LC_OK;
    };
    LC_TRY(place(wide, 0, 0));
    LC_TRY(place(silu, L.in_split, L.in_split));
    LC_TRY(place(plain, L.act_end, L.in_split));
    LC_TRY(dense_weight_init(&L.in, (const bf16*)d, total, W, ld));
    g.ld = total - L.in_split;
    g.ld_dt = L.in_split;
    if (space) { g.off_k = g.off_v + inner; g.off_q = g.off_k + sb.kv_heads * sb.dim; }
    // attention
    if (sa.qk_norm == QkNorm::PerHead) {
        LC_TRY(model_gain_f32(m, pl + "q.norm", sa.dim, &a.q_norm));
        LC_TRY(model_gain_f32(m, pl + "k.norm", sa.dim, &a.k_norm));
    }
    if (sa.conv_taps) LC_TRY(conv_table(m, pl, {nq, nk, nv}, sa.conv_taps, &a.conv));
    if (sa.rot.dims) LC_TRY(rot_table(m, sa.rot, &a.rot));
    // recurrence
    LC_TRY(model_gain_f32(m, pr + "norm", inner, &b.o_norm));
    if (space) {
        LC_TRY(model_gain_f32(m, pr + "conv", g.channels * g.taps, &b.conv));
        LC_TRY(model_gain_f32(m, pr + "conv.b", g.channels, &b.conv_b));
        LC_TRY(model_gain_f32(m, pr + "dt_bias", sb.heads, &b.dt_bias));
        LC_TRY(model_gain_f32(m, pr + "D", sb.heads, &b.skip));
        LC_TRY(changed_gain(m, pr + "A_log", sb.heads, [](float v) { return std::exp(v); }, &b.a_exp));
    } else {
        std::vector<float> table((size_t)sb.heads * 3);  // factors, then their logarithms
        for (int h = 0; h < sb.heads; h++) {
            table[2 * h] = (float)sb.decay[h];
            table[2 * h + 1] = (float)(sb.decay[h] - (double)table[2 * h]);
            table[2 * sb.heads + h] = (float)std::fmax(std::log(sb.decay[h]), -1e4);  // far below where exp ends, and still a number
        }
        void* dec = nullptr;
        LC_TRY(zalloc(st, &dec, table.size() * 4));
        LC_CUDA(cudaMemcpyAsync(dec, table.data(), table.size() * 4, cudaMemcpyHostToDevice, m->stream));
        LC_CUDA(cudaStreamSynchronize(m->stream));
        b.decay = (const float2*)dec;
        b.log_decay = (const float*)dec + 2 * sb.heads;
    }
    // outputs
    L.mixed_off = sa.heads * a.ep;
    L.mixed_ld = L.mixed_off + round8(inner);
    const PackMap heads{sa.vdim, a.ep, 0, 0};
    if (L.s.combine == Combine::Normed) {
        LC_TRY(model_gain_f32(m, pl + "out", W, &L.out_norm[0]));
        LC_TRY(model_gain_f32(m, pr + "out", W, &L.out_norm[1]));
        if (2 * L.mixed_off == L.mixed_ld) {  // rows of equal length: one batch of two
            LC_TRY(talloc(st, &d, (size_t)W * L.mixed_ld * 2));
            DevTensor* t = nullptr;
            LC_TRY(matrix(m, pl + "o", W, sa.heads * sa.vdim, &t));
            LC_TRY(launch_pack((const bf16*)t->view, W, sa.heads * sa.vdim, (bf16*)d, L.mixed_off, PackMap(), heads, false, m->stream));
            LC_TRY(matrix(m, pr + "o", W, inner, &t));
            LC_TRY(launch_pack((const bf16*)t->view, W, inner, (bf16*)d + (size_t)W * L.mixed_off, L.mixed_off, PackMap(), PackMap(), false, m->stream));
            return dense_weight_init(&L.out, (const bf16*)d, W, L.mixed_off, L.mixed_off, 2, (size_t)W * L.mixed_off);
        }
        LC_TRY(plain_weight(m, pl + "o", W, sa.heads * sa.vdim, &L.out, heads, L.mixed_off));
        return plain_weight(m, pr + "o", W, inner, &L.out2);
    }
    LC_TRY(talloc(st, &d, (size_t)W * L.mixed_ld * 2));
    DevTensor* t = nullptr;
    LC_TRY(matrix(m, pl + "o", W, sa.heads * sa.vdim, &t));
    LC_TRY(launch_pack((const bf16*)t->view, W, sa.heads * sa.vdim, (bf16*)d, L.mixed_ld, PackMap(), heads, false, m->stream));
    LC_TRY(matrix(m, pr + "o", W, inner, &t));
    LC_TRY(launch_pack((const bf16*)t->view, W, inner, (bf16*)d + L.mixed_off, L.mixed_ld, PackMap(), PackMap(), false, m->stream));
    return dense_weight_init(&L.out, (const bf16*)d, W, L.mixed_ld, L.mixed_ld);
}

// The experts' matrices `parts` [n, k] as one batch; several parts: their rows in turn.
int32_t expert_weights(lc_model* m, const std::string& p, const std::vector<const char*>& parts, int experts, int n, int k, DenseWeight* w) {
    const int ld = round8(k), np = (int)parts.size();
    const size_t each = (size_t)np * n * ld;
    void* d = nullptr;
    LC_TRY(talloc(*m->stack, &d, experts * each * 2));
    for (int e = 0; e < experts; e++)
        for (int i = 0; i < np; i++) {
            DevTensor* t = nullptr;
            LC_TRY(matrix(m, p + "e" + std::to_string(e) + "." + parts[i], n, k, &t));
            LC_TRY(launch_pack((const bf16*)t->view, n, k, (bf16*)d + e * each + (size_t)i * ld, ld, PackMap{1, np, 0, 0}, PackMap(), false, m->stream));
        }
    return dense_weight_init(w, (const bf16*)d, np * n, k, ld, experts, each);
}

int32_t bind_ffn(lc_model* m, StackLayer& L, const std::string& p) {
    LayerStack& st = *m->stack;
    const LayerSpec& s = L.s;
    const int W = st.spec.width, ld = round8(W);
    if (s.ffn == FfnKind::Relu2) {
        LC_TRY(plain_weight(m, p + "up", s.ff, W, &L.up));
        return plain_weight(m, p + "down", W, s.ff, &L.down);
    }
    if (s.ffn == FfnKind::GatedSilu || s.ffn == FfnKind::GatedGelu) {
        void* d = nullptr;
        LC_TRY(talloc(st, &d, (size_t)2 * s.ff * ld * 2));
        const char* part[2] = {"gate", "up"};
        for (int i = 0; i < 2; i++) {
            DevTensor* t = nullptr;
            LC_TRY(matrix(m, p + part[i], s.ff, W, &t));
            LC_TRY(launch_pack((const bf16*)t->view, s.ff, W, (bf16*)d + (size_t)i * ld, ld, PackMap{1, 2, 0, 0}, PackMap(), false, m->stream));
        }
        LC_TRY(dense_weight_init(&L.up, (const bf16*)d, 2 * s.ff, W, ld));
        return plain_weight(m, p + "down", W, s.ff, &L.down);
    }
    const MoeSpec& e = s.moe;
    std::vector<std::string> names = {p + "router"};
    std::vector<int> rows = {e.outputs()}, offs;
    if (e.shared_ff) {
        names.insert(names.end(), {p + "shared.sg", p + "shared.up"});
        rows.insert(rows.end(), {1, e.shared_ff});
        LC_TRY(plain_weight(m, p + "shared.down", W, e.shared_ff, &L.shared_down));
    }
    LC_TRY(fused_weight(m, names, rows, W, &L.route, &offs, e.shared_ff ? 32 : 8));
    L.off_gate = e.shared_ff ? offs[1] : 0;
    L.route_split = e.shared_ff ? offs[2] : (L.route.n + 31) / 32 * 32;
    LC_TRY(model_gain_f32(m, p + "correction", e.outputs(), &L.correction));
    LC_TRY(expert_weights(m, p, e.gated ? std::vector<const char*>{"gate", "up"} : std::vector<const char*>{"up"}, e.experts, e.ff, W, &L.up));
    LC_TRY(expert_weights(m, p, {"down"}, e.experts, W, e.ff, &L.down));
    L.expert_bytes = (uint64_t)(e.gated ? 3 : 2) * e.ff * W * 2;
    m->expert_bytes_all += L.expert_bytes * e.experts;
    m->expert_bytes_each = 1;  // d_moe_touched counts bytes
    return LC_OK;
}

size_t elt(const LayerStack& st) { return st.f32 ? 4 : 2; }

int32_t product(lc_model* m, const DenseWeight& w, const void* x, int ldx, int T, void* out, int ldo, bool out_f32 = false, DenseEpilogue epi = DENSE_STORE,
                DenseArgs extra = DenseArgs()) {
    LayerStack& st = *m->stack;
    DenseArgs a = extra;
    a.w = &w; a.x = x; a.ldx = ldx; a.x_rows = a.x_rows ? a.x_rows : m->t_cap; a.T = T; a.out = out; a.ldo = ldo; a.out_f32 = out_f32; a.epi = epi; a.f32 = st.f32;
    m->launches_in_call += 1;
    return launch_dense(a, st.ws, m->stream);
}
const void* at(const LayerStack& st, const void* base, size_t elems) { return (const uint8_t*)base + elems * elt(st); }

int32_t delta_block(lc_model* m, MixerUnit& L, const void* x, int ldx, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    const MixerSpec& s = L.s;
    const int nd = s.heads * s.dim, nv = s.heads * s.vdim;
    LC_TRY(product(m, L.in, x, ldx, T, st.proj, L.in.n));
    DenseArgs e;
    e.e0 = L.a_exp; e.e1 = L.dt_bias; e.e_div = s.dim;
    LC_TRY(product(m, L.a2, at(st, st.proj, (size_t)L.off_a), L.in.n, T, st.log_decay, nd, true, DENSE_LOG_DECAY, e));
    LC_TRY(product(m, L.g2, at(st, st.proj, (size_t)L.off_g), L.in.n, T, st.gate, nv));
    DeltaArgs d;
    d.g = L.dg; d.proj = st.proj; d.conv = L.conv; d.ring = L.ring; d.state = L.state; d.tok_seq = m->d_tok_seq; d.tok_pos = m->d_tok_pos; d.T = T;
    d.qk = st.qk; d.v = st.v; d.log_decay = st.log_decay; d.o = st.o; d.norm_w = L.o_norm; d.gate = st.gate;
    d.out = st.mixed; d.ldo = round8(nv); d.f32 = st.f32;
    if (decode_step) {
        LC_TRY(launch_delta_step(d, m->stream));
        m->launches_in_call += 1;
    } else {
        LC_TRY(launch_delta_prep(d, m->stream));
        d.runs = st.d_short_runs; d.n_runs = st.n_short_runs;
        d.chunks = st.d_chunks; d.n_chunks = st.n_chunks; d.chunk_runs = st.d_chunk_runs; d.n_chunk_runs = st.n_chunk_runs;
        if (d.n_runs) LC_TRY(launch_delta_scan(d, m->stream));
        if (d.n_chunk_runs) LC_TRY(launch_delta_chunks(d, (float*)st.chunk_scratch.p, m->stream));
        HeadNormArgs o;
        o.o = st.o; o.heads = s.heads; o.n = s.vdim; o.T = T; o.eps = st.spec.eps; o.w = L.o_norm; o.gate = st.gate; o.ld_gate = nv; o.out = st.mixed; o.ldo = d.ldo; o.f32 = st.f32;
        LC_TRY(launch_head_norm(o, m->stream));
        m->launches_in_call += 2 + (d.n_runs ? 1 : 0) + (d.n_chunk_runs ? 2 : 0);
    }
    return product(m, L.out, st.mixed, d.ldo, T, st.y, st.spec.width, true);
}

int32_t general_delta_block(lc_model* m, MixerUnit& L, const void* x, int ldx, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    const MixerSpec& s = L.s;
    const int n = s.heads * s.dim, ld_act = L.in.n - L.in_split;
    DenseArgs in, e;
    in.split = L.in_split; in.act_end = L.act_end; in.out2 = st.proj; in.ldo2 = ld_act;
    LC_TRY(product(m, L.in, x, ldx, T, st.projf, L.in_split, true, DENSE_SPLIT_TANH, in));
    e.e1 = L.dt_bias; e.scale = (float)s.decay_scale;
    LC_TRY(product(m, L.a2, st.proj, ld_act, T, st.log_decay, n, true, DENSE_SIGMOID_DECAY, e));
    GeneralArgs d;
    d.g = L.gg; d.proj = st.projf; d.a_bias = L.a_bias; d.log_decay = st.log_decay; d.state = L.state; d.tok_seq = m->d_tok_seq; d.tok_pos = m->d_tok_pos; d.T = T; d.o = st.o;
    d.norm_w = L.o_norm; d.gate = at(st, st.proj, (size_t)L.off_g); d.ld_gate = ld_act; d.out = st.mixed; d.ldo = round8(n); d.f32 = st.f32;
    if (decode_step) {
        LC_TRY(launch_general_step(d, m->stream));
        m->launches_in_call += 1;
    } else {
        d.runs = st.d_short_runs; d.n_runs = st.n_short_runs;
        d.chunks = st.d_chunks; d.n_chunks = st.n_chunks; d.chunk_runs = st.d_chunk_runs; d.n_chunk_runs = st.n_chunk_runs;
        if (d.n_runs) LC_TRY(launch_general_scan(d, m->stream));
        if (d.n_chunk_runs) LC_TRY(launch_general_chunks(d, (float*)st.chunk_scratch.p, m->stream));
        if (d.n_runs) {  // the chunks norm and gate their own tokens
            HeadNormArgs o;
            if (d.n_chunk_runs) { o.runs = d.runs; o.n_runs = d.n_runs; o.longest = st.longest_short; }
            o.o = st.o; o.heads = s.heads; o.n = s.dim; o.T = T; o.eps = st.spec.eps; o.w = L.o_norm; o.w_stride = s.dim; o.gate = d.gate; o.ld_gate = ld_act; o.out = st.mixed;
            o.ldo = d.ldo; o.f32 = st.f32;
            LC_TRY(launch_head_norm(o, m->stream));
        }
        m->launches_in_call += (d.n_runs ? 2 : 0) + (d.n_chunk_runs ? 3 : 0);
    }
    return product(m, L.out, st.mixed, d.ldo, T, st.y, st.spec.width, true);
}

int32_t latent_block(lc_model* m, MixerUnit& L, const void* x, int ldx, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    const LatentShape& g = L.lg;
    LC_TRY(product(m, L.in, x, ldx, T, st.projf, L.in.n, true));
    LatentArgs a;
    a.g = g; a.proj = st.projf; a.ld_proj = L.in.n; a.q_rank = L.s.q_rank; a.off_c = L.off_c; a.off_r = L.off_r; a.q_norm = L.q_norm; a.c_norm = L.c_norm;
    a.eps = st.spec.eps; a.rot = L.rot; a.cq = st.cq; a.ld_cq = round8(L.s.q_rank); a.cache = L.cache; a.page_tokens = m->page_tokens; a.page_table = m->d_page_table;
    a.tok_seq = m->d_tok_seq; a.tok_pos = m->d_tok_pos; a.pages_per_seq = m->pages_per_seq; a.T = T; a.q = st.q; a.q_abs = st.q_abs; a.o = st.o_lat; a.f32 = st.f32;
    LC_TRY(launch_latent_prep(a, m->stream));
    m->launches_in_call += 1;
    const int ldq = g.heads * g.ld_q, ldc = g.heads * g.cp, lde = g.heads * L.ep;
    LC_TRY(product(m, L.uq, st.cq, a.ld_cq, T, st.q, ldq));
    const int few = decode_step || !st.prefill_tiles ? T : st.n_short;
    if (few > 0) {
        DenseArgs b;
        b.x_batch = (size_t)g.ld_q; b.out_batch = (size_t)g.cp;
        LC_TRY(product(m, L.uk_t, st.q, ldq, few, st.q_abs, ldc, false, DENSE_STORE, b));
        a.T = few;
        int launches = 0;
        LC_TRY(launch_latent_attention(a, st.pieces, st.pieces_bytes, &launches, m->stream));
        m->launches_in_call += launches;
        b.x_batch = (size_t)g.cp; b.out_batch = (size_t)L.ep;
        LC_TRY(product(m, L.uv, st.o_lat, ldc, few, st.mixed, lde, false, DENSE_STORE, b));
    }
    if (few < T)
        for (const LayerStack::Group& gr : st.groups) {
            LC_TRY(launch_latent_gather(a, st.d_lat_ctx + gr.ctx0, gr.n_ctx, gr.longest, st.ctx_c.p, m->stream));
            DenseArgs c;
            c.x_rows = gr.rows;
            LC_TRY(product(m, L.uk_all, st.ctx_c.p, g.cp + g.rp, gr.rows, st.ctx_k.p, g.heads * g.dp, false, DENSE_STORE, c));
            LC_TRY(product(m, L.uv_all, st.ctx_c.p, g.cp + g.rp, gr.rows, st.ctx_v.p, lde, false, DENSE_STORE, c));
            LatentPrefill p;
            p.tiles = st.d_lat_tiles + gr.tile0; p.c = st.ctx_c.p; p.k = st.ctx_k.p; p.v = st.ctx_v.p; p.out = st.mixed; p.ep = L.ep;
            LC_TRY(launch_latent_prefill(a, p, gr.n_tiles, m->stream));
            m->launches_in_call += 2;
        }
    return product(m, L.out, st.mixed, lde, T, st.y, st.spec.width, true);
}

// Preparation and attention of `a`'s tokens; the caller has set where they come from and where the output goes.
int32_t attend(lc_model* m, const MixerUnit& L, const MixerUnit& src, AttnArgs a, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    a.g = L.ag; a.proj = st.projf; a.off_k = L.off_k; a.off_v = L.off_v; a.q_norm = L.q_norm; a.k_norm = L.k_norm; a.eps = st.spec.eps; a.rot = L.rot;
    a.conv = L.conv; a.ring = (float*)L.ring; a.one_each = decode_step;
    a.q = st.q; a.k_cache = src.k_cache; a.v_cache = src.v_cache; a.page_tokens = m->page_tokens; a.page_table = m->d_page_table; a.tok_seq = m->d_tok_seq;
    a.tok_pos = m->d_tok_pos; a.pages_per_seq = m->pages_per_seq; a.T = T; a.sink = L.sink; a.f32 = st.f32;
    a.q_factor = L.q_factor; a.head_gate = L.off_hg >= 0 ? st.projf + L.off_hg : nullptr;
    LC_TRY(launch_attn_prep(a, m->stream));
    m->launches_in_call += 1;
    if (L.ag.taps > 0 && !decode_step) {
        LC_TRY(launch_attn_keep(a, st.d_runs, st.n_runs, m->stream));
        m->launches_in_call += 1;
    }
    const int few = decode_step || !st.prefill_tiles ? T : st.n_short;
    a.T = few;
    if (few > 0) {
        LC_TRY(launch_attn_tokens(a, st.attn, m->stream));
        m->launches_in_call += 1;
    }
    if (few < T) {
        LC_TRY(launch_attn_tiles(a, st.d_attn_tiles, st.n_attn_tiles, m->stream));
        m->launches_in_call += 1;
    }
    return LC_OK;
}

int32_t attention_block(lc_model* m, MixerUnit& L, const void* x, int ldx, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    DenseArgs in, out;
    in.e1 = L.in_bias; out.e1 = L.out_bias;
    LC_TRY(product(m, L.in, x, ldx, T, st.projf, L.in.n, true, L.in_bias ? DENSE_BIAS : DENSE_STORE, in));
    AttnArgs a;
    a.ld_proj = L.in.n; a.out = st.mixed; a.ldo = L.ag.heads * L.ep;
    LC_TRY(attend(m, L, L.s.kv_from < 0 ? L : st.layers[(size_t)L.s.kv_from].mix[0], a, T, decode_step));
    return product(m, L.out, st.mixed, a.ldo, T, st.y, st.spec.width, true, L.out_bias ? DENSE_BIAS : DENSE_STORE, out);
}

int32_t recur(lc_model* m, const MixerUnit& L, LinearArgs a, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    a.g = L.ng; a.proj = st.proj; a.dt = st.projf; a.conv = L.conv; a.conv_b = L.conv_b; a.dt_bias = L.dt_bias; a.a_exp = L.a_exp; a.skip = L.skip; a.log_decay = L.log_decay; a.decay = L.decay;
    a.ring = L.ring; a.in = st.lin; a.state = L.state; a.tok_seq = m->d_tok_seq; a.tok_pos = m->d_tok_pos; a.T = T; a.o = st.o; a.norm_w = L.o_norm; a.f32 = st.f32;
    int launches = 1;
    if (decode_step) {
        LC_TRY(launch_linear_step(a, &launches, m->stream));
    } else {
        a.runs = st.d_short_runs; a.n_runs = st.n_short_runs; a.chunk_runs = st.d_chunk_runs; a.n_chunk_runs = st.n_chunk_runs; a.all_runs = st.d_runs; a.n_all_runs = st.n_runs;
        LC_TRY(launch_linear_runs(a, &launches, m->stream));
    }
    LC_TRY(launch_linear_output(a, m->stream));
    m->launches_in_call += launches;
    return LC_OK;
}

// Attention and a linear recurrence side by side; Normed: their outputs in y and y2.
int32_t pair_block(lc_model* m, StackLayer& L, const void* x, int ldx, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    DenseArgs in;
    const int ld_act = L.in.n - L.in_split;
    in.split = L.in_split; in.act_end = L.act_end; in.out2 = st.proj; in.ldo2 = ld_act;
    LC_TRY(product(m, L.in, x, ldx, T, st.projf, L.in_split, true, DENSE_SPLIT_SILU, in));
    const bool normed = L.s.combine == Combine::Normed;
    AttnArgs a;
    a.ld_proj = L.in_split; a.out = st.mixed; a.ldo = L.mixed_ld; a.out_scale = normed ? 1.0f : L.s.mix_scale[0];
    if (L.s.mix[0].out_gate) { a.gate = at(st, st.proj, (size_t)L.mix[0].off_g); a.ld_gate = ld_act; }
    LC_TRY(attend(m, L.mix[0], L.mix[0], a, T, decode_step));
    LinearArgs b;
    b.out = (void*)at(st, st.mixed, (size_t)L.mixed_off); b.ldo = L.mixed_ld; b.out_scale = normed ? 1.0f : L.s.mix_scale[1];
    LC_TRY(recur(m, L.mix[1], b, T, decode_step));
    if (normed && L.out.batch == 2) {
        DenseArgs o;
        o.x_batch = (size_t)L.mixed_off; o.out_batch = (size_t)m->t_cap * st.spec.width;
        return product(m, L.out, st.mixed, L.mixed_ld, T, st.y, st.spec.width, true, DENSE_STORE, o);
    }
    LC_TRY(product(m, L.out, st.mixed, L.mixed_ld, T, st.y, st.spec.width, true));
    return normed ? product(m, L.out2, b.out, L.mixed_ld, T, st.y2, st.spec.width, true) : LC_OK;
}

// x += norm(proj(gelu(gate x) * the layer's part of the token's row)): the two products; x as activations is in `xa`.
int32_t side_block(lc_model* m, int l, int T) {
    LayerStack& st = *m->stack;
    const StackLayer& L = st.layers[(size_t)l];
    const int n = st.spec.side_dim, ld = round8(n);
    DenseArgs e;
    e.table = st.side_embed + (size_t)l * n; e.table_ld = (int)st.layers.size() * n; e.table_rows = st.spec.vocab; e.ids = m->d_tokens;
    LC_TRY(product(m, L.side_gate, st.xa, st.width_p, T, st.side, ld, false, DENSE_GELU_TABLE, e));
    return product(m, L.side_proj, st.side, ld, T, st.y, st.spec.width, true);
}

// What the residual sum (or a probe) needs to finish the mixture's output.
MoeSum moe_sum(const LayerStack& st, const StackLayer& L, const void* x, int ldx) {
    const MoeSpec& e = L.s.moe;
    MoeSum r;
    r.rows = st.moe_rows; r.ld_rows = round8(st.spec.width); r.sel = st.moe_sel; r.pos = st.moe_pos; r.off = st.plan.off; r.weight = st.moe_w; r.top = e.top; r.experts = e.experts;
    r.h = x; r.ld_h = ldx;
    if (e.shared_ff) { r.gate = st.moe_z + L.off_gate; r.ld_gate = L.route_split; }
    return r;
}

PairSum pair_sum(const LayerStack& st, const StackLayer& L) {
    PairSum r;
    r.y2 = st.y2; r.w0 = L.out_norm[0]; r.w1 = L.out_norm[1];
    return r;
}

int32_t moe_block(lc_model* m, StackLayer& L, const void* x, int ldx, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    const MoeSpec& e = L.s.moe;
    DenseArgs r;
    const int ldf = round8(e.ff), lds = round8(e.shared_ff);
    r.split = L.route_split; r.out2 = st.ffn; r.ldo2 = lds;
    LC_TRY(product(m, L.route, x, ldx, T, st.moe_z, L.route_split, true, DENSE_SPLIT_RELU2, r));
    ExpertPlan plan = st.plan;
    // tiles that hold the usual expert's tokens
    const int usual = (T * e.top + e.outputs() - 1) / e.outputs();
    plan.tile_rows = usual <= 12 ? 16 : usual <= 24 ? 32 : usual <= 48 ? 64 : usual <= 96 ? 128 : 256;
    plan.most_rows = T * e.top;
    plan.most_tiles = std::min(st.plan_tiles, std::min(plan.most_rows, e.experts + plan.most_rows / plan.tile_rows));
    ChoiceArgs c;
    c.m = e; c.z = st.moe_z; c.ld_z = L.route_split; c.T = T; c.correction = L.correction; c.sel = st.moe_sel; c.pos = st.moe_pos; c.weight = st.moe_w; c.counts = st.moe_counts;
    c.plan = plan; c.touched = decode_step ? m->d_moe_touched : nullptr; c.touched_bytes = L.expert_bytes;
    LC_TRY(launch_expert_choice(c, m->stream));
    m->launches_in_call += 1;
    DenseArgs g;
    g.plan = &plan; g.gather = true;
    const void* in = x;
    int ld_in = ldx;
    if (!st.f32 && plan.tile_rows > kGatheredRows) {
        in = st.moe_in; ld_in = st.width_p;
        LC_TRY(launch_expert_gather(moe_sum(st, L, x, ldx), st.spec.width, T, st.moe_in, ld_in, m->stream));
        m->launches_in_call += 1;
        g.gather = false; g.x_rows = st.moe_slots;
    }
    LC_TRY(product(m, L.up, in, ld_in, T, st.moe_up, ldf, false, e.gated ? DENSE_GATED_SILU : DENSE_RELU2, g));
    if (e.shared_ff) LC_TRY(product(m, L.shared_down, st.ffn, lds, T, st.y, st.spec.width, true));
    g.gather = false; g.x_rows = st.moe_slots;
    return product(m, L.down, st.moe_up, ldf, T, st.moe_rows, round8(st.spec.width), false, DENSE_STORE, g);
}

int32_t ffn_block(lc_model* m, StackLayer& L, const void* x, int ldx, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    if (L.s.ffn == FfnKind::Moe) return moe_block(m, L, x, ldx, T, decode_step);
    const int ldf = round8(L.s.ff);
    LC_TRY(product(m, L.up, x, ldx, T, st.ffn, ldf, false, L.s.ffn == FfnKind::GatedSilu ? DENSE_GATED_SILU : L.s.ffn == FfnKind::GatedGelu ? DENSE_GATED_GELU : DENSE_RELU2));
    return product(m, L.down, st.ffn, ldf, T, st.y, st.spec.width, true);
}

// The layers' input: the residual itself in f32 models without norms on inputs, else the activations made from it.
const void* layer_input(lc_model* m, int* ld) {
    LayerStack& st = *m->stack;
    *ld = st.xa ? st.width_p : st.spec.width;
    return st.xa ? st.xa : (const void*)m->d_hidden;
}

}  // namespace

int32_t stack_bind(lc_model* m) {
    LayerStack& st = *m->stack;
    const ArchSpec& sp = st.spec;
    LC_TRY(dense_workspace_alloc(&st.ws));
    st.layers.resize(sp.layers.size());
    for (size_t i = 0; i < sp.layers.size(); i++) {
        StackLayer& L = st.layers[i];
        L.s = sp.layers[i];
        const std::string p = "l" + std::to_string(i) + ".";
        for (int j = 0; j < L.s.mixers(); j++) L.mix[j].s = L.s.mix[j];
        MixerUnit& u = L.mix[0];
        if (L.s.combine != Combine::Single) LC_TRY(bind_pair(m, L, p + "mix."));
        else if (u.s.kind == MixerKind::ChannelDelta) LC_TRY(bind_delta(m, u, p + "mix."));
        else if (u.s.kind == MixerKind::LatentAttention) LC_TRY(bind_latent(m, u, p + "mix."));
        else if (u.s.kind == MixerKind::GeneralDelta) LC_TRY(bind_general_delta(m, u, p + "mix."));
        else LC_TRY(bind_attention(m, u, p + "mix."));
        auto norms = [&](const std::string& name, const float** in, const float** out) -> int32_t {
            if (sp.norm_inputs) LC_TRY(norm_gain(m, name, in));
            if (!sp.norm_outputs) return LC_OK;
            return norm_gain(m, sp.norm_inputs ? name + "b" : name, out);
        };
        LC_TRY(norms(p + "norm1", &L.norm1_in, &L.norm1_out));
        if (L.s.ffn != FfnKind::None) {
            LC_TRY(bind_ffn(m, L, p + "mlp."));
            LC_TRY(norms(p + "norm2", &L.norm2_in, &L.norm2_out));
        }
        if (sp.depth_average) LC_TRY(model_gain_f32(m, p + "dwa", (int)i + 2, &L.dwa));
        if (sp.side_dim) {
            LC_TRY(plain_weight(m, p + "side.gate", sp.side_dim, sp.width, &L.side_gate));
            LC_TRY(plain_weight(m, p + "side.proj", sp.width, sp.side_dim, &L.side_proj));
            LC_TRY(model_gain_f32(m, p + "side.norm", sp.width, &L.side_norm));
        }
        LC_TRY(block_weights(m, {&u.in, &u.out, &u.a2, &u.g2, &u.uq, &u.uk_t, &u.uv, &u.uk_all, &u.uv_all, &L.in, &L.out, &L.out2, &L.up, &L.down, &L.route, &L.shared_down,
                                 &L.side_gate, &L.side_proj}));
    }
    DevTensor* e = nullptr;
    LC_TRY(matrix(m, "embed", sp.vocab, sp.width, &e));
    st.embed = (const bf16*)e->view;
    m->embed = e;
    if (sp.side_dim) {
        LC_TRY(matrix(m, "side.embed", sp.vocab, (int)sp.layers.size() * sp.side_dim, &e));
        st.side_embed = (const bf16*)e->view;
    }
    if (sp.bigram.buckets) {
        LC_TRY(matrix(m, "bigram", (int)sp.bigram.buckets + 1, sp.width, &e));
        st.bigram = (const bf16*)e->view;
    }
    st.packed.clear();  // the tables are read as they are
    LC_TRY(norm_gain(m, "final.norm", &st.final_norm));
    LC_TRY(plain_weight(m, "head", sp.vocab, sp.width, &st.head));
    return block_weights(m, {&st.head});
}

int32_t stack_alloc(lc_model* m) {
    LayerStack& st = *m->stack;
    const size_t T = (size_t)m->t_cap, e = elt(st);
    st.width_p = round8(st.spec.width);
    st.prefill_tiles = st.delta_chunks = !st.f32;
    int experts = 0, top = 0;
    size_t z = 0, hidden = 8, attn_part = 0;
    size_t proj = 8, projf = 8, gate = 8, mixed = 8, cq = 8, q = 8, qa = 8, ffn = 8, ld = 8, qk = 8, v = 8;
    size_t lin = 0;
    auto alloc_mixer = [&](MixerUnit& L) -> int32_t {
        const MixerSpec& s = L.s;
        if (s.kind == MixerKind::ChannelDelta) {
            const size_t nv = (size_t)s.heads * s.vdim, S = (size_t)s.heads * s.dim * s.vdim, ring = (size_t)s.conv_taps * L.dg.channels;
            proj = std::max(proj, (size_t)L.in.n);
            gate = std::max(gate, nv);
            mixed = std::max(mixed, (size_t)round8((int)nv));
            ld = std::max(ld, (size_t)s.heads * s.dim);
            qk = std::max(qk, (size_t)2 * s.kv_heads * s.dim);
            v = std::max(v, nv);
            LC_TRY(zalloc(st, (void**)&L.state, (size_t)m->max_seqs * S * 4));
            LC_TRY(zalloc(st, &L.ring, (size_t)m->max_seqs * ring * e));
            st.delta_chunks = st.delta_chunks && delta_chunks_apply(L.dg, st.f32);
            st.chunk_bytes = std::max(st.chunk_bytes, delta_chunk_bytes(L.dg));
            st.state_bytes_per_seq += S * 4 + ring * e;
        } else if (s.kind == MixerKind::GeneralDelta) {
            const size_t n = (size_t)s.heads * s.dim, S = n * s.dim;
            proj = std::max(proj, (size_t)(L.in.n - L.in_split));
            projf = std::max(projf, (size_t)L.in_split);
            mixed = std::max(mixed, (size_t)round8((int)n));
            ld = std::max(ld, n);
            v = std::max(v, n);
            LC_TRY(zalloc(st, (void**)&L.state, (size_t)m->max_seqs * S * 4));
            st.delta_chunks = st.delta_chunks && general_chunks_apply(L.gg, s.decay_scale, st.f32);
            st.chunk_bytes = std::max(st.chunk_bytes, general_chunk_bytes(L.gg));
            st.state_bytes_per_seq += S * 4;
        } else if (s.kind == MixerKind::Attention) {
            const AttnShape& g = L.ag;
            projf = std::max(projf, (size_t)L.in.n);
            q = std::max(q, (size_t)g.heads * g.dp);
            mixed = std::max(mixed, (size_t)g.heads * g.ep);
            st.prefill_tiles = st.prefill_tiles && attn_tiles_apply(g, st.f32);
            attn_part = std::max(attn_part, attn_part_bytes(g));
            if (g.taps) {
                const size_t ring = (size_t)g.taps * ((g.heads + g.kv_heads) * g.dim + g.kv_heads * g.vdim);
                LC_TRY(zalloc(st, &L.ring, (size_t)m->max_seqs * ring * 4));
                st.state_bytes_per_seq += ring * 4;
            }
            if (s.kv_from < 0) {
                const size_t rows = (size_t)m->pages_total * m->page_tokens * g.kv_heads;
                LC_TRY(zalloc(st, &L.k_cache, rows * g.k_pitch * e));
                LC_TRY(zalloc(st, &L.v_cache, rows * g.v_pitch * e));
                st.cache_bytes_per_token += (size_t)g.kv_heads * (g.k_pitch + g.v_pitch) * e;
            }
        } else if (s.kind == MixerKind::LinearState) {
            const LinearShape& g = L.ng;
            const size_t S = (size_t)g.heads * g.dim * g.vdim, ring = (size_t)g.taps * g.channels;
            v = std::max(v, (size_t)g.heads * g.vdim);
            lin = std::max(lin, (size_t)g.ld_in);
            LC_TRY(zalloc(st, (void**)&L.state, (size_t)m->max_seqs * S * 4));
            if (ring) LC_TRY(zalloc(st, &L.ring, (size_t)m->max_seqs * ring * e));
            st.delta_chunks = st.delta_chunks && linear_chunks_apply(g, st.f32);
            st.state_bytes_per_seq += S * 4 + ring * e;
        } else {
            const LatentShape& g = L.lg;
            projf = std::max(projf, (size_t)L.in.n);
            cq = std::max(cq, (size_t)round8(s.q_rank));
            q = std::max(q, (size_t)g.heads * g.ld_q);
            qa = std::max(qa, (size_t)g.heads * g.cp);
            mixed = std::max(mixed, (size_t)g.heads * L.ep);
            const size_t row = (size_t)(g.cp + g.rp) * e;
            st.prefill_tiles = st.prefill_tiles && latent_prefill_applies(g, L.ep, st.f32);
            st.ctx_c_row = std::max(st.ctx_c_row, (size_t)(g.cp + g.rp));
            st.ctx_k_row = std::max(st.ctx_k_row, (size_t)g.heads * g.dp);
            st.ctx_v_row = std::max(st.ctx_v_row, (size_t)g.heads * L.ep);
            st.pieces_bytes = std::max(st.pieces_bytes, latent_pieces_bytes(g, m->max_seqs));
            LC_TRY(zalloc(st, &L.cache, (size_t)m->pages_total * m->page_tokens * row));
            st.cache_bytes_per_token += row;
        }
        return LC_OK;
    };
    bool pairs = false;
    for (StackLayer& L : st.layers) {
        const LayerSpec& ls = L.s;
        for (int j = 0; j < ls.mixers(); j++) LC_TRY(alloc_mixer(L.mix[j]));
        if (ls.combine != Combine::Single) {
            proj = std::max(proj, (size_t)(L.in.n - L.in_split));
            projf = std::max(projf, (size_t)L.in_split);
            mixed = std::max(mixed, (size_t)L.mixed_ld);
            pairs = pairs || ls.combine == Combine::Normed;
        }
        if (ls.ffn == FfnKind::Moe) {
            experts = std::max(experts, ls.moe.experts); top = std::max(top, ls.moe.top);
            z = std::max(z, (size_t)L.route_split);
            hidden = std::max(hidden, (size_t)round8(ls.moe.ff));
            ffn = std::max(ffn, (size_t)round8(ls.moe.shared_ff));
        } else if (ls.ffn != FfnKind::None) ffn = std::max(ffn, (size_t)round8(ls.ff));
    }
    if (experts) {
        st.moe_slots = (int)T * top;
        st.plan_tiles = experts + st.moe_slots / 16;
        LC_TRY(zalloc(st, (void**)&st.moe_z, T * z * 4)); LC_TRY(zalloc(st, (void**)&st.moe_w, T * top * 4));
        LC_TRY(zalloc(st, (void**)&st.moe_sel, T * top * 4)); LC_TRY(zalloc(st, (void**)&st.moe_pos, T * top * 4));
        LC_TRY(zalloc(st, (void**)&st.moe_counts, ((size_t)experts + 1) * 4));
        LC_TRY(zalloc(st, &st.moe_up, (size_t)st.moe_slots * hidden * e)); LC_TRY(zalloc(st, &st.moe_rows, (size_t)st.moe_slots * st.width_p * e));
        if (!st.f32) LC_TRY(zalloc(st, &st.moe_in, (size_t)st.moe_slots * st.width_p * e));
        LC_TRY(zalloc(st, (void**)&st.plan.tiles, (size_t)st.plan_tiles * sizeof(ExpertTile))); LC_TRY(zalloc(st, (void**)&st.plan.n_tiles, 4));
        LC_TRY(zalloc(st, (void**)&st.plan.off, ((size_t)experts + 1) * 4)); LC_TRY(zalloc(st, (void**)&st.plan.lists, (size_t)experts * T * 4));
        st.plan.list_stride = (int)T;
        LC_TRY(dalloc(&m->d_moe_touched, 1));
        LC_CUDA(cudaMemsetAsync(m->d_moe_touched, 0, 8, m->stream));
    }
    if (attn_part) {
        st.attn.part_bytes = attn_part;
        st.attn.n_tickets = 12 * sm_count();
        LC_TRY(zalloc(st, (void**)&st.attn.part, attn_part)); LC_TRY(zalloc(st, (void**)&st.attn.tickets, (size_t)st.attn.n_tickets * 4));
        LC_TRY(zalloc(st, (void**)&st.d_attn_tiles, T * sizeof(AttnTile)));
    }
    if (!st.f32 || st.spec.norm_inputs) LC_TRY(zalloc(st, &st.xa, T * st.width_p * e));
    LC_TRY(zalloc(st, &st.proj, T * proj * e)); LC_TRY(zalloc(st, (void**)&st.projf, T * projf * 4));
    LC_TRY(zalloc(st, &st.gate, T * gate * e)); LC_TRY(zalloc(st, &st.mixed, T * mixed * e));
    LC_TRY(zalloc(st, &st.cq, T * cq * e)); LC_TRY(zalloc(st, &st.q, T * q * e));
    LC_TRY(zalloc(st, &st.q_abs, T * qa * e)); LC_TRY(zalloc(st, &st.o_lat, T * qa * e));
    LC_TRY(zalloc(st, &st.ffn, T * ffn * e)); LC_TRY(zalloc(st, &st.last, (size_t)m->head_rows * st.width_p * e));
    if (lin) LC_TRY(zalloc(st, &st.lin, T * lin * e));
    if (st.bigram) LC_TRY(zalloc(st, (void**)&st.last_token, (size_t)m->max_seqs * 4));
    if (st.spec.depth_average) LC_TRY(zalloc(st, (void**)&st.depth, (st.layers.size() + 1) * T * st.spec.width * 4));
    if (st.spec.side_dim) LC_TRY(zalloc(st, &st.side, T * round8(st.spec.side_dim) * e));
    LC_TRY(zalloc(st, (void**)&st.y, (pairs ? 2 : 1) * T * st.spec.width * 4));
    if (pairs) st.y2 = st.y + T * st.spec.width;
    LC_TRY(zalloc(st, (void**)&st.log_decay, T * ld * 4));
    LC_TRY(zalloc(st, (void**)&st.qk, T * qk * 4)); LC_TRY(zalloc(st, (void**)&st.v, T * v * 4)); LC_TRY(zalloc(st, (void**)&st.o, T * v * 4));
    LC_TRY(zalloc(st, (void**)&st.d_runs, T * sizeof(SeqRun)));
    LC_TRY(zalloc(st, (void**)&st.d_short_runs, T * sizeof(SeqRun))); LC_TRY(zalloc(st, (void**)&st.d_chunks, T * sizeof(DeltaChunk)));
    LC_TRY(zalloc(st, (void**)&st.d_chunk_runs, T * sizeof(DeltaChunkRun)));
    LC_TRY(zalloc(st, (void**)&st.d_lat_tiles, T * sizeof(LatentTile))); LC_TRY(zalloc(st, (void**)&st.d_lat_ctx, T * sizeof(LatentContext)));
    if (st.pieces_bytes) LC_TRY(zalloc(st, &st.pieces, st.pieces_bytes));
    return LC_OK;
}

void stack_free(lc_model* m) {
    if (!m->stack) return;
    for (void* p : m->stack->owned) cudaFree(p);
    for (void* p : m->stack->temps) cudaFree(p);
    for (DevBuf* b : {&m->stack->ctx_c, &m->stack->ctx_k, &m->stack->ctx_v, &m->stack->chunk_scratch}) b->release();
    dense_workspace_free(&m->stack->ws);
}

// Cache and state a one-token step at position `ctx` reads and writes.
uint64_t stack_step_bytes(const lc_model* m, int ctx) {
    const LayerStack& st = *m->stack;
    uint64_t b = 2 * st.state_bytes_per_seq + (uint64_t)st.layers.size() * st.spec.side_dim * 2 + (st.bigram ? (uint64_t)st.spec.width * 2 : 0);
    for (const StackLayer& layer : st.layers) {
        const MixerUnit& L = layer.mix[0];
        if (L.s.kind == MixerKind::LatentAttention) b += (uint64_t)(ctx + 1) * (L.lg.cp + L.lg.rp) * elt(st);
        if (L.s.kind != MixerKind::Attention) continue;
        const int window = L.ag.window > 0 ? L.ag.window : ctx + 1, lo = std::max(0, ctx + 1 - window), seen = ctx + 1 - lo + std::min(L.ag.keep_first, lo);
        b += (uint64_t)seen * L.ag.kv_heads * (L.ag.dp + L.ag.ep) * elt(st);
    }
    return b;
}

uint64_t stack_table_bytes(const lc_model* m) {
    const ArchSpec& sp = m->stack->spec;
    return (uint64_t)sp.vocab * sp.layers.size() * sp.side_dim * 2 + (sp.bigram.buckets ? (uint64_t)(sp.bigram.buckets + 1) * sp.width * 2 : 0);
}

// What a call's tokens mean to the layers: runs of consecutive positions, those of at least kTileRun tokens also as tiles
// over contexts of their own.  The caller orders the runs so that the short ones come first.
int32_t stack_upload_runs(lc_model* m, const std::vector<int32_t>& seq, const std::vector<int32_t>& pos) {
    LayerStack& st = *m->stack;
    std::vector<SeqRun> runs;
    for (size_t i = 0; i < seq.size(); i++) {
        if (runs.empty() || seq[i] != seq[i - 1] || pos[i] != pos[i - 1] + 1) runs.push_back(SeqRun{(int32_t)i, 0, seq[i], pos[i]});
        runs.back().n++;
    }
    st.n_runs = (int)runs.size();
    LC_CUDA(cudaMemcpyAsync(st.d_runs, runs.data(), runs.size() * sizeof(SeqRun), cudaMemcpyHostToDevice, m->stream));
    std::vector<SeqRun> shorts;
    std::vector<DeltaChunk> chunks;
    std::vector<DeltaChunkRun> chunk_runs;
    for (const SeqRun& r : runs) {
        if (!st.delta_chunks || r.n < kChunkRun) { shorts.push_back(r); continue; }
        chunk_runs.push_back(DeltaChunkRun{r, (int32_t)chunks.size(), (r.n + kDeltaChunk - 1) / kDeltaChunk});
        for (int t = 0; t < r.n; t += kDeltaChunk) chunks.push_back(DeltaChunk{r.tok0 + t, std::min(kDeltaChunk, r.n - t)});
    }
    st.longest_short = 0;
    for (const SeqRun& r : shorts) st.longest_short = std::max(st.longest_short, r.n);
    st.n_short_runs = (int)shorts.size(); st.n_chunks = (int)chunks.size(); st.n_chunk_runs = (int)chunk_runs.size();
    if (!shorts.empty()) LC_CUDA(cudaMemcpyAsync(st.d_short_runs, shorts.data(), shorts.size() * sizeof(SeqRun), cudaMemcpyHostToDevice, m->stream));
    if (!chunks.empty()) {
        LC_CUDA(cudaMemcpyAsync(st.d_chunks, chunks.data(), chunks.size() * sizeof(DeltaChunk), cudaMemcpyHostToDevice, m->stream));
        LC_CUDA(cudaMemcpyAsync(st.d_chunk_runs, chunk_runs.data(), chunk_runs.size() * sizeof(DeltaChunkRun), cudaMemcpyHostToDevice, m->stream));
        if (st.chunk_bytes) LC_TRY(st.chunk_scratch.reserve(std::max(chunks.size(), (size_t)m->t_cap / kDeltaChunk) * st.chunk_bytes));
    }
    st.groups.clear();
    st.n_short = (int)seq.size();
    st.n_attn_tiles = 0;
    std::vector<LatentTile> tiles;
    std::vector<LatentContext> ctx;
    size_t first = 0;
    while (first < runs.size() && runs[first].n < kTileRun) first++;
    if (st.prefill_tiles && first < runs.size()) st.n_short = runs[first].tok0;
    if (st.prefill_tiles && st.d_attn_tiles && first < runs.size()) {
        std::vector<AttnTile> at;
        for (size_t i = first; i < runs.size(); i++)
            for (int t = 0; t < runs[i].n; t += 64) at.push_back(AttnTile{runs[i].tok0 + t, std::min(64, runs[i].n - t), runs[i].seq, runs[i].pos0 + t});
        st.n_attn_tiles = (int)at.size();
        LC_CUDA(cudaMemcpyAsync(st.d_attn_tiles, at.data(), at.size() * sizeof(AttnTile), cudaMemcpyHostToDevice, m->stream));
        LC_CUDA(cudaStreamSynchronize(m->stream));
    }
    if (st.prefill_tiles && st.ctx_c_row && first < runs.size()) {
        int most = 0;
        for (size_t i = first; i < runs.size(); i++) {
            const SeqRun& r = runs[i];
            const int len = r.pos0 + r.n;
            if (st.groups.empty() || st.groups.back().rows + len > kContextRows) st.groups.push_back({(int)tiles.size(), 0, (int)ctx.size(), 0, 0, 0});
            LayerStack::Group& gr = st.groups.back();
            for (int t = 0; t < r.n; t += 64) { tiles.push_back(LatentTile{r.tok0 + t, std::min(64, r.n - t), r.pos0 + t, gr.rows}); gr.n_tiles++; }
            ctx.push_back(LatentContext{r.seq, len, gr.rows});
            gr.n_ctx++;
            gr.rows += len;
            gr.longest = std::max(gr.longest, len);
            most = std::max(most, gr.rows);
        }
        LC_CUDA(cudaMemcpyAsync(st.d_lat_tiles, tiles.data(), tiles.size() * sizeof(LatentTile), cudaMemcpyHostToDevice, m->stream));
        LC_CUDA(cudaMemcpyAsync(st.d_lat_ctx, ctx.data(), ctx.size() * sizeof(LatentContext), cudaMemcpyHostToDevice, m->stream));
        const size_t rows = (size_t)std::max(most, std::min(kContextRows, m->t_cap));
        LC_TRY(st.ctx_c.reserve(rows * st.ctx_c_row * 2));
        LC_TRY(st.ctx_k.reserve(rows * st.ctx_k_row * 2));
        LC_TRY(st.ctx_v.reserve(rows * st.ctx_v_row * 2));
    }
    LC_CUDA(cudaStreamSynchronize(m->stream));  // the copies read vectors that die with this frame
    return LC_OK;
}

int32_t stack_mixer(lc_model* m, int l, const void* x, int ldx, int T, bool decode_step) {
    StackLayer& L = m->stack->layers[l];
    if (L.s.combine != Combine::Single) return pair_block(m, L, x, ldx, T, decode_step);
    switch (L.mix[0].s.kind) {
        case MixerKind::ChannelDelta: return delta_block(m, L.mix[0], x, ldx, T, decode_step);
        case MixerKind::LatentAttention: return latent_block(m, L.mix[0], x, ldx, T, decode_step);
        case MixerKind::GeneralDelta: return general_delta_block(m, L.mix[0], x, ldx, T, decode_step);
        default: return attention_block(m, L.mix[0], x, ldx, T, decode_step);
    }
}

int32_t stack_run_layers(lc_model* m, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    const int W = st.spec.width;
    int ldx = 0;
    const void* x = layer_input(m, &ldx);
    EmbedArgs e;
    e.table = st.embed; e.rows = st.spec.vocab; e.width = W; e.T = T; e.ids = m->d_tokens; e.scale = st.spec.embed_scale; e.eps = st.spec.eps; e.w = st.layers[0].norm1_in;
    e.x = m->d_hidden; e.copy = st.depth; e.act = st.xa; e.ld_act = st.width_p; e.f32 = st.f32;
    e.pair.table = st.bigram; e.pair.rows = st.spec.bigram; e.pair.tok_seq = m->d_tok_seq; e.pair.tok_pos = m->d_tok_pos; e.pair.last = st.last_token; e.pair.one_each = decode_step;
    LC_TRY(launch_embed_rows(e, m->stream));
    m->launches_in_call += 1;
    if (st.bigram && !decode_step) {
        LC_TRY(launch_keep_tokens(st.d_runs, st.n_runs, m->d_tokens, st.last_token, m->stream));
        m->launches_in_call += 1;
    }
    const size_t plane = (size_t)m->t_cap * W;
    ResidualArgs r;
    r.y = st.y; r.eps = st.spec.eps; r.width = W; r.T = T; r.x = m->d_hidden; r.ld_act = st.width_p; r.f32 = st.f32;
    for (size_t l = 0; l < st.layers.size(); l++) {
        StackLayer& L = st.layers[l];
        const bool ffn = L.s.ffn != FfnKind::None, last = l + 1 == st.layers.size(), side = st.spec.side_dim > 0;
        const float* after = last ? nullptr : st.layers[l + 1].norm1_in;  // the norm ahead of the next layer; the last sum is read in f32
        // plain_next: the sum itself is read next, not its norm
        auto sum = [&](const float* w, const float* next, bool moe, bool pair, bool plain_next, bool end) -> int32_t {
            r.depth = DepthSum();
            if (end && st.depth) { r.depth.past = st.depth; r.depth.keep = st.depth + (l + 1) * plane; r.depth.stride = plane; r.depth.c = L.dwa; r.depth.n = (int)l + 1; }
            r.w = w; r.w_next = plain_next ? nullptr : next; r.act = st.spec.norm_inputs && !plain_next && !next ? nullptr : st.xa;
            r.moe = moe ? moe_sum(st, L, x, ldx) : MoeSum();
            r.pair = pair ? pair_sum(st, L) : PairSum();
            m->launches_in_call += 1;
            return launch_residual(r, m->stream);
        };
        LC_TRY(stack_mixer(m, (int)l, x, ldx, T, decode_step));
        LC_TRY(sum(L.norm1_out, ffn ? L.norm2_in : after, false, L.s.combine == Combine::Normed, side && !ffn, !side && !ffn));
        if (ffn) {
            LC_TRY(ffn_block(m, L, x, ldx, T, decode_step));
            LC_TRY(sum(L.norm2_out, after, L.s.ffn == FfnKind::Moe, false, side, !side));
        }
        if (!side) continue;
        LC_TRY(side_block(m, (int)l, T));
        LC_TRY(sum(L.side_norm, after, false, false, false, true));
    }
    return LC_OK;
}

// One sublayer on the f32 rows already in d_hidden (its output, before the norm, in `y`): for layer-level checks.
int32_t stack_probe(lc_model* m, int l, int T, bool ffn, float** y) {
    LayerStack& st = *m->stack;
    int ldx = st.spec.width;
    const void* x = m->d_hidden;
    if (!st.f32) {
        x = layer_input(m, &ldx);
        LC_TRY(launch_act_rows(m->d_hidden, st.spec.width, T, st.xa, st.width_p, m->stream));
    }
    LC_CHECK(!ffn || st.layers[l].s.ffn != FfnKind::None, LC_ERR_INVALID, "layer %d has no feed-forward", l);
    *y = st.y;
    StackLayer& L = st.layers[l];
    ResidualArgs r;
    r.y = st.y; r.eps = st.spec.eps; r.width = st.spec.width; r.T = T; r.ld_act = st.width_p; r.f32 = st.f32;
    if (!ffn) {
        LC_TRY(stack_mixer(m, l, x, ldx, T, false));
        if (L.s.combine != Combine::Normed) return LC_OK;
        r.pair = pair_sum(st, L);
        return launch_residual(r, m->stream);
    }
    LC_TRY(ffn_block(m, L, x, ldx, T, false));
    if (L.s.ffn != FfnKind::Moe) return LC_OK;
    r.moe = moe_sum(st, L, x, ldx);
    return launch_residual(r, m->stream);
}

int32_t stack_head(lc_model* m, int n, const int32_t* idx, float* logits) {
    LayerStack& st = *m->stack;
    LC_TRY(launch_norm_rows(m->d_hidden, idx, st.final_norm, st.spec.eps, st.spec.width, n, st.last, st.width_p, st.f32, m->stream));
    m->launches_in_call += 1;
    DenseArgs e;
    e.scale = st.spec.logit_scale; e.cap = st.spec.logit_softcap; e.x_rows = m->head_rows;
    return product(m, st.head, st.last, st.width_p, n, logits, st.spec.vocab, true, DENSE_LOGITS, e);
}

}  // namespace lc
