// The layers of a checkpoint-directory design on the device: binding of the weights, the cache and state they keep, and the
// launches of one pass over T tokens.  Per layer:
//   ChannelDelta     in = q | k | v | a1 | g1 | b (one product)  ->  a2 (log decay in its epilogue), g2  ->  convolutions + unit
//                    vectors -> recurrence -> per-head norm and gate -> out
//   LatentAttention  in = dq | dkv (one product)  ->  latent norms, key rotation, cache append  ->  uq -> (per head) uk^T
//                    -> attention over the latents -> (per head) uv -> out
//   Relu2            up (squared relu in its epilogue) -> down
// each followed by x += rms_norm(y) w, which also writes the activations the next product reads.
#include <cmath>
#include <cstring>
#include "lc_model.h"

namespace lc {

namespace {

typedef __nv_bfloat16 bf16;
constexpr int kContextRows = 16384;  // rows of projected keys and values at a time (one longer context is taken whole)

int32_t zalloc(LayerStack& st, void** p, size_t bytes) {
    uint8_t* q = nullptr;
    LC_TRY(dalloc(&q, bytes));
    st.owned.push_back(q);
    LC_CUDA(cudaMemsetAsync(q, 0, std::max<size_t>(bytes, 16), stream()));
    *p = q;
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
int32_t fused_weight(lc_model* m, const std::vector<std::string>& names, const std::vector<int>& rows, int k, DenseWeight* w, std::vector<int>* offs) {
    int total = 0;
    for (int r : rows) { offs->push_back(total); total += round8(r); }
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

int32_t bind_delta(lc_model* m, StackLayer& L, const std::string& p) {
    LayerStack& st = *m->stack;
    const LayerSpec& s = L.s;
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
    // the three convolutions' taps as one f32 table
    void* cp = nullptr;
    LC_TRY(zalloc(st, &cp, (size_t)L.dg.channels * s.conv_taps * 4));
    const char* cn[3] = {"q.conv", "k.conv", "v.conv"};
    const int cc[3] = {nk, nk, nv};
    size_t at = 0;
    for (int i = 0; i < 3; i++) {
        const float* g = nullptr;
        LC_TRY(model_gain_f32(m, p + cn[i], cc[i] * s.conv_taps, &g));
        LC_CUDA(cudaMemcpyAsync((float*)cp + at, g, (size_t)cc[i] * s.conv_taps * 4, cudaMemcpyDeviceToDevice, m->stream));
        at += (size_t)cc[i] * s.conv_taps;
    }
    L.conv = (const float*)cp;
    const float* alog = nullptr;
    LC_TRY(model_gain_f32(m, p + "A_log", s.heads, &alog));
    std::vector<float> h((size_t)s.heads);
    LC_CUDA(cudaMemcpyAsync(h.data(), alog, h.size() * 4, cudaMemcpyDeviceToHost, m->stream));
    LC_CUDA(cudaStreamSynchronize(m->stream));
    for (float& v : h) v = std::exp(v);
    void* ae = nullptr;
    LC_TRY(zalloc(st, &ae, h.size() * 4));
    LC_CUDA(cudaMemcpyAsync(ae, h.data(), h.size() * 4, cudaMemcpyHostToDevice, m->stream));
    LC_CUDA(cudaStreamSynchronize(m->stream));
    L.a_exp = (const float*)ae;
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

int32_t bind_latent(lc_model* m, StackLayer& L, const std::string& p) {
    LayerStack& st = *m->stack;
    LayerSpec& s = L.s;
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

int32_t delta_block(lc_model* m, StackLayer& L, const void* x, int ldx, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    const LayerSpec& s = L.s;
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
        LC_TRY(launch_delta_output(d, m->stream));
        m->launches_in_call += 2 + (d.n_runs ? 1 : 0) + (d.n_chunk_runs ? 2 : 0);
    }
    return product(m, L.out, st.mixed, d.ldo, T, st.y, st.spec.width, true);
}

int32_t latent_block(lc_model* m, StackLayer& L, const void* x, int ldx, int T, bool decode_step) {
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

int32_t relu2_block(lc_model* m, StackLayer& L, const void* x, int ldx, int T) {
    LayerStack& st = *m->stack;
    const int ldf = round8(L.s.ff);
    LC_TRY(product(m, L.up, x, ldx, T, st.ffn, ldf, false, DENSE_RELU2));
    return product(m, L.down, st.ffn, ldf, T, st.y, st.spec.width, true);
}

// The layers' input: the residual itself in f32, or its bf16 copy.
const void* layer_input(lc_model* m, int* ld) {
    LayerStack& st = *m->stack;
    *ld = st.f32 ? st.spec.width : st.width_p;
    return st.f32 ? (const void*)m->d_hidden : st.xa;
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
        if (L.s.mixer == MixerKind::ChannelDelta) LC_TRY(bind_delta(m, L, p + "mix."));
        else LC_TRY(bind_latent(m, L, p + "mix."));
        LC_TRY(model_gain_f32(m, p + "norm1", sp.width, &L.norm1));
        if (L.s.ffn != FfnKind::None) {
            LC_TRY(plain_weight(m, p + "mlp.up", L.s.ff, sp.width, &L.up));
            LC_TRY(plain_weight(m, p + "mlp.down", sp.width, L.s.ff, &L.down));
            LC_TRY(model_gain_f32(m, p + "norm2", sp.width, &L.norm2));
        }
        LC_TRY(block_weights(m, {&L.in, &L.out, &L.up, &L.down, &L.a2, &L.g2, &L.uq, &L.uk_t, &L.uv, &L.uk_all, &L.uv_all}));
    }
    DevTensor* e = nullptr;
    LC_TRY(matrix(m, "embed", sp.vocab, sp.width, &e));
    st.embed = (const bf16*)e->view;
    st.packed.clear();  // the embedding table is read as it is
    m->embed = e;
    LC_TRY(model_gain_f32(m, "final.norm", sp.width, &st.final_norm));
    LC_TRY(plain_weight(m, "head", sp.vocab, sp.width, &st.head));
    return block_weights(m, {&st.head});
}

int32_t stack_alloc(lc_model* m) {
    LayerStack& st = *m->stack;
    const size_t T = (size_t)m->t_cap, e = elt(st);
    st.width_p = round8(st.spec.width);
    st.prefill_tiles = st.delta_chunks = !st.f32;
    size_t proj = 8, projf = 8, gate = 8, mixed = 8, cq = 8, q = 8, qa = 8, ffn = 8, ld = 8, qk = 8, v = 8;
    for (StackLayer& L : st.layers) {
        const LayerSpec& s = L.s;
        if (s.mixer == MixerKind::ChannelDelta) {
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
        if (s.ffn != FfnKind::None) ffn = std::max(ffn, (size_t)round8(s.ff));
    }
    if (!st.f32) LC_TRY(zalloc(st, &st.xa, T * st.width_p * e));
    LC_TRY(zalloc(st, &st.proj, T * proj * e)); LC_TRY(zalloc(st, (void**)&st.projf, T * projf * 4));
    LC_TRY(zalloc(st, &st.gate, T * gate * e)); LC_TRY(zalloc(st, &st.mixed, T * mixed * e));
    LC_TRY(zalloc(st, &st.cq, T * cq * e)); LC_TRY(zalloc(st, &st.q, T * q * e));
    LC_TRY(zalloc(st, &st.q_abs, T * qa * e)); LC_TRY(zalloc(st, &st.o_lat, T * qa * e));
    LC_TRY(zalloc(st, &st.ffn, T * ffn * e)); LC_TRY(zalloc(st, &st.last, (size_t)m->head_rows * st.width_p * e));
    LC_TRY(zalloc(st, (void**)&st.y, T * st.spec.width * 4)); LC_TRY(zalloc(st, (void**)&st.log_decay, T * ld * 4));
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
    st.n_short_runs = (int)shorts.size(); st.n_chunks = (int)chunks.size(); st.n_chunk_runs = (int)chunk_runs.size();
    if (!shorts.empty()) LC_CUDA(cudaMemcpyAsync(st.d_short_runs, shorts.data(), shorts.size() * sizeof(SeqRun), cudaMemcpyHostToDevice, m->stream));
    if (!chunks.empty()) {
        LC_CUDA(cudaMemcpyAsync(st.d_chunks, chunks.data(), chunks.size() * sizeof(DeltaChunk), cudaMemcpyHostToDevice, m->stream));
        LC_CUDA(cudaMemcpyAsync(st.d_chunk_runs, chunk_runs.data(), chunk_runs.size() * sizeof(DeltaChunkRun), cudaMemcpyHostToDevice, m->stream));
        LC_TRY(st.chunk_scratch.reserve(std::max(chunks.size(), (size_t)m->t_cap / kDeltaChunk) * st.chunk_bytes));
    }
    st.groups.clear();
    st.n_short = (int)seq.size();
    std::vector<LatentTile> tiles;
    std::vector<LatentContext> ctx;
    size_t first = 0;
    while (first < runs.size() && runs[first].n < kTileRun) first++;
    if (st.prefill_tiles && first < runs.size()) {
        st.n_short = runs[first].tok0;
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
    return L.s.mixer == MixerKind::ChannelDelta ? delta_block(m, L, x, ldx, T, decode_step) : latent_block(m, L, x, ldx, T, decode_step);
}
int32_t stack_ffn(lc_model* m, int l, const void* x, int ldx, int T) { return relu2_block(m, m->stack->layers[l], x, ldx, T); }

int32_t stack_run_layers(lc_model* m, int T, bool decode_step) {
    LayerStack& st = *m->stack;
    const int W = st.spec.width;
    int ldx = 0;
    const void* x = layer_input(m, &ldx);
    LC_TRY(launch_embed_rows(st.embed, st.spec.vocab, W, m->d_tokens, T, m->d_hidden, st.xa, st.width_p, m->stream));
    m->launches_in_call += 1;
    for (size_t l = 0; l < st.layers.size(); l++) {
        LC_TRY(stack_mixer(m, (int)l, x, ldx, T, decode_step));
        LC_TRY(launch_norm_residual(st.y, st.layers[l].norm1, st.spec.eps, W, T, m->d_hidden, st.xa, st.width_p, m->stream));
        m->launches_in_call += 1;
        if (st.layers[l].s.ffn == FfnKind::None) continue;
        LC_TRY(stack_ffn(m, (int)l, x, ldx, T));
        LC_TRY(launch_norm_residual(st.y, st.layers[l].norm2, st.spec.eps, W, T, m->d_hidden, st.xa, st.width_p, m->stream));
        m->launches_in_call += 1;
    }
    return LC_OK;
}

// One sublayer on the f32 rows already in d_hidden (its output, before the norm, in `y`): for layer-level checks.
int32_t stack_probe(lc_model* m, int l, int T, bool ffn, float** y) {
    LayerStack& st = *m->stack;
    int ldx = 0;
    const void* x = layer_input(m, &ldx);
    if (!st.f32) LC_TRY(launch_act_rows(m->d_hidden, st.spec.width, T, st.xa, st.width_p, m->stream));
    LC_CHECK(!ffn || st.layers[l].s.ffn != FfnKind::None, LC_ERR_INVALID, "layer %d has no feed-forward", l);
    LC_TRY(ffn ? stack_ffn(m, l, x, ldx, T) : stack_mixer(m, l, x, ldx, T, false));
    *y = st.y;
    return LC_OK;
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
