// Launch interface of the layers that checkpoint-directory designs are made of (bf16 weights; activations bf16, or f32 when
// the model runs in true 32-bit), and what a model of such layers keeps on the device.
#pragma once
#include <cuda_bf16.h>
#include <map>
#include <memory>
#include <vector>
#include "lc_arch.h"
#include "lc_common.cuh"

namespace lc {

inline int round8(int v) { return (v + 7) & ~7; }

// ---- dense16.cu: y = x W^T over bf16 weights -----------------------------------------------------------------------------
// `batch` matrices of n rows and k columns (one per head in the batched products), rows ld elements apart (ld % 8 == 0).
struct DenseWeight {
    const __nv_bfloat16* data = nullptr;
    int n = 0, k = 0, ld = 0, batch = 1;
    size_t batch_stride = 0;
    const unsigned char* tiles = nullptr;  // the tensor-core form: [matrix][n / 128][k / 64] blocks of 128 rows x 128 bytes, swizzled, zero-padded
};
int32_t dense_weight_init(DenseWeight* w, const __nv_bfloat16* data, int n, int k, int ld, int batch = 1, size_t batch_stride = 0);
// Rewrites the plain matrix into blocks at dst (dense_tile_bytes of them), after which `data` is no longer read.
size_t dense_tile_bytes(const DenseWeight& w);
int32_t dense_weight_tile(DenseWeight* w, void* dst, cudaStream_t s);

enum DenseEpilogue {
    DENSE_STORE = 0,
    DENSE_RELU2 = 1,      // max(y, 0)^2
    DENSE_LOG_DECAY = 2,  // -e0[row / e_div] * softplus(y + e1[row]), 32-bit
    DENSE_LOGITS = 3,     // y * scale, then cap * tanh(. / cap) when cap > 0
    DENSE_GATED_SILU = 4, // rows in pairs (2i: gate, 2i + 1: up): out row i = silu(gate) * up
    DENSE_SPLIT_RELU2 = 5, // rows below `split` as they are, in 32-bit, to `out`; the others squared relu, in the activations' type, to out2
    DENSE_SPLIT_SILU = 6,  // the same with silu up to row `act_end`, and the rest as they are
    DENSE_GELU_TABLE = 7,  // gelu (tanh form) times element `row` of the token's row in a table (0 for ids outside it)
    DENSE_GATED_GELU = 8,  // as DENSE_GATED_SILU with gelu (tanh form)
    DENSE_BIAS = 9,        // y + e1[row]
    DENSE_SPLIT_TANH = 10, // as DENSE_SPLIT_SILU with tanh
    DENSE_SIGMOID_DECAY = 11  // -scale * sigmoid(y + e1[row])
};
// A product of one of several matrices per token (experts): the tokens come as tiles of rows that share a matrix.
struct ExpertTile { int32_t expert, first, rows, row0; };  // rows first .. first + rows - 1 of the expert's list; row0: the first one's row in expert order
struct ExpertPlan {
    ExpertTile* tiles = nullptr;
    int32_t* n_tiles = nullptr;
    int32_t* off = nullptr;        // [experts + 1] rows of the experts before (expert order)
    int32_t* lists = nullptr;      // [experts][list_stride] token of every row
    int list_stride = 0;
    int tile_rows = 16;            // most rows of a tile: 16, 32, 64, 128 or 256
    int most_tiles = 0, most_rows = 0;  // bounds of this call (what the device finds is not known to the host)
};
struct DenseArgs {
    const DenseWeight* w = nullptr;
    const void* x = nullptr;      // [x_rows][..] activations, bf16 or (f32 = true) float; row t of matrix b at x + b * x_batch + t * ldx
    int ldx = 0, x_rows = 0;      // x_rows: rows the buffer has (>= T)
    size_t x_batch = 0;
    int T = 0;
    void* out = nullptr;          // row t of matrix b at out + b * out_batch + t * ldo
    int ldo = 0;
    size_t out_batch = 0;
    bool out_f32 = false;         // otherwise the activations' type
    DenseEpilogue epi = DENSE_STORE;
    const float* e0 = nullptr;
    const float* e1 = nullptr;
    int e_div = 1;
    float scale = 1.0f, cap = 0.0f;
    void* out2 = nullptr;         // DENSE_SPLIT_*
    int ldo2 = 0, split = 0;      // split: a multiple of 32
    int act_end = 0;              // DENSE_SPLIT_SILU, DENSE_SPLIT_TANH
    const __nv_bfloat16* table = nullptr;  // DENSE_GELU_TABLE: rows table_ld apart
    int table_ld = 0, table_rows = 0;
    const int64_t* ids = nullptr;
    const ExpertPlan* plan = nullptr;  // matrix = expert; output rows in expert order, input rows too unless `gather`
    bool gather = false;          // input row of a tile's row = its token
    bool f32 = false;
};
// Scratch of the shares of k that several CTAs sum, and the tensor maps over activation buffers seen so far.
struct DenseWorkspace {
    float* partial = nullptr;
    size_t partial_bytes = 0;
    unsigned* tickets = nullptr;
    int max_tickets = 0;
    struct Map { alignas(64) unsigned char b[128]; };
    std::map<std::vector<uint64_t>, std::unique_ptr<Map>> maps;
};
int32_t dense_workspace_alloc(DenseWorkspace* ws);
void dense_workspace_free(DenseWorkspace* ws);
int32_t launch_dense(const DenseArgs& a, DenseWorkspace& ws, cudaStream_t s);

// ---- mixers.cu -------------------------------------------------------------------------------------------------------
// Consecutive tokens of one sequence inside a call: rows tok0 .. tok0 + n - 1, the first at position pos0.
struct SeqRun { int32_t tok0, n, seq, pos0; };

// Copies a weight into a padded layout: element (r, c) of [rows, cols] goes to row map(r), column map(c), where a map sends
// index i of groups of `len` to group * stride + i, entries from `split` on moved up by `shift`; `transpose` swaps rows and
// columns inside each row group (dst row = group * stride + column, dst column = index inside the group).
struct PackMap { int len = 0, stride = 0, split = 0, shift = 0; };
int32_t launch_pack(const __nv_bfloat16* src, int rows, int cols, __nv_bfloat16* dst, int ld, PackMap row, PackMap col, bool transpose, cudaStream_t s);

// x[t] = embed[ids[t]] * scale in f32 (+ the row of the token pair); act != null: the same as activations, through rms_norm(.) * w
// when w is given.  ids outside the table give zero rows
struct PairEmbed {
    const __nv_bfloat16* table = nullptr;  // [buckets + 1][width]; null: none
    BigramSpec rows;
    const int32_t *tok_seq = nullptr, *tok_pos = nullptr;
    int32_t* last = nullptr;               // [slot] the sequence's last token of earlier calls
    bool one_each = false;                 // every token is the only one of its sequence: `last` is brought up to date too
};
struct EmbedArgs {
    const __nv_bfloat16* table = nullptr;
    int rows = 0, width = 0, T = 0;
    const int64_t* ids = nullptr;
    float scale = 1.0f, eps = 1e-6f;
    const float* w = nullptr;
    float *x = nullptr, *copy = nullptr;   // copy: a second one, or null
    void* act = nullptr;
    int ld_act = 0;
    bool f32 = false;
    PairEmbed pair;
};
int32_t launch_embed_rows(const EmbedArgs& a, cudaStream_t s);
// act[t] = bf16(x[t])
int32_t launch_act_rows(const float* x, int width, int T, void* act, int ld_act, cudaStream_t s);
// The output of a mixture of experts at one token: gate * y + sum over the choices of weight * (expert's row, or the input for
// identity experts).
struct MoeSum {
    const void* rows = nullptr;      // experts' outputs in expert order (activations); null: no mixture
    int ld_rows = 0;
    const int32_t *sel = nullptr, *pos = nullptr, *off = nullptr;  // [T][top] expert and place in its list; [experts + 1]
    const float* weight = nullptr;   // [T][top]
    int top = 0, experts = 0;
    const void* h = nullptr;         // [T][ld_h] the mixture's input
    int ld_h = 0;
    const float* gate = nullptr;     // [T] rows ld_gate apart, before the sigmoid; null: y is not read
    int ld_gate = 0;
};
// The output of two mixers side by side: (rms_norm(y) * w0 + rms_norm(y2) * w1) / 2.
struct PairSum {
    const float *y2 = nullptr, *w0 = nullptr, *w1 = nullptr;  // y2 null: no pair
};
// What leaves a layer: sum_j c[j] X_j over n rows of earlier results (planes `stride` apart) and, with c[n], this one, kept in `keep`.
struct DepthSum {
    const float *past = nullptr, *c = nullptr;
    float* keep = nullptr;                                    // null: no sum over depth
    size_t stride = 0;
    int n = 0;
};
// x[t] += rms_norm(y[t]) * w, or += y[t] without w; act != null: the sum as activations, through rms_norm(.) * w_next when that is
// given.  With a mixture or a pair y is first replaced by its output (x null: nothing more happens).
struct ResidualArgs {
    float* y = nullptr;
    const float *w = nullptr, *w_next = nullptr;
    float eps = 1e-6f;
    int width = 0, T = 0;
    float* x = nullptr;
    void* act = nullptr;
    int ld_act = 0;
    bool f32 = false;
    MoeSum moe;
    PairSum pair;
    DepthSum depth;                    // only without w
};
int32_t launch_residual(const ResidualArgs& a, cudaStream_t s);
// out[i] = rms_norm(x[idx ? idx[i] : i]) * w as activations
int32_t launch_norm_rows(const float* x, const int32_t* idx, const float* w, float eps, int width, int n, void* out, int ldo, bool f32, cudaStream_t s);
// last[slot] = the last token of every run, behind the embedding
int32_t launch_keep_tokens(const SeqRun* runs, int n_runs, const int64_t* ids, int32_t* last, cudaStream_t s);

// Per head: o / rms(o) * w * sigmoid(gate), as activations.
struct HeadNormArgs {
    const float* o = nullptr;          // [T][heads * n]
    int heads = 0, n = 0, T = 0;
    float eps = 1e-6f;
    const float* w = nullptr;          // heads w_stride apart (0: shared)
    int w_stride = 0;
    const void* gate = nullptr;        // [T][ld_gate] activations, before the sigmoid
    int ld_gate = 0;
    void* out = nullptr;               // [T][ldo] activations
    int ldo = 0;
    bool f32 = false;
    const SeqRun* runs = nullptr;      // only the tokens of these runs; longest: the most tokens of one
    int n_runs = 0, longest = 0;
};
int32_t launch_head_norm(const HeadNormArgs& a, cudaStream_t s);

// Gated delta rule with one decay per key channel.  `proj` rows hold q | k | v | ... | beta logits as projected; the inputs of
// the short convolutions of the last `taps` positions live in `ring` [slot][taps][channels], entry position % taps.
struct DeltaShape { int heads, kv_heads, dim, vdim, taps, ld, off_k, off_v, off_b, channels; float unit_eps, eps; };
constexpr int kDeltaChunk = 64;
struct DeltaChunk { int32_t tok0, n; };                       // up to kDeltaChunk consecutive tokens of a run
struct DeltaChunkRun { SeqRun run; int32_t chunk0, n_chunks; };
struct DeltaArgs {
    DeltaShape g;
    const void* proj = nullptr;
    const float* conv = nullptr;       // [channels][taps], the last column weighs the current token
    void* ring = nullptr;
    float* state = nullptr;            // [slot][heads][dim][vdim]
    const int32_t *tok_seq = nullptr, *tok_pos = nullptr;
    int T = 0;
    float* qk = nullptr;               // [T][2][kv_heads * dim] unit vectors, q scaled by dim^-1/2
    float* v = nullptr;                // [T][heads * vdim]
    const float* log_decay = nullptr;  // [T][heads * dim]
    float* o = nullptr;                // [T][heads * vdim]
    const SeqRun* runs = nullptr;      // walked token by token
    int n_runs = 0;
    const DeltaChunk* chunks = nullptr;         // longer runs (delta_chunk.cu)
    const DeltaChunkRun* chunk_runs = nullptr;
    int n_chunks = 0, n_chunk_runs = 0;
    const float* norm_w = nullptr;     // [vdim]
    const void* gate = nullptr;        // [T][heads * vdim] before the sigmoid
    void* out = nullptr;               // [T][ldo] activations
    int ldo = 0;
    bool f32 = false;
};
int32_t launch_delta_prep(const DeltaArgs& a, cudaStream_t s);   // convolutions, silu, unit vectors
int32_t launch_delta_scan(const DeltaArgs& a, cudaStream_t s);   // the recurrence over every run; leaves state and ring for the next call
int32_t launch_delta_step(const DeltaArgs& a, cudaStream_t s);   // the two with norm and gate for one new token per sequence (rows of tok_seq / tok_pos)

// delta_chunk.cu: the recurrence over `chunk_runs`, in chunks; scratch of delta_chunk_bytes per chunk
bool delta_chunks_apply(const DeltaShape& g, bool f32);
size_t delta_chunk_bytes(const DeltaShape& g);
int32_t launch_delta_chunks(const DeltaArgs& a, float* scratch, cudaStream_t s);

#ifdef __CUDACC__
// The inputs of a run's last `taps` positions, for the convolutions of the next call: head h's v channels, and the q and k
// channels of its key head once per group.
template <typename A>
__device__ __forceinline__ void delta_keep_inputs(const DeltaArgs& a, const SeqRun& run, int h, int tid, int threads) {
    const DeltaShape& g = a.g;
    const int rep = g.heads / g.kv_heads, kh = h / rep;
    A* ring = (A*)a.ring + (size_t)run.seq * g.taps * g.channels;
    const A* proj = (const A*)a.proj;
    const int m = run.n < g.taps ? run.n : g.taps, per = g.vdim + (h % rep == 0 ? 2 * g.dim : 0);
    for (int i = tid; i < m * per; i += threads) {
        const int j = i / per, c = i - j * per;
        int column, channel;
        if (c < g.vdim) { column = g.off_v + h * g.vdim + c; channel = 2 * g.kv_heads * g.dim + h * g.vdim + c; }
        else if (c < g.vdim + g.dim) { column = kh * g.dim + c - g.vdim; channel = column; }
        else { column = g.off_k + kh * g.dim + c - g.vdim - g.dim; channel = g.kv_heads * g.dim + kh * g.dim + c - g.vdim - g.dim; }
        const int t = run.n - 1 - j;
        ring[(size_t)((run.pos0 + t) % g.taps) * g.channels + channel] = proj[(size_t)(run.tok0 + t) * g.ld + column];
    }
}
#endif

// Cache of latent attention: per page page_tokens rows [kv_rank | pad | rot_dim | pad] of the activations' type.
struct LatentShape { int heads, dim, rot, rank, ld_q, dp, cp, rp, rot_pairs; float scale; };  // dp, cp, rp: dim, rank, rot rounded up to 8
struct LatentArgs {
    LatentShape g;
    const float* proj = nullptr;       // [T][ld_proj]: query latent | kv latent | rotated key part
    int ld_proj = 0, q_rank = 0, off_c = 0, off_r = 0;
    const float *q_norm = nullptr, *c_norm = nullptr;
    float eps = 1e-6f;
    const float2* rot = nullptr;       // [position][rot_pairs] (cos, sin)
    void* cq = nullptr;                // [T][ld_cq]
    int ld_cq = 0;
    void* cache = nullptr;
    int page_tokens = 16;
    const int32_t *page_table = nullptr, *tok_seq = nullptr, *tok_pos = nullptr;
    int pages_per_seq = 0, T = 0;
    const void* q = nullptr;           // [T][heads][ld_q]: unrotated part at 0, part to rotate at dp
    const void* q_abs = nullptr;       // [T][heads][cp]: the unrotated part carried through the key projection
    void* o = nullptr;                 // [T][heads][cp]: weighted sums of latents
    bool f32 = false;
};
int32_t launch_latent_prep(const LatentArgs& a, cudaStream_t s);
int32_t launch_rot_table(const double* freq_dev, int pairs, double magnitude, int positions, float2* out, cudaStream_t s);
// ---- latent_attention.cu ---------------------------------------------------------------------------------------------
// Tokens 0 .. T - 1 of `a`, each over its own context through q_abs / q, into o.  scratch: partial sums of context pieces.
size_t latent_pieces_bytes(const LatentShape& g, int tokens);
int32_t launch_latent_attention(const LatentArgs& a, void* scratch, size_t scratch_bytes, int* launches, cudaStream_t s);
// Runs of many tokens: up to 64 consecutive tokens (rows tok0 .. of the call, first position pos0) whose sequence's gathered
// context starts at row row0 of c / k / v.
struct LatentTile { int32_t tok0, n, pos0, row0; };
struct LatentContext { int32_t seq, len, row0; };
struct LatentPrefill {
    const LatentTile* tiles = nullptr;
    const void *c = nullptr, *k = nullptr, *v = nullptr;  // [rows][cp + rp], [rows][heads * dp], [rows][heads * ep]
    void* out = nullptr;                                  // [T][heads * ep]
    int ep = 0;
};
bool latent_prefill_applies(const LatentShape& g, int ep, bool f32);
int32_t launch_latent_gather(const LatentArgs& a, const LatentContext* ctx, int n_ctx, int longest, void* out, cudaStream_t s);
int32_t launch_latent_prefill(const LatentArgs& a, const LatentPrefill& p, int n_tiles, cudaStream_t s);

// ---- gqa_attention.cu: attention over the keys and values of a paged cache, [page][kv head][page_tokens][pitch] ----------------
struct AttnShape {
    int heads, kv_heads, dim, vdim, dp, ep, rot_dims;  // dp, ep: dim, vdim rounded up to 8
    float scale, cap;                                  // cap > 0: scores through cap * tanh(. / cap)
    int window, keep_first;                            // MaskSpec
    QkNorm norm;
    AttnPairs pairs;
    int taps;                                          // of the convolutions on q, k and v (0: none; then norm is not AllHeads)
    int k_pitch, v_pitch, k_swz, v_swz;                // cache rows (attn_cache_layout): elements apart; 7: chunks swizzled by position
};
void attn_cache_layout(AttnShape* g, bool f32);
struct AttnArgs {
    AttnShape g;
    const float* proj = nullptr;       // [T][ld_proj] q | k | v
    int ld_proj = 0, off_k = -1, off_v = 0;  // off_k < 0: the layer has no keys and values of its own
    const float *q_norm = nullptr, *k_norm = nullptr;
    const float* conv = nullptr;       // [channels q | k | v][taps], the last column weighs the current token
    float* ring = nullptr;             // [slot][taps][channels]: the inputs of the last `taps` positions, entry position % taps
    bool one_each = false;             // every token is the only one of its sequence: attn_prep also keeps its inputs
    float eps = 1e-6f;
    const float2* rot = nullptr;       // [position][rot_dims / 2] (cos, sin)
    void* q = nullptr;                 // [T][heads][dp]
    void *k_cache = nullptr, *v_cache = nullptr;
    int page_tokens = 16;
    const int32_t *page_table = nullptr, *tok_seq = nullptr, *tok_pos = nullptr;
    int pages_per_seq = 0, T = 0;
    const float* sink = nullptr;       // [heads] or null
    const void* gate = nullptr;        // [T][ld_gate] activations, heads vdim apart: sigmoid(gate) on the output; null: none
    int ld_gate = 0;
    const float* head_gate = nullptr;  // [T][ld_proj] one number per head: sigmoid(.) on the head's output; null: none
    const float* q_factor = nullptr;   // [position] on the queries; null: none
    float out_scale = 1.0f;
    void* out = nullptr;               // [T][ldo], heads ep apart
    int ldo = 0;
    bool f32 = false;
};
int32_t launch_attn_prep(const AttnArgs& a, cudaStream_t s);   // convolutions, norms of q and k, rotation, cache append
int32_t launch_attn_keep(const AttnArgs& a, const SeqRun* runs, int n_runs, cudaStream_t s);  // the runs' last inputs, behind attn_prep
struct AttnScratch { float* part = nullptr; size_t part_bytes = 0; unsigned* tickets = nullptr; int n_tickets = 0; };
size_t attn_part_bytes(const AttnShape& g);
int32_t launch_attn_tokens(const AttnArgs& a, const AttnScratch& sc, cudaStream_t s);  // tokens 0 .. T - 1, each over its own context
// up to 64 consecutive tokens (rows tok0 .. of the call, first position pos0)
struct AttnTile { int32_t tok0, n, seq, pos0; };
bool attn_tiles_apply(const AttnShape& g, bool f32);
int32_t launch_attn_tiles(const AttnArgs& a, const AttnTile* tiles, int n_tiles, cudaStream_t s);

// ---- linear_state.cu: S_t = decay_t S_(t-1) + step_t k_t v_t^T, o_t = S_t^T q_t (+ skip v_t), per head, S in f32 -------------------------
struct LinearShape {
    LinearKind kind;
    int heads, groups, dim, vdim;      // q, k: groups x dim; v: heads x vdim
    int ld, off_v, off_k, off_q, off_g;  // columns of the projected rows: v, k, q (StateSpace: before the convolution), gate
    int ld_dt, off_dt;                 // StateSpace: where the steps are projected to
    int taps, channels, ld_in;         // StateSpace: channels v | k | q, one after the other from off_v on; ld_in: rows of `in`
    int norm_parts;
    float eps;
};
struct LinearArgs {
    LinearShape g;
    const void* proj = nullptr;        // [T][ld] activations
    const float* dt = nullptr;         // [T][ld_dt] 32-bit part of the projection
    const float *conv = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *a_exp = nullptr, *skip = nullptr;  // StateSpace; a_exp = e^A_log
    const float* log_decay = nullptr;  // Constant: [heads]
    const float2* decay = nullptr;     // Constant: [heads] the factors as sums of two floats: one float's rounding would add up over thousands of tokens
    void* ring = nullptr;              // [slot][taps][channels] activations
    void* in = nullptr;                // StateSpace: [T][ld_in] v | k | q behind convolution and silu
    float* state = nullptr;            // [slot][heads][dim][vdim]
    const int32_t *tok_seq = nullptr, *tok_pos = nullptr;
    int T = 0;
    float* o = nullptr;                // [T][heads * vdim]
    const SeqRun* runs = nullptr;      // walked token by token
    int n_runs = 0;
    const DeltaChunkRun* chunk_runs = nullptr;  // in chunks of kDeltaChunk tokens
    int n_chunk_runs = 0;
    const SeqRun* all_runs = nullptr;  // all of them, for the inputs that the next call's convolutions need
    int n_all_runs = 0;
    const float* norm_w = nullptr;     // [heads * vdim]
    float out_scale = 1.0f;
    void* out = nullptr;               // [T][ldo] activations
    int ldo = 0;
    bool f32 = false;
};
bool linear_chunks_apply(const LinearShape& g, bool f32);
int32_t launch_linear_runs(const LinearArgs& a, int* launches, cudaStream_t s);  // convolutions, the recurrence over all runs, the kept inputs
int32_t launch_linear_step(const LinearArgs& a, int* launches, cudaStream_t s);  // the same for one token per sequence
int32_t launch_linear_output(const LinearArgs& a, cudaStream_t s);               // gate and norm

// ---- general_delta.cu: S_t = diag(w) S_(t-1) - (a u) (u^T S_(t-1)) + k v^T, o_t = S_t^T r, per head, S in f32; u = k / sqrt(|k|^2 + unit_eps),
// a = sigmoid(. + a_bias), all of r, k, v, a and the state dim wide -----------------------------------------------------------------------
struct GeneralShape {
    int heads, dim;
    int ld, off_k, off_v, off_a;       // columns of the projected rows (r at 0)
    float unit_eps, eps;
};
constexpr int kGeneralChunk = 32;      // tokens per step of the chunked form
struct GeneralArgs {
    GeneralShape g;
    const float* proj = nullptr;       // [T][ld] r | k | v | a
    const float* a_bias = nullptr;     // [heads * dim]
    const float* log_decay = nullptr;  // [T][heads * dim], ln w
    float* state = nullptr;            // [slot][heads][dim][dim]
    const int32_t *tok_seq = nullptr, *tok_pos = nullptr;
    int T = 0;
    float* o = nullptr;                // [T][heads * dim]
    const SeqRun* runs = nullptr;      // walked token by token
    int n_runs = 0;
    const DeltaChunk* chunks = nullptr;         // longer runs
    const DeltaChunkRun* chunk_runs = nullptr;
    int n_chunks = 0, n_chunk_runs = 0;
    const float* norm_w = nullptr;     // step and chunks: norm, gate and output as in HeadNormArgs
    const void* gate = nullptr;
    int ld_gate = 0;
    void* out = nullptr;
    int ldo = 0;
    bool f32 = false;
};
bool general_chunks_apply(const GeneralShape& g, double decay_scale, bool f32);
size_t general_chunk_bytes(const GeneralShape& g);               // scratch per chunk of kDeltaChunk tokens
int32_t launch_general_scan(const GeneralArgs& a, cudaStream_t s);
int32_t launch_general_chunks(const GeneralArgs& a, float* scratch, cudaStream_t s);  // with norm and gate
int32_t launch_general_step(const GeneralArgs& a, cudaStream_t s);  // one token per sequence, with norm and gate

// ---- expert_choice.cu: routing ---------------------------------------------------------------------------------------------
struct ChoiceArgs {
    MoeSpec m;
    const float* z = nullptr;          // [T][ld_z] router logits
    int ld_z = 0, T = 0;
    const float* correction = nullptr; // [outputs]
    int32_t *sel = nullptr, *pos = nullptr;  // [T][top] expert, its place in the expert's list (experts with matrices)
    float* weight = nullptr;           // [T][top]
    int32_t* counts = nullptr;         // [experts] + one ticket word, zero between launches
    ExpertPlan plan;
    unsigned long long* touched = nullptr;  // += touched_bytes for every expert that received a token
    unsigned long long touched_bytes = 0;
};
int32_t launch_expert_choice(const ChoiceArgs& a, cudaStream_t s);
// The bf16 rows m.h of T tokens, each copied to its rows of `out` (expert order, ldo apart).
int32_t launch_expert_gather(const MoeSum& m, int width, int T, void* out, int ldo, cudaStream_t s);

// ---- a stack of such layers (layers.cu) --------------------------------------------------------------------------------
struct MixerUnit {
    MixerSpec s;
    DenseWeight in, out;            // (two mixers side by side: StackLayer has these)
    // ChannelDelta: `in` = q | k | v | a1 | g1 | b
    DenseWeight a2, g2;
    DeltaShape dg{};
    int off_a = 0, off_g = 0;       // off_g also: the output gate of GeneralDelta and Attention, in the activations' part
    const float *conv = nullptr, *a_exp = nullptr, *dt_bias = nullptr, *o_norm = nullptr;
    float* state = nullptr;
    void* ring = nullptr;
    // LatentAttention: `in` = dq | dkv
    DenseWeight uq, uk_t, uv;       // one token at a time: key projection transposed per head, value projection per head
    DenseWeight uk_all, uv_all;     // whole contexts: all heads at once
    LatentShape lg{};
    int off_r = 0, off_c = 0, ep = 0;
    const float *q_norm = nullptr, *c_norm = nullptr;
    const float2* rot = nullptr;
    void* cache = nullptr;
    // Attention: `in` = q | k | v (q alone when another layer's cache is read)
    AttnShape ag{};
    int off_k = -1, off_v = 0;
    const float *k_norm = nullptr, *sink = nullptr;
    void *k_cache = nullptr, *v_cache = nullptr;
    const float *in_bias = nullptr, *out_bias = nullptr, *q_factor = nullptr;
    int off_hg = -1;                // the gates per head
    // GeneralDelta: `in` = r | k | v | a (32-bit, below in_split) | w1 | g; a2 = w2, dt_bias = its bias
    GeneralShape gg{};
    int in_split = 0, act_end = 0;
    const float* a_bias = nullptr;
    // LinearState
    LinearShape ng{};
    const float *conv_b = nullptr, *skip = nullptr, *log_decay = nullptr;
    const float2* decay = nullptr;
};
struct StackLayer {
    LayerSpec s;
    MixerUnit mix[2];
    // two mixers side by side: what both read projected by one product, 32-bit rows below in_split, activations behind it (silu up
    // to row act_end); their outputs lie side by side in rows of mixed_ld, the second one's from mixed_off on, and leave through
    // `out` together (Scaled) or through one matrix each (Normed)
    DenseWeight in, out, out2;
    int in_split = 0, act_end = 0, mixed_off = 0, mixed_ld = 0;
    const float* out_norm[2] = {nullptr, nullptr};
    // norms of the sublayers' inputs (null: none) and outputs
    const float *norm1_in = nullptr, *norm1_out = nullptr, *norm2_in = nullptr, *norm2_out = nullptr;
    DenseWeight up, down;              // GatedSilu: `up` = gate and up rows in turn
    // Moe: `up` and `down` of all experts; `route` = router | gate of the shared expert | (from row route_split on) its up
    DenseWeight route, shared_down;
    int off_gate = 0, route_split = 0;
    const float* correction = nullptr;
    uint64_t expert_bytes = 0;         // one expert's matrices
    const float* dwa = nullptr;        // weights of the sum over depth
    // token input
    DenseWeight side_gate, side_proj;
    const float* side_norm = nullptr;
};
struct LayerStack {
    ArchSpec spec;
    bool f32 = false;                  // true 32-bit activations and cache
    std::vector<StackLayer> layers;
    DenseWeight head;
    const __nv_bfloat16* embed = nullptr;
    const __nv_bfloat16 *side_embed = nullptr, *bigram = nullptr;
    int32_t* last_token = nullptr;     // [slot], for the pair embedding
    float* depth = nullptr;            // [layers + 1][t_cap][width]: the call's embedding and layers' results
    const float* final_norm = nullptr;
    DenseWorkspace ws;
    std::vector<void*> owned;
    std::vector<void*> temps;          // plain copies of weights, dropped once their blocks exist
    std::vector<std::string> packed;   // checkpoint tensors whose bytes live on in blocks only
    std::vector<std::pair<RotarySpec, const float2*>> rot_tables;
    std::vector<std::pair<QueryTemperature, const float*>> q_factors;
    uint64_t cache_bytes_per_token = 0, state_bytes_per_seq = 0;
    // step buffers for t_cap tokens
    int width_p = 0;
    void *xa = nullptr, *proj = nullptr, *gate = nullptr, *mixed = nullptr, *cq = nullptr, *q = nullptr, *q_abs = nullptr, *o_lat = nullptr, *ffn = nullptr, *last = nullptr,
         *side = nullptr, *lin = nullptr;
    float *y = nullptr, *y2 = nullptr, *projf = nullptr, *log_decay = nullptr, *qk = nullptr, *v = nullptr, *o = nullptr;
    SeqRun* d_runs = nullptr;
    int n_runs = 0;
    // gated delta rule of the call: short runs walk token by token, long ones in chunks (when every such layer has that form)
    bool delta_chunks = false;
    SeqRun* d_short_runs = nullptr;
    DeltaChunk* d_chunks = nullptr;
    DeltaChunkRun* d_chunk_runs = nullptr;
    int n_short_runs = 0, n_chunks = 0, n_chunk_runs = 0, longest_short = 0;
    size_t chunk_bytes = 0;            // scratch per chunk, widest layer
    DevBuf chunk_scratch;
    // latent attention of the call: its first n_short tokens attend one by one, the others in tiles over projected contexts,
    // in groups whose contexts fit the context buffers
    struct Group { int tile0, n_tiles, ctx0, n_ctx, rows, longest; };
    int n_short = 0;
    std::vector<Group> groups;
    LatentTile* d_lat_tiles = nullptr;
    LatentContext* d_lat_ctx = nullptr;
    AttnTile* d_attn_tiles = nullptr;
    int n_attn_tiles = 0;
    AttnScratch attn;
    // mixtures of experts
    float *moe_z = nullptr, *moe_w = nullptr;
    int32_t *moe_sel = nullptr, *moe_pos = nullptr, *moe_counts = nullptr;
    void *moe_up = nullptr, *moe_rows = nullptr, *moe_in = nullptr;  // the experts' hidden rows, outputs and (bf16) inputs, in expert order
    ExpertPlan plan;
    int plan_tiles = 0, moe_slots = 0;  // room of the tile list; rows of moe_up and moe_rows
    void* pieces = nullptr;
    size_t pieces_bytes = 0;
    bool prefill_tiles = false;        // every attention layer has a tile form
    size_t ctx_c_row = 0, ctx_k_row = 0, ctx_v_row = 0;  // widest rows of the context buffers, in elements
    DevBuf ctx_c, ctx_k, ctx_v;
};

}  // namespace lc
