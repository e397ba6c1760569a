// What one model handle of the C ABI holds, shared by the engine (engine.cu: life cycle, cache, batching, decode loop) and
// the layers of the checkpoint-directory designs (layers.cu).
#pragma once
#include <algorithm>
#include <map>
#include <memory>
#include <string>
#include <vector>
#include "lc_arch.h"
#include "lc_kernels.h"
#include "lc_mixers.h"

namespace lc {

struct DevTensor {
    uint32_t typ = 0;
    std::vector<uint64_t> dims;
    void* dev = nullptr;   // owning pointer (null when the bytes live inside a fused buffer)
    void* view = nullptr;  // where the bytes are
    size_t nbytes = 0;
    size_t rows = 0, cols = 0;
};

struct LayerW {
    QWeight qkv, o, gate, up, down;
    QWeight q, k, v;  // used when the three cannot be fused
    bool fused_qkv = false;
    const float* attn_norm = nullptr;
    const float* ffn_norm = nullptr;
    void* fused_buf = nullptr;
    // mixture-of-experts FFN (no counterpart in the reference): f32 router [n_experts, H], the experts' three matrices,
    // and -- when every expert is Q4_K with a tensor map -- device arrays of those maps for the one-launch grouped product
    const float* router = nullptr;
    std::vector<QWeight> egate, eup, edown;
    void *tm_gate = nullptr, *tm_up = nullptr, *tm_down = nullptr;
    bool grouped_ok = false;
};

constexpr int kPrefillChunk = 512;
constexpr int kTileRun = 16;             // runs of fewer tokens attend token by token
constexpr int kChunkRun = 32;            // runs of fewer tokens walk the gated delta rule token by token
constexpr int kStackChunk = 2048;      // tokens per pass of a checkpoint-directory design
constexpr int kTokTile = 8;
constexpr int kMoeGroupedTokens = 64;  // calls of at most this many tokens run the experts as one grouped launch

}  // namespace lc

using namespace lc;

struct lc_model {
    std::unique_ptr<LayerStack> stack;  // set: the layers of a checkpoint-directory design (layers.cu) instead of the Llama blocks below
    lc_model_config cfg{};
    int device = 0;
    cudaStream_t stream = nullptr;
    std::map<std::string, DevTensor> tensors;
    bool finalized = false;
    std::vector<LayerW> layers;
    QWeight head;
    const DevTensor* embed = nullptr;
    const float* final_norm = nullptr;
    std::vector<void*> owned;  // f32 copies of norm gains etc.

    // geometry: H, L, hd are the model's; nh, nkv, F, V, nqkv are THIS RANK'S part when the model is cut across ranks
    // (tp > 1: heads, kv heads, FFN rows and vocabulary rows divided by tp; experts e0 .. e0 + El - 1 of a mixture layer)
    int H = 0, L = 0, nh = 0, nkv = 0, hd = 0, F = 0, V = 0, nqkv = 0;
    int tp = 1, rank = 0, v0 = 0, e0 = 0, El = 0;
    bool use_dist = false;               // the ranks are other processes (lc_dist_init); else members lists them, or tp == 1
    std::vector<lc_model*> members;      // rank 0 of an in-process group: every rank's handle in rank order (itself first)
    lc_model* leader = nullptr;          // a rank > 0 of such a group
    float* d_part = nullptr;             // where the column-cut products leave their partial rows for the sum over the ranks
    long long* d_key = nullptr;          // greedy pick of the local vocabulary slice as (total-order key << 32 | global index)
    long long* d_key_max = nullptr;
    float* d_logits_all = nullptr;       // dist: the ranks' logit slices gathered for the host
    PrefillTile* d_tiles = nullptr;      // the call's tokens as runs of up to 64 consecutive positions of one sequence
    int n_tiles = 0;
    float* pending_dst = nullptr;        // where the next sum over the ranks has to land
    bool pending_pushed = false;         // ... and whether the product already sent its rows to the ranks
    GemvPush push_desc;
    int head_rows = 1;                   // rows the head works on at a time (logits and picks have room for as many)
    int page_tokens = 16, pages_per_seq = 0, pages_total = 0, max_seqs = 1, t_cap = 0;
    size_t kv_elt = 2;

    // KV cache
    std::vector<void*> k_pools, v_pools;  // per layer
    struct alignas(64) TmapBytes { unsigned char b[128]; };
    std::vector<TmapBytes> k_tmaps, v_tmaps;  // per layer: tensor maps over the key and value pools (f16 pools of 128-dim heads)
    bool k_tmaps_ok = false;
    std::vector<int> free_pages;
    std::vector<std::vector<int>> seq_pages;
    std::vector<int> seq_len;
    std::vector<char> seq_open;          // slots handed out by lc_seq_open
    int32_t* d_page_table = nullptr;
    std::vector<int32_t> h_page_table;
    bool page_table_dirty = true;

    // step buffers
    int64_t* d_tokens = nullptr;
    int32_t *d_tok_seq = nullptr, *d_tok_pos = nullptr, *d_tok_rope = nullptr, *d_last_idx = nullptr;
    float *d_hidden = nullptr, *d_hidden2 = nullptr, *d_qkv = nullptr, *d_attn = nullptr, *d_ffn = nullptr;
    float *d_last = nullptr, *d_logits = nullptr;
    bool seeded = false;          // lc_model_set_seed: stochastic sampling allowed, draws from seeded_uniform(seed, draws++)
    uint64_t seed = 0, draws = 0;
    int64_t* d_next = nullptr;
    int64_t* d_out_tokens = nullptr;
    size_t out_tokens_cap = 0;
    int32_t* d_step_ctr = nullptr;
    unsigned long long* d_stream_slots = nullptr;  // cross-CTA merge slots of the single-token attention kernel (zero between launches)
    // mixture-of-experts scratch: the router's picks and weights per token, per-expert slot counts and lists, the slots'
    // FFN hidden rows and outputs (calls of up to kMoeGroupedTokens tokens), every expert's output plane (larger calls)
    int32_t *d_moe_sel = nullptr, *d_moe_cnt = nullptr, *d_moe_lists = nullptr;
    float *d_moe_w = nullptr, *d_moe_h = nullptr, *d_moe_y = nullptr, *d_moe_yall = nullptr;
    GemvPlanes moe_planes_x, moe_planes_h;  // fixed-point activations of the grouped launches: the layer's input per token, the experts' hidden rows per slot
    unsigned long long* d_moe_touched = nullptr;  // experts that received a token, summed over layers and steps since the last read
    uint64_t expert_bytes_each = 0, expert_bytes_all = 0;
    double touched_per_step = 0.0;
    void* d_attn_scratch = nullptr;
    GemmWorkspace gemm_ws;  // f16 activation halves for the many-token tensor-core product
    bool any_unfused_qkv = false;  // some layer's q/k/v differ in type
    float* d_qkv_parts = nullptr;  // then: [T][nq] | [T][nkv hd] | [T][nkv hd] before they are interleaved into d_qkv
    int* d_attn_counters = nullptr;
    size_t attn_scratch_bytes = 0;
    unsigned long long* d_sanity = nullptr;

    std::map<int, cudaGraphExec_t> decode_graphs;
    int graph_nodes = 0;
    cudaEvent_t ev0 = nullptr, ev1 = nullptr;

    lc_counters ctr{};
    uint64_t launches_in_call = 0;

    // What the device-side per-token metadata currently describes (a decode step for these sequences at
    // these cache positions), so that consecutive one-token calls only have to send the token ids.
    bool meta_valid = false;
    std::vector<int> meta_seqs, meta_pos;
    // pinned staging for the per-step host <-> device traffic
    int64_t* pin_tokens = nullptr;
    int64_t* pin_next = nullptr;
    float* pin_logits = nullptr;
};

namespace lc {

struct DeviceGuard {
    int prev = 0;
    bool ok = false;
    explicit DeviceGuard(int dev) {
        if (cudaGetDevice(&prev) == cudaSuccess && cudaSetDevice(dev) == cudaSuccess) ok = true;
    }
    ~DeviceGuard() { if (ok) cudaSetDevice(prev); }
};

template <typename T>
inline int32_t dalloc(T** p, size_t count) {
    void* q = nullptr;
    cudaError_t e = cudaMalloc(&q, std::max<size_t>(count * sizeof(T), 16));
    if (e != cudaSuccess) {
        (void)cudaGetLastError();
        set_error("device allocation of %zu bytes failed: %s", count * sizeof(T), cudaGetErrorString(e));
        return LC_ERR_OOM;
    }
    *p = (T*)q;
    return LC_OK;
}

// A vector as f32 on the device (engine.cu).
int32_t model_gain_f32(lc_model* m, const std::string& name, int expect, const float** out);

// layers.cu: the layers of a checkpoint-directory design
int32_t stack_bind(lc_model* m);   // weights
int32_t stack_alloc(lc_model* m);  // cache, state and step buffers, sized by the handle's pool and slots
void stack_free(lc_model* m);
uint64_t stack_step_bytes(const lc_model* m, int ctx);
uint64_t stack_table_bytes(const lc_model* m);  // of tables of which a step reads one row per token (the embedding apart)
int32_t stack_upload_runs(lc_model* m, const std::vector<int32_t>& seq, const std::vector<int32_t>& pos);
int32_t stack_run_layers(lc_model* m, int T, bool decode_step);
int32_t stack_head(lc_model* m, int n, const int32_t* idx, float* logits);  // logits of rows idx (null: rows 0 .. n - 1)
int32_t stack_probe(lc_model* m, int l, int T, bool ffn, float** y);

}  // namespace lc
