// Attention of query heads over shared key/value heads in a paged cache, under a window with kept first tokens (MaskSpec) and
// with a sink: exp(sink[head]) joins the softmax denominator, without key or value.  Scores may be bounded by a tanh, outputs gated.
//   attn_prep_kernel    RMS norm over all of a token's q and over all of its k, rotation of halves, cache append
//   attn_head_prep_kernel  the same for norms per head or none: short convolutions, norm ahead of the rotation or behind it, either
//                       pairing, a factor per position on the queries
//   attn_plain_kernel   any shape, f32 arithmetic throughout; models in true 32-bit
//   attn_tokens_kernel  few tokens per sequence (decode): the query heads of one kv head of one token are the rows of the
//                       products; every warp walks key tiles of its own
//   attn_tiles_kernel   runs of many tokens: 64 consecutive queries of one head over key tiles of 64
// Both tile kernels walk only tiles that hold a visible key: those of the kept first tokens, then those from the window's
// lower edge on.  Scores, softmax and sums are f32; the weights enter the second product as two bf16 halves.
// Cache rows hold the key after norm and rotation, so a layer without projections of its own reads another layer's cache.  The
// rows of one page and kv head lie together in the form in which shared memory wants them (ldmatrix without bank conflicts): a
// row of a multiple of 64 elements has its 16-byte chunks at chunk ^ (position & 7), any other row is padded.  So a tile comes
// with one bulk copy per page for its keys and one for its values.
#include <algorithm>
#include <cmath>
#include <type_traits>
#include "lc_mixers.h"
#include "lc_mma.cuh"
#include "lc_tma.cuh"

namespace lc {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

// First key of the window and the number of kept keys before it.
struct Seen { int lo, keep; };
__device__ __forceinline__ Seen seen_from(const AttnShape& g, int pos) {
    Seen s;
    s.lo = g.window > 0 ? max(0, pos - g.window + 1) : 0;
    s.keep = min(g.keep_first, s.lo);
    return s;
}
// The tiles of `size` keys that hold a visible key, in order: n_first tiles from the start, then from tile `base` on.
struct Tiles {
    int n_first, base, n;
    __device__ __forceinline__ int at(int i) const { return i < n_first ? i : base + i - n_first; }
};
__device__ __forceinline__ Tiles tiles_of(const Seen& s, int last, int size) {
    Tiles t;
    t.base = s.lo / size;
    t.n_first = min((s.keep + size - 1) / size, t.base);
    t.n = t.n_first + last / size - t.base + 1;
    return t;
}

// A score in log2 units, bounded: k.x * tanh(dot * scale / cap) with k = (cap, 2 scale / cap) times log2 e.
__device__ __forceinline__ float2 cap_constants(const AttnShape& g) { return make_float2(g.cap * kLog2e, g.cap > 0.0f ? 2.0f * g.scale / g.cap * kLog2e : 0.0f); }
__device__ __forceinline__ float capped(float dot, float2 k) { return k.x - k.x * __fdividef(2.0f, 1.0f + exp2f(dot * k.y)); }
// The factor on all of head h of token t's output.
__device__ __forceinline__ float head_factor(const AttnArgs& a, size_t t, int h) { return a.head_gate ? sigmoid_f(a.head_gate[t * a.ld_proj + h]) : 1.0f; }
// The factor on element c of head h of token t's output.
template <typename A>
__device__ __forceinline__ float out_factor(const AttnArgs& a, size_t t, int h, int c) {
    return a.gate && c < a.g.vdim ? a.out_scale * sigmoid_f(act_f<A>(((const A*)a.gate)[t * a.ld_gate + (size_t)h * a.g.vdim + c])) : a.out_scale;
}
__device__ __forceinline__ float4 finished(const AttnArgs& a, size_t t, int h, int c, float4 x) {
    if (!a.gate && a.out_scale == 1.0f) return x;
    return make_float4(x.x * out_factor<bf16>(a, t, h, c), x.y * out_factor<bf16>(a, t, h, c + 1), x.z * out_factor<bf16>(a, t, h, c + 2), x.w * out_factor<bf16>(a, t, h, c + 3));
}

// Where element i of the cache row of position `pos` lies (swz: 7 or 0).
__device__ __forceinline__ int cell_of(int i, int pos, int swz) { return (((i >> 3) ^ (pos & swz)) << 3) + (i & 7); }
// Requests the keys and values of positions key .. key + n - 1 of one kv head (one thread).
__device__ __forceinline__ void request_rows(const AttnArgs& a, const int32_t* pt, int kvh, int key, int n, bf16* k_dst, bf16* v_dst, uint64_t* bar) {
    const AttnShape& g = a.g;
    while (n > 0) {
        const int page = key / a.page_tokens, slot = key - page * a.page_tokens, take = min(n, a.page_tokens - slot);
        const size_t row = ((size_t)pt[page] * g.kv_heads + kvh) * a.page_tokens + slot;
        bulk_load(k_dst, (const bf16*)a.k_cache + row * g.k_pitch, (uint32_t)(take * g.k_pitch * 2), bar);
        bulk_load(v_dst, (const bf16*)a.v_cache + row * g.v_pitch, (uint32_t)(take * g.v_pitch * 2), bar);
        key += take; n -= take;
        k_dst += take * g.k_pitch; v_dst += take * g.v_pitch;
    }
}

template <typename A> __device__ __forceinline__ void put4(A* p, float4 v);
template <> __device__ __forceinline__ void put4<float>(float* p, float4 v) { *(float4*)p = v; }
template <> __device__ __forceinline__ void put4<bf16>(bf16* p, float4 v) { *(uint2*)p = make_uint2(pack2(v.x, v.y), pack2(v.z, v.w)); }

// One CTA per token and share of its elements; VEC = 4: dim, vdim and the rotated half are multiples of four.
template <typename A, int VEC>
__global__ void __launch_bounds__(256) attn_prep_kernel(const AttnArgs a) {
    __shared__ float sh[32], sh2[32];
    pdl_launch_dependents();
    pdl_wait();
    const AttnShape& g = a.g;
    const int t = blockIdx.x, seq = a.tok_seq[t], pos = a.tok_pos[t], nq = g.heads * g.dim, nk = g.kv_heads * g.dim, half = g.rot_dims / 2;
    const bool own = a.off_k >= 0;
    const float *q = a.proj + (size_t)t * a.ld_proj, *k = q + (own ? a.off_k : 0), *v = q + a.off_v;
    const int page = a.page_table[(size_t)seq * a.pages_per_seq + pos / a.page_tokens], slot = pos % a.page_tokens;
    const float2* tab = a.rot + (size_t)pos * half;
    auto squares = [&](const float* x, int n) {
        float ss = 0.0f;
        if constexpr (VEC == 4) {
#pragma unroll 4
            for (int i = threadIdx.x * 4; i < n; i += 1024) {
                const float4 u = *(const float4*)(x + i);
                ss = fmaf(u.x, u.x, fmaf(u.y, u.y, fmaf(u.z, u.z, fmaf(u.w, u.w, ss))));
            }
        } else {
            for (int i = threadIdx.x; i < n; i += 256) ss = fmaf(x[i], x[i], ss);
        }
        return ss;
    };
    float sq = squares(q, nq), sk = own ? squares(k, nk) : 0.0f;
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) sh2[threadIdx.x >> 5] = sk;
    sq = block_sum_once(sq, sh);  // its barrier publishes the other warps' shares too
    sk = 0.0f;
    for (int w = 0; w < 8; w++) sk += sh2[w];
    const float rq = 1.0f / sqrtf(sq / (float)nq + a.eps), rk = own ? 1.0f / sqrtf(sk / (float)nk + a.eps) : 0.0f;
    // items of a head: VEC pairs of the rotated part, then VEC elements of the rest
    const int pairs = half / VEC, per = pairs + (g.dim - g.rot_dims) / VEC, start = blockIdx.y * 256 + threadIdx.x, step = gridDim.y * 256;
    auto item = [&](const float* x, const float* w, float r, A* row, int swz, int i) {
        auto dst = [&](int c) { return row + cell_of(c, pos, swz); };
        if constexpr (VEC == 4) {
            auto normed = [&](int c) {
                const float4 u = *(const float4*)(x + c), b = *(const float4*)(w + c);
                return make_float4(u.x * r * b.x, u.y * r * b.y, u.z * r * b.z, u.w * r * b.w);
            };
            if (i < pairs) {
                const float4 u = normed(4 * i), z = normed(half + 4 * i), cs0 = *(const float4*)(tab + 4 * i), cs1 = *(const float4*)(tab + 4 * i + 2);
                put4<A>(dst(4 * i), make_float4(u.x * cs0.x - z.x * cs0.y, u.y * cs0.z - z.y * cs0.w, u.z * cs1.x - z.z * cs1.y, u.w * cs1.z - z.w * cs1.w));
                put4<A>(dst(half + 4 * i), make_float4(z.x * cs0.x + u.x * cs0.y, z.y * cs0.z + u.y * cs0.w, z.z * cs1.x + u.z * cs1.y, z.w * cs1.z + u.w * cs1.w));
            } else {
                const int c = g.rot_dims + 4 * (i - pairs);
                put4<A>(dst(c), normed(c));
            }
        } else {
            if (i < pairs) {
                const float u = x[i] * r * w[i], z = x[half + i] * r * w[half + i];
                const float2 cs = tab[i];
                *dst(i) = to_act<A>(u * cs.x - z * cs.y);
                *dst(half + i) = to_act<A>(z * cs.x + u * cs.y);
            } else {
                const int c = g.rot_dims + i - pairs;
                *dst(c) = to_act<A>(x[c] * r * w[c]);
            }
        }
    };
    A* qo = (A*)a.q + (size_t)t * g.heads * g.dp;
    for (int i = start; i < g.heads * per; i += step) {
        const int h = i / per;
        item(q + h * g.dim, a.q_norm + h * g.dim, rq, qo + h * g.dp, 0, i - h * per);
    }
    if (!own) return;
    const size_t row0 = (size_t)page * g.kv_heads * a.page_tokens + slot;
    for (int i = start; i < g.kv_heads * per; i += step) {
        const int h = i / per;
        item(k + h * g.dim, a.k_norm + h * g.dim, rk, (A*)a.k_cache + (row0 + (size_t)h * a.page_tokens) * g.k_pitch, g.k_swz, i - h * per);
    }
    const int vper = g.vdim / VEC;
    for (int i = start; i < g.kv_heads * vper; i += step) {
        const int h = i / vper, c = (i - h * vper) * VEC;
        A* dst = (A*)a.v_cache + (row0 + (size_t)h * a.page_tokens) * g.v_pitch + cell_of(c, pos, g.v_swz);
        if constexpr (VEC == 4) put4<A>(dst, *(const float4*)(v + h * g.vdim + c));
        else dst[0] = to_act<A>(v[h * g.vdim + c]);
    }
}

// Norms per head: one warp per (stretch of tokens, head): the heads of q, then of k, then of v.  A lane owns four neighbouring
// elements, from 4 (lane + 32 p) on, and keeps its channels' last inputs while it walks the stretch (TAPS of them; 0: no
// convolution; -1: any number, re-read).  AHEAD: tokens whose rows, angles and pages are fetched together; behind the last one it
// is taken again, with the same result.
template <typename A, int TAPS, int NQ, int AHEAD>
__global__ void __launch_bounds__(256, NQ > 1 ? 1 : TAPS == 0 ? 4 : 3) attn_head_prep_kernel(const AttnArgs a, int stretch) {
    constexpr int kWin = TAPS > 1 ? TAPS - 1 : 1, kTaps = TAPS > 0 ? TAPS : 1, kTurn = NQ == 1 && TAPS == 0 ? 4 : 2;
    __shared__ float s_x[8][128 * NQ];
    pdl_launch_dependents();
    pdl_wait();
    const AttnShape& g = a.g;
    const int warp = warp_index(), lane = threadIdx.x & 31, unit = blockIdx.y * 8 + warp;
    if (unit >= g.heads + (a.off_k >= 0 ? 2 * g.kv_heads : 0)) return;
    const bool is_q = unit < g.heads, is_v = unit >= g.heads + g.kv_heads;
    const int h = is_q ? unit : is_v ? unit - g.heads - g.kv_heads : unit - g.heads, n = is_v ? g.vdim : g.dim, half = g.rot_dims / 2;
    const int nq = g.heads * g.dim, nk = g.kv_heads * g.dim, channels = nq + nk + g.kv_heads * g.vdim;
    const int ch0 = (is_q ? 0 : is_v ? nq + nk : nq) + h * n, col0 = (is_q ? 0 : is_v ? a.off_v : a.off_k) + h * n;
    const int taps = TAPS > 0 ? TAPS : g.taps;
    const bool vec = (n & 3) == 0;  // then a lane's elements exist together and lie 16-byte aligned in the projected rows
    const bool near = g.pairs == AttnPairs::Neighbours && !is_v, near4 = near && (half & 1) == 0;
    // halves whose partners lie a whole number of lanes apart: exchanged between lanes, angles fetched ahead
    const bool apart = kTurn == 4 && !is_v && half > 0 && !near && (half & 3) == 0;
    auto four_at = [&](const float* row, int c, float (&x)[4]) {
        if (vec) {
            const float4 u = c < n ? *(const float4*)(row + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            x[0] = u.x; x[1] = u.y; x[2] = u.z; x[3] = u.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; e++) x[e] = c + e < n ? row[c + e] : 0.0f;
        }
    };
    auto angles_at = [&](int pos, int c, float2 (&cs)[kTurn]) {  // of the pairs (c, c + 1) and (c + 2, c + 3), or of the four elements
#pragma unroll
        for (int i = 0; i < kTurn; i++) cs[i] = make_float2(1.0f, 0.0f);
        if constexpr (kTurn == 4)
            if (apart) {
                if (c >= 2 * half) return;
                const float4* p = (const float4*)(a.rot + (size_t)pos * half + (c < half ? c : c - half));
                const float4 u = __ldg(p), z = __ldg(p + 1);
                cs[0] = make_float2(u.x, u.y); cs[1] = make_float2(u.z, u.w); cs[2] = make_float2(z.x, z.y); cs[3] = make_float2(z.z, z.w);
                return;
            }
        const float2* tab = a.rot + (size_t)pos * half + c / 2;
        if (near4) {
            if (c < 2 * half) { const float4 u = __ldg((const float4*)tab); cs[0] = make_float2(u.x, u.y); cs[1] = make_float2(u.z, u.w); }
        } else if (near) {
            if (c < 2 * half) cs[0] = __ldg(tab);
            if (c + 2 < 2 * half) cs[1] = __ldg(tab + 1);
        }
    };
    const int t0 = blockIdx.x * stretch, t1 = min(a.T, t0 + stretch);
    float w[NQ][4][kTaps], win[NQ][4][kWin], gain[NQ][4];  // win[.][.][j]: the input j + 1 tokens back
    const float* gw = is_q ? a.q_norm : a.k_norm;
#pragma unroll
    for (int p = 0; p < NQ; p++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int c = 4 * (lane + 32 * p) + e;
            if constexpr (TAPS > 0)
#pragma unroll
                for (int j = 0; j < TAPS; j++) w[p][e][j] = c < n ? a.conv[(size_t)(ch0 + c) * TAPS + j] : 0.0f;
            gain[p][e] = g.norm != QkNorm::PerHead || is_v ? 1.0f : c < n ? gw[c] : 0.0f;
        }
    int prev_seq = -1, prev_pos = -1;
    float ahead[AHEAD][NQ][4];
    float2 turn[AHEAD][NQ][kTurn];
    int seq_a[AHEAD], pos_a[AHEAD], page_a[AHEAD];
    for (int tb = t0; tb < t1; tb += AHEAD) {
#pragma unroll
        for (int v = 0; v < AHEAD; v++) {
            const int t = min(tb + v, t1 - 1);
            seq_a[v] = a.tok_seq[t]; pos_a[v] = a.tok_pos[t];
            const float* row = a.proj + (size_t)t * a.ld_proj + col0;
#pragma unroll
            for (int p = 0; p < NQ; p++) {
                four_at(row, 4 * (lane + 32 * p), ahead[v][p]);
                angles_at(pos_a[v], 4 * (lane + 32 * p), turn[v][p]);
            }
            page_a[v] = is_q ? 0 : __ldg(a.page_table + (size_t)seq_a[v] * a.pages_per_seq + pos_a[v] / a.page_tokens);
        }
#pragma unroll
        for (int v = 0; v < AHEAD; v++) {
            const int t = min(tb + v, t1 - 1), seq = seq_a[v], pos = pos_a[v];
            // where the inputs j tokens back are: the call's rows as far as they belong to this run, the ring before that (zero before the start)
            auto back_row = [&](int j) {
                const int tt = max(t - j, 0);
                const bool here = t - j >= 0 && a.tok_seq[tt] == seq && a.tok_pos[tt] == pos - j;
                return here ? a.proj + (size_t)tt * a.ld_proj + col0 : a.ring + ((size_t)seq * taps + (pos >= j ? (pos - j) % taps : 0)) * channels + ch0;
            };
            float x[NQ][4];
            if constexpr (TAPS > 0)
                if (seq != prev_seq || pos != prev_pos + 1) {
#pragma unroll
                    for (int j = 1; j < TAPS; j++) {
                        const float* r = back_row(j);
#pragma unroll
                        for (int p = 0; p < NQ; p++)
#pragma unroll
                            for (int e = 0; e < 4; e++) {
                                const int c = 4 * (lane + 32 * p) + e;
                                win[p][e][j - 1] = pos >= j && c < n ? r[c] : 0.0f;
                            }
                    }
                }
            float ss = 0.0f;
#pragma unroll
            for (int p = 0; p < NQ; p++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const float u = ahead[v][p][e];
                    float y = u;
                    if constexpr (TAPS > 0) {
                        y = 0.0f;
#pragma unroll
                        for (int j = TAPS - 1; j > 0; j--) y = fmaf(w[p][e][TAPS - 1 - j], win[p][e][j - 1], y);
                        y = fmaf(w[p][e][TAPS - 1], u, y);
#pragma unroll
                        for (int j = TAPS - 2; j > 0; j--) win[p][e][j] = win[p][e][j - 1];
                        win[p][e][0] = u;
                    } else if constexpr (TAPS < 0) {
                        y = 0.0f;
                        const int c = 4 * (lane + 32 * p) + e;
                        if (c < n)
                            for (int j = taps - 1; j >= 0; j--) {
                                const float z = j == 0 ? u : pos >= j ? back_row(j)[c] : 0.0f;
                                y = fmaf(a.conv[(size_t)(ch0 + c) * taps + taps - 1 - j], z, y);
                            }
                    }
                    x[p][e] = y;
                    ss = fmaf(y, y, ss);
                }
            if (TAPS != 0 && a.one_each)
#pragma unroll
                for (int p = 0; p < NQ; p++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int c = 4 * (lane + 32 * p) + e;
                        if (c < n) a.ring[((size_t)seq * taps + pos % taps) * channels + ch0 + c] = ahead[v][p][e];
                    }
            prev_seq = seq; prev_pos = pos;
            if (!is_v) {
                if (g.norm == QkNorm::PerHead) {
                    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)n + a.eps);
#pragma unroll
                    for (int p = 0; p < NQ; p++)
#pragma unroll
                        for (int e = 0; e < 4; e++) x[p][e] *= r * gain[p][e];
                }
                if (near) {
#pragma unroll
                    for (int p = 0; p < NQ; p++)
#pragma unroll
                        for (int e = 0; e < 4; e += 2) {
                            const float2 cs = turn[v][p][e / 2];
                            const float y = x[p][e], z = x[p][e + 1];
                            x[p][e] = y * cs.x - z * cs.y;
                            x[p][e + 1] = z * cs.x + y * cs.y;
                        }
                } else if (kTurn == 4 && apart) {
                    const int c = 4 * lane, from = c < half ? lane + half / 4 : lane - half / 4;
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const float other = __shfl_sync(0xffffffffu, x[0][e], from & 31);
                        const float2 cs = turn[v][0][kTurn == 4 ? e : 0];
                        if (c < 2 * half) x[0][e] = x[0][e] * cs.x + (c < half ? -other : other) * cs.y;
                    }
                } else if (half > 0) {
                    const float2* tab = a.rot + (size_t)pos * half;
                    __syncwarp();
#pragma unroll
                    for (int p = 0; p < NQ; p++) *(float4*)(s_x[warp] + 4 * (lane + 32 * p)) = make_float4(x[p][0], x[p][1], x[p][2], x[p][3]);
                    __syncwarp();
#pragma unroll
                    for (int p = 0; p < NQ; p++)
#pragma unroll
                        for (int e = 0; e < 4; e++) {
                            const int c = 4 * (lane + 32 * p) + e;
                            if (c >= 2 * half) continue;
                            const float2 cs = tab[c < half ? c : c - half];
                            x[p][e] = c < half ? x[p][e] * cs.x - s_x[warp][c + half] * cs.y : x[p][e] * cs.x + s_x[warp][c - half] * cs.y;
                        }
                }
                if (g.norm == QkNorm::PerHeadAfter) {
                    ss = 0.0f;
#pragma unroll
                    for (int p = 0; p < NQ; p++)
#pragma unroll
                        for (int e = 0; e < 4; e++) ss = fmaf(x[p][e], x[p][e], ss);
                    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)n + a.eps);
#pragma unroll
                    for (int p = 0; p < NQ; p++)
#pragma unroll
                        for (int e = 0; e < 4; e++) x[p][e] *= r;
                }
            }
            if (is_q && a.q_factor) {
                const float f = __ldg(a.q_factor + pos);
#pragma unroll
                for (int p = 0; p < NQ; p++)
#pragma unroll
                    for (int e = 0; e < 4; e++) x[p][e] *= f;
            }
            A* dst;
            int swz = 0;
            if (is_q) dst = (A*)a.q + ((size_t)t * g.heads + h) * g.dp;
            else {
                const size_t at = ((size_t)page_a[v] * g.kv_heads + h) * a.page_tokens + pos % a.page_tokens;
                dst = is_v ? (A*)a.v_cache + at * g.v_pitch : (A*)a.k_cache + at * g.k_pitch;
                swz = is_v ? g.v_swz : g.k_swz;
            }
#pragma unroll
            for (int p = 0; p < NQ; p++) {
                const int c = 4 * (lane + 32 * p);
                if (c >= n) continue;
                A* d = dst + cell_of(c, pos, swz);
                if (vec) put4<A>(d, make_float4(x[p][0], x[p][1], x[p][2], x[p][3]));
                else
#pragma unroll
                    for (int e = 0; e < 4; e++)
                        if (c + e < n) d[e] = to_act<A>(x[p][e]);
            }
        }
    }
}

// The inputs of a run's last `taps` positions, for the convolutions of the next call.
__global__ void __launch_bounds__(256) attn_keep_kernel(const AttnArgs a, const SeqRun* __restrict__ runs) {
    pdl_launch_dependents();
    pdl_wait();
    const AttnShape& g = a.g;
    const SeqRun run = runs[blockIdx.x];
    const int nq = g.heads * g.dim, nk = g.kv_heads * g.dim, channels = nq + nk + g.kv_heads * g.vdim, ch = blockIdx.y * 256 + threadIdx.x;
    if (ch >= channels) return;
    const int col = ch < nq ? ch : ch < nq + nk ? a.off_k + ch - nq : a.off_v + ch - nq - nk;
    for (int t = max(0, run.n - g.taps); t < run.n; t++)
        a.ring[((size_t)run.seq * g.taps + (run.pos0 + t) % g.taps) * channels + ch] = a.proj[(size_t)(run.tok0 + t) * a.ld_proj + col];
}

// One CTA per (head, token), a key per thread.
constexpr int kPlainThreads = 128;
template <typename A>
__global__ void __launch_bounds__(kPlainThreads) attn_plain_kernel(const AttnArgs a) {
    extern __shared__ float smf[];
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const AttnShape& g = a.g;
    const int h = blockIdx.x, t = blockIdx.y, seq = a.tok_seq[t], pos = a.tok_pos[t], kvh = h / (g.heads / g.kv_heads);
    float *s_q = smf, *s_o = s_q + g.dim, *s_p = s_o + g.vdim;
    size_t* s_row = (size_t*)(s_p + kPlainThreads + ((g.dim + g.vdim) & 1));
    const A* q = (const A*)a.q + ((size_t)t * g.heads + h) * g.dp;
    for (int i = threadIdx.x; i < g.dim; i += kPlainThreads) s_q[i] = act_f<A>(q[i]);
    for (int i = threadIdx.x; i < g.vdim; i += kPlainThreads) s_o[i] = 0.0f;
    __syncthreads();
    const int32_t* pt = a.page_table + (size_t)seq * a.pages_per_seq;
    const Seen sn = seen_from(g, pos);
    const int n = sn.keep + pos - sn.lo + 1;  // visible keys: the kept ones, then the window
    float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.0f : 0.0f;
    for (int k0 = 0; k0 < n; k0 += kPlainThreads) {
        const int i = k0 + threadIdx.x, key = i < sn.keep ? i : sn.lo + i - sn.keep;
        float sc = -INFINITY;
        if (i < n) {
            const size_t row = ((size_t)pt[key / a.page_tokens] * g.kv_heads + kvh) * a.page_tokens + key % a.page_tokens;
            s_row[threadIdx.x] = row;
            const A* kr = (const A*)a.k_cache + row * g.k_pitch;
            float d = 0.0f;
            for (int c = 0; c < g.dim; c++) d = fmaf(s_q[c], act_f<A>(kr[cell_of(c, key, g.k_swz)]), d);
            sc = d * g.scale;
            if (g.cap > 0.0f) sc = g.cap * tanhf(sc / g.cap);
        }
        const float mt = fmaxf(m, block_max(sc, red));
        const float p = i < n ? expf(sc - mt) : 0.0f, corr = expf(m - mt);
        s_p[threadIdx.x] = p;
        l = l * corr + block_sum(p, red);
        m = mt;
        const int nk = min(kPlainThreads, n - k0);
        for (int c = threadIdx.x; c < g.vdim; c += kPlainThreads) {
            float o = 0.0f;
            for (int j = 0; j < nk; j++) {
                const int at = k0 + j, key = at < sn.keep ? at : sn.lo + at - sn.keep;
                o = fmaf(s_p[j], act_f<A>(((const A*)a.v_cache)[s_row[j] * g.v_pitch + cell_of(c, key, g.v_swz)]), o);
            }
            s_o[c] = fmaf(s_o[c], corr, o);
        }
        __syncthreads();
    }
    A* out = (A*)a.out + (size_t)t * a.ldo + (size_t)h * g.ep;
    const float hf = head_factor(a, t, h);
    for (int c = threadIdx.x; c < g.ep; c += kPlainThreads) out[c] = to_act<A>(c < g.vdim ? s_o[c] / l * hf * out_factor<A>(a, t, h, c) : 0.0f);
}

// ---- few tokens per sequence ------------------------------------------------------------------------------------------------
// A CTA of four warps takes up to 16 query heads of one kv head of one token and a piece of its key tiles (16 keys each); the
// warps deal the tiles among themselves, each with its own ring of copies in flight and its own running softmax, and meet at
// the end.  Several pieces: the CTA that finishes last merges them.
constexpr int kPartCells = 12;  // CTAs per SM whose partial sums there is room for
constexpr int kDecKeys = 16, kDecStages = 2, kDecWarps = 4, kMaxPieces = 32;
struct AttnParts { float *o, *ml; unsigned* tickets; };  // [token][kv head][row block][piece][16][ep], [..][16][2] (log2 units)

template <int NV, bool CAP>
__global__ void __launch_bounds__(32 * kDecWarps) attn_tokens_kernel(const AttnArgs a, const AttnParts pt_out, int* error_flag) {
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ float s_ml[kDecWarps][16][2], s_scale[kMaxPieces][16];
    __shared__ uint64_t s_full[kDecWarps][kDecStages];
    __shared__ int s_last;
    const AttnShape& g = a.g;
    const int d16 = (g.dp + 15) & ~15, qp = d16 + 8, qb = qp * 2, kb_row = g.k_pitch * 2, vb_row = g.v_pitch * 2;
    const int tid = threadIdx.x, warp = warp_index(), lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
    const int rep = g.heads / g.kv_heads, blocks = (rep + 15) / 16, t = blockIdx.x, kvh = blockIdx.y / blocks, r0 = (blockIdx.y % blocks) * 16, nh = min(16, rep - r0),
              h0 = kvh * rep + r0, pieces = gridDim.z;
    bf16 *s_q = (bf16*)smem, *s_k = s_q + 16 * qp + (size_t)warp * kDecStages * kDecKeys * (g.k_pitch + g.v_pitch), *s_v = s_k + kDecStages * kDecKeys * g.k_pitch;
    uint64_t* full = s_full[warp];
    if (lane == 0) {
        for (int i = 0; i < kDecStages; i++) mbar_init(&full[i], 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    pdl_launch_dependents();
    __syncwarp();
    pdl_wait();
    const int seq = a.tok_seq[t], pos = a.tok_pos[t];
    const Seen sn = seen_from(g, pos);
    const Tiles tl = tiles_of(sn, pos, kDecKeys);
    const int per = (tl.n + pieces - 1) / pieces, i0 = blockIdx.z * per, i1 = min(tl.n, i0 + per), mine = i1 > i0 + warp ? (i1 - i0 - warp + kDecWarps - 1) / kDecWarps : 0;
    const int32_t* pt = a.page_table + (size_t)seq * a.pages_per_seq;
    const uint32_t q_sm = smem_u32(s_q), k_sm = smem_u32(s_k), v_sm = smem_u32(s_v);
    auto load = [&](int j) {
        if (lane == 0 && j < mine) {
            const int st = j % kDecStages, key = tl.at(i0 + warp + j * kDecWarps) * kDecKeys, n = min(kDecKeys, pos + 1 - key);
            mbar_expect_tx(&full[st], (uint32_t)(n * (g.k_pitch + g.v_pitch) * 2));
            request_rows(a, pt, kvh, key, n, s_k + st * kDecKeys * g.k_pitch, s_v + st * kDecKeys * g.v_pitch, &full[st]);
        }
    };
    for (int j = 0; j < kDecStages; j++) load(j);
    for (int i = tid; i < 16 * (d16 / 8); i += 32 * kDecWarps) {
        const int r = i / (d16 / 8), c = (i - r * (d16 / 8)) * 8;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < nh && c < g.dp) v = *(const uint4*)((const bf16*)a.q + ((size_t)t * g.heads + h0 + r) * g.dp + c);
        *(uint4*)(s_q + r * qp + c) = v;
    }
    __syncthreads();
    float o[NV][4], m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < NV; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const float sc = g.scale * kLog2e;
    const float2 ck = cap_constants(g);
    const uint32_t qa = q_sm + (uint32_t)((lane & 15) * qb + (lane >> 4) * 16);
    const int krow = (lane & 7) + ((lane >> 4) << 3), kx = krow & g.k_swz, kc = (lane >> 3) & 1, vx = lane & 15 & g.v_swz, vc = lane >> 4;
    for (int j = 0; j < mine; j++) {
        const int st = j % kDecStages, key0 = tl.at(i0 + warp + j * kDecWarps) * kDecKeys;
        if (!mbar_wait(&full[st], (uint32_t)(j / kDecStages) & 1)) atomicCAS(error_flag, 0, 15);
        if (key0 + kDecKeys > pos + 1) {  // the rows behind the token: their weights are zero, the values have to be finite
            for (int i = lane; i < (key0 + kDecKeys - pos - 1) * (g.v_pitch / 8); i += 32) *(uint4*)(s_v + (st * kDecKeys + pos + 1 - key0) * g.v_pitch + i * 8) = make_uint4(0u, 0u, 0u, 0u);
            __syncwarp();
        }
        float s[2][4];
#pragma unroll
        for (int i = 0; i < 2; i++) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
        const uint32_t ka = k_sm + (uint32_t)((st * kDecKeys + krow) * kb_row);
#pragma unroll 4
        for (int k = 0; k < d16 / 16; k++) {
            uint32_t q4[4], kb[4];
            ldsm4(qa + k * 32, q4);
            ldsm4(ka + (uint32_t)(((2 * k + kc) ^ kx) << 4), kb);
            mma_bf16(s[0], q4, kb[0], kb[1]);
            mma_bf16(s[1], q4, kb[2], kb[3]);
        }
        const bool edge = key0 + kDecKeys > pos + 1 || key0 < sn.lo;
        float mx[2] = {m_run[0], m_run[1]};
#pragma unroll
        for (int i = 0; i < 2; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                s[i][e] = CAP ? capped(s[i][e], ck) : s[i][e] * sc;
                if (edge) {
                    const int key = key0 + 8 * i + 2 * t4 + (e & 1);
                    if (key > pos || (key < sn.lo && key >= sn.keep)) s[i][e] = -INFINITY;
                }
                mx[e >> 1] = fmaxf(mx[e >> 1], s[i][e]);
            }
        float corr[2], sum[2] = {0.0f, 0.0f};
#pragma unroll
        for (int r = 0; r < 2; r++) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));  // finite: every tile holds a visible key
            corr[r] = exp2f(m_run[r] - mx[r]);
            m_run[r] = mx[r];
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int i = 0; i < 2; i++) {
            float p[4];
#pragma unroll
            for (int e = 0; e < 4; e++) { p[e] = exp2f(s[i][e] - m_run[e >> 1]); sum[e >> 1] += p[e]; }
            split2(p[0], p[1], ph[2 * i], pl[2 * i]);
            split2(p[2], p[3], ph[2 * i + 1], pl[2 * i + 1]);
        }
#pragma unroll
        for (int r = 0; r < 2; r++) l_run[r] = l_run[r] * corr[r] + sum[r];  // this lane's share of the row
#pragma unroll
        for (int r = 0; r < 2; r++) corr[r] = r == 0 || nh > 8 ? corr[r] : 1.0f;
        if (__any_sync(0xffffffffu, corr[0] != 1.0f || corr[1] != 1.0f))
#pragma unroll
            for (int i = 0; i < NV; i++) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
        const uint32_t va = v_sm + (uint32_t)((st * kDecKeys + (lane & 15)) * vb_row);
#pragma unroll
        for (int np = 0; np < NV / 2; np++) {
            if (16 * np >= g.ep) break;
            uint32_t b[4];
            ldsm4t(va + (uint32_t)(((2 * np + vc) ^ vx) << 4), b);
            mma_bf16(o[2 * np], ph, b[0], b[1]);
            mma_bf16(o[2 * np + 1], ph, b[2], b[3]);
            mma_bf16(o[2 * np], pl, b[0], b[1]);
            mma_bf16(o[2 * np + 1], pl, b[2], b[3]);
        }
        __syncwarp();
        load(j + kDecStages);
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    }
    __syncthreads();  // the copies' buffers become the warps' sums: [warp][16][ep]
    float* s_o = (float*)(s_q + 16 * qp);
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int row = g8 + 8 * r;
        if (row < nh) {
            if (t4 == 0) { s_ml[warp][row][0] = m_run[r]; s_ml[warp][row][1] = l_run[r]; }
#pragma unroll
            for (int i = 0; i < NV; i++)
                if (8 * i < g.ep) *(float2*)(s_o + ((size_t)warp * 16 + row) * g.ep + 8 * i + 2 * t4) = make_float2(o[i][2 * r], o[i][2 * r + 1]);
        }
    }
    __syncthreads();
    auto sink_of = [&](int row) { return a.sink ? a.sink[h0 + row] * kLog2e : -INFINITY; };
    if (tid < nh) {  // the warps' factors; with one piece also the sink and the division
        float m = pieces == 1 ? sink_of(tid) : -INFINITY;
        for (int w = 0; w < kDecWarps; w++) m = fmaxf(m, s_ml[w][tid][0]);
        float l = pieces == 1 && a.sink ? exp2f(sink_of(tid) - m) : 0.0f, f[kDecWarps];
        for (int w = 0; w < kDecWarps; w++) {
            f[w] = m == -INFINITY ? 0.0f : exp2f(s_ml[w][tid][0] - m);
            l += f[w] * s_ml[w][tid][1];
        }
        const float last = pieces == 1 ? head_factor(a, t, h0 + tid) / l : 1.0f;
        for (int w = 0; w < kDecWarps; w++) s_scale[w][tid] = f[w] * last;
        if (pieces > 1) {
            float* ml = pt_out.ml + ((((size_t)t * gridDim.y + blockIdx.y) * pieces + blockIdx.z) * 16 + tid) * 2;
            ml[0] = m; ml[1] = l;
        }
    }
    __syncthreads();
    const int vec = g.ep / 4;
    const size_t cell = (size_t)t * gridDim.y + blockIdx.y;
    for (int i = tid; i < nh * vec; i += 32 * kDecWarps) {
        const int row = i / vec, c = (i - row * vec) * 4;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int w = 0; w < kDecWarps; w++) {
            const float f = s_scale[w][row];
            const float4 v = *(const float4*)(s_o + ((size_t)w * 16 + row) * g.ep + c);
            x.x = fmaf(f, v.x, x.x); x.y = fmaf(f, v.y, x.y); x.z = fmaf(f, v.z, x.z); x.w = fmaf(f, v.w, x.w);
        }
        if (pieces == 1) put4<bf16>((bf16*)a.out + (size_t)t * a.ldo + (size_t)(h0 + row) * g.ep + c, finished(a, t, h0 + row, c, x));
        else *(float4*)(pt_out.o + ((cell * pieces + blockIdx.z) * 16 + row) * g.ep + c) = x;
    }
    if (pieces == 1) return;
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        s_last = atomicAdd(pt_out.tickets + cell, 1u) == (unsigned)pieces - 1;
        if (s_last) pt_out.tickets[cell] = 0;
        __threadfence();
    }
    __syncthreads();
    if (!s_last) return;
    for (int row = warp; row < nh; row += kDecWarps) {  // a lane per piece
        const float* ml = pt_out.ml + ((cell * pieces + min(lane, pieces - 1)) * 16 + row) * 2;
        const float pm = lane < pieces ? __ldcg(ml) : -INFINITY, pl = lane < pieces ? __ldcg(ml + 1) : 0.0f, sk = sink_of(row), m = fmaxf(warp_max(pm), sk);
        const float f = pm == -INFINITY ? 0.0f : exp2f(pm - m), l = warp_sum(f * pl) + (a.sink ? exp2f(sk - m) : 0.0f);
        if (lane < pieces) s_scale[lane][row] = f / l * head_factor(a, t, h0 + row);
    }
    __syncthreads();
    for (int i = tid; i < nh * vec; i += 32 * kDecWarps) {
        const int row = i / vec, c = (i - row * vec) * 4;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        const float* src = pt_out.o + (cell * pieces * 16 + row) * g.ep + c;
#pragma unroll 8
        for (int p = 0; p < pieces; p++) {
            const float f = s_scale[p][row];
            const float4 v = __ldcg((const float4*)(src + (size_t)p * 16 * g.ep));
            x.x = fmaf(f, v.x, x.x); x.y = fmaf(f, v.y, x.y); x.z = fmaf(f, v.z, x.z); x.w = fmaf(f, v.w, x.w);
        }
        put4<bf16>((bf16*)a.out + (size_t)t * a.ldo + (size_t)(h0 + row) * g.ep + c, finished(a, t, h0 + row, c, x));
    }
}

// ---- runs of many tokens ----------------------------------------------------------------------------------------------------
constexpr int kKeys = 64;
template <int NV, bool CAP>
__global__ void __launch_bounds__(128) attn_tiles_kernel(const AttnArgs a, const AttnTile* __restrict__ tiles, int* error_flag) {
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ uint64_t full[2];
    const AttnShape& g = a.g;
    const int d16 = (g.dp + 15) & ~15, qp = d16 + 8, qb = qp * 2, kb_row = g.k_pitch * 2, vb_row = g.v_pitch * 2;
    bf16 *s_q = (bf16*)smem, *s_k = s_q + 64 * qp, *s_v = s_k + 2 * kKeys * g.k_pitch;
    const int tid = threadIdx.x, warp = warp_index(), lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
    if (tid == 0) {
        mbar_init(&full[0], 1);
        mbar_init(&full[1], 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    pdl_launch_dependents();
    pdl_wait();
    const AttnTile tl = tiles[gridDim.x - 1 - blockIdx.x];  // the tiles with the longest contexts first
    const int h = blockIdx.y, kvh = h / (g.heads / g.kv_heads), last = tl.pos0 + tl.n - 1;
    const Seen sn = seen_from(g, tl.pos0);  // of the first query: no other sees an earlier window
    Tiles kt = tiles_of(sn, last, kKeys);
    kt.n_first = min((g.keep_first + kKeys - 1) / kKeys, kt.base);
    kt.n = kt.n_first + last / kKeys - kt.base + 1;
    const int32_t* pt = a.page_table + (size_t)tl.seq * a.pages_per_seq;
    const uint32_t q_sm = smem_u32(s_q), k_sm = smem_u32(s_k), v_sm = smem_u32(s_v);
    auto load = [&](int i) {  // warp 0: a lane per 16 keys
        if (warp != 0 || i >= kt.n) return;
        const int key0 = kt.at(i) * kKeys, n = min(kKeys, last + 1 - key0), buf = i & 1;
        if (lane == 0) mbar_expect_tx(&full[buf], (uint32_t)(n * (g.k_pitch + g.v_pitch) * 2));
        __syncwarp();
        if (lane * 16 < n) request_rows(a, pt, kvh, key0 + lane * 16, min(16, n - lane * 16), s_k + (buf * kKeys + lane * 16) * g.k_pitch, s_v + (buf * kKeys + lane * 16) * g.v_pitch, &full[buf]);
        __syncwarp();
    };
    __syncwarp();
    load(0);
    load(1);
    for (int i = tid; i < 64 * (d16 / 8); i += 128) {
        const int r = i / (d16 / 8), c = (i - r * (d16 / 8)) * 8;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < tl.n && c < g.dp) v = *(const uint4*)((const bf16*)a.q + ((size_t)(tl.tok0 + r) * g.heads + h) * g.dp + c);
        *(uint4*)(s_q + r * qp + c) = v;
    }
    __syncthreads();
    float o[NV][4], m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < NV; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const float sc = g.scale * kLog2e;
    const float2 ck = cap_constants(g);
    const int q0 = warp * 16, pa = tl.pos0 + q0, pb = min(pa + 15, last), qpos[2] = {pa + g8, pa + g8 + 8};
    const int wlo_a = g.window > 0 ? max(0, pa - g.window + 1) : 0, wlo_b = g.window > 0 ? max(0, pb - g.window + 1) : 0;
    const int qlo[2] = {g.window > 0 ? qpos[0] - g.window + 1 : 0, g.window > 0 ? qpos[1] - g.window + 1 : 0};
    const int krow = (lane & 7) + ((lane >> 4) << 3), kx = krow & g.k_swz, kc = (lane >> 3) & 1, vx = lane & 15 & g.v_swz, vc = lane >> 4;
    for (int i = 0; i < kt.n; i++) {
        const int buf = i & 1, key0 = kt.at(i) * kKeys;
        if (!mbar_wait(&full[buf], (uint32_t)(i >> 1) & 1)) atomicCAS(error_flag, 0, 16);
        if (key0 + kKeys > last + 1) {  // the rows behind the last query: their weights are zero, the values have to be finite
            for (int c = tid; c < (key0 + kKeys - last - 1) * (g.v_pitch / 8); c += 128) *(uint4*)(s_v + (buf * kKeys + last + 1 - key0) * g.v_pitch + c * 8) = make_uint4(0u, 0u, 0u, 0u);
            __syncthreads();
        }
        if (q0 < tl.n && key0 <= pb && (key0 + kKeys > wlo_a || key0 < g.keep_first)) {
            float s[8][4];
#pragma unroll
            for (int n = 0; n < 8; n++) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.0f;
            const uint32_t qa = q_sm + (uint32_t)((q0 + (lane & 15)) * qb + (lane >> 4) * 16), ka = k_sm + (uint32_t)((buf * kKeys + krow) * kb_row);
#pragma unroll 2
            for (int k = 0; k < d16 / 16; k++) {
                uint32_t q4[4];
                ldsm4(qa + k * 32, q4);
#pragma unroll
                for (int n = 0; n < 4; n++) {
                    uint32_t kb[4];
                    ldsm4(ka + (uint32_t)(16 * n * kb_row + (((2 * k + kc) ^ kx) << 4)), kb);
                    mma_bf16(s[2 * n], q4, kb[0], kb[1]);
                    mma_bf16(s[2 * n + 1], q4, kb[2], kb[3]);
                }
            }
            const bool edge = key0 + kKeys - 1 > pa || key0 < wlo_b;
            float mx[2] = {m_run[0], m_run[1]}, base[2], corr[2], sum[2] = {0.0f, 0.0f};
#pragma unroll
            for (int n = 0; n < 8; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    float v = CAP ? capped(s[n][e], ck) : s[n][e] * sc;
                    if (edge) {
                        const int key = key0 + 8 * n + 2 * t4 + (e & 1), r = e >> 1;
                        if (key > qpos[r] || (key < qlo[r] && key >= g.keep_first)) v = -INFINITY;
                    }
                    s[n][e] = v;
                    mx[e >> 1] = fmaxf(mx[e >> 1], v);
                }
#pragma unroll
            for (int r = 0; r < 2; r++) {
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
                base[r] = mx[r] == -INFINITY ? 0.0f : mx[r];  // a query whose window starts behind this tile has seen no key yet
                corr[r] = exp2f(m_run[r] - base[r]);
                m_run[r] = mx[r];
            }
            uint32_t ph[4][4], pl[4][4];
#pragma unroll
            for (int n = 0; n < 8; n++) {
                float p[4];
#pragma unroll
                for (int e = 0; e < 4; e++) { p[e] = exp2f(s[n][e] - base[e >> 1]); sum[e >> 1] += p[e]; }
                const int ks = n >> 1, hs = (n & 1) * 2;
                split2(p[0], p[1], ph[ks][hs], pl[ks][hs]);
                split2(p[2], p[3], ph[ks][hs + 1], pl[ks][hs + 1]);
            }
#pragma unroll
            for (int r = 0; r < 2; r++) l_run[r] = l_run[r] * corr[r] + sum[r];  // this lane's share of the row
#pragma unroll
            for (int n = 0; n < NV; n++) { o[n][0] *= corr[0]; o[n][1] *= corr[0]; o[n][2] *= corr[1]; o[n][3] *= corr[1]; }
            const uint32_t va = v_sm + (uint32_t)((buf * kKeys + (lane & 15)) * vb_row);
#pragma unroll
            for (int ks = 0; ks < 4; ks++)
#pragma unroll
                for (int np = 0; np < NV / 2; np++) {
                    if (16 * np >= g.ep) break;
                    uint32_t b[4];
                    ldsm4t(va + (uint32_t)(16 * ks * vb_row + (((2 * np + vc) ^ vx) << 4)), b);
                    mma_bf16(o[2 * np], ph[ks], b[0], b[1]);
                    mma_bf16(o[2 * np + 1], ph[ks], b[2], b[3]);
                    mma_bf16(o[2 * np], pl[ks], b[0], b[1]);
                    mma_bf16(o[2 * np + 1], pl[ks], b[2], b[3]);
                }
        }
        __syncthreads();
        load(i + 2);
    }
    const float sink = a.sink ? a.sink[h] * kLog2e : -INFINITY;
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int row = q0 + g8 + 8 * r;
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
        if (row >= tl.n) continue;
        const float m = fmaxf(m_run[r], sink), f = exp2f(m_run[r] - m), inv = f / (l_run[r] * f + (a.sink ? exp2f(sink - m) : 0.0f)) * head_factor(a, tl.tok0 + row, h);
        bf16* dst = (bf16*)a.out + (size_t)(tl.tok0 + row) * a.ldo + (size_t)h * g.ep + 2 * t4;
#pragma unroll
        for (int n = 0; n < NV; n++) {
            if (8 * n >= g.ep) continue;
            float2 x = make_float2(o[n][2 * r] * inv, o[n][2 * r + 1] * inv);
            if (a.gate || a.out_scale != 1.0f) {
                const int c = 8 * n + 2 * t4;
                x.x *= out_factor<bf16>(a, tl.tok0 + row, h, c);
                x.y *= out_factor<bf16>(a, tl.tok0 + row, h, c + 1);
            }
            *(uint32_t*)(dst + 8 * n) = pack2(x.x, x.y);
        }
    }
}

int value_tiles(int ep) { return ep <= 32 ? 4 : ep <= 64 ? 8 : ep <= 96 ? 12 : ep <= 128 ? 16 : 32; }
size_t tokens_smem(const AttnShape& g) {
    const size_t qp = ((g.dp + 15) & ~15) + 8;
    return (16 * qp + (size_t)kDecWarps * std::max((size_t)kDecStages * kDecKeys * (g.k_pitch + g.v_pitch), (size_t)16 * g.ep * 2)) * 2;
}
size_t tiles_smem(const AttnShape& g) {
    const size_t qp = ((g.dp + 15) & ~15) + 8;
    return (64 * qp + 2 * kKeys * ((size_t)g.k_pitch + g.v_pitch)) * 2;
}
int pitch_of(int n8, bool f32, int* swz) {
    const int chunks = n8 / 8;
    *swz = !f32 && chunks % 8 == 0 ? 7 : 0;
    if (f32 || *swz) return n8;
    return chunks % 2 ? n8 + 16 : n8 + 8;  // an odd number of chunks; an odd row is followed by a chunk of zeros, since products take 16 columns
}
bool tensor_form(const AttnShape& g, bool f32) { return !f32 && g.ep <= 256 && tokens_smem(g) <= kMaxSmem - 4096 && tiles_smem(g) <= kMaxSmem - 1024; }
template <typename A, int TAPS>
int32_t head_prep_taps(const AttnArgs& a, cudaStream_t s) {
    const int widest = std::max(a.g.dim, a.g.vdim);
    auto go = [&](auto kern, int stretch) -> int32_t {
        const dim3 grid((unsigned)((a.T + stretch - 1) / stretch), (unsigned)((a.g.heads + (a.off_k >= 0 ? 2 * a.g.kv_heads : 0) + 7) / 8));
        LC_CUDA(launch_pdl(kern, grid, dim3(256), 0, s, a, stretch));
        return LC_OK;
    };
    LC_CHECK(widest <= 512, LC_ERR_UNSUPPORTED, "attention: heads of %d and %d dimensions (at most 512)", a.g.dim, a.g.vdim);
    if constexpr (sizeof(A) == 2 && TAPS >= 0)
        if (a.T >= 256 && widest <= 128) return go(attn_head_prep_kernel<A, TAPS, 1, 2>, TAPS ? 16 : 4);
    const int stretch = a.T < 256 ? 1 : 8;
    return widest <= 128 ? go(attn_head_prep_kernel<A, TAPS, 1, 1>, stretch) : widest <= 256 ? go(attn_head_prep_kernel<A, TAPS, 2, 1>, stretch)
                                                                                             : go(attn_head_prep_kernel<A, TAPS, 4, 1>, stretch);
}
template <typename A>
int32_t head_prep(const AttnArgs& a, cudaStream_t s) {
    LC_CHECK(a.off_k >= 0 || a.g.taps == 0, LC_ERR_UNSUPPORTED, "attention: convolutions over another layer's cache");
    switch (a.g.taps) {
        case 0: return head_prep_taps<A, 0>(a, s);
        case 2: return head_prep_taps<A, 2>(a, s);
        case 3: return head_prep_taps<A, 3>(a, s);
        case 4: return head_prep_taps<A, 4>(a, s);
        default: return head_prep_taps<A, -1>(a, s);
    }
}
int cells(const AttnShape& g) { return g.kv_heads * ((g.heads / g.kv_heads + 15) / 16); }

}  // namespace

void attn_cache_layout(AttnShape* g, bool f32) {
    g->k_pitch = pitch_of(g->dp, f32, &g->k_swz);
    g->v_pitch = pitch_of(g->ep, f32, &g->v_swz);
}

int32_t launch_attn_keep(const AttnArgs& a, const SeqRun* runs, int n_runs, cudaStream_t s) {
    const int channels = (a.g.heads + a.g.kv_heads) * a.g.dim + a.g.kv_heads * a.g.vdim;
    LC_CUDA(launch_pdl(attn_keep_kernel, dim3((unsigned)n_runs, (unsigned)((channels + 255) / 256)), dim3(256), 0, s, a, runs));
    return LC_OK;
}

int32_t launch_attn_prep(const AttnArgs& a, cudaStream_t s) {
    const AttnShape& g = a.g;
    if (g.norm != QkNorm::AllHeads) return a.f32 ? head_prep<float>(a, s) : head_prep<bf16>(a, s);
    LC_CHECK(g.pairs == AttnPairs::Halves && g.taps == 0 && !a.q_factor, LC_ERR_UNSUPPORTED, "attention: norms over all heads with neighbouring pairs, convolutions or factors on queries");
    const bool vec = g.dim % 4 == 0 && g.vdim % 4 == 0 && g.rot_dims % 8 == 0;
    // few tokens: several CTAs each, all of which sum the whole rows
    const dim3 grid((unsigned)a.T, (unsigned)(a.T < 32 ? std::max(1, std::min(8, (g.heads + g.kv_heads) * g.dim / 1024)) : 1));
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(launch_pdl(kern, grid, dim3(256), 0, s, a));
        return LC_OK;
    };
    if (a.f32) return vec ? go(attn_prep_kernel<float, 4>) : go(attn_prep_kernel<float, 1>);
    return vec ? go(attn_prep_kernel<bf16, 4>) : go(attn_prep_kernel<bf16, 1>);
}

size_t attn_part_bytes(const AttnShape& g) {
    return (size_t)kPartCells * sm_count() * 16 * ((size_t)g.ep + 2) * sizeof(float);
}

int32_t launch_attn_tokens(const AttnArgs& a, const AttnScratch& sc, cudaStream_t s) {
    const AttnShape& g = a.g;
    if (a.T <= 0) return LC_OK;
    if (!tensor_form(g, a.f32)) {
        const size_t smem = (size_t)(g.dim + g.vdim + 2 + kPlainThreads) * 4 + kPlainThreads * sizeof(size_t);
        LC_CHECK(smem <= kMaxSmem, LC_ERR_UNSUPPORTED, "attention: heads of %d and %d dimensions", g.dim, g.vdim);
        const dim3 grid((unsigned)g.heads, (unsigned)a.T);
        auto go = [&](auto kern) -> int32_t {
            LC_CUDA(ensure_smem_limit((const void*)kern, smem));
            LC_CUDA(launch_pdl(kern, grid, dim3(kPlainThreads), smem, s, a));
            return LC_OK;
        };
        return a.f32 ? go(attn_plain_kernel<float>) : go(attn_plain_kernel<bf16>);
    }
    const int n = cells(g), cap = a.pages_per_seq * a.page_tokens;
    const int span = g.window > 0 ? std::min(cap, g.window) / kDecKeys + 2 + std::min(cap, g.keep_first) / kDecKeys : (cap + kDecKeys - 1) / kDecKeys;  // most tiles of a token
    // pieces: fewest turns of a warp over the waves of CTAs (a CTA's start and end cost about four), merging costs a little more
    const size_t smem = tokens_smem(g);
    const int resident = sm_count() * std::max(1, (int)std::min<size_t>(4, (kMaxSmem + 1024) / (smem + 4096)));
    int pieces = 1;
    long best = -1;
    for (int c = 1; c <= std::min(kMaxPieces, (span + kDecWarps - 1) / kDecWarps); c++) {
        if (c > 1 && (a.T * n > sc.n_tickets || (size_t)a.T * n * c * 16 * ((size_t)g.ep + 2) * sizeof(float) > sc.part_bytes)) break;
        const long waves = ((long)a.T * n * c + resident - 1) / resident, cost = waves * (((span + c - 1) / c + kDecWarps - 1) / kDecWarps + 4) + (c > 1 ? 3 : 0);
        if (best < 0 || cost < best) { best = cost; pieces = c; }
    }
    AttnParts p;
    p.o = sc.part;
    p.ml = sc.part + (size_t)a.T * n * pieces * 16 * g.ep;
    p.tickets = sc.tickets;
    const dim3 grid((unsigned)a.T, (unsigned)n, (unsigned)pieces);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3(32 * kDecWarps), smem, s, a, p, gemv_error_flag_dev()));
        return LC_OK;
    };
    auto of = [&](auto nv) -> int32_t { return g.cap > 0.0f ? go(attn_tokens_kernel<decltype(nv)::value, true>) : go(attn_tokens_kernel<decltype(nv)::value, false>); };
    switch (value_tiles(g.ep)) {
        case 4: return of(std::integral_constant<int, 4>());
        case 8: return of(std::integral_constant<int, 8>());
        case 12: return of(std::integral_constant<int, 12>());
        case 16: return of(std::integral_constant<int, 16>());
        default: return of(std::integral_constant<int, 32>());
    }
}

bool attn_tiles_apply(const AttnShape& g, bool f32) { return tensor_form(g, f32); }

int32_t launch_attn_tiles(const AttnArgs& a, const AttnTile* tiles, int n_tiles, cudaStream_t s) {
    const size_t smem = tiles_smem(a.g);
    const dim3 grid((unsigned)n_tiles, (unsigned)a.g.heads);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3(128), smem, s, a, tiles, gemv_error_flag_dev()));
        return LC_OK;
    };
    auto of = [&](auto nv) -> int32_t { return a.g.cap > 0.0f ? go(attn_tiles_kernel<decltype(nv)::value, true>) : go(attn_tiles_kernel<decltype(nv)::value, false>); };
    switch (value_tiles(a.g.ep)) {
        case 4: return of(std::integral_constant<int, 4>());
        case 8: return of(std::integral_constant<int, 8>());
        case 12: return of(std::integral_constant<int, 12>());
        case 16: return of(std::integral_constant<int, 16>());
        default: return of(std::integral_constant<int, 32>());
    }
}

}  // namespace lc
