// Linear recurrences with one decay per head (LinearShape): S_t = e^(l_t) S_(t-1) + b_t k_t v_t^T, o_t = S_t^T q_t + skip v_t.
// Constant: l from the config, b = 1, q, k, v already through silu (the product's epilogue).  StateSpace: b = softplus(dt + bias),
// l = -a b, q and k shared by the heads of a group; v, k and q come through a short convolution with bias and silu.
// S, l, b and all sums are f32; q, k and v are activations (A = bf16, or float when a model runs in true 32-bit).
//   linear_conv_kernel    convolutions of a call's tokens
//   linear_scan_kernel    the recurrence token by token: short runs, f32 models
//   linear_chunk_kernel   long runs, 64 tokens at a time on the tensor cores.  With G_t the sum of l inside the chunk,
//                           o_t = e^(G_t) S0^T q_t + sum_(s <= t) (q_t . k_s) e^(G_t - G_s) b_s v_s,
//                           S = e^(G_end) S0 + sum_s k_s (e^(G_end - G_s) b_s v_s)^T;
//                         q, k and v enter as they are, the f32 factors (weights, scaled values, S0) as two bf16 halves
//   linear_step_kernel    one token per sequence: convolution, recurrence; many items: linear_ring_kernel behind linear_conv_kernel
//   linear_output_kernel  gate and norm: Constant rms_norm(o) w sigmoid(gate) over all heads, StateSpace rms_norm(o silu(gate)) w in parts
#include <algorithm>
#include <cmath>
#include "lc_mixers.h"
#include "lc_mma.cuh"
#include "lc_tma.cuh"
#include "lc_umma.cuh"

namespace lc {

namespace {

// of activations: with the quick exponential and division where the result is rounded to bf16
template <typename A> __device__ __forceinline__ float sigmoid_of(float v) {
    if constexpr (sizeof(A) == 2) return __fdividef(1.0f, 1.0f + __expf(-v));
    else return 1.0f / (1.0f + expf(-v));
}
template <typename A> __device__ __forceinline__ float silu_any(float v) { return v * sigmoid_of<A>(v); }
__device__ __forceinline__ float softplus_of(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
// (b, l) of head h at token t
__device__ __forceinline__ float2 step_decay(const LinearArgs& a, size_t t, int h) {
    if (a.g.kind == LinearKind::Constant) return make_float2(1.0f, a.log_decay[h]);
    const float b = softplus_of(a.dt[t * a.g.ld_dt + a.g.off_dt + h] + a.dt_bias[h]);
    return make_float2(b, -a.a_exp[h] * b);
}
// e^l as a sum of two floats
__device__ __forceinline__ float2 decay_of(const LinearArgs& a, int h, float l) { return a.g.kind == LinearKind::Constant ? a.decay[h] : make_float2(expf(l), 0.0f); }
__device__ __forceinline__ float decayed(float s, float2 d) { return fmaf(s, d.x, s * d.y); }
// Rows of v | k | q that the recurrence reads.
template <typename A> struct Rows { const A* p; int ld, v, k, q; };
template <typename A>
__device__ __forceinline__ Rows<A> rows_of(const LinearArgs& a) {
    const LinearShape& g = a.g;
    if (g.kind == LinearKind::Constant) return {(const A*)a.proj, g.ld, g.off_v, g.off_k, g.off_q};
    return {(const A*)a.in, g.ld_in, 0, g.heads * g.vdim, g.heads * g.vdim + g.groups * g.dim};
}

template <typename A> __device__ __forceinline__ float2 two(const A* p);
template <> __device__ __forceinline__ float2 two<float>(const float* p) { return *(const float2*)p; }
template <> __device__ __forceinline__ float2 two<bf16>(const bf16* p) { return __bfloat1622float2(*(const __nv_bfloat162*)p); }
template <typename A> __device__ __forceinline__ void put_two(A* p, float2 v);
template <> __device__ __forceinline__ void put_two<float>(float* p, float2 v) { *(float2*)p = v; }
template <> __device__ __forceinline__ void put_two<bf16>(bf16* p, float2 v) { *(uint32_t*)p = pack2(v.x, v.y); }
template <typename A> __device__ __forceinline__ float4 four(const A* p);
template <> __device__ __forceinline__ float4 four<float>(const float* p) { return *(const float4*)p; }
template <> __device__ __forceinline__ float4 four<bf16>(const bf16* p) {
    const uint2 v = *(const uint2*)p;
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xFFFF0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xFFFF0000u));
}
template <typename A> __device__ __forceinline__ void put_four(A* p, float4 v);
template <> __device__ __forceinline__ void put_four<float>(float* p, float4 v) { *(float4*)p = v; }
template <> __device__ __forceinline__ void put_four<bf16>(bf16* p, float4 v) { *(uint2*)p = make_uint2(pack2(v.x, v.y), pack2(v.z, v.w)); }

// A thread walks `stretch` tokens of two neighbouring channels and keeps their last inputs in registers (TAPS of them; 0: any
// number, re-read).  Inputs of earlier positions come from the call's rows as far as they belong to the same run, from the ring
// before that, and are zero before the sequence's start.  one_each: every token is the only one of its sequence; its inputs enter the
// ring here (an entry that no convolution of this call reads).
template <typename A, int TAPS>
__global__ void __launch_bounds__(128) linear_conv_kernel(const LinearArgs a, int stretch, int one_each) {
    pdl_launch_dependents();
    pdl_wait();
    const LinearShape& g = a.g;
    const int c = (blockIdx.y * 128 + threadIdx.x) * 2;
    if (c >= g.channels) return;
    const bool both = c + 1 < g.channels;
    const int taps = TAPS > 0 ? TAPS : g.taps;
    constexpr int kT = TAPS > 0 ? TAPS : 1;
    const A* in = (const A*)a.proj + g.off_v + c;
    const A* ring = (const A*)a.ring + c;
    const float2 bias = make_float2(a.conv_b[c], both ? a.conv_b[c + 1] : 0.0f);
    auto weight = [&](int j) { return make_float2(a.conv[(size_t)c * taps + j], both ? a.conv[(size_t)(c + 1) * taps + j] : 0.0f); };
    float w[2][kT], win[2][kT];  // win[.][j]: the input j + 1 tokens back
    if constexpr (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < TAPS; j++) {
            const float2 v = weight(j);
            w[0][j] = v.x; w[1][j] = v.y;
            win[0][j] = win[1][j] = 0.0f;
        }
    }
    const int t0 = blockIdx.x * stretch, t1 = min(a.T, t0 + stretch);
    int prev_seq = -1, prev_pos = -1;
    constexpr int kAhead = 4;  // tokens whose inputs are fetched together
    for (int tb = t0; tb < t1; tb += kAhead) {
        float2 ahead[kAhead];
        int seq_a[kAhead], pos_a[kAhead];
#pragma unroll
        for (int v = 0; v < kAhead; v++) {
            const int t = min(tb + v, t1 - 1);
            seq_a[v] = a.tok_seq[t]; pos_a[v] = a.tok_pos[t];
            ahead[v] = two<A>(in + (size_t)t * g.ld);
        }
#pragma unroll
        for (int v = 0; v < kAhead; v++) {
            const int t = tb + v;
            if (t >= t1) break;
            const int seq = seq_a[v], pos = pos_a[v];
            auto back = [&](int j) {
                if (pos - j < 0) return make_float2(0.0f, 0.0f);
                const int tt = t - j;
                if (tt >= 0 && a.tok_seq[tt] == seq && a.tok_pos[tt] == pos - j) return two<A>(in + (size_t)tt * g.ld);
                const A* r = ring + ((size_t)seq * taps + (pos - j) % taps) * g.channels;
                return make_float2(act_f<A>(r[0]), both ? act_f<A>(r[1]) : 0.0f);
            };
            const float2 u = ahead[v];
            float2 y = bias;
            if constexpr (TAPS > 0) {
                if (seq != prev_seq || pos != prev_pos + 1) {
#pragma unroll
                    for (int j = 1; j < TAPS; j++) {  // all of them on their way at once
                        const int tt = max(t - j, 0);
                        const bool here = t - j >= 0 && a.tok_seq[tt] == seq && a.tok_pos[tt] == pos - j;
                        const A* r = here ? in + (size_t)tt * g.ld : ring + ((size_t)seq * TAPS + (pos >= j ? (pos - j) % TAPS : 0)) * g.channels;
                        win[0][j - 1] = pos >= j ? act_f<A>(r[0]) : 0.0f;
                        win[1][j - 1] = pos >= j && both ? act_f<A>(r[1]) : 0.0f;
                    }
                }
#pragma unroll
                for (int j = TAPS - 1; j > 0; j--) { y.x = fmaf(w[0][TAPS - 1 - j], win[0][j - 1], y.x); y.y = fmaf(w[1][TAPS - 1 - j], win[1][j - 1], y.y); }
                y.x = fmaf(w[0][TAPS - 1], u.x, y.x); y.y = fmaf(w[1][TAPS - 1], u.y, y.y);
#pragma unroll
                for (int j = TAPS - 1; j > 0; j--) { win[0][j] = win[0][j - 1]; win[1][j] = win[1][j - 1]; }
                win[0][0] = u.x; win[1][0] = u.y;
                prev_seq = seq; prev_pos = pos;
            } else {
                for (int j = taps - 1; j >= 0; j--) {
                    const float2 v = j == 0 ? u : back(j), cw = weight(taps - 1 - j);
                    y.x = fmaf(cw.x, v.x, y.x); y.y = fmaf(cw.y, v.y, y.y);
                }
            }
            put_two<A>((A*)a.in + (size_t)t * g.ld_in + c, make_float2(silu_any<A>(y.x), silu_any<A>(y.y)));
            if (one_each) {
                A* r = (A*)a.ring + ((size_t)seq * taps + pos % taps) * g.channels + c;
                r[0] = to_act<A>(u.x);
                if (both) r[1] = to_act<A>(u.y);
            }
        }
    }
}

// The inputs of a run's last `taps` positions, for the convolutions of the next call.
template <typename A>
__global__ void __launch_bounds__(256) linear_keep_kernel(const LinearArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const LinearShape& g = a.g;
    const SeqRun run = a.all_runs[blockIdx.x];
    const int c = blockIdx.y * 256 + threadIdx.x;
    if (c >= g.channels) return;
    for (int t = max(0, run.n - g.taps); t < run.n; t++)
        ((A*)a.ring)[((size_t)run.seq * g.taps + (run.pos0 + t) % g.taps) * g.channels + c] = ((const A*)a.proj)[(size_t)(run.tok0 + t) * g.ld + g.off_v + c];
}

// A CTA of four warps owns 32 value columns of one head of one run; four lanes share a column's `dim` state entries (DPL each:
// float4 groups dealt round robin), eight columns per warp.
constexpr int kScanTok = 16;  // tokens staged in shared memory at a time
template <typename A, int DPL>
__global__ void __launch_bounds__(128) linear_scan_kernel(const LinearArgs a) {
    constexpr int DP = DPL * 4;
    extern __shared__ __align__(16) float sm[];
    float *s_q = sm, *s_k = s_q + kScanTok * DP, *s_v = s_k + kScanTok * DP, *s_b = s_v + kScanTok * 32;
    float2* s_g = (float2*)(s_b + kScanTok);
    pdl_launch_dependents();
    pdl_wait();
    const LinearShape& g = a.g;
    const SeqRun run = a.runs[blockIdx.x];
    const int h = blockIdx.y, kg = h / (g.heads / g.groups);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r4 = lane & 3, col = warp * 8 + (lane >> 2), e = blockIdx.z * 32 + col;
    float* st = a.state + ((size_t)run.seq * g.heads + h) * g.dim * g.vdim;
    const Rows<A> src = rows_of<A>(a);
    const float skip = a.skip ? a.skip[h] : 0.0f;
    float S[DPL];
#pragma unroll
    for (int i = 0; i < DPL; i++) {
        const int d = (i >> 2) * 16 + r4 * 4 + (i & 3);
        S[i] = (run.pos0 > 0 && d < g.dim && e < g.vdim) ? st[(size_t)d * g.vdim + e] : 0.0f;
    }
    for (int c0 = 0; c0 < run.n; c0 += kScanTok) {
        const int m = min(kScanTok, run.n - c0);
        __syncthreads();
        for (int i = threadIdx.x; i < m * DP; i += 128) {
            const int t = i / DP, d = i - t * DP;
            const A* row = src.p + (size_t)(run.tok0 + c0 + t) * src.ld + kg * g.dim + d;
            s_q[i] = d < g.dim ? act_f<A>(row[src.q]) : 0.0f;
            s_k[i] = d < g.dim ? act_f<A>(row[src.k]) : 0.0f;
        }
        for (int i = threadIdx.x; i < m * 32; i += 128) {
            const int t = i >> 5, c = blockIdx.z * 32 + (i & 31);
            s_v[i] = c < g.vdim ? act_f<A>(src.p[(size_t)(run.tok0 + c0 + t) * src.ld + src.v + h * g.vdim + c]) : 0.0f;
        }
        if (threadIdx.x < m) {
            const float2 bl = step_decay(a, (size_t)(run.tok0 + c0 + threadIdx.x), h);
            s_b[threadIdx.x] = bl.x;
            s_g[threadIdx.x] = decay_of(a, h, bl.y);
        }
        __syncthreads();
        for (int t = 0; t < m; t++) {
            const float4 *q4 = (const float4*)(s_q + t * DP), *k4 = (const float4*)(s_k + t * DP);
            const float v = s_v[t * 32 + col], u = s_b[t] * v;
            const float2 decay = s_g[t];
            float o = 0.0f;
#pragma unroll
            for (int i = 0; i < DPL / 4; i++) {
                const float4 kv = k4[i * 4 + r4], qv = q4[i * 4 + r4];
                const float kk[4] = {kv.x, kv.y, kv.z, kv.w}, qq[4] = {qv.x, qv.y, qv.z, qv.w};
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    S[4 * i + j] = fmaf(kk[j], u, decayed(S[4 * i + j], decay));
                    o = fmaf(S[4 * i + j], qq[j], o);
                }
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (r4 == 0 && e < g.vdim) a.o[(size_t)(run.tok0 + c0 + t) * g.heads * g.vdim + h * g.vdim + e] = fmaf(skip, v, o);
        }
    }
#pragma unroll
    for (int i = 0; i < DPL; i++) {
        const int d = (i >> 2) * 16 + r4 * 4 + (i & 3);
        if (d < g.dim && e < g.vdim) st[(size_t)d * g.vdim + e] = S[i];
    }
}

// ---- long runs --------------------------------------------------------------------------------------------------------------
// A CTA of eight warps walks the chunks of one run for 32 value columns of one head.  Per chunk a warp owns 16 tokens and 16 columns
// of the read-outs, and an eighth of S (DP: `dim` padded; 32 key rows: a quarter, in four warps), which stays in registers as the
// accumulators of its update; its halves are published for the next chunk's read-outs.
constexpr int kC = kDeltaChunk, kCols = 32, kVP = kCols + 8;
__host__ __device__ constexpr size_t chunk_smem(int dp) {
    return (size_t)(2 * 2 * kC * (dp + 8) + 2 * kC * kVP + 2 * dp * kVP + 2 * kC * kVP) * 2 + 6 * kC * sizeof(float);
}
constexpr int kChunkThreads = 256;
template <int DP>
__global__ void __launch_bounds__(kChunkThreads, DP <= 128 ? 2 : 1) linear_chunk_kernel(const LinearArgs a) {
    constexpr int QP = DP + 8, kMT = DP / 16, kOwnM = kMT >= 8 ? kMT / 8 : 1, kOwnN = kMT >= 8 ? 4 : 2;
    static_assert(kMT >= 2, "at least two tiles of key rows");
    extern __shared__ __align__(16) unsigned char smem[];
    bf16 *s_q = (bf16*)smem, *s_k = s_q + 2 * kC * QP, *s_v = s_k + 2 * kC * QP, *s_S = s_v + 2 * kC * kVP, *s_w = s_S + 2 * DP * kVP;
    float* s_sums = (float*)(s_w + 2 * kC * kVP);  // of this chunk and the next: G in log2 units as a sum of two floats, the steps
    pdl_launch_dependents();
    pdl_wait();
    const LinearShape& g = a.g;
    const DeltaChunkRun cr = a.chunk_runs[blockIdx.x];
    const int h = blockIdx.y, kg = h / (g.heads / g.groups), e0 = blockIdx.z * kCols;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
    const Rows<bf16> src = rows_of<bf16>(a);
    const float skip = a.skip ? a.skip[h] : 0.0f;
    float* st = a.state + ((size_t)cr.run.seq * g.heads + h) * g.dim * g.vdim;
    // this warp's tokens (16 rb ..) and columns of the read-outs; the two warps of a scheduler (warp & 3) share the triangle evenly
    const int rb = warp < 4 ? warp : 7 - warp, ch = (warp >> 2) * 16;
    const bool owner = kMT >= 4 || warp < 4;
    const int m0 = kMT >= 8 ? warp * kOwnM : kMT == 4 ? warp & 3 : warp & 1, n0 = kMT >= 8 ? 0 : kMT == 4 ? (warp >> 2) * 2 : (warp >> 1 & 1) * 2;
    const uint32_t q_sm = smem_u32(s_q), k_sm = smem_u32(s_k), v_sm = smem_u32(s_v), S_sm = smem_u32(s_S), w_sm = smem_u32(s_w);
    auto load = [&](int c) {
        const int buf = c & 1, left = cr.run.n - c * kC;
        const bf16* row = src.p + (size_t)(cr.run.tok0 + c * kC) * src.ld;
        for (int i = tid; i < kC * (DP / 8); i += kChunkThreads) {
            const int t = i / (DP / 8), d = (i - t * (DP / 8)) * 8;
            const bool in = t < left && d < g.dim;
            const bf16* p = row + (in ? (size_t)t * src.ld + kg * g.dim + d : 0);
            const uint32_t at = (uint32_t)((buf * kC + t) * QP + d) * 2;
            cp16(q_sm + at, p + (in ? src.q : 0), in ? 16 : 0);
            cp16(k_sm + at, p + (in ? src.k : 0), in ? 16 : 0);
        }
        for (int i = tid; i < kC * (kCols / 8); i += kChunkThreads) {
            const int t = i / (kCols / 8), e = (i & (kCols / 8 - 1)) * 8;
            const bool in = t < left && e0 + e < g.vdim;
            cp16(v_sm + (uint32_t)((buf * kC + t) * kVP + e) * 2, row + (in ? (size_t)t * src.ld + src.v + h * g.vdim + e0 + e : 0), in ? 16 : 0);
        }
        cp_commit();
    };
    float2 bl[2];  // warp 0: step and log decay of tokens 2 lane, 2 lane + 1 of the chunk to come; behind the run's end neither
    auto fetch = [&](int c) {
        if (warp == 0)
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int t = c * kC + 2 * lane + j;
                bl[j] = t < cr.run.n ? step_decay(a, (size_t)(cr.run.tok0 + t), h) : make_float2(0.0f, 0.0f);
            }
    };
    auto sums = [&](int c) {
        if (warp != 0) return;
        float* g2 = s_sums + (c & 1) * 3 * kC;
        const double l0 = (double)bl[0].y * 1.4426950408889634, l1 = (double)bl[1].y * 1.4426950408889634;
        double sum = l0 + l1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += up;
        }
        const double at[2] = {sum - l1, sum};
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const float hi = (float)at[j];
            g2[2 * lane + j] = hi;
            g2[kC + 2 * lane + j] = (float)(at[j] - (double)hi);
            g2[2 * kC + 2 * lane + j] = bl[j].x;
        }
    };
    load(0);
    fetch(0);
    sums(0);
    float S[kOwnM][kOwnN][4];
#pragma unroll
    for (int i = 0; i < kOwnM; i++)
#pragma unroll
        for (int n = 0; n < kOwnN; n++)
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int d = (m0 + i) * 16 + g8 + 8 * r, e = e0 + (n0 + n) * 8 + 2 * t4;
                float2 v = make_float2(0.0f, 0.0f);
                if (owner && cr.run.pos0 > 0 && d < g.dim && e < g.vdim) v = *(const float2*)(st + (size_t)d * g.vdim + e);
                S[i][n][2 * r] = v.x; S[i][n][2 * r + 1] = v.y;
            }
    auto publish = [&]() {
        if (!owner) return;
#pragma unroll
        for (int i = 0; i < kOwnM; i++)
#pragma unroll
            for (int n = 0; n < kOwnN; n++)
#pragma unroll
                for (int r = 0; r < 2; r++) {
                    uint32_t hi, lo;
                    split2(S[i][n][2 * r], S[i][n][2 * r + 1], hi, lo);
                    bf16* dst = s_S + ((m0 + i) * 16 + g8 + 8 * r) * kVP + (n0 + n) * 8 + 2 * t4;
                    *(uint32_t*)dst = hi;
                    *(uint32_t*)(dst + DP * kVP) = lo;
                }
    };
    publish();
    const int krow = (lane & 7) + ((lane >> 4) << 3), kcol = ((lane >> 3) & 1) * 8, vrow = lane & 15, vcol = (lane >> 4) * 8;
    for (int c = 0; c < cr.n_chunks; c++) {
        const int buf = c & 1;
        const float *s_gh = s_sums + buf * 3 * kC, *s_gl = s_gh + kC, *s_b = s_gl + kC;
        cp_wait<0>();
        __syncthreads();  // the chunk's rows, G and S are there; nobody reads the other buffers any more
        if (c + 1 < cr.n_chunks) { load(c + 1); fetch(c + 1); }
        const float eh = s_gh[kC - 1], el = s_gl[kC - 1], keep = exp2f(eh + el);
        for (int i = tid; i < kC * (kCols / 2); i += kChunkThreads) {  // values on their way into S
            const int t = i / (kCols / 2), e = (i & (kCols / 2 - 1)) * 2;
            const float f = s_b[t] * exp2f((eh - s_gh[t]) + (el - s_gl[t]));
            const float2 v = two<bf16>(s_v + (buf * kC + t) * kVP + e);
            uint32_t hi, lo;
            split2(v.x * f, v.y * f, hi, lo);
            *(uint32_t*)(s_w + t * kVP + e) = hi;
            *(uint32_t*)(s_w + (kC + t) * kVP + e) = lo;
        }
        float p[8][4], o[2][4], oi[2][4];
#pragma unroll
        for (int n = 0; n < 8; n++) p[n][0] = p[n][1] = p[n][2] = p[n][3] = 0.0f;
#pragma unroll
        for (int n = 0; n < 2; n++) o[n][0] = o[n][1] = o[n][2] = o[n][3] = oi[n][0] = oi[n][1] = oi[n][2] = oi[n][3] = 0.0f;
#pragma unroll 2
        for (int kk = 0; kk < DP / 16; kk++) {
            uint32_t q4[4];
            ldsm4(q_sm + (uint32_t)((buf * kC + 16 * rb + vrow) * QP + 16 * kk + vcol) * 2, q4);
#pragma unroll
            for (int n = 0; n < 4; n++) {
                if (n > rb) break;
                uint32_t kb[4];
                ldsm4(k_sm + (uint32_t)((buf * kC + 16 * n + krow) * QP + 16 * kk + kcol) * 2, kb);
                mma_bf16(p[2 * n], q4, kb[0], kb[1]);
                mma_bf16(p[2 * n + 1], q4, kb[2], kb[3]);
            }
#pragma unroll
            for (int half = 0; half < 2; half++) {
                uint32_t sb[4];
                ldsm4t(S_sm + (uint32_t)((half * DP + 16 * kk + vrow) * kVP + ch + vcol) * 2, sb);
                mma_bf16(oi[0], q4, sb[0], sb[1]);
                mma_bf16(oi[1], q4, sb[2], sb[3]);
            }
        }
        const int tr[2] = {16 * rb + g8, 16 * rb + g8 + 8};
        const float gh[2] = {s_gh[tr[0]], s_gh[tr[1]]}, gl[2] = {s_gl[tr[0]], s_gl[tr[1]]};
#pragma unroll
        for (int ks = 0; ks < 4; ks++) {
            if (ks > rb) break;
            uint32_t ph[4], pl[4];
#pragma unroll
            for (int hs = 0; hs < 2; hs++) {
                const int s0 = 16 * ks + 8 * hs + 2 * t4;
                float f[4];
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const int s = s0 + (j & 1), r = j >> 1;
                    f[j] = s <= tr[r] ? p[2 * ks + hs][j] * s_b[s] * exp2f((gh[r] - s_gh[s]) + (gl[r] - s_gl[s])) : 0.0f;
                }
                split2(f[0], f[1], ph[2 * hs], pl[2 * hs]);
                split2(f[2], f[3], ph[2 * hs + 1], pl[2 * hs + 1]);
            }
            uint32_t b[4];
            ldsm4t(v_sm + (uint32_t)((buf * kC + 16 * ks + vrow) * kVP + ch + vcol) * 2, b);
            mma_bf16(o[0], ph, b[0], b[1]);
            mma_bf16(o[1], ph, b[2], b[3]);
            mma_bf16(o[0], pl, b[0], b[1]);
            mma_bf16(o[1], pl, b[2], b[3]);
        }
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int t = c * kC + tr[r];
            if (t >= cr.run.n) continue;
            const float f = exp2f(gh[r] + gl[r]);
            float* dst = a.o + (size_t)(cr.run.tok0 + t) * g.heads * g.vdim + h * g.vdim + e0 + ch + 2 * t4;
#pragma unroll
            for (int n = 0; n < 2; n++) {
                if (e0 + ch + 8 * n >= g.vdim) break;
                const float2 v = two<bf16>(s_v + (buf * kC + tr[r]) * kVP + ch + 8 * n + 2 * t4);
                *(float2*)(dst + 8 * n) = make_float2(fmaf(f, oi[n][2 * r], o[n][2 * r]) + skip * v.x, fmaf(f, oi[n][2 * r + 1], o[n][2 * r + 1]) + skip * v.y);
            }
        }
        if (c + 1 < cr.n_chunks) sums(c + 1);
        __syncthreads();  // the scaled values are there, S has been read
        if (!owner) continue;
#pragma unroll
        for (int i = 0; i < kOwnM; i++)
#pragma unroll
            for (int n = 0; n < kOwnN; n++) { S[i][n][0] *= keep; S[i][n][1] *= keep; S[i][n][2] *= keep; S[i][n][3] *= keep; }
#pragma unroll
        for (int ks = 0; ks < 4; ks++) {
            uint32_t wb[2][kOwnN / 2][4];
#pragma unroll
            for (int half = 0; half < 2; half++)
#pragma unroll
                for (int n = 0; n < kOwnN / 2; n++) ldsm4t(w_sm + (uint32_t)((half * kC + 16 * ks + vrow) * kVP + n0 * 8 + 16 * n + vcol) * 2, wb[half][n]);
#pragma unroll
            for (int i = 0; i < kOwnM; i++) {
                uint32_t kt[4];  // keys transposed: rows are key dimensions, columns tokens
                ldsm4t(k_sm + (uint32_t)((buf * kC + 16 * ks + krow) * QP + (m0 + i) * 16 + kcol) * 2, kt);
#pragma unroll
                for (int half = 0; half < 2; half++)
#pragma unroll
                    for (int n = 0; n < kOwnN / 2; n++) {
                        mma_bf16(S[i][2 * n], kt, wb[half][n][0], wb[half][n][1]);
                        mma_bf16(S[i][2 * n + 1], kt, wb[half][n][2], wb[half][n][3]);
                    }
            }
        }
        publish();
    }
#pragma unroll
    for (int i = 0; i < kOwnM; i++)
#pragma unroll
        for (int n = 0; n < kOwnN; n++)
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int d = (m0 + i) * 16 + g8 + 8 * r, e = e0 + (n0 + n) * 8 + 2 * t4;
                if (owner && d < g.dim && e < g.vdim) *(float2*)(st + (size_t)d * g.vdim + e) = make_float2(S[i][n][2 * r], S[i][n][2 * r + 1]);
            }
}

// ---- one token per sequence -----------------------------------------------------------------------------------------------------
// One CTA per (head, token); a thread owns VEC neighbouring value columns and every `groups`-th key row, kept in registers (ROWS of
// them; 0: re-read).  The ring entry written here is not one that any head reads in this step.
constexpr int kStepThreads = 256;
template <typename A, int VEC, int ROWS>
__global__ void __launch_bounds__(kStepThreads) linear_step_kernel(const LinearArgs a) {
    extern __shared__ float sm[];
    pdl_launch_dependents();
    pdl_wait();
    const LinearShape& g = a.g;
    const int h = blockIdx.x, t = blockIdx.y, rep = g.heads / g.groups, kg = h / rep, seq = a.tok_seq[t], pos = a.tok_pos[t], tid = threadIdx.x;
    const int cols = g.vdim / VEC, groups = kStepThreads / cols, c = tid % cols, gr = tid / cols;
    float *s_q = sm, *s_k = s_q + g.dim, *s_v = s_k + g.dim, *s_o = s_v + g.vdim;
    float* st = a.state + ((size_t)seq * g.heads + h) * g.dim * g.vdim + c * VEC;
    const bool live = pos > 0, mine = gr < groups;
    float S[ROWS > 0 ? ROWS : 1][VEC];
    auto load = [&](int d, float (&v)[VEC]) {
#pragma unroll
        for (int j = 0; j < VEC; j++) v[j] = 0.0f;
        if (!live) return;
        if constexpr (VEC == 4) { const float4 x = *(const float4*)(st + (size_t)d * g.vdim); v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; }
        else v[0] = st[(size_t)d * g.vdim];
    };
    if (ROWS > 0 && mine) {  // the state's reads travel while the inputs are made
#pragma unroll
        for (int i = 0; i < ROWS; i++)
            if (gr + i * groups < g.dim) load(gr + i * groups, S[i]);
    }
    const float2 bl = step_decay(a, (size_t)t, h);
    const A* proj = (const A*)a.proj + (size_t)t * g.ld;
    for (int i = tid; i < 2 * g.dim + g.vdim; i += kStepThreads) {
        const int part = i < g.dim ? 0 : i < 2 * g.dim ? 1 : 2;  // q, k, v
        const int at = part == 0 ? kg * g.dim + i : part == 1 ? kg * g.dim + i - g.dim : h * g.vdim + i - 2 * g.dim;
        const A cur = proj[(part == 0 ? g.off_q : part == 1 ? g.off_k : g.off_v) + at];
        float y = act_f<A>(cur);
        if (g.kind == LinearKind::StateSpace) {
            const int channel = (part == 0 ? g.off_q : part == 1 ? g.off_k : g.off_v) - g.off_v + at;
            A* ring = (A*)a.ring + (size_t)seq * g.taps * g.channels + channel;
            const float* w = a.conv + (size_t)channel * g.taps;
            float acc = a.conv_b[channel];
            for (int j = g.taps - 1; j > 0; j--)
                if (pos - j >= 0) acc = fmaf(w[g.taps - 1 - j], act_f<A>(ring[(size_t)((pos - j) % g.taps) * g.channels]), acc);
            y = act_f<A>(to_act<A>(silu_any<A>(fmaf(w[g.taps - 1], y, acc))));  // the type that runs of tokens keep it in
            if (part == 2 || h % rep == 0) ring[(size_t)(pos % g.taps) * g.channels] = cur;
        }
        sm[i] = y;
    }
    const float2 decay = decay_of(a, h, bl.y);
    __syncthreads();
    if (mine) {
        float u[VEC], o[VEC];
#pragma unroll
        for (int j = 0; j < VEC; j++) { u[j] = bl.x * s_v[c * VEC + j]; o[j] = 0.0f; }
        auto turn = [&](int d, float (&v)[VEC]) {
            const float k = s_k[d], q = s_q[d];
#pragma unroll
            for (int j = 0; j < VEC; j++) { v[j] = fmaf(k, u[j], decayed(v[j], decay)); o[j] = fmaf(v[j], q, o[j]); }
            if constexpr (VEC == 4) *(float4*)(st + (size_t)d * g.vdim) = make_float4(v[0], v[1], v[2], v[3]);
            else st[(size_t)d * g.vdim] = v[0];
        };
        if constexpr (ROWS > 0) {
#pragma unroll
            for (int i = 0; i < ROWS; i++)
                if (gr + i * groups < g.dim) turn(gr + i * groups, S[i]);
        } else {
            for (int d = gr; d < g.dim; d += groups) { load(d, S[0]); turn(d, S[0]); }
        }
#pragma unroll
        for (int j = 0; j < VEC; j++) s_o[gr * g.vdim + c * VEC + j] = o[j];
    }
    __syncthreads();
    const float skip = a.skip ? a.skip[h] : 0.0f;
    for (int e = tid; e < g.vdim; e += kStepThreads) {
        float o = skip * s_v[e];
        for (int i = 0; i < groups; i++) o += s_o[i * g.vdim + e];
        a.o[((size_t)t * g.heads + h) * g.vdim + e] = o;
    }
}

// The same for many (head, token) items: one CTA per SM walks them with the states in a ring of bulk copies, so that reads, sums and
// writes of neighbouring items overlap.  The ninth warp's lane 0 issues the copies: a state and the item's rows of q, k and v in (behind
// the convolutions), the new state out.  A stage is filled again once its store has been read.
constexpr int kRingThreads = kStepThreads + 32;
struct RingShape { int stages, state_bytes, stage_bytes; };  // a stage: state | q | k | v
template <typename A>
__global__ void __launch_bounds__(kRingThreads, 1) linear_ring_kernel(const LinearArgs a, const RingShape rs, int* error_flag) {
    extern __shared__ __align__(128) unsigned char ring_smem[];
    __shared__ uint64_t s_full[8], s_done[8];
    pdl_launch_dependents();
    const LinearShape& g = a.g;
    const int tid = threadIdx.x, items = g.heads * a.T, rep = g.heads / g.groups, mine = items > (int)blockIdx.x ? (items - (int)blockIdx.x - 1) / (int)gridDim.x + 1 : 0;
    float* s_o = (float*)(ring_smem + (size_t)rs.stages * rs.stage_bytes);  // [2][groups][vdim]
    if (tid == 0) {
        for (int i = 0; i < rs.stages; i++) { mbar_init(&s_full[i], 1); mbar_init(&s_done[i], kStepThreads); }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    auto head_of = [&](int j) { return (int)((blockIdx.x + j * gridDim.x) % g.heads); };
    auto token_of = [&](int j) { return (int)((blockIdx.x + j * gridDim.x) / g.heads); };
    const size_t state_elems = (size_t)g.dim * g.vdim;
    if (tid >= kStepThreads) {
        const int lane = tid & 31;
        const Rows<A> src = rows_of<A>(a);
        int seqs = 0, seqs0 = -32;  // of items seqs0 .. seqs0 + 31, a lane each
        auto seq_of = [&](int j) {
            if (j >= seqs0 + 32) { seqs0 = j; seqs = j + lane < mine ? a.tok_seq[token_of(j + lane)] : 0; }
            return __shfl_sync(0xffffffffu, seqs, j - seqs0);
        };
        auto load = [&](int j, int seq) {
            if (lane != 0) return;
            const int h = head_of(j), t = token_of(j), kg = h / rep, st = j % rs.stages;
            unsigned char* dst = ring_smem + (size_t)st * rs.stage_bytes;
            const A* row = src.p + (size_t)t * src.ld;
            const uint32_t nd = (uint32_t)(g.dim * sizeof(A)), nv = (uint32_t)(g.vdim * sizeof(A));
            mbar_expect_tx(&s_full[st], (uint32_t)rs.state_bytes + 2 * nd + nv);
            bulk_load(dst, a.state + ((size_t)seq * g.heads + h) * state_elems, (uint32_t)rs.state_bytes, &s_full[st]);
            bulk_load(dst + rs.state_bytes, row + src.q + kg * g.dim, nd, &s_full[st]);
            bulk_load(dst + rs.state_bytes + nd, row + src.k + kg * g.dim, nd, &s_full[st]);
            bulk_load(dst + rs.state_bytes + 2 * nd, row + src.v + h * g.vdim, nv, &s_full[st]);
        };
        // seqs of an item are needed twice, at its load and at its store: the ring of the last loads' slots
        int slot[8];
#pragma unroll
        for (int i = 0; i < 8; i++) slot[i] = 0;
        int loaded = 0, stored = 0;
        auto load_next = [&]() {
            const int seq = seq_of(loaded);
#pragma unroll
            for (int i = 0; i < 8; i++)
                if (i == loaded % rs.stages) slot[i] = seq;
            load(loaded, seq);
            loaded++;
        };
        while (loaded < min(mine, rs.stages)) load_next();
        bool ok = true;
        for (; stored < mine; stored++) {
            const int st = stored % rs.stages;
            if (!mbar_wait(&s_done[st], (uint32_t)(stored / rs.stages) & 1)) { ok = false; break; }
            int seq = 0;
#pragma unroll
            for (int i = 0; i < 8; i++)
                if (i == st) seq = slot[i];
            if (lane == 0) {
                bulk_store(a.state + ((size_t)seq * g.heads + head_of(stored)) * state_elems, ring_smem + (size_t)st * rs.stage_bytes, (uint32_t)rs.state_bytes);
                bulk_commit();
            }
            if (stored > 0 && loaded < mine) {  // the stage before this one has been written out
                if (lane == 0) bulk_wait_read<1>();
                __syncwarp();
                load_next();
            }
        }
        if (lane == 0) {
            if (!ok) {
                atomicCAS(error_flag, 0, 17);
                for (int j = stored; j < loaded; j++) mbar_wait(&s_full[j % rs.stages], (uint32_t)(j / rs.stages) & 1);
            }
            bulk_wait<0>();
        }
        return;
    }
    const int cols = g.vdim / 4, groups = kStepThreads / cols, c = tid % cols, gr = tid / cols;
    // what an item's factors are made of, fetched one item ahead
    auto fetch = [&](int j, float2& bl, int& pos) {
        if (j >= mine) return;
        bl = step_decay(a, (size_t)token_of(j), head_of(j));
        pos = a.tok_pos[token_of(j)];
    };
    float2 bl = make_float2(0.0f, 0.0f);
    int pos = 0;
    fetch(0, bl, pos);
    bool ok = true;
    for (int j = 0; j < mine; j++) {
        const int st = j % rs.stages, h = head_of(j), t = token_of(j);
        float2 bl_next = bl;
        int pos_next = pos;
        fetch(j + 1, bl_next, pos_next);
        const float2 decay = pos > 0 ? decay_of(a, h, bl.y) : make_float2(0.0f, 0.0f);
        if (ok && !mbar_wait(&s_full[st], (uint32_t)(j / rs.stages) & 1)) { ok = false; atomicCAS(error_flag, 0, 17); }  // every thread goes on to the barriers
        float* S = (float*)(ring_smem + (size_t)st * rs.stage_bytes);
        const A *q = (const A*)(S + state_elems), *k = q + g.dim, *v = k + g.dim;
        float* so = s_o + (j & 1) * groups * g.vdim;
        if (gr < groups) {
            float4 u = make_float4(bl.x * act_f<A>(v[4 * c]), bl.x * act_f<A>(v[4 * c + 1]), bl.x * act_f<A>(v[4 * c + 2]), bl.x * act_f<A>(v[4 * c + 3]));
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
            for (int d = gr; d < g.dim; d += groups) {
                float4* at = (float4*)(S + (size_t)d * g.vdim) + c;
                float4 x = *at;
                if (pos == 0) x = make_float4(0.f, 0.f, 0.f, 0.f);
                const float kk = act_f<A>(k[d]), qq = act_f<A>(q[d]);
                x.x = fmaf(kk, u.x, decayed(x.x, decay)); x.y = fmaf(kk, u.y, decayed(x.y, decay));
                x.z = fmaf(kk, u.z, decayed(x.z, decay)); x.w = fmaf(kk, u.w, decayed(x.w, decay));
                o.x = fmaf(x.x, qq, o.x); o.y = fmaf(x.y, qq, o.y); o.z = fmaf(x.z, qq, o.z); o.w = fmaf(x.w, qq, o.w);
                *at = x;
            }
            *((float4*)(so + gr * g.vdim) + c) = o;
        }
        const float skip = a.skip ? a.skip[h] : 0.0f;
        float own = 0.0f;
        if (tid < g.vdim) own = skip * act_f<A>(v[tid]);
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        mbar_arrive(&s_done[st]);
        asm volatile("bar.sync 1, %0;" ::"n"(kStepThreads) : "memory");
        if (tid < g.vdim) {
            for (int i = 0; i < groups; i++) own += so[i * g.vdim + tid];
            a.o[((size_t)t * g.heads + h) * g.vdim + tid] = own;
        }
        bl = bl_next; pos = pos_next;
    }
}

// One CTA per (token, part of the norm); linear_output4_kernel: rows and parts are multiples of four.
template <typename A>
__global__ void __launch_bounds__(512) linear_output4_kernel(const LinearArgs a) {
    __shared__ float sh[32];
    pdl_launch_dependents();
    pdl_wait();
    const LinearShape& g = a.g;
    const int inner = g.heads * g.vdim, n = inner / g.norm_parts, e0 = blockIdx.y * n;
    const size_t t = blockIdx.x;
    const bool gate_first = g.kind == LinearKind::StateSpace;
    const float *o = a.o + t * inner + e0, *w = a.norm_w + e0;
    const A* gate = (const A*)a.proj + t * g.ld + g.off_g + e0;
    A* dst = (A*)a.out + t * a.ldo + e0;
    constexpr int kHeld = 2;  // vectors of a thread that stay in registers between the passes
    auto value = [&](int e, float4& z) {
        float4 v = *(const float4*)(o + e);
        z = four<A>(gate + e);
        if (gate_first) { v.x *= silu_any<A>(z.x); v.y *= silu_any<A>(z.y); v.z *= silu_any<A>(z.z); v.w *= silu_any<A>(z.w); }
        return v;
    };
    float4 v[kHeld], z[kHeld];
    float ss = 0.0f;
    auto square = [&](float4 x) { ss = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, ss)))); };
#pragma unroll
    for (int i = 0; i < kHeld; i++) {
        const int e = (threadIdx.x + i * blockDim.x) * 4;
        if (e < n) v[i] = value(e, z[i]);
        else v[i] = z[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        square(v[i]);
    }
    for (int e = (threadIdx.x + kHeld * blockDim.x) * 4; e < n; e += blockDim.x * 4) { float4 y; square(value(e, y)); }
    const float r = a.out_scale / sqrtf(block_sum_once(ss, sh) / (float)n + g.eps);
    auto put = [&](int e, float4 x, float4 y) {
        const float4 b = *(const float4*)(w + e);
        x.x *= r * b.x; x.y *= r * b.y; x.z *= r * b.z; x.w *= r * b.w;
        if (!gate_first) { x.x *= sigmoid_of<A>(y.x); x.y *= sigmoid_of<A>(y.y); x.z *= sigmoid_of<A>(y.z); x.w *= sigmoid_of<A>(y.w); }
        put_four<A>(dst + e, x);
    };
#pragma unroll
    for (int i = 0; i < kHeld; i++) {
        const int e = (threadIdx.x + i * blockDim.x) * 4;
        if (e < n) put(e, v[i], z[i]);
    }
    for (int e = (threadIdx.x + kHeld * blockDim.x) * 4; e < n; e += blockDim.x * 4) { float4 y; const float4 x = value(e, y); put(e, x, y); }
}
template <typename A>
__global__ void __launch_bounds__(256) linear_output_kernel(const LinearArgs a) {
    __shared__ float sh[32];
    pdl_launch_dependents();
    pdl_wait();
    const LinearShape& g = a.g;
    const int inner = g.heads * g.vdim, n = inner / g.norm_parts, e0 = blockIdx.y * n;
    const size_t t = blockIdx.x;
    const bool gate_first = g.kind == LinearKind::StateSpace;
    const float* o = a.o + t * inner + e0;
    const A* gate = (const A*)a.proj + t * g.ld + g.off_g + e0;
    auto value = [&](int e) { return gate_first ? o[e] * silu_any<A>(act_f<A>(gate[e])) : o[e]; };
    constexpr int kHeld = 8;  // elements of a thread that stay in registers between the passes
    float v[kHeld], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < kHeld; i++) {
        const int e = threadIdx.x + i * blockDim.x;
        v[i] = e < n ? value(e) : 0.0f;
        ss = fmaf(v[i], v[i], ss);
    }
    for (int e = threadIdx.x + kHeld * blockDim.x; e < n; e += blockDim.x) { const float x = value(e); ss = fmaf(x, x, ss); }
    const float r = a.out_scale / sqrtf(block_sum_once(ss, sh) / (float)n + g.eps);
    A* dst = (A*)a.out + t * a.ldo + e0;
    auto put = [&](int e, float x) {
        x *= r * a.norm_w[e0 + e];
        dst[e] = to_act<A>(gate_first ? x : x * sigmoid_of<A>(act_f<A>(gate[e])));
    };
#pragma unroll
    for (int i = 0; i < kHeld; i++) {
        const int e = threadIdx.x + i * blockDim.x;
        if (e < n) put(e, v[i]);
    }
    for (int e = threadIdx.x + kHeld * blockDim.x; e < n; e += blockDim.x) put(e, value(e));
}

int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

template <typename A>
int32_t conv_dispatch(const LinearArgs& a, bool one_each, cudaStream_t s) {
    const int stretch = a.T < 256 ? 1 : 16;
    const dim3 grid((unsigned)((a.T + stretch - 1) / stretch), (unsigned)((a.g.channels + 255) / 256));
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(launch_pdl(kern, grid, dim3(128), 0, s, a, stretch, one_each ? 1 : 0));
        return LC_OK;
    };
    switch (a.g.taps) {
        case 2: return go(linear_conv_kernel<A, 2>);
        case 3: return go(linear_conv_kernel<A, 3>);
        case 4: return go(linear_conv_kernel<A, 4>);
        default: return go(linear_conv_kernel<A, 0>);
    }
}

template <typename A>
int32_t scan_dispatch(const LinearArgs& a, cudaStream_t s) {
    const dim3 grid((unsigned)a.n_runs, (unsigned)a.g.heads, (unsigned)((a.g.vdim + 31) / 32));
    const int dp = padded_dim(a.g.dim);
    const size_t smem = (size_t)kScanTok * (2 * dp + 32 + 3) * sizeof(float);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3(128), smem, s, a));
        return LC_OK;
    };
    switch (dp) {
        case 32: return go(linear_scan_kernel<A, 8>);
        case 64: return go(linear_scan_kernel<A, 16>);
        case 128: return go(linear_scan_kernel<A, 32>);
        default: return go(linear_scan_kernel<A, 64>);
    }
}

int32_t chunk_dispatch(const LinearArgs& a, cudaStream_t s) {
    const dim3 grid((unsigned)a.n_chunk_runs, (unsigned)a.g.heads, (unsigned)((a.g.vdim + kCols - 1) / kCols));
    const int dp = padded_dim(a.g.dim);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, chunk_smem(dp)));
        LC_CUDA(launch_pdl(kern, grid, dim3(kChunkThreads), chunk_smem(dp), s, a));
        return LC_OK;
    };
    switch (dp) {
        case 32: return go(linear_chunk_kernel<32>);
        case 64: return go(linear_chunk_kernel<64>);
        case 128: return go(linear_chunk_kernel<128>);
        default: return go(linear_chunk_kernel<256>);
    }
}

template <typename A>
int32_t step_dispatch(const LinearArgs& a, cudaStream_t s) {
    const int vec = a.g.vdim % 4 == 0 ? 4 : 1, cols = a.g.vdim / vec;
    LC_CHECK(cols <= kStepThreads, LC_ERR_UNSUPPORTED, "linear recurrence: %d value dimensions per head", a.g.vdim);
    const int groups = kStepThreads / cols, rows = (a.g.dim + groups - 1) / groups;
    const size_t smem = (size_t)(2 * a.g.dim + a.g.vdim + groups * a.g.vdim) * sizeof(float);
    const dim3 grid((unsigned)a.g.heads, (unsigned)a.T);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3(kStepThreads), smem, s, a));
        return LC_OK;
    };
    if (vec == 4) return rows <= 4 ? go(linear_step_kernel<A, 4, 4>) : rows <= 8 ? go(linear_step_kernel<A, 4, 8>) : rows <= 16 ? go(linear_step_kernel<A, 4, 16>) : go(linear_step_kernel<A, 4, 0>);
    return rows <= 16 ? go(linear_step_kernel<A, 1, 16>) : go(linear_step_kernel<A, 1, 0>);
}

// How the ring of states fits; stages 0: it does not, or there are too few items for it.
RingShape ring_shape(const LinearArgs& a) {
    const LinearShape& g = a.g;
    const int elt = a.f32 ? 4 : 2, groups = g.vdim >= 4 ? kStepThreads / (g.vdim / 4) : 0;
    RingShape r{0, g.dim * g.vdim * 4, 0};
    if (g.dim % 8 || g.vdim % 8 || g.vdim > kStepThreads || g.heads * a.T < 2 * sm_count()) return r;
    r.stage_bytes = (r.state_bytes + (2 * g.dim + g.vdim) * elt + 127) / 128 * 128;
    const int room = (int)kMaxSmem - 1024 - 2 * groups * g.vdim * 4, stages = room / r.stage_bytes;
    r.stages = stages < 3 ? 0 : std::min(stages, 6);
    return r;
}
template <typename A>
int32_t ring_dispatch(const LinearArgs& a, int* launches, cudaStream_t s) {
    if (a.g.kind == LinearKind::StateSpace) { LC_TRY(conv_dispatch<A>(a, true, s)); ++*launches; }
    const RingShape r = ring_shape(a);
    const size_t smem = (size_t)r.stages * r.stage_bytes + (size_t)2 * (kStepThreads / (a.g.vdim / 4)) * a.g.vdim * 4;
    LC_CUDA(ensure_smem_limit((const void*)linear_ring_kernel<A>, smem));
    LC_CUDA(launch_pdl(linear_ring_kernel<A>, dim3((unsigned)std::min(a.g.heads * a.T, sm_count())), dim3(kRingThreads), smem, s, a, r, gemv_error_flag_dev()));
    ++*launches;
    return LC_OK;
}

}  // namespace

bool linear_chunks_apply(const LinearShape& g, bool f32) { return !f32 && g.dim % 8 == 0 && g.vdim % 8 == 0 && g.dim <= 256; }

int32_t launch_linear_runs(const LinearArgs& a, int* launches, cudaStream_t s) {
    LC_CHECK(a.g.dim <= 256, LC_ERR_UNSUPPORTED, "linear recurrence: %d state dimensions per head (at most 256)", a.g.dim);
    const bool conv = a.g.kind == LinearKind::StateSpace;
    if (conv) { LC_TRY(a.f32 ? conv_dispatch<float>(a, false, s) : conv_dispatch<bf16>(a, false, s)); ++*launches; }
    if (a.n_runs) { LC_TRY(a.f32 ? scan_dispatch<float>(a, s) : scan_dispatch<bf16>(a, s)); ++*launches; }
    if (a.n_chunk_runs) { LC_TRY(chunk_dispatch(a, s)); ++*launches; }
    if (!conv) return LC_OK;
    const dim3 grid((unsigned)a.n_all_runs, (unsigned)((a.g.channels + 255) / 256));
    if (a.f32) LC_CUDA(launch_pdl(linear_keep_kernel<float>, grid, dim3(256), 0, s, a));
    else LC_CUDA(launch_pdl(linear_keep_kernel<bf16>, grid, dim3(256), 0, s, a));
    ++*launches;
    return LC_OK;
}
int32_t launch_linear_step(const LinearArgs& a, int* launches, cudaStream_t s) {
    if (ring_shape(a).stages) return a.f32 ? ring_dispatch<float>(a, launches, s) : ring_dispatch<bf16>(a, launches, s);
    ++*launches;
    return a.f32 ? step_dispatch<float>(a, s) : step_dispatch<bf16>(a, s);
}
int32_t launch_linear_output(const LinearArgs& a, cudaStream_t s) {
    const int n = a.g.heads * a.g.vdim / a.g.norm_parts;
    if (n % 4 == 0 && a.ldo % 4 == 0 && a.g.off_g % 4 == 0 && (uintptr_t)a.norm_w % 16 == 0) {
        const dim3 grid((unsigned)a.T, (unsigned)a.g.norm_parts), block((unsigned)std::max(32, std::min(512, (n / 8 + 31) / 32 * 32)));
        if (a.f32) LC_CUDA(launch_pdl(linear_output4_kernel<float>, grid, block, 0, s, a));
        else LC_CUDA(launch_pdl(linear_output4_kernel<bf16>, grid, block, 0, s, a));
        return LC_OK;
    }
    const dim3 grid((unsigned)a.T, (unsigned)a.g.norm_parts), block((unsigned)std::min(256, (n + 31) / 32 * 32));
    if (a.f32) LC_CUDA(launch_pdl(linear_output_kernel<float>, grid, block, 0, s, a));
    else LC_CUDA(launch_pdl(linear_output_kernel<bf16>, grid, block, 0, s, a));
    return LC_OK;
}

}  // namespace lc
