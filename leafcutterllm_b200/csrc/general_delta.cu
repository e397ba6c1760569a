// A delta rule whose removal is apart from its writing: per head, over a state S of dim x dim in f32,
//   S_t = D_t S_(t-1) - b_t z_t^T + k_t v_t^T,   z_t = S_(t-1)^T u_t,   o_t = S_t^T r_t,
// with D_t = diag(w_t), u_t the unit key and b_t = a_t u_t (every key channel has its own rate a).
//   general_scan_kernel   runs of few tokens, and models in true 32-bit: token by token
//   general_step_kernel   one token per sequence: recurrence, norm and gate of one head of one token per CTA; the state is read and
//                         written once and stays in registers between
//   general_chunk_kernel, general_carry_kernel   longer runs, kGeneralChunk tokens at a time:
// Inside a chunk let G_t be the sum of the log decays up to token t (per key channel) and S0 the state before the chunk.  Unrolled,
//   z_t = (e^G_(t-1) u_t)^T S0 + sum_(s < t) (Auk_ts v_s - Aub_ts z_s),   Axy_ts = sum_d x_t e^(G_(t-1) - G_s) y_s,
//   o_t = (e^G_t r_t)^T S0 + sum_(s <= t) (Brk_ts v_s - Brb_ts z_s),      Brx_ts = sum_d r_t e^(G_t - G_s) x_s.
// Solving the triangular system for its two right-hand sides, Z = W S0 + Y with
//   W = (I + Aub)^-1 (e^G_(t-1) u),   Y = (I + Aub)^-1 Auk V,
// turns the chunk into one product per state and value column:
//   [S; O] = [M; R] S0 + [C; P],   M = diag(e^G_end) - Bh^T W,  C = Kh^T V - Bh^T Y,  R = e^G r - Brb W,  P = Brk V - Brb Y,
// with Kh, Bh = e^(G_end - G_s) k_s, b_s.  general_chunk_kernel leaves M, R, C and P (all chunks of all heads at once),
// general_carry_kernel walks the chunks (one CTA per run, head and 32 value columns).
// The exponents are taken relative to the chunk's middle, G_t - G_m and G_m - G_s: with log decays of at most `decay_scale` per token
// they stay below 16 decay_scale, so every factor is an ordinary number.
#include <algorithm>
#include <cmath>
#include "lc_mixers.h"
#include "lc_mma.cuh"
#include "lc_tma.cuh"

namespace lc {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

// ---- token by token ---------------------------------------------------------------------------------------------------------
// A CTA of four warps owns 32 value columns of one head of one run; four lanes share a column's state entries (DPL each: float4
// groups dealt round robin), eight columns per warp.
constexpr int kScanTok = 16;  // tokens staged in shared memory at a time
template <int DPL>
__global__ void __launch_bounds__(128) general_scan_kernel(const GeneralArgs a) {
    constexpr int DP = DPL * 4;
    extern __shared__ __align__(16) float sm[];
    float *s_r = sm, *s_k = s_r + kScanTok * DP, *s_w = s_k + kScanTok * DP, *s_b = s_w + kScanTok * DP, *s_v = s_b + kScanTok * DP, *s_rk = s_v + kScanTok * 32;
    pdl_launch_dependents();
    pdl_wait();
    const GeneralShape& g = a.g;
    const SeqRun run = a.runs[blockIdx.x];
    const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r4 = lane & 3, col = warp * 8 + (lane >> 2), e = blockIdx.z * 32 + col, n = g.heads * g.dim;
    float* st = a.state + ((size_t)run.seq * g.heads + h) * g.dim * g.dim;
    float S[DPL];
#pragma unroll
    for (int i = 0; i < DPL; i++) {
        const int d = (i >> 2) * 16 + r4 * 4 + (i & 3);
        S[i] = (run.pos0 > 0 && d < g.dim && e < g.dim) ? st[(size_t)d * g.dim + e] : 0.0f;
    }
    for (int c0 = 0; c0 < run.n; c0 += kScanTok) {
        const int m = min(kScanTok, run.n - c0);
        __syncthreads();
        for (int t = warp; t < m; t += 4) {  // a warp per token: its operands and its key's length
            const size_t tok = (size_t)(run.tok0 + c0 + t);
            const float *p = a.proj + tok * g.ld + h * g.dim, *l = a.log_decay + tok * n + h * g.dim;
            float ss = 0.0f;
            for (int d = lane; d < DP; d += 32) {
                const bool ok = d < g.dim;
                const float k = ok ? p[g.off_k + d] : 0.0f;
                s_r[t * DP + d] = ok ? p[d] : 0.0f;
                s_k[t * DP + d] = k;
                s_w[t * DP + d] = ok ? expf(l[d]) : 0.0f;
                s_b[t * DP + d] = ok ? k * sigmoid_f(p[g.off_a + d] + a.a_bias[h * g.dim + d]) : 0.0f;
                ss = fmaf(k, k, ss);
            }
            const int c = blockIdx.z * 32 + lane;
            s_v[t * 32 + lane] = c < g.dim ? p[g.off_v + c] : 0.0f;
            ss = warp_sum(ss);
            if (lane == 0) s_rk[t] = 1.0f / (ss + g.unit_eps);  // once for the unit key that is looked for, once for the one that is removed
        }
        __syncthreads();
        for (int t = 0; t < m; t++) {
            const float4 *r4p = (const float4*)(s_r + t * DP), *k4p = (const float4*)(s_k + t * DP), *w4p = (const float4*)(s_w + t * DP), *b4p = (const float4*)(s_b + t * DP);
            float kk[DPL], z = 0.0f;
#pragma unroll
            for (int i = 0; i < DPL / 4; i++) {
                const float4 kv = k4p[i * 4 + r4];
                kk[4 * i] = kv.x; kk[4 * i + 1] = kv.y; kk[4 * i + 2] = kv.z; kk[4 * i + 3] = kv.w;
#pragma unroll
                for (int j = 0; j < 4; j++) z = fmaf(S[4 * i + j], kk[4 * i + j], z);
            }
            z += __shfl_xor_sync(0xffffffffu, z, 1);
            z += __shfl_xor_sync(0xffffffffu, z, 2);
            z *= s_rk[t];
            const float v = s_v[t * 32 + col];
            float o = 0.0f;
#pragma unroll
            for (int i = 0; i < DPL / 4; i++) {
                const float4 rv = r4p[i * 4 + r4], wv = w4p[i * 4 + r4], bv = b4p[i * 4 + r4];
                const float rr[4] = {rv.x, rv.y, rv.z, rv.w}, ww[4] = {wv.x, wv.y, wv.z, wv.w}, bb[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    S[4 * i + j] = fmaf(kk[4 * i + j], v, fmaf(ww[j], S[4 * i + j], -bb[j] * z));
                    o = fmaf(S[4 * i + j], rr[j], o);
                }
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (r4 == 0 && e < g.dim) a.o[(size_t)(run.tok0 + c0 + t) * n + h * g.dim + e] = o;
        }
    }
#pragma unroll
    for (int i = 0; i < DPL; i++) {
        const int d = (i >> 2) * 16 + r4 * 4 + (i & 3);
        if (d < g.dim && e < g.dim) st[(size_t)d * g.dim + e] = S[i];
    }
}

// ---- one token per sequence -------------------------------------------------------------------------------------------------
// With y = S^T (w r):  o = y - z (b . r) + v (k . r), so the state is walked once; a thread owns VEC neighbouring value columns and
// every `groups`-th key row, kept in registers (ROWS of them; 0: re-read for the update).  Thread i < dim also owns channel i.
template <typename A, int VEC, int ROWS, int THREADS>
__global__ void __launch_bounds__(THREADS) general_step_kernel(const GeneralArgs a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[32], s_sum[3][THREADS / 32];
    pdl_launch_dependents();
    pdl_wait();
    const GeneralShape& g = a.g;
    const int h = blockIdx.x, t = blockIdx.y, seq = a.tok_seq[t], tid = threadIdx.x, dim = g.dim, cols = dim / VEC, groups = THREADS / cols;
    float *s_k = sm, *s_w = s_k + dim, *s_wr = s_w + dim, *s_b = s_wr + dim, *s_v = s_b + dim, *s_z = s_v + dim, *s_y = s_z + groups * dim;
    const int c = tid % cols, gr = tid / cols;
    float* st = a.state + ((size_t)seq * g.heads + h) * dim * dim + c * VEC;
    const bool live = a.tok_pos[t] > 0, mine = gr < groups;
    float S[ROWS > 0 ? ROWS : 1][VEC];
    auto load = [&](int d, float (&v)[VEC]) {
#pragma unroll
        for (int j = 0; j < VEC; j++) v[j] = 0.0f;
        if (d >= dim || !live) return;
        if constexpr (VEC == 4) { const float4 f = *(const float4*)(st + (size_t)d * dim); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
        else v[0] = st[(size_t)d * dim];
    };
    auto store = [&](int d, const float (&v)[VEC]) {
        if constexpr (VEC == 4) *(float4*)(st + (size_t)d * dim) = make_float4(v[0], v[1], v[2], v[3]);
        else st[(size_t)d * dim] = v[0];
    };
    if (ROWS > 0 && mine) {
#pragma unroll
        for (int i = 0; i < ROWS; i++) load(gr + i * groups, S[i]);
    }
    float r = 0.0f, k = 0.0f, v = 0.0f, lw = 0.0f, ra = 0.0f, gate = 0.0f, norm = 0.0f;
    if (tid < dim) {
        const int ch = h * dim + tid;
        const float* p = a.proj + (size_t)t * g.ld + ch;
        r = p[0]; k = p[g.off_k]; v = p[g.off_v]; ra = p[g.off_a] + a.a_bias[ch];
        lw = a.log_decay[(size_t)t * g.heads * dim + ch];
        gate = act_f<A>(((const A*)a.gate)[(size_t)t * a.ld_gate + ch]);
        norm = a.norm_w[ch];
    }
    const float w = expf(lw), b = sigmoid_f(ra) * k;  // b still without the key's length
    if (tid < dim) { s_k[tid] = k; s_w[tid] = w; s_wr[tid] = w * r; s_b[tid] = b; s_v[tid] = v; }
    const float kk = warp_sum(k * k), kr = warp_sum(k * r), br = warp_sum(b * r);
    if ((tid & 31) == 0) { s_sum[0][tid >> 5] = kk; s_sum[1][tid >> 5] = kr; s_sum[2][tid >> 5] = br; }
    __syncthreads();
    float dz[VEC], dy[VEC];
#pragma unroll
    for (int j = 0; j < VEC; j++) dz[j] = dy[j] = 0.0f;
    auto look = [&](int d, const float (&x)[VEC]) {
        const float kd = s_k[d], wr = s_wr[d];
#pragma unroll
        for (int j = 0; j < VEC; j++) { dz[j] = fmaf(x[j], kd, dz[j]); dy[j] = fmaf(x[j], wr, dy[j]); }
    };
    if (mine) {
        if constexpr (ROWS > 0) {
#pragma unroll
            for (int i = 0; i < ROWS; i++)
                if (gr + i * groups < dim) look(gr + i * groups, S[i]);
        } else {
            for (int d = gr; d < dim; d += groups) { float x[VEC]; load(d, x); look(d, x); }
        }
#pragma unroll
        for (int j = 0; j < VEC; j++) { s_z[gr * dim + c * VEC + j] = dz[j]; s_y[gr * dim + c * VEC + j] = dy[j]; }
    }
    __syncthreads();
    float o = 0.0f;
    if (tid < dim) {
        float z = 0.0f, y = 0.0f, n2 = g.unit_eps, sr = 0.0f, sb = 0.0f;
        for (int i = 0; i < (dim + 31) / 32; i++) { n2 += s_sum[0][i]; sr += s_sum[1][i]; sb += s_sum[2][i]; }
        for (int i = 0; i < groups; i++) { z += s_z[i * dim + tid]; y += s_y[i * dim + tid]; }
        z /= n2;  // both unit keys' lengths
        o = y - z * sb + v * sr;
        s_z[tid] = z;
    }
    const float ss = block_sum(o * o, red);  // also publishes z
    if (mine) {
        float z[VEC], u[VEC];
#pragma unroll
        for (int j = 0; j < VEC; j++) { z[j] = s_z[c * VEC + j]; u[j] = s_v[c * VEC + j]; }
        auto change = [&](int d, float (&x)[VEC]) {
            const float wd = s_w[d], bd = s_b[d], kd = s_k[d];
#pragma unroll
            for (int j = 0; j < VEC; j++) x[j] = fmaf(kd, u[j], fmaf(wd, x[j], -bd * z[j]));
            store(d, x);
        };
        if constexpr (ROWS > 0) {
#pragma unroll
            for (int i = 0; i < ROWS; i++)
                if (gr + i * groups < dim) change(gr + i * groups, S[i]);
        } else {
            for (int d = gr; d < dim; d += groups) { float x[VEC]; load(d, x); change(d, x); }
        }
    }
    if (tid < dim) ((A*)a.out)[(size_t)t * a.ldo + h * dim + tid] = to_act<A>(o / sqrtf(ss / (float)dim + g.eps) * norm * sigmoid_f(gate));
}

// ---- chunks -------------------------------------------------------------------------------------------------------------------
constexpr int kT = kGeneralChunk, kPitch = kT + 4, kHalves = kDeltaChunk / kT, kThreads = 384, kWarps = kThreads / 32;
// What general_chunk_kernel leaves of one (chunk, head), in floats: rows 0 .. dp - 1 belong to the state, dp .. dp + 31 to the tokens.
struct ItemLayout {
    int dp;
    __host__ __device__ int rows() const { return dp + kT; }
    __host__ __device__ size_t co() const { return (size_t)dp * rows(); }           // M | R: [dp][rows] (transposed); C | P: [dp / 32][rows][32]
    __host__ __device__ size_t size() const { return 2 * co(); }
};

__device__ __forceinline__ void get4(float (&x)[4], const float* p) {
    const float4 f = *(const float4*)p;
    x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
}

template <int DP>
__global__ void __launch_bounds__(kThreads, DP <= 64 ? 2 : 1) general_chunk_kernel(const GeneralArgs a, float* __restrict__ scratch) {
    constexpr int kQuads = (DP / 4 + kWarps - 1) / kWarps;  // fours of channels per warp
    extern __shared__ __align__(16) float sm[];
    // channel-major [DP][kPitch]: u e^(G_(t-1) - G_m), r e^(G_t - G_m), k e^(G_m - G_t), b e^(G_m - G_t)
    float *s_u = sm, *s_r = s_u + DP * kPitch, *s_k = s_r + DP * kPitch, *s_b = s_k + DP * kPitch;
    float *s_v = s_b + DP * kPitch, *s_x = s_v + kT * DP;                             // [kT][DP] v; [kT][2 DP] W | Y
    float *s_auk = s_x + 2 * kT * DP, *s_aub = s_auk + kT * kPitch, *s_brk = s_aub + kT * kPitch, *s_brb = s_brk + kT * kPitch;
    float *s_cm = s_brb + kT * kPitch, *s_ce = s_cm + DP, *s_ge = s_ce + DP;          // e^G_m, e^(G_end - G_m), e^G_end
    float* s_len = s_ge + DP;                                                         // [kWarps][32]
    pdl_launch_dependents();
    pdl_wait();
    const GeneralShape& g = a.g;
    const DeltaChunk ck = a.chunks[blockIdx.x / kHalves];
    const int sub = blockIdx.x % kHalves, n = min(kT, ck.n - sub * kT), h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, dim = g.dim;
    if (n <= 0) return;
    const size_t tok0 = (size_t)ck.tok0 + sub * kT;
    const ItemLayout L{DP};
    float* out = scratch + ((size_t)blockIdx.x * g.heads + h) * L.size();
    const bool vec = dim % 4 == 0;
    auto four = [&](const float* p, int d, bool ok, float (&x)[4]) {
        if (vec) {
            const float4 f = ok && d < dim ? *(const float4*)(p + d) : make_float4(0.f, 0.f, 0.f, 0.f);
            x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
        } else {
#pragma unroll
            for (int j = 0; j < 4; j++) x[j] = ok && d + j < dim ? p[d + j] : 0.0f;
        }
    };
    {  // a lane per token
        const bool ok = lane < n;
        const size_t tok = tok0 + (ok ? lane : 0);
        const float *p = a.proj + tok * g.ld + h * dim, *l = a.log_decay + tok * g.heads * dim + h * dim, *ab = a.a_bias + h * dim;
        float k[kQuads][4], ss = 0.0f;
#pragma unroll
        for (int i = 0; i < kQuads; i++) {
            const int d = 4 * (warp + i * kWarps);
            if (d < DP) four(p + g.off_k, d, ok, k[i]);
            else k[i][0] = k[i][1] = k[i][2] = k[i][3] = 0.0f;
#pragma unroll
            for (int j = 0; j < 4; j++) ss = fmaf(k[i][j], k[i][j], ss);
        }
        s_len[warp * 32 + lane] = ss;
        for (int i = tid; i < kT * DP / 4; i += kThreads) {
            const int t = i / (DP / 4), e = (i - t * (DP / 4)) * 4;
            float v[4];
            four(a.proj + (tok0 + (t < n ? t : 0)) * g.ld + g.off_v + h * dim, e, t < n, v);
            *(float4*)(s_v + t * DP + e) = make_float4(v[0], v[1], v[2], v[3]);
        }
        __syncthreads();
        ss = g.unit_eps;
#pragma unroll
        for (int w = 0; w < kWarps; w++) ss += s_len[w * 32 + lane];
        const float rk = 1.0f / sqrtf(ss);
#pragma unroll
        for (int i = 0; i < kQuads; i++) {
            const int d0 = 4 * (warp + i * kWarps);
            if (d0 >= DP) break;
            float r[4], ld[4], ra[4], bias[4];
            four(p, d0, ok, r);
            four(l, d0, ok, ld);
            four(p + g.off_a, d0, ok, ra);
            four(ab, d0, true, bias);
#pragma unroll
            for (int j = 0; j < 4; j++) {
                float G = ld[j] * kLog2e;
#pragma unroll
                for (int o = 1; o < 32; o *= 2) {
                    const float y = __shfl_up_sync(0xffffffffu, G, o);
                    if (lane >= o) G += y;
                }
                const float up = __shfl_up_sync(0xffffffffu, G, 1), gp = lane > 0 ? up : 0.0f, gm = __shfl_sync(0xffffffffu, G, kT / 2 - 1), ge = __shfl_sync(0xffffffffu, G, 31);
                const float u = k[i][j] * rk, back = exp2f(gm - G);
                const int d = d0 + j, at = d * kPitch + lane;
                s_u[at] = u * exp2f(gp - gm);
                s_r[at] = r[j] * exp2f(G - gm);
                s_k[at] = k[i][j] * back;
                s_b[at] = sigmoid_f(ra[j] + bias[j]) * u * back;
                if (lane == 0) { s_cm[d] = exp2f(gm); s_ce[d] = exp2f(ge - gm); s_ge[d] = exp2f(ge); }
            }
        }
    }
    __syncthreads();
    // the four triangles, one 4 x 4 tile of two of them per thread and quarter of the channels
    if (tid < 288) {
        const int kq = tid & 3, pair = (tid >> 2) & 1;
        int ti = 0, tj = tid >> 3;
        while (tj > ti) { tj -= ti + 1; ti++; }
        const float *x = (pair ? s_r : s_u) + 4 * ti, *yk = s_k + 4 * tj, *yb = s_b + 4 * tj;
        float ak[4][4] = {}, ab[4][4] = {};
#pragma unroll 4
        for (int d = kq; d < DP; d += 4) {
            float xt[4], ks[4], bs[4];
            get4(xt, x + d * kPitch); get4(ks, yk + d * kPitch); get4(bs, yb + d * kPitch);
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) { ak[i][j] = fmaf(xt[i], ks[j], ak[i][j]); ab[i][j] = fmaf(xt[i], bs[j], ab[i][j]); }
        }
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) {
                ak[i][j] += __shfl_xor_sync(0xffffffffu, ak[i][j], 1);
                ak[i][j] += __shfl_xor_sync(0xffffffffu, ak[i][j], 2);
                ab[i][j] += __shfl_xor_sync(0xffffffffu, ab[i][j], 1);
                ab[i][j] += __shfl_xor_sync(0xffffffffu, ab[i][j], 2);
                const int t = 4 * ti + i, s = 4 * tj + j;
                if (s > t || (s == t && !pair)) ak[i][j] = ab[i][j] = 0.0f;
            }
        float *mk = pair ? s_brk : s_auk, *mb = pair ? s_brb : s_aub;
#pragma unroll
        for (int i = 0; i < 4; i++)
            if (kq == i) {
                *(float4*)(mk + (4 * ti + i) * kPitch + 4 * tj) = make_float4(ak[i][0], ak[i][1], ak[i][2], ak[i][3]);
                *(float4*)(mb + (4 * ti + i) * kPitch + 4 * tj) = make_float4(ab[i][0], ab[i][1], ab[i][2], ab[i][3]);
            }
    }
    __syncthreads();
    // forward substitution, one column of W or Y per thread
    for (int col = tid; col < 2 * DP; col += kThreads) {
        float x[kT];
        if (col < DP) {
            const float cm = s_cm[col];
#pragma unroll
            for (int t = 0; t < kT; t += 4) {
                float q[4];
                get4(q, s_u + col * kPitch + t);
#pragma unroll
                for (int j = 0; j < 4; j++) x[t + j] = q[j] * cm;
            }
        } else {
            float v[kT];
#pragma unroll
            for (int t = 0; t < kT; t++) v[t] = s_v[t * DP + col - DP];
#pragma unroll
            for (int t = 0; t < kT; t++) {
                float p[2] = {0.0f, 0.0f};
#pragma unroll
                for (int s = 0; s < t; s += 4) {
                    float m[4];
                    get4(m, s_auk + t * kPitch + s);
#pragma unroll
                    for (int j = 0; j < 4; j++)
                        if (s + j < t) p[j & 1] = fmaf(m[j], v[s + j], p[j & 1]);
                }
                x[t] = p[0] + p[1];
            }
        }
#pragma unroll
        for (int t = 0; t < kT; t++) {
            float p[2] = {0.0f, 0.0f};
#pragma unroll
            for (int s = 0; s < t; s += 4) {
                float m[4];
                get4(m, s_aub + t * kPitch + s);
#pragma unroll
                for (int j = 0; j < 4; j++)
                    if (s + j < t) p[j & 1] = fmaf(m[j], x[s + j], p[j & 1]);
            }
            x[t] -= p[0] + p[1];
            s_x[t * 2 * DP + col] = x[t];
        }
    }
    __syncthreads();
    // M, R, C and P in tiles of 4 x 4
    constexpr int kCols = DP / 4, kTasks = (DP + kT) / 4 * kCols;
    for (int task = tid; task < kTasks; task += kThreads) {
        const int e0 = task % kCols * 4, row0 = task / kCols * 4;
        const bool token = row0 >= DP;
        const int t0 = row0 - DP;
        const float *lk = token ? s_brk + t0 * kPitch : s_k + row0 * kPitch, *lb = token ? s_brb + t0 * kPitch : s_b + row0 * kPitch;
        const int end = token ? t0 + 4 : kT;
        float m[4][4] = {}, c[4][4] = {};
        for (int s = 0; s < end; s += 4) {
            float xb[4][4], xk[4][4];
#pragma unroll
            for (int i = 0; i < 4; i++) { get4(xb[i], lb + i * kPitch + s); get4(xk[i], lk + i * kPitch + s); }
#pragma unroll
            for (int j = 0; j < 4; j++) {
                float w[4], y[4], v[4];
                get4(w, s_x + (s + j) * 2 * DP + e0); get4(y, s_x + (s + j) * 2 * DP + DP + e0); get4(v, s_v + (s + j) * DP + e0);
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int q = 0; q < 4; q++) {
                        m[i][q] = fmaf(-xb[i][j], w[q], m[i][q]);
                        c[i][q] = fmaf(xk[i][j], v[q], c[i][q]);
                        c[i][q] = fmaf(-xb[i][j], y[q], c[i][q]);
                    }
            }
        }
        if (token) {
#pragma unroll
            for (int q = 0; q < 4; q++) {
                float r[4];
                get4(r, s_r + (e0 + q) * kPitch + t0);
                const float cm = s_cm[e0 + q];
#pragma unroll
                for (int i = 0; i < 4; i++) m[i][q] = fmaf(r[i], cm, m[i][q]);
            }
        } else {
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const float ce = s_ce[row0 + i];
#pragma unroll
                for (int q = 0; q < 4; q++) { m[i][q] = fmaf(m[i][q], ce, e0 + q == row0 + i ? s_ge[row0 + i] : 0.0f); c[i][q] *= ce; }
            }
        }
        float* co = out + L.co() + (size_t)(e0 / 32) * L.rows() * 32 + e0 % 32;
#pragma unroll
        for (int i = 0; i < 4; i++) {
            *(float4*)(out + (size_t)(e0 + i) * L.rows() + row0) = make_float4(m[0][i], m[1][i], m[2][i], m[3][i]);
            *(float4*)(co + (size_t)(row0 + i) * 32) = make_float4(c[i][0], c[i][1], c[i][2], c[i][3]);
        }
    }
}

// A product of (dp + 32) x dp by dp x 32 per chunk, in 4 x 4 tiles; the operands of the chunk behind the next one travel meanwhile.
template <int DP>
__global__ void __launch_bounds__(2 * DP + 64) general_carry_kernel(const GeneralArgs a, const float* __restrict__ scratch, int* error_flag) {
    constexpr int kRows = DP + kT, kMr = DP * kRows, kCo = kRows * 32;
    extern __shared__ __align__(128) float sm[];
    __shared__ uint64_t full[2];
    float *s_mr = sm, *s_co = s_mr + 2 * kMr, *s_S = s_co + 2 * kCo;
    const int tid = threadIdx.x, rg = tid >> 3, eg = tid & 7;
    if (tid == 0) {
        mbar_init(&full[0], 1);
        mbar_init(&full[1], 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    pdl_launch_dependents();
    __syncthreads();
    pdl_wait();
    const GeneralShape& g = a.g;
    const DeltaChunkRun cr = a.chunk_runs[blockIdx.x];
    const int h = blockIdx.y, e0 = blockIdx.z * 32, chunks = (cr.run.n + kT - 1) / kT;
    const ItemLayout L{DP};
    float* st = a.state + ((size_t)cr.run.seq * g.heads + h) * g.dim * g.dim;
    auto request = [&](int c) {  // one thread
        const float* src = scratch + ((size_t)(cr.chunk0 * kHalves + c) * g.heads + h) * L.size();
        mbar_expect_tx(&full[c & 1], (uint32_t)(kMr + kCo) * 4);
        bulk_load(s_mr + (c & 1) * kMr, src, (uint32_t)kMr * 4, &full[c & 1]);
        bulk_load(s_co + (c & 1) * kCo, src + L.co() + (size_t)blockIdx.z * kCo, (uint32_t)kCo * 4, &full[c & 1]);
    };
    if (tid == 0) {
        request(0);
        if (chunks > 1) request(1);
    }
    const bool owner = 4 * rg < DP;  // of state rows; the others make the tokens' read-outs
    float S[4][4] = {};
    auto publish = [&]() {
#pragma unroll
        for (int i = 0; i < 4; i++) *(float4*)(s_S + (4 * rg + i) * 32 + 4 * eg) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
    };
    if (owner) {
        if (cr.run.pos0 > 0)
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const int d = 4 * rg + i, e = e0 + 4 * eg + j;
                    if (d < g.dim && e < g.dim) S[i][j] = st[(size_t)d * g.dim + e];
                }
        publish();
    }
    __syncthreads();
    for (int c = 0; c < chunks; c++) {
        const float *mr = s_mr + (c & 1) * kMr + 4 * rg, *co = s_co + (c & 1) * kCo + 4 * rg * 32 + 4 * eg, *sp = s_S + 4 * eg;
        if (!mbar_wait(&full[c & 1], (uint32_t)(c >> 1) & 1) && tid == 0) atomicExch(error_flag, 17);
#pragma unroll
        for (int i = 0; i < 4; i++) get4(S[i], co + i * 32);
#pragma unroll 8
        for (int d = 0; d < DP; d++) {
            float x[4], y[4];
            get4(x, mr + d * kRows);
            get4(y, sp + d * 32);
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) S[i][j] = fmaf(x[i], y[j], S[i][j]);
        }
        __syncthreads();
        if (tid == 0 && c + 2 < chunks) request(c + 2);
        if (owner) publish();
        else {
            const int t0 = c * kT + 4 * rg - DP;
#pragma unroll
            for (int i = 0; i < 4; i++) {
                if (t0 + i >= cr.run.n) break;
                float* o = a.o + (size_t)(cr.run.tok0 + t0 + i) * g.heads * g.dim + h * g.dim + e0 + 4 * eg;
#pragma unroll
                for (int j = 0; j < 4; j++)
                    if (e0 + 4 * eg + j < g.dim) o[j] = S[i][j];
            }
        }
        __syncthreads();
    }
    if (owner)
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int d = 4 * rg + i, e = e0 + 4 * eg + j;
                if (d < g.dim && e < g.dim) st[(size_t)d * g.dim + e] = S[i][j];
            }
}

int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : 128; }
size_t chunk_smem(int dp) { return ((size_t)4 * dp * kPitch + 3 * kT * dp + 4 * kT * kPitch + 3 * dp + 32 * kWarps) * sizeof(float); }
size_t carry_smem(int dp) { return ((size_t)2 * dp * (dp + kT) + 2 * (dp + kT) * 32 + dp * 32) * sizeof(float); }

template <typename A>
int32_t step_dispatch(const GeneralArgs& a, cudaStream_t s) {
    const int dim = a.g.dim, vec = dim % 4 == 0 ? 4 : 1, cols = dim / vec, threads = vec == 4 && dim * dim >= 8192 ? 512 : 256;
    const int groups = threads / cols, rows = (dim + groups - 1) / groups;
    const size_t smem = (size_t)(5 * dim + 2 * groups * dim) * sizeof(float);
    const dim3 grid((unsigned)a.g.heads, (unsigned)a.T);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3((unsigned)threads), smem, s, a));
        return LC_OK;
    };
    if (threads == 512) return rows <= 8 ? go(general_step_kernel<A, 4, 8, 512>) : go(general_step_kernel<A, 4, 0, 512>);
    if (vec == 4) return rows <= 4 ? go(general_step_kernel<A, 4, 4, 256>) : rows <= 8 ? go(general_step_kernel<A, 4, 8, 256>) : go(general_step_kernel<A, 4, 0, 256>);
    return rows <= 16 ? go(general_step_kernel<A, 1, 16, 256>) : go(general_step_kernel<A, 1, 0, 256>);
}

}  // namespace

bool general_chunks_apply(const GeneralShape& g, double decay_scale, bool f32) { return !f32 && g.dim <= 128 && decay_scale * kT / 2 <= 30.0; }
size_t general_chunk_bytes(const GeneralShape& g) { return ItemLayout{padded_dim(g.dim)}.size() * g.heads * kHalves * sizeof(float); }

int32_t launch_general_scan(const GeneralArgs& a, cudaStream_t s) {
    const int dim = a.g.dim, dpl = dim <= 32 ? 8 : dim <= 64 ? 16 : dim <= 128 ? 32 : 64;
    LC_CHECK(dim <= 256, LC_ERR_UNSUPPORTED, "delta rule: %d dimensions per head (at most 256)", dim);
    const size_t smem = (size_t)kScanTok * (4 * 4 * dpl + 32 + 1) * sizeof(float);
    const dim3 grid((unsigned)a.n_runs, (unsigned)a.g.heads, (unsigned)((dim + 31) / 32));
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3(128), smem, s, a));
        return LC_OK;
    };
    switch (dpl) {
        case 8: return go(general_scan_kernel<8>);
        case 16: return go(general_scan_kernel<16>);
        case 32: return go(general_scan_kernel<32>);
        default: return go(general_scan_kernel<64>);
    }
}

int32_t launch_general_chunks(const GeneralArgs& a, float* scratch, cudaStream_t s) {
    auto go = [&](auto chunk, auto carry, int dp) -> int32_t {
        const dim3 g1((unsigned)(a.n_chunks * kHalves), (unsigned)a.g.heads), g2((unsigned)a.n_chunk_runs, (unsigned)a.g.heads, (unsigned)(dp / 32));
        LC_CUDA(ensure_smem_limit((const void*)chunk, chunk_smem(dp)));
        LC_CUDA(ensure_smem_limit((const void*)carry, carry_smem(dp)));
        LC_CUDA(launch_pdl(chunk, g1, dim3(kThreads), chunk_smem(dp), s, a, scratch));
        LC_CUDA(launch_pdl(carry, g2, dim3((unsigned)(2 * dp + 64)), carry_smem(dp), s, a, (const float*)scratch, gemv_error_flag_dev()));
        return LC_OK;
    };
    switch (padded_dim(a.g.dim)) {
        case 32: return go(general_chunk_kernel<32>, general_carry_kernel<32>, 32);
        case 64: return go(general_chunk_kernel<64>, general_carry_kernel<64>, 64);
        default: return go(general_chunk_kernel<128>, general_carry_kernel<128>, 128);
    }
}

int32_t launch_general_step(const GeneralArgs& a, cudaStream_t s) { return a.f32 ? step_dispatch<float>(a, s) : step_dispatch<__nv_bfloat16>(a, s); }

}  // namespace lc
