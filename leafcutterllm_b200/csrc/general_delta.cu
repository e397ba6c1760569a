// A delta rule whose removal is apart from its writing: per head, over a state S of dim x dim in f32,
//   S_t = D_t S_(t-1) - b_t z_t^T + k_t v_t^T,   z_t = S_(t-1)^T u_t,   o_t = S_t^T r_t,
// with D_t = diag(w_t), u_t the unit key and b_t = a_t u_t (every key channel has its own rate a).
//   general_scan_kernel   runs of few tokens, and models in true 32-bit: token by token
//   general_step_kernel   one token per sequence: recurrence, norm and gate of one head of one token per CTA; the state is read and
//                         written once and stays in registers between
//   general_chunk_kernel, general_carry_kernel, general_read_kernel   longer runs, kGeneralChunk tokens at a time:
// Inside a chunk let G_t be the sum of the log decays up to token t (per key channel) and S0 the state before the chunk.  Unrolled,
//   z_t = (e^G_(t-1) u_t)^T S0 + sum_(s < t) (Auk_ts v_s - Aub_ts z_s),   Axy_ts = sum_d x_t e^(G_(t-1) - G_s) y_s,
//   o_t = (e^G_t r_t)^T S0 + sum_(s <= t) (Brk_ts v_s - Brb_ts z_s),      Brx_ts = sum_d r_t e^(G_t - G_s) x_s.
// Solving the triangular system for its two right-hand sides, Z = W S0 + Y with
//   W = (I + Aub)^-1 (e^G_(t-1) u),   Y = (I + Aub)^-1 Auk V,
// makes the chunk linear in the state before it:
//   S = M S0 + C,  O = R S0 + P,   M = diag(e^G_end) - Bh^T W,  C = Kh^T V - Bh^T Y,  R = e^G r - Brb W,  P = Brk V - Brb Y,
// with Kh, Bh = e^(G_end - G_s) k_s, b_s.  general_chunk_kernel leaves M, R, C and P (all chunks of all heads at once),
// general_carry_kernel walks the chunks' states (one CTA per run, head and 32 value columns), general_read_kernel makes the read-outs
// (all at once again), their norm and gate.
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
    const int h = blockIdx.y, warp = warp_index(), lane = threadIdx.x & 31, r4 = lane & 3, col = warp * 8 + (lane >> 2), e = blockIdx.z * 32 + col, n = g.heads * g.dim;
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
constexpr int kT = kGeneralChunk, kPitch = kT + 4, kHalves = kDeltaChunk / kT;
// What general_chunk_kernel leaves of one (chunk, head), in floats.
struct ItemLayout {
    int dp;
    __host__ __device__ size_t m() const { return 0; }                             // [dp][dp], transposed
    __host__ __device__ size_t c() const { return (size_t)dp * dp; }               // [dp / 32][dp][32]; replaced by S0
    __host__ __device__ size_t r() const { return (size_t)2 * dp * dp; }           // [dp][kT], transposed
    __host__ __device__ size_t p() const { return r() + (size_t)dp * kT; }         // [kT][dp]
    __host__ __device__ size_t size() const { return p() + (size_t)dp * kT; }
};

__device__ __forceinline__ void get4(float (&x)[4], const float* p) {
    const float4 f = *(const float4*)p;
    x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
}
// A warp's lanes over 4 x 4 tiles: LaneGrid<16> 2 rows of tiles by 16 columns, <8> 4 by 8.  Neighbouring lanes share a column and
// every other lane a row, so that 16-byte loads of either operand reach the banks two lanes at a time.
template <int COLS>
struct LaneGrid {
    static constexpr int kRows = 32 / COLS;
    __device__ static __forceinline__ int row(int lane) { return (lane & 1) | (COLS == 8 ? (lane >> 4) << 1 : 0); }
    __device__ static __forceinline__ int col(int lane) { return (lane >> 1) & (COLS - 1); }
};
constexpr int cols_per_warp(int dp) { return dp >= 64 ? 16 : 8; }
constexpr int chunk_threads(int dp) { return dp <= 64 ? 192 : 384; }
constexpr int chunk_ctas(int dp) { return dp <= 64 ? 3 : 1; }

template <int DP>
__global__ void __launch_bounds__(chunk_threads(DP), chunk_ctas(DP)) general_chunk_kernel(const GeneralArgs a, float* __restrict__ scratch) {
    constexpr int kThreads = chunk_threads(DP), kWarps = kThreads / 32, kQuads = (DP / 4 + kWarps - 1) / kWarps;  // fours of channels per warp
    typedef LaneGrid<cols_per_warp(DP)> Lanes;
    constexpr int kColBlocks = DP / 4 / cols_per_warp(DP);
    extern __shared__ __align__(16) float sm[];
    // channel-major [DP][kPitch]: u e^(G_(t-1) - G_m), r e^(G_t - G_m), k e^(G_m - G_t), b e^(G_m - G_t); the first two are read side by side
    float *s_u = sm, *s_r = s_u + DP * kPitch + 16, *s_k = s_r + DP * kPitch, *s_b = s_k + DP * kPitch;
    float *s_v = s_b + DP * kPitch, *s_y = s_v + kT * DP, *s_w = s_u;                 // [kT][DP] v, Y, W (in place of u)
    float *s_auk = s_y + kT * DP, *s_aub = s_auk + kT * kPitch, *s_brk = s_aub + kT * kPitch, *s_brb = s_brk + kT * kPitch;
    float *s_cm = s_brb + kT * kPitch, *s_ce = s_cm + DP, *s_ge = s_ce + DP;          // e^G_m, e^(G_end - G_m), e^G_end
    float* s_len = s_ge + DP;                                                         // [kWarps][32]
    pdl_launch_dependents();
    pdl_wait();
    const GeneralShape& g = a.g;
    const DeltaChunk ck = a.chunks[blockIdx.x / kHalves];
    const int sub = blockIdx.x % kHalves, n = min(kT, ck.n - sub * kT), h = blockIdx.y, tid = threadIdx.x, warp = warp_index(), lane = tid & 31, dim = g.dim;
    if (n <= 0) return;
    const size_t tok0 = (size_t)ck.tok0 + sub * kT;
    const ItemLayout L{DP};
    float* out = scratch + ((size_t)blockIdx.x * g.heads + h) * L.size();
    const bool vec = dim % 4 == 0;
    {
        // the operands' rows as they lie, [kT][kStage] in the places that their channel-major forms take afterwards
        constexpr int kStage = DP + 4;
        const float *p = a.proj + tok0 * g.ld + h * dim, *l = a.log_decay + tok0 * g.heads * dim + h * dim, *ab = a.a_bias + h * dim;
        const size_t ld_l = (size_t)g.heads * dim;
        for (int i = tid; i < kT * DP / 4; i += kThreads) {
            const int t = i / (DP / 4), d = (i - t * (DP / 4)) * 4, at = t * kStage + d;
            const float *row = p + (size_t)t * g.ld + d, *lrow = l + t * ld_l + d;
            if (vec) {
                const int bytes = t < n && d < dim ? 16 : 0;  // 0: zeros
                const size_t o = bytes ? 0 : (size_t)t * g.ld + d, ol = bytes ? 0 : t * ld_l + d;
                cp16(smem_u32(s_k + at), row - o + g.off_k, bytes);
                cp16(smem_u32(s_u + at), lrow - ol, bytes);
                cp16(smem_u32(s_r + at), row - o, bytes);
                cp16(smem_u32(s_b + at), row - o + g.off_a, bytes);
                cp16(smem_u32(s_v + t * DP + d), row - o + g.off_v, bytes);
            } else {
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const bool ok = t < n && d + j < dim;
                    s_k[at + j] = ok ? row[g.off_k + j] : 0.0f;
                    s_u[at + j] = ok ? lrow[j] : 0.0f;
                    s_r[at + j] = ok ? row[j] : 0.0f;
                    s_b[at + j] = ok ? row[g.off_a + j] : 0.0f;
                    s_v[t * DP + d + j] = ok ? row[g.off_v + j] : 0.0f;
                }
            }
        }
        cp_commit();
        float k[kQuads][4], G[kQuads][4], r[kQuads][4], ra[kQuads][4], ss = 0.0f;  // a lane per token, fours of channels per warp
#pragma unroll
        for (int i = 0; i < kQuads; i++) {
            const int d0 = 4 * (warp + i * kWarps);
#pragma unroll
            for (int j = 0; j < 4; j++) ra[i][j] = d0 + j < dim ? __ldg(ab + d0 + j) : 0.0f;
        }
        cp_wait<0>();
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kQuads; i++) {
            const int d0 = 4 * (warp + i * kWarps), at = lane * kStage + d0;
            if (d0 >= DP) break;
            float z[4];
            get4(k[i], s_k + at); get4(G[i], s_u + at); get4(r[i], s_r + at); get4(z, s_b + at);
#pragma unroll
            for (int j = 0; j < 4; j++) { ss = fmaf(k[i][j], k[i][j], ss); ra[i][j] += z[j]; }
        }
        s_len[warp * 32 + lane] = ss;
        __syncthreads();
        ss = g.unit_eps;
#pragma unroll
        for (int w = 0; w < kWarps; w++) ss += s_len[w * 32 + lane];
        const float rk = 1.0f / sqrtf(ss);
#pragma unroll
        for (int i = 0; i < kQuads; i++) {
            const int d0 = 4 * (warp + i * kWarps);
            if (d0 >= DP) break;
#pragma unroll
            for (int j = 0; j < 4; j++) G[i][j] *= kLog2e;
#pragma unroll
            for (int o = 1; o < 32; o *= 2)
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const float y = __shfl_up_sync(0xffffffffu, G[i][j], o);
                    if (lane >= o) G[i][j] += y;
                }
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const float up = __shfl_up_sync(0xffffffffu, G[i][j], 1), gp = lane > 0 ? up : 0.0f, gm = __shfl_sync(0xffffffffu, G[i][j], kT / 2 - 1),
                            ge = __shfl_sync(0xffffffffu, G[i][j], 31);
                const float u = k[i][j] * rk, back = exp2f(gm - G[i][j]);
                const int d = d0 + j, at = d * kPitch + lane;
                s_u[at] = u * exp2f(gp - gm);
                s_r[at] = r[i][j] * exp2f(G[i][j] - gm);
                s_k[at] = k[i][j] * back;
                s_b[at] = __fdividef(u, 1.0f + __expf(-ra[i][j])) * back;
                if (lane == 0) { s_cm[d] = exp2f(gm); s_ce[d] = exp2f(ge - gm); s_ge[d] = exp2f(ge); }
            }
        }
    }
    __syncthreads();
    // the four triangles, a 4 x 4 tile of two of them per thread and share of the channels
    constexpr int kShares = kWarps >= 9 ? 4 : 2, kTiles = 16 / kShares;  // tiles per warp
    if (warp * kTiles < 36) {
        const int pair = lane & 1, share = lane / (2 * kTiles), tile = min(warp * kTiles + (lane >> 1) % kTiles, 35);
        int ti = 0, tj = tile;
        while (tj > ti) { tj -= ti + 1; ti++; }
        const int d0 = 4 * (share & 1) + DP / 2 * (share >> 1);  // shares of neighbouring channel fours: other banks
        const float *x = (pair ? s_r : s_u) + 4 * ti + d0 * kPitch, *yk = s_k + 4 * tj + d0 * kPitch, *yb = s_b + 4 * tj + d0 * kPitch;
        float ak[4][4] = {}, ab[4][4] = {};
#pragma unroll 4
        for (int i = 0; i < DP / kShares; i++) {
            const int d = (i & 3) + (i >> 2) * 8;
            float xt[4], ks[4], bs[4];
            get4(xt, x + d * kPitch); get4(ks, yk + d * kPitch); get4(bs, yb + d * kPitch);
#pragma unroll
            for (int p = 0; p < 4; p++)
#pragma unroll
                for (int q = 0; q < 4; q++) { ak[p][q] = fmaf(xt[p], ks[q], ak[p][q]); ab[p][q] = fmaf(xt[p], bs[q], ab[p][q]); }
        }
        float *mk = pair ? s_brk : s_auk, *mb = pair ? s_brb : s_aub;
#pragma unroll
        for (int p = 0; p < 4; p++) {
#pragma unroll
            for (int q = 0; q < 4; q++) {
#pragma unroll
                for (int o = 2 * kTiles; o < 32; o *= 2) {
                    ak[p][q] += __shfl_xor_sync(0xffffffffu, ak[p][q], o);
                    ab[p][q] += __shfl_xor_sync(0xffffffffu, ab[p][q], o);
                }
                const int t = 4 * ti + p, s = 4 * tj + q;
                if (s > t || (s == t && !pair)) ak[p][q] = ab[p][q] = 0.0f;
            }
            if ((p & (kShares - 1)) == share) {
                *(float4*)(mk + (4 * ti + p) * kPitch + 4 * tj) = make_float4(ak[p][0], ak[p][1], ak[p][2], ak[p][3]);
                *(float4*)(mb + (4 * ti + p) * kPitch + 4 * tj) = make_float4(ab[p][0], ab[p][1], ab[p][2], ab[p][3]);
            }
        }
    }
    __syncthreads();
    // Auk V, tiles of 4 x 4
    for (int u = warp; u < kT / 4 / Lanes::kRows * kColBlocks; u += kWarps) {
        const int t0 = 4 * (u / kColBlocks * Lanes::kRows + Lanes::row(lane)), e0 = 4 * (u % kColBlocks * cols_per_warp(DP) + Lanes::col(lane));
        float y[4][4] = {};
        for (int s = 0; s <= t0; s += 4) {
            float m[4][4];
#pragma unroll
            for (int i = 0; i < 4; i++) get4(m[i], s_auk + (t0 + i) * kPitch + s);
#pragma unroll
            for (int j = 0; j < 4; j++) {
                float v[4];
                get4(v, s_v + (s + j) * DP + e0);
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int q = 0; q < 4; q++) y[i][q] = fmaf(m[i][j], v[q], y[i][q]);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; i++) *(float4*)(s_y + (t0 + i) * DP + e0) = make_float4(y[i][0], y[i][1], y[i][2], y[i][3]);
    }
    __syncthreads();
    // forward substitution, one column of W or Y per thread
    {
        float x[kT];
        if (tid < DP) {
            const float cm = s_cm[tid];
#pragma unroll
            for (int t = 0; t < kT; t += 4) {
                float q[4];
                get4(q, s_u + tid * kPitch + t);
#pragma unroll
                for (int j = 0; j < 4; j++) x[t + j] = q[j] * cm;
            }
        } else if (tid < 2 * DP) {
#pragma unroll
            for (int t = 0; t < kT; t++) x[t] = s_y[t * DP + tid - DP];
        }
        __syncthreads();  // W takes the place of u
        if (tid < 2 * DP) {
            float* dst = tid < DP ? s_w + tid : s_y + tid - DP;
            dst[0] = x[0];
#pragma unroll
            for (int t = 1; t < kT; t++) {
                float p[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
                for (int s = 0; s < t; s += 4) {
                    float m[4];
                    get4(m, s_aub + t * kPitch + s);
#pragma unroll
                    for (int j = 0; j < 4; j++)
                        if (s + j < t) p[j] = fmaf(m[j], x[s + j], p[j]);
                }
                x[t] -= (p[0] + p[1]) + (p[2] + p[3]);
                dst[t * DP] = x[t];
            }
        }
    }
    __syncthreads();
    // M and C (state rows), R and P (token rows): eight rows by four columns per thread
    constexpr int kUnitRows = 8 * Lanes::kRows;
    for (int u = warp; u < (DP + kT) / kUnitRows * kColBlocks; u += kWarps) {
        const int base = u / kColBlocks * kUnitRows, e0 = 4 * (u % kColBlocks * cols_per_warp(DP) + Lanes::col(lane));
        const bool token = base >= DP;
        const int row0 = (token ? base - DP : base) + 4 * Lanes::row(lane), step = 4 * Lanes::kRows;  // rows row0 .. + 3 and row0 + step .. + 3
        const float *lk = (token ? s_brk : s_k) + row0 * kPitch, *lb = (token ? s_brb : s_b) + row0 * kPitch;
        const int end = token ? row0 + step + 4 : kT;
        float m[8][4] = {}, c[8][4] = {};
#pragma unroll 1
        for (int s = 0; s < end; s += 2) {
            float2 xb[8], xk[8];
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const int at = ((i >> 2) * step + (i & 3)) * kPitch + s;
                // a token's upper rows end before the lower ones; what lies behind their end was not written
                const bool live = !token || i >= 4 || s < row0 + 4;
                xb[i] = live ? *(const float2*)(lb + at) : make_float2(0.0f, 0.0f);
                xk[i] = live ? *(const float2*)(lk + at) : make_float2(0.0f, 0.0f);
            }
#pragma unroll
            for (int j = 0; j < 2; j++) {
                float w[4], y[4], v[4];
                get4(w, s_w + (s + j) * DP + e0); get4(y, s_y + (s + j) * DP + e0); get4(v, s_v + (s + j) * DP + e0);
#pragma unroll
                for (int i = 0; i < 8; i++) {
                    const float b = j ? -xb[i].y : -xb[i].x, k = j ? xk[i].y : xk[i].x;
#pragma unroll
                    for (int q = 0; q < 4; q++) {
                        m[i][q] = fmaf(b, w[q], m[i][q]);
                        c[i][q] = fmaf(k, v[q], c[i][q]);
                        c[i][q] = fmaf(b, y[q], c[i][q]);
                    }
                }
            }
        }
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int row = row0 + half * step, i0 = 4 * half;
            if (token) {
#pragma unroll
                for (int q = 0; q < 4; q++) {
                    float r[4];
                    get4(r, s_r + (e0 + q) * kPitch + row);
                    const float cm = s_cm[e0 + q];
                    *(float4*)(out + L.r() + (size_t)(e0 + q) * kT + row) = make_float4(fmaf(r[0], cm, m[i0][q]), fmaf(r[1], cm, m[i0 + 1][q]), fmaf(r[2], cm, m[i0 + 2][q]), fmaf(r[3], cm, m[i0 + 3][q]));
                }
#pragma unroll
                for (int i = 0; i < 4; i++) *(float4*)(out + L.p() + (size_t)(row + i) * DP + e0) = make_float4(c[i0 + i][0], c[i0 + i][1], c[i0 + i][2], c[i0 + i][3]);
            } else {
                float ce[4];
                get4(ce, s_ce + row);
#pragma unroll
                for (int q = 0; q < 4; q++) {
                    float x[4];
#pragma unroll
                    for (int i = 0; i < 4; i++) x[i] = fmaf(m[i0 + i][q], ce[i], e0 + q == row + i ? s_ge[row + i] : 0.0f);
                    *(float4*)(out + L.m() + (size_t)(e0 + q) * DP + row) = make_float4(x[0], x[1], x[2], x[3]);
                }
                float* co = out + L.c() + (size_t)(e0 / 32) * DP * 32 + e0 % 32;
#pragma unroll
                for (int i = 0; i < 4; i++) *(float4*)(co + (size_t)(row + i) * 32) = make_float4(c[i0 + i][0] * ce[i], c[i0 + i][1] * ce[i], c[i0 + i][2] * ce[i], c[i0 + i][3] * ce[i]);
            }
        }
    }
}

// S = M S0 + C, one product of dp x dp by dp x 32 per chunk in 4 x 4 tiles, by two groups of warps that share its sum; the operands of
// the next chunk travel meanwhile.  The state before every chunk takes the place of its C.
template <int DP>
__global__ void __launch_bounds__(4 * DP) general_carry_kernel(const GeneralArgs a, float* __restrict__ scratch, int* error_flag) {
    constexpr int kM = DP * DP, kC = DP * 32;
    typedef LaneGrid<8> Lanes;
    extern __shared__ __align__(128) float sm[];
    __shared__ uint64_t full[2];
    float *s_m = sm, *s_c = s_m + 2 * kM, *s_S = s_c + 2 * kC, *s_part = s_S + kC;
    const int tid = threadIdx.x, lane = tid & 31, group = warp_index() / (DP / 16), warp = warp_index() - group * (DP / 16), d0 = 16 * warp + 4 * Lanes::row(lane), e = 4 * Lanes::col(lane);
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
    const int h = blockIdx.y, e0 = blockIdx.z * 32 + e, chunks = (cr.run.n + kT - 1) / kT;
    const ItemLayout L{DP};
    float* st = a.state + ((size_t)cr.run.seq * g.heads + h) * g.dim * g.dim;
    auto item = [&](int c) { return scratch + ((size_t)(cr.chunk0 * kHalves + c) * g.heads + h) * L.size(); };
    auto request = [&](int c) {  // one thread
        const float* src = item(c);
        mbar_expect_tx(&full[c & 1], (uint32_t)(kM + kC) * 4);
        bulk_load(s_m + (c & 1) * kM, src + L.m(), (uint32_t)kM * 4, &full[c & 1]);
        bulk_load(s_c + (c & 1) * kC, src + L.c() + (size_t)blockIdx.z * kC, (uint32_t)kC * 4, &full[c & 1]);
    };
    if (tid == 0) {
        request(0);
        if (chunks > 1) request(1);
    }
    float S[4][4] = {};  // of group 0: rows d0 .., columns e0 ..
    auto publish = [&]() {
#pragma unroll
        for (int i = 0; i < 4; i++) *(float4*)(s_S + (d0 + i) * 32 + e) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
    };
    if (group == 0) {
        if (cr.run.pos0 > 0)
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++)
                    if (d0 + i < g.dim && e0 + j < g.dim) S[i][j] = st[(size_t)(d0 + i) * g.dim + e0 + j];
        publish();
    }
    __syncthreads();
    for (int c = 0; c < chunks; c++) {
        const float *mp = s_m + (c & 1) * kM + d0 + group * (DP / 2) * DP, *sp = s_S + e + group * (DP / 2) * 32;
        if (!mbar_wait(&full[c & 1], (uint32_t)(c >> 1) & 1) && tid == 0) atomicCAS(error_flag, 0, 18);
        float acc[4][4] = {};
        if (group == 0) {
            float* keep = item(c) + L.c() + (size_t)blockIdx.z * kC + e;
            const float* add = s_c + (c & 1) * kC + e;
#pragma unroll
            for (int i = 0; i < 4; i++) {
                *(float4*)(keep + (d0 + i) * 32) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
                get4(acc[i], add + (d0 + i) * 32);
            }
        }
#pragma unroll 8
        for (int d = 0; d < DP / 2; d++) {
            float x[4], y[4];
            get4(x, mp + d * DP);
            get4(y, sp + d * 32);
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
        }
        if (group == 1)
#pragma unroll
            for (int i = 0; i < 4; i++) *(float4*)(s_part + (d0 + i) * 32 + e) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        __syncthreads();
        if (tid == 2 * DP && c + 2 < chunks) request(c + 2);
        if (group == 0) {
#pragma unroll
            for (int i = 0; i < 4; i++) {
                float p[4];
                get4(p, s_part + (d0 + i) * 32 + e);
#pragma unroll
                for (int j = 0; j < 4; j++) S[i][j] = acc[i][j] + p[j];
            }
            publish();
        }
        __syncthreads();
    }
    if (group == 0)
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++)
                if (d0 + i < g.dim && e0 + j < g.dim) st[(size_t)(d0 + i) * g.dim + e0 + j] = S[i][j];
}

// O = R S0 + P of one (chunk, head), norm and gate.
template <int DP>
__global__ void __launch_bounds__(2 * DP) general_read_kernel(const GeneralArgs a, const float* __restrict__ scratch, int* error_flag) {
    typedef LaneGrid<cols_per_warp(DP)> Lanes;
    constexpr int kColBlocks = DP / 4 / cols_per_warp(DP);
    extern __shared__ __align__(128) float sm[];
    __shared__ uint64_t full;
    __shared__ float s_ss[kColBlocks][kT];
    float *s_S = sm, *s_R = sm + DP * DP;
    const int tid = threadIdx.x, warp = warp_index(), lane = tid & 31, cb = warp % kColBlocks;
    const int t0 = 4 * (warp / kColBlocks * Lanes::kRows + Lanes::row(lane)), e0 = 4 * (cb * cols_per_warp(DP) + Lanes::col(lane));
    if (tid == 0) {
        mbar_init(&full, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    pdl_launch_dependents();
    __syncthreads();
    pdl_wait();
    const GeneralShape& g = a.g;
    const DeltaChunk ck = a.chunks[blockIdx.x / kHalves];
    const int sub = blockIdx.x % kHalves, n = min(kT, ck.n - sub * kT), h = blockIdx.y;
    if (n <= 0) return;
    const size_t tok0 = (size_t)ck.tok0 + sub * kT;
    const ItemLayout L{DP};
    const float* src = scratch + ((size_t)blockIdx.x * g.heads + h) * L.size();
    if (tid == 0) {  // S0 and R lie one behind the other
        mbar_expect_tx(&full, (uint32_t)(DP * DP + DP * kT) * 4);
        bulk_load(s_S, src + L.c(), (uint32_t)(DP * DP + DP * kT) * 4, &full);
    }
    const bool vec = g.dim % 4 == 0;
    float o[4][4], gate[4][4], w[4];
#pragma unroll
    for (int i = 0; i < 4; i++) {
        get4(o[i], src + L.p() + (size_t)(t0 + i) * DP + e0);
        const bf16* gp = (const bf16*)a.gate + (tok0 + min(t0 + i, n - 1)) * a.ld_gate + (size_t)h * g.dim + e0;
        if (vec) {
            const uint2 u = e0 < g.dim ? *(const uint2*)gp : make_uint2(0u, 0u);
            gate[i][0] = __uint_as_float(u.x << 16); gate[i][1] = __uint_as_float(u.x & 0xFFFF0000u);
            gate[i][2] = __uint_as_float(u.y << 16); gate[i][3] = __uint_as_float(u.y & 0xFFFF0000u);
        } else
#pragma unroll
            for (int j = 0; j < 4; j++) gate[i][j] = e0 + j < g.dim ? __bfloat162float(gp[j]) : 0.0f;
    }
#pragma unroll
    for (int j = 0; j < 4; j++) w[j] = e0 + j < g.dim ? a.norm_w[h * g.dim + e0 + j] : 0.0f;
    if (!mbar_wait(&full, 0) && tid == 0) atomicCAS(error_flag, 0, 19);
    const float *rp = s_R + t0, *sp = s_S + (e0 / 32) * DP * 32 + e0 % 32;
#pragma unroll 8
    for (int d = 0; d < DP; d++) {
        float x[4], y[4];
        get4(x, rp + d * kT);
        get4(y, sp + d * 32);
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) o[i][j] = fmaf(x[i], y[j], o[i][j]);
    }
    float ss[4];
#pragma unroll
    for (int i = 0; i < 4; i++) {
        ss[i] = fmaf(o[i][0], o[i][0], fmaf(o[i][1], o[i][1], fmaf(o[i][2], o[i][2], o[i][3] * o[i][3])));
#pragma unroll
        for (int m = 2; m < 2 * cols_per_warp(DP); m *= 2) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], m);
    }
    if constexpr (kColBlocks > 1) {
        if (Lanes::col(lane) == 0)
#pragma unroll
            for (int i = 0; i < 4; i++) s_ss[cb][t0 + i] = ss[i];
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 4; i++) {
            ss[i] = 0.0f;
#pragma unroll
            for (int b = 0; b < kColBlocks; b++) ss[i] += s_ss[b][t0 + i];
        }
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        if (t0 + i >= n) break;
        const float r = 1.0f / sqrtf(ss[i] / (float)g.dim + g.eps);
        float y[4];
#pragma unroll
        for (int j = 0; j < 4; j++) y[j] = __fdividef(o[i][j] * r * w[j], 1.0f + __expf(-gate[i][j]));
        bf16* dst = (bf16*)a.out + (tok0 + t0 + i) * a.ldo + (size_t)h * g.dim + e0;
        if (vec) {
            if (e0 < g.dim) *(uint2*)dst = make_uint2(pack2(y[0], y[1]), pack2(y[2], y[3]));
        } else
#pragma unroll
            for (int j = 0; j < 4; j++)
                if (e0 + j < g.dim) dst[j] = __float2bfloat16_rn(y[j]);
    }
}

int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : 128; }
size_t chunk_smem(int dp) { return ((size_t)4 * dp * kPitch + 16 + 2 * kT * dp + 4 * kT * kPitch + 3 * dp + chunk_threads(dp)) * sizeof(float); }
size_t carry_smem(int dp) { return ((size_t)2 * dp * dp + 4 * dp * 32) * sizeof(float); }
size_t read_smem(int dp) { return ((size_t)dp * dp + dp * kT) * sizeof(float); }

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

template <int DP>
static int32_t run_chunks(const GeneralArgs& a, float* scratch, cudaStream_t s) {
    const dim3 all((unsigned)(a.n_chunks * kHalves), (unsigned)a.g.heads), walk((unsigned)a.n_chunk_runs, (unsigned)a.g.heads, (unsigned)(DP / 32));
    LC_CUDA(ensure_smem_limit((const void*)general_chunk_kernel<DP>, chunk_smem(DP)));
    LC_CUDA(ensure_smem_limit((const void*)general_carry_kernel<DP>, carry_smem(DP)));
    LC_CUDA(ensure_smem_limit((const void*)general_read_kernel<DP>, read_smem(DP)));
    LC_CUDA(launch_pdl(general_chunk_kernel<DP>, all, dim3(chunk_threads(DP)), chunk_smem(DP), s, a, scratch));
    LC_CUDA(launch_pdl(general_carry_kernel<DP>, walk, dim3(4 * DP), carry_smem(DP), s, a, scratch, gemv_error_flag_dev()));
    LC_CUDA(launch_pdl(general_read_kernel<DP>, all, dim3(2 * DP), read_smem(DP), s, a, (const float*)scratch, gemv_error_flag_dev()));
    return LC_OK;
}
int32_t launch_general_chunks(const GeneralArgs& a, float* scratch, cudaStream_t s) {
    switch (padded_dim(a.g.dim)) {
        case 32: return run_chunks<32>(a, scratch, s);
        case 64: return run_chunks<64>(a, scratch, s);
        default: return run_chunks<128>(a, scratch, s);
    }
}

int32_t launch_general_step(const GeneralArgs& a, cudaStream_t s) { return a.f32 ? step_dispatch<float>(a, s) : step_dispatch<__nv_bfloat16>(a, s); }

}  // namespace lc
