// The gated delta rule over long runs, 64 tokens at a time, in f32 throughout (mixers.cu walks short runs token by token).
//
// Inside a chunk let G_t be the sum of the log decays up to token t (per key channel, G <= 0) and S0 the state before the
// chunk.  Unrolling the recurrence gives, with products over key channels d,
//   A_ts = sum_d k_t k_s e^(G_t - G_s)  (s < t),     B_ts = sum_d q_t k_s e^(G_t - G_s)  (s <= t),
//   u_t = beta_t (v_t - S0^T (e^(G_t) k_t) - sum_(s < t) A_ts u_s),
//   o_t = S0^T (e^(G_t) q_t) + sum_(s <= t) B_ts u_s,      S = e^(G_end) S0 + sum_s (e^(G_end - G_s) k_s) u_s^T.
// The triangular system does not involve S0 when it is solved for its two right-hand sides, so
//   delta_chunk_kernel  (all chunks of all heads at once) leaves W = (I + beta A)^-1 beta (e^G k) and Ub = (I + beta A)^-1 beta v
//                       beside e^G q, e^(G_end - G) k, B and e^(G_end);
//   delta_carry_kernel  (one CTA per run, head and 32 value columns) walks the chunks: U = Ub - W S0, O = (e^G q) S0 + B U,
//                       S = e^(G_end) S0 + (e^(G_end - G) k)^T U.
// No exponent is ever positive: a 4 x 4 tile of A and B below the diagonal factors its decay at the last token before the
// tile's rows, e^(G_t - G_r) e^(G_r - G_s) with s <= r < t, and the tiles on the diagonal take each pair's difference.
#include <algorithm>
#include <cmath>
#include "lc_mixers.h"
#include "lc_tma.cuh"

namespace lc {

namespace {

constexpr int kC = kDeltaChunk;
constexpr int kP = kC + 4;           // pitch of the channel-major arrays
constexpr int kCols = 32;            // value columns of a carrying CTA
constexpr float kLog2e = 1.4426950408889634f;

// Scratch of one (chunk, head), in floats.
struct ChunkLayout {
    int dp, e;
    __host__ __device__ size_t wq() const { return 0; }                                // [dp][128]: W of the 64 tokens, then e^G q
    __host__ __device__ size_t kh() const { return (size_t)dp * 128; }                 // [64][dp]
    __host__ __device__ size_t bt() const { return kh() + (size_t)kC * dp; }           // [64 s][64 t]
    __host__ __device__ size_t ub() const { return bt() + (size_t)kC * kC; }           // [64][e]
    __host__ __device__ size_t ge() const { return ub() + (size_t)kC * e; }            // [dp]
    __host__ __device__ size_t size() const { return ge() + (size_t)dp; }
};
__host__ __device__ inline int padded_cols(int vdim) { return (vdim + kCols - 1) / kCols * kCols; }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

constexpr int kChunkThreads = 288;  // 136 lower tiles of 4 x 4 pairs, each in two halves of the channels: 272
template <int DP>
__global__ void __launch_bounds__(kChunkThreads, 2) delta_chunk_kernel(const DeltaArgs a, float* __restrict__ scratch) {
    extern __shared__ __align__(16) float sm[];
    float *s_k = sm, *s_q = s_k + DP * kP, *s_G = s_q + DP * kP, *s_b = s_G + DP * kP;
    float* s_A = DP * kP >= kC * kC ? s_q : s_b + kC;  // takes the place of q once q has been used
    pdl_launch_dependents();
    pdl_wait();
    const DeltaShape& g = a.g;
    const DeltaChunk ck = a.chunks[blockIdx.x];
    const int h = blockIdx.y, kh = h / (g.heads / g.kv_heads), tid = threadIdx.x;
    const ChunkLayout L{DP, padded_cols(g.vdim)};
    float* out = scratch + ((size_t)blockIdx.x * g.heads + h) * L.size();
    // channel-major copies; rows past the chunk's tokens and channels past dim are zero (no key, no decay)
    const int nk = g.kv_heads * g.dim;
    if (g.dim % 4 == 0) {
        for (int i = tid; i < kC * DP / 4; i += kChunkThreads) {
            const int t = i & (kC - 1), d = i / kC * 4;
            float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q, l = q;
            if (t < ck.n && d < g.dim) {
                const size_t tok = (size_t)(ck.tok0 + t);
                q = *(const float4*)(a.qk + tok * 2 * nk + kh * g.dim + d);
                k = *(const float4*)(a.qk + (tok * 2 + 1) * nk + kh * g.dim + d);
                l = *(const float4*)(a.log_decay + tok * g.heads * g.dim + h * g.dim + d);
            }
            const float qq[4] = {q.x, q.y, q.z, q.w}, kk[4] = {k.x, k.y, k.z, k.w}, ll[4] = {l.x, l.y, l.z, l.w};
#pragma unroll
            for (int j = 0; j < 4; j++) { s_q[(d + j) * kP + t] = qq[j]; s_k[(d + j) * kP + t] = kk[j]; s_G[(d + j) * kP + t] = ll[j] * kLog2e; }
        }
    } else {
        for (int i = tid; i < kC * DP; i += kChunkThreads) {
            const int t = i & (kC - 1), d = i / kC;
            float q = 0.0f, k = 0.0f, l = 0.0f;
            if (t < ck.n && d < g.dim) {
                const size_t tok = (size_t)(ck.tok0 + t);
                q = a.qk[tok * 2 * nk + kh * g.dim + d];
                k = a.qk[(tok * 2 + 1) * nk + kh * g.dim + d];
                l = a.log_decay[tok * g.heads * g.dim + h * g.dim + d] * kLog2e;
            }
            s_q[d * kP + t] = q; s_k[d * kP + t] = k; s_G[d * kP + t] = l;
        }
    }
    for (int i = tid; i < kC; i += kChunkThreads)
        s_b[i] = i < ck.n ? sigmoid_f(__bfloat162float(((const __nv_bfloat16*)a.proj)[(size_t)(ck.tok0 + i) * g.ld + g.off_b + h])) : 0.0f;
    __syncthreads();
    for (int d = tid; d < DP; d += kChunkThreads) {
        float sum = 0.0f;
        for (int t = 0; t < kC; t += 4) {
            float4 v = *(float4*)(s_G + d * kP + t);
            v.x = sum += v.x; v.y = sum += v.y; v.z = sum += v.z; v.w = sum += v.w;
            *(float4*)(s_G + d * kP + t) = v;
        }
    }
    __syncthreads();
    // A and B, one tile per thread and half of the channels
    float ta[4][4] = {}, tb[4][4] = {};
    int ti = 0, tj = 0;
    const bool tile = tid < 272;
    if (tile) {
        int rest = tid >> 1;
        while (rest > ti) { rest -= ti + 1; ti++; }
        tj = rest;
        const int d0 = (tid & 1) * (DP / 2), d1 = d0 + DP / 2;
        if (ti != tj) {
            for (int d = d0; d < d1; d++) {
                const float4 kt = *(const float4*)(s_k + d * kP + 4 * ti), qt = *(const float4*)(s_q + d * kP + 4 * ti), gt = *(const float4*)(s_G + d * kP + 4 * ti);
                const float4 ks = *(const float4*)(s_k + d * kP + 4 * tj), gs = *(const float4*)(s_G + d * kP + 4 * tj);
                const float r = s_G[d * kP + 4 * ti - 1];
                const float ft[4] = {exp2f(gt.x - r), exp2f(gt.y - r), exp2f(gt.z - r), exp2f(gt.w - r)};
                const float x[4] = {ks.x * exp2f(r - gs.x), ks.y * exp2f(r - gs.y), ks.z * exp2f(r - gs.z), ks.w * exp2f(r - gs.w)};
                const float y[4] = {kt.x * ft[0], kt.y * ft[1], kt.z * ft[2], kt.w * ft[3]}, z[4] = {qt.x * ft[0], qt.y * ft[1], qt.z * ft[2], qt.w * ft[3]};
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) { ta[i][j] = fmaf(y[i], x[j], ta[i][j]); tb[i][j] = fmaf(z[i], x[j], tb[i][j]); }
            }
        } else {
            for (int d = d0; d < d1; d++)
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const float kt = s_k[d * kP + 4 * ti + i], qt = s_q[d * kP + 4 * ti + i], gt = s_G[d * kP + 4 * ti + i];
#pragma unroll
                    for (int j = 0; j <= i; j++) {
                        const float x = s_k[d * kP + 4 * ti + j] * exp2f(gt - s_G[d * kP + 4 * ti + j]);
                        if (j < i) ta[i][j] = fmaf(kt, x, ta[i][j]);
                        tb[i][j] = fmaf(qt, x, tb[i][j]);
                    }
                }
        }
        // the two halves sit in neighbouring lanes; the last warp has 16 lanes with tiles
        const unsigned m = tid < 256 ? 0xffffffffu : 0xffffu;
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) {
                ta[i][j] += __shfl_xor_sync(m, ta[i][j], 1);
                tb[i][j] += __shfl_xor_sync(m, tb[i][j], 1);
            }
        // B goes out as [s][t] with zeros above the diagonal: one half writes the tile, the other the tile across the diagonal
        float* bt = out + L.bt();
#pragma unroll
        for (int j = 0; j < 4; j++) {
            if ((tid & 1) == 0) *(float4*)(bt + (4 * tj + j) * kC + 4 * ti) = make_float4(tb[0][j], tb[1][j], tb[2][j], tb[3][j]);
            else if (ti != tj) *(float4*)(bt + (4 * ti + j) * kC + 4 * tj) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    for (int i = tid; i < kC * DP; i += kChunkThreads) {
        const int d = i % DP, t = i / DP;
        out[L.kh() + i] = s_k[d * kP + t] * exp2f(s_G[d * kP + kC - 1] - s_G[d * kP + t]);
    }
    for (int i = tid; i < DP * kC / 4; i += kChunkThreads) {
        const int t = (i & (kC / 4 - 1)) * 4, d = i / (kC / 4);
        const float4 q = *(const float4*)(s_q + d * kP + t), e = *(const float4*)(s_G + d * kP + t);
        *(float4*)(out + L.wq() + (size_t)d * 128 + 64 + t) = make_float4(q.x * exp2f(e.x), q.y * exp2f(e.y), q.z * exp2f(e.z), q.w * exp2f(e.w));
    }
    for (int d = tid; d < DP; d += kChunkThreads) out[L.ge() + d] = exp2f(s_G[d * kP + kC - 1]);
    __syncthreads();  // q has been used
    if (tile && (tid & 1) == 0)
#pragma unroll
        for (int i = 0; i < 4; i++) *(float4*)(s_A + (4 * ti + i) * kC + 4 * tj) = make_float4(ta[i][0], ta[i][1], ta[i][2], ta[i][3]);
    __syncthreads();
    // forward substitution, one column of the right-hand sides per thread; entries of A on and above the diagonal are not used
    for (int c = tid; c < DP + L.e; c += kChunkThreads) {
        float x[kC];
        const bool is_w = c < DP;
        const int col = is_w ? c : c - DP;
        if (is_w) {
#pragma unroll
            for (int t = 0; t < kC; t += 4) {
                const float4 k = *(const float4*)(s_k + col * kP + t), e = *(const float4*)(s_G + col * kP + t);
                x[t] = k.x * exp2f(e.x); x[t + 1] = k.y * exp2f(e.y); x[t + 2] = k.z * exp2f(e.z); x[t + 3] = k.w * exp2f(e.w);
            }
        } else {
            const float* v = a.v + (size_t)ck.tok0 * g.heads * g.vdim + h * g.vdim + col;
#pragma unroll
            for (int t = 0; t < kC; t++) x[t] = t < ck.n && col < g.vdim ? v[(size_t)t * g.heads * g.vdim] : 0.0f;
        }
#pragma unroll
        for (int t = 0; t < kC; t++) {
            float p[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int s = 0; s < t; s += 4) {
                const float4 row = *(const float4*)(s_A + t * kC + s);
                p[0] = fmaf(row.x, x[s], p[0]);
                if (s + 1 < t) p[1] = fmaf(row.y, x[s + 1], p[1]);
                if (s + 2 < t) p[2] = fmaf(row.z, x[s + 2], p[2]);
                if (s + 3 < t) p[3] = fmaf(row.w, x[s + 3], p[3]);
            }
            x[t] = s_b[t] * (x[t] - ((p[0] + p[1]) + (p[2] + p[3])));
        }
        if (is_w) {
#pragma unroll
            for (int t = 0; t < kC; t += 4) *(float4*)(out + L.wq() + (size_t)col * 128 + t) = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
        } else {
#pragma unroll
            for (int t = 0; t < kC; t++) out[L.ub() + (size_t)t * L.e + col] = x[t];
        }
    }
}

__device__ __forceinline__ void copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void fma4x4(float (&c)[4][4], const float4& x, const float4& y) {
    const float p[4] = {x.x, x.y, x.z, x.w}, q[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) c[i][j] = fmaf(p[i], q[j], c[i][j]);
}

constexpr int kCarryThreads = 256;  // a 128 x 32 product in 4 x 4 tiles
template <int DP>
__global__ void __launch_bounds__(kCarryThreads) delta_carry_kernel(const DeltaArgs a, const float* __restrict__ scratch) {
    extern __shared__ __align__(16) float sm[];
    float *s_wq = sm, *s_kh = s_wq + 2 * DP * 128, *s_bt = s_kh + kC * DP, *s_ub = s_bt + kC * kC, *s_u = s_ub + kC * kCols, *s_S = s_u + kC * kCols,
          *s_ge = s_S + DP * kCols;
    pdl_launch_dependents();
    pdl_wait();
    const DeltaShape& g = a.g;
    const DeltaChunkRun cr = a.chunk_runs[blockIdx.x];
    const int h = blockIdx.y, e0 = blockIdx.z * kCols, tid = threadIdx.x, tg = tid >> 3, eg = tid & 7;
    const ChunkLayout L{DP, padded_cols(g.vdim)};
    float* st = a.state + ((size_t)cr.run.seq * g.heads + h) * g.dim * g.vdim;
    auto base = [&](int c) { return scratch + ((size_t)(cr.chunk0 + c) * g.heads + h) * L.size(); };
    auto load_wq = [&](int c) {
        const float* src = base(c) + L.wq();
        float* dst = s_wq + (c & 1) * DP * 128;
        for (int i = tid; i < DP * 32; i += kCarryThreads) copy16(dst + i * 4, src + i * 4);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto load_rest = [&](int c) {
        const float* b = base(c);
        for (int i = tid; i < kC * DP / 4; i += kCarryThreads) copy16(s_kh + i * 4, b + L.kh() + i * 4);
        for (int i = tid; i < kC * kC / 4; i += kCarryThreads) copy16(s_bt + i * 4, b + L.bt() + i * 4);
        for (int i = tid; i < kC * kCols / 4; i += kCarryThreads) copy16(s_ub + i * 4, b + L.ub() + (size_t)(i >> 3) * L.e + e0 + (i & 7) * 4);
        for (int i = tid; i < DP / 4; i += kCarryThreads) copy16(s_ge + i * 4, b + L.ge() + i * 4);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_wq(0);
    load_rest(0);
    // this thread's part of the state: key rows 4 tg .., value columns e0 + 4 eg ..
    const bool owner = 4 * tg < DP;
    float S[4][4];
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int d = 4 * tg + i, e = e0 + 4 * eg + j;
            S[i][j] = cr.run.pos0 > 0 && d < g.dim && e < g.vdim ? st[(size_t)d * g.vdim + e] : 0.0f;
        }
    auto publish = [&]() {
        if (owner)
#pragma unroll
            for (int i = 0; i < 4; i++) *(float4*)(s_S + (4 * tg + i) * kCols + 4 * eg) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
    };
    publish();
    for (int c = 0; c < cr.n_chunks; c++) {
        if (c + 1 < cr.n_chunks) { load_wq(c + 1); asm volatile("cp.async.wait_group 2;" ::: "memory"); }
        else asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const float* wq = s_wq + (c & 1) * DP * 128;
        float acc[4][4] = {};
#pragma unroll 8
        for (int d = 0; d < DP; d++) fma4x4(acc, *(const float4*)(wq + d * 128 + 4 * tg), *(const float4*)(s_S + d * kCols + 4 * eg));
        if (c + 1 < cr.n_chunks) asm volatile("cp.async.wait_group 1;" ::: "memory");
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (tg < 16) {
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const float4 b = *(const float4*)(s_ub + (4 * tg + i) * kCols + 4 * eg);
                *(float4*)(s_u + (4 * tg + i) * kCols + 4 * eg) = make_float4(b.x - acc[i][0], b.y - acc[i][1], b.z - acc[i][2], b.w - acc[i][3]);
            }
        }
        __syncthreads();
        if (owner) {
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const float ge = s_ge[4 * tg + i];
#pragma unroll
                for (int j = 0; j < 4; j++) S[i][j] *= ge;
            }
#pragma unroll 8
            for (int s = 0; s < kC; s++) fma4x4(S, *(const float4*)(s_kh + s * DP + 4 * tg), *(const float4*)(s_u + s * kCols + 4 * eg));
        }
        if (tg >= 16) {  // the tokens' read-outs: rows 4 (tg - 16) ..
            const int t0 = 4 * (tg - 16);
#pragma unroll 4
            for (int s = 0; s < t0 + 4; s++) fma4x4(acc, *(const float4*)(s_bt + s * kC + t0), *(const float4*)(s_u + s * kCols + 4 * eg));
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const int t = c * kC + t0 + i;
                if (t >= cr.run.n) continue;
                float* o = a.o + (size_t)(cr.run.tok0 + t) * g.heads * g.vdim + h * g.vdim + e0 + 4 * eg;
#pragma unroll
                for (int j = 0; j < 4; j++)
                    if (e0 + 4 * eg + j < g.vdim) o[j] = acc[i][j];
            }
        }
        __syncthreads();
        publish();
        if (c + 1 < cr.n_chunks) load_rest(c + 1);
    }
    if (owner)
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int d = 4 * tg + i, e = e0 + 4 * eg + j;
                if (d < g.dim && e < g.vdim) st[(size_t)d * g.vdim + e] = S[i][j];
            }
    if (blockIdx.z == 0) delta_keep_inputs<__nv_bfloat16>(a, cr.run, h, tid, kCarryThreads);
}

int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : 128; }
size_t chunk_smem(int dp) { return ((size_t)3 * dp * kP + kC + (dp * kP >= kC * kC ? 0 : kC * kC)) * sizeof(float); }
size_t carry_smem(int dp) { return ((size_t)2 * dp * 128 + kC * dp + kC * kC + 2 * kC * kCols + dp * kCols + dp) * sizeof(float); }

}  // namespace

bool delta_chunks_apply(const DeltaShape& g, bool f32) { return !f32 && g.dim <= 128; }
size_t delta_chunk_bytes(const DeltaShape& g) { return ChunkLayout{padded_dim(g.dim), padded_cols(g.vdim)}.size() * g.heads * sizeof(float); }

int32_t launch_delta_chunks(const DeltaArgs& a, float* scratch, cudaStream_t s) {
    const dim3 g1((unsigned)a.n_chunks, (unsigned)a.g.heads), g2((unsigned)a.n_chunk_runs, (unsigned)a.g.heads, (unsigned)(padded_cols(a.g.vdim) / kCols));
    auto go = [&](auto chunk, auto carry, int dp) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)chunk, chunk_smem(dp)));
        LC_CUDA(ensure_smem_limit((const void*)carry, carry_smem(dp)));
        LC_CUDA(launch_pdl(chunk, g1, dim3(kChunkThreads), chunk_smem(dp), s, a, scratch));
        LC_CUDA(launch_pdl(carry, g2, dim3(kCarryThreads), carry_smem(dp), s, a, (const float*)scratch));
        return LC_OK;
    };
    switch (padded_dim(a.g.dim)) {
        case 32: return go(delta_chunk_kernel<32>, delta_carry_kernel<32>, 32);
        case 64: return go(delta_chunk_kernel<64>, delta_carry_kernel<64>, 64);
        default: return go(delta_chunk_kernel<128>, delta_carry_kernel<128>, 128);
    }
}

}  // namespace lc
