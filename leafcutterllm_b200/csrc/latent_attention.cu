// Latent attention: every head's key is the projection of ONE cached latent per token (plus a rotated part all heads share) and
// its value another projection of the same latent.  The key projection is moved onto the query and the value projection behind
// the weighted sum, so for FEW tokens the kernels attend with `heads` queries per token over rows [latent | rotated part] of
// the paged cache and return, per head, the weighted sum of latents.  For MANY tokens of a sequence that costs more than
// projecting the context once: the latents are gathered, keys and values of all heads projected by two ordinary products, and
// the prefill kernel attends over those.
#include <algorithm>
#include <cmath>
#include "lc_mixers.h"
#include "lc_mma.cuh"
#include "lc_tma.cuh"
#include "lc_umma.cuh"

namespace lc {

namespace {

// Any shape, any type, f32 arithmetic throughout: one CTA per (token, head), keys in tiles of one per thread.
constexpr int kPlainThreads = 128;
template <typename A>
__global__ void __launch_bounds__(kPlainThreads) latent_attention_plain_kernel(const LatentArgs a) {
    extern __shared__ float sm[];
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const LatentShape& g = a.g;
    const int h = blockIdx.x, t = blockIdx.y, seq = a.tok_seq[t], pos = a.tok_pos[t], ld = g.cp + g.rp;
    float *s_q = sm, *s_o = s_q + ld, *s_p = s_o + g.cp;
    int* s_row = (int*)(s_p + kPlainThreads);
    const A* qa = (const A*)a.q_abs + ((size_t)t * g.heads + h) * g.cp;
    const A* qr = (const A*)a.q + ((size_t)t * g.heads + h) * g.ld_q + g.dp;
    for (int i = threadIdx.x; i < g.cp; i += kPlainThreads) { s_q[i] = i < g.rank ? act_f<A>(qa[i]) : 0.0f; s_o[i] = 0.0f; }
    for (int i = threadIdx.x; i < g.rp; i += kPlainThreads) {
        float v = i < g.rot ? act_f<A>(qr[i]) : 0.0f;
        if (i < 2 * g.rot_pairs) {
            const float2 cs = a.rot[(size_t)pos * g.rot_pairs + i / 2];
            const float u = act_f<A>(qr[i & ~1]), w = act_f<A>(qr[i | 1]);
            v = (i & 1) ? w * cs.x + u * cs.y : u * cs.x - w * cs.y;
        }
        s_q[g.cp + i] = v;
    }
    __syncthreads();
    const int32_t* pt = a.page_table + (size_t)seq * a.pages_per_seq;
    const A* cache = (const A*)a.cache;
    float m = -INFINITY, l = 0.0f;
    for (int k0 = 0; k0 <= pos; k0 += kPlainThreads) {
        const int key = k0 + threadIdx.x;
        float sc = -INFINITY;
        if (key <= pos) {
            const int row = pt[key / a.page_tokens] * a.page_tokens + key % a.page_tokens;
            s_row[threadIdx.x] = row;
            const A* kr = cache + (size_t)row * ld;
            float d = 0.0f;
            for (int i = 0; i < ld; i++) d = fmaf(s_q[i], act_f<A>(kr[i]), d);
            sc = d * g.scale;
        }
        const float mt = fmaxf(m, block_max(sc, red));
        const float p = key <= pos ? expf(sc - mt) : 0.0f, corr = expf(m - mt);
        s_p[threadIdx.x] = p;
        l = l * corr + block_sum(p, red);
        m = mt;
        const int n = min(kPlainThreads, pos + 1 - k0);
        for (int i = threadIdx.x; i < g.cp; i += kPlainThreads) {
            float o = s_o[i] * corr;
            for (int j = 0; j < n; j++) o = fmaf(s_p[j], act_f<A>(cache[(size_t)s_row[j] * ld + i]), o);
            s_o[i] = o;
        }
        __syncthreads();
    }
    A* out = (A*)a.o + ((size_t)t * g.heads + h) * g.cp;
    for (int i = threadIdx.x; i < g.cp; i += kPlainThreads) out[i] = to_act<A>(s_o[i] / l);
}

// ---- tensor-core forms (bf16) -------------------------------------------------------------------------------------------
// element i of a rotated part whose row starts at r
__device__ __forceinline__ float rotated(const bf16* r, const float2* tab, int pairs, int n, int i) {
    if (i >= n) return 0.0f;
    if (i >= 2 * pairs) return __bfloat162float(r[i]);
    const float2 cs = tab[i / 2];
    const float u = __bfloat162float(r[i & ~1]), w = __bfloat162float(r[i | 1]);
    return (i & 1) ? w * cs.x + u * cs.y : u * cs.x - w * cs.y;
}
constexpr int kKeys = 64;  // keys per tile of the prefill kernel

// Few tokens per sequence: the queries of 16 * MT heads of ONE token are the rows of the products, the cached rows (latent |
// rotated part) the keys and, without the rotated part, the values.  The context is cut into gridDim.z pieces and walked in
// tiles of 32 keys by three kinds of warps:
//   producer (1)   a lane per key: looks up the cached row and requests it with one bulk copy, four tiles in flight; keys past
//                  the token's position repeat its own row (their weight is zero, but the row has to be finite);
//   scores (8)     a warp takes all rows, sixteen keys and a quarter of the rows' elements; the partial scores meet in shared
//                  memory, then a few threads per row do the online softmax and write the weights, high and low halves;
//   sums (8)       a warp takes all rows and 8 * NCT latent columns, one tile behind the scores.
// Waits are bounded; one that runs out raises the library's device error flag (every loop has a fixed count and goes on).
struct LatentPieces { float *o, *ml; };  // [token][piece][heads][cp] sums, [token][piece][heads][2] maximum (log2 units) and weight sum
constexpr int kDecodeKeys = 32, kDecodeTiles = 4, kDecodeThreads = 17 * 32, kPPitch = kDecodeKeys + 8, kPartPitch = kDecodeKeys + 4;
template <int MT, int NCT>
__global__ void __launch_bounds__(kDecodeThreads, 1) latent_decode_kernel(const LatentArgs a, const LatentPieces pc, int* error_flag) {
    constexpr int ROWS = 16 * MT, KQ = 4;
    constexpr int KPT = ROWS * kDecodeKeys / 256, TPR = kDecodeKeys / KPT;  // keys per softmax thread, threads per row
    extern __shared__ __align__(128) unsigned char smem[];
    const LatentShape& g = a.g;
    const int d = g.cp + g.rp, d32 = (d + 31) & ~31, pitch = d32 + 8, row_bytes = pitch * 2;
    bf16 *s_q = (bf16*)smem, *s_k = s_q + ROWS * pitch, *s_p = s_k + kDecodeTiles * kDecodeKeys * pitch;  // s_p: [2 tiles][high, low][ROWS][kPPitch]
    float *s_part = (float*)(s_p + 4 * ROWS * kPPitch), *s_corr = s_part + KQ * ROWS * kPartPitch, *s_l = s_corr + 2 * ROWS;
    uint64_t *full = (uint64_t*)(s_l + ROWS), *empty = full + kDecodeTiles, *p_full = empty + kDecodeTiles, *p_empty = p_full + 2;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
    const int t = blockIdx.x, h0 = blockIdx.y * ROWS, nh = min(ROWS, g.heads - h0);
    if (tid == 0) {
        for (int i = 0; i < kDecodeTiles; i++) { mbar_init(&full[i], 1); mbar_init(&empty[i], 8); }
        for (int i = 0; i < 2; i++) { mbar_init(&p_full[i], 8); mbar_init(&p_empty[i], 8); }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    pdl_launch_dependents();
    pdl_wait();
    const int seq = a.tok_seq[t], pos = a.tok_pos[t], pieces = gridDim.z;
    const int tiles = pos / kDecodeKeys + 1, per = (tiles + pieces - 1) / pieces, kt0 = blockIdx.z * per, n = min(tiles, kt0 + per) - kt0;
    const size_t out_row = ((size_t)t * pieces + blockIdx.z) * g.heads;
    if (n <= 0) {
        for (int i = tid; i < nh; i += kDecodeThreads) { pc.ml[(out_row + h0 + i) * 2] = -INFINITY; pc.ml[(out_row + h0 + i) * 2 + 1] = 0.0f; }
        return;
    }
    auto wait = [&](uint64_t* bar, int phase) { if (!mbar_wait(bar, (uint32_t)phase & 1)) atomicCAS(error_flag, 0, 14); };
    const uint32_t q_sm = smem_u32(s_q), k_sm = smem_u32(s_k), p_sm = smem_u32(s_p);
    // queries: the part carried through the key projection as it is, the other part rotated; zeros behind every row
    for (int i = tid; i < ROWS * (g.cp / 8); i += kDecodeThreads) {
        const int r = i / (g.cp / 8), c = i - r * (g.cp / 8);
        cp16(q_sm + (uint32_t)(r * row_bytes + c * 16), (const bf16*)a.q_abs + ((size_t)t * g.heads + h0 + min(r, nh - 1)) * g.cp + c * 8, r < nh ? 16 : 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    const bf16 zero = __float2bfloat16_rn(0.0f);
    for (int i = tid; i < kDecodeTiles * kDecodeKeys * (pitch - d); i += kDecodeThreads) s_k[(i / (pitch - d)) * pitch + d + i % (pitch - d)] = zero;
    const float2* tab = a.rot + (size_t)pos * g.rot_pairs;
    for (int i = tid; i < ROWS * (pitch - g.cp); i += kDecodeThreads) {
        const int r = i / (pitch - g.cp), c = i - r * (pitch - g.cp);
        s_q[r * pitch + g.cp + c] = r < nh && c < g.rp ? __float2bfloat16_rn(rotated((const bf16*)a.q + ((size_t)t * g.heads + h0 + r) * g.ld_q + g.dp, tab, g.rot_pairs, g.rot, c)) : zero;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();

    if (warp == 16) {
        const int32_t* pt = a.page_table + (size_t)seq * a.pages_per_seq;
        auto row_of = [&](int i) {
            const int kp = min((kt0 + i) * kDecodeKeys + lane, pos);
            return (size_t)pt[kp / a.page_tokens] * a.page_tokens + kp % a.page_tokens;
        };
        size_t row = row_of(0);
        for (int i = 0; i < n; i++) {
            const size_t cur = row;
            row = row_of(i + 1);
            const int b = i % kDecodeTiles;
            if (i >= kDecodeTiles) wait(&empty[b], i / kDecodeTiles - 1);
            if (lane == 0) mbar_expect_tx(&full[b], (uint32_t)(kDecodeKeys * d * 2));
            __syncwarp();
            bulk_load(s_k + (size_t)(b * kDecodeKeys + lane) * pitch, (const bf16*)a.cache + cur * d, (uint32_t)(d * 2), &full[b]);
        }
    } else if (warp < 8) {
        const int kg = warp & 1, kq = warp >> 1, steps = d32 / 16, st0 = steps * kq / KQ, st1 = steps * (kq + 1) / KQ;
        const int srow = tid / TPR, skey = (tid % TPR) * KPT;
        const float sc = g.scale * 1.4426950408889634f;
        float m_run = -INFINITY, l_run = 0.0f;
        const uint32_t qa = q_sm + (uint32_t)((lane & 15) * row_bytes + (lane >> 4) * 16);
        for (int i = 0; i < n; i++) {
            const int b = i % kDecodeTiles;
            wait(&full[b], i / kDecodeTiles);
            float s[MT][2][4];
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int j = 0; j < 2; j++) s[m][j][0] = s[m][j][1] = s[m][j][2] = s[m][j][3] = 0.0f;
            const uint32_t ka = k_sm + (uint32_t)((b * kDecodeKeys + kg * 16 + (lane & 7) + ((lane >> 4) << 3)) * row_bytes + ((lane >> 3) & 1) * 16);
#pragma unroll 3
            for (int st = st0; st < st1; st++) {
                uint32_t kb[4];
                ldsm4(ka + st * 32, kb);
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    uint32_t aq[4];
                    ldsm4(qa + (uint32_t)(16 * m * row_bytes) + st * 32, aq);
                    mma_bf16(s[m][0], aq, kb[0], kb[1]);
                    mma_bf16(s[m][1], aq, kb[2], kb[3]);
                }
            }
            asm volatile("bar.sync 1, 256;" ::: "memory");  // the previous tile's partial scores have been read
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int j = 0; j < 2; j++)
#pragma unroll
                    for (int r = 0; r < 2; r++)
                        *(float2*)(s_part + (kq * ROWS + 16 * m + g8 + 8 * r) * kPartPitch + kg * 16 + 8 * j + 2 * t4) = make_float2(s[m][j][2 * r], s[m][j][2 * r + 1]);
            asm volatile("bar.sync 1, 256;" ::: "memory");
            float v[KPT];
#pragma unroll
            for (int j = 0; j < KPT; j++) v[j] = 0.0f;
#pragma unroll
            for (int q = 0; q < KQ; q++)
#pragma unroll
                for (int j = 0; j < KPT; j += 2) {
                    const float2 x = *(const float2*)(s_part + (q * ROWS + srow) * kPartPitch + skey + j);
                    v[j] += x.x; v[j + 1] += x.y;
                }
            float mx = m_run;
#pragma unroll
            for (int j = 0; j < KPT; j++) {
                v[j] = (kt0 + i) * kDecodeKeys + skey + j <= pos ? v[j] * sc : -INFINITY;
                mx = fmaxf(mx, v[j]);
            }
#pragma unroll
            for (int w = 1; w < TPR; w <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
            const float corr = exp2f(m_run - mx);  // mx is finite: a tile starts at or before the token's position
            m_run = mx;
            float sum = 0.0f;
#pragma unroll
            for (int j = 0; j < KPT; j++) { v[j] = exp2f(v[j] - mx); sum += v[j]; }
#pragma unroll
            for (int w = 1; w < TPR; w <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
            l_run = l_run * corr + sum;
            const int pb = i & 1;
            if (i >= 2) wait(&p_empty[pb], i / 2 - 1);
            if (tid % TPR == 0) s_corr[pb * ROWS + srow] = corr;
            bf16* ph = s_p + (size_t)(2 * pb) * ROWS * kPPitch + srow * kPPitch + skey;
#pragma unroll
            for (int j = 0; j < KPT; j += 2) {
                uint32_t hi, lo;
                split2(v[j], v[j + 1], hi, lo);
                *(uint32_t*)(ph + j) = hi;
                *(uint32_t*)(ph + ROWS * kPPitch + j) = lo;
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full[pb]);
        }
        if (tid % TPR == 0) {
            s_l[srow] = l_run;
            if (pieces > 1 && srow < nh) { pc.ml[(out_row + h0 + srow) * 2] = m_run; pc.ml[(out_row + h0 + srow) * 2 + 1] = l_run; }
        }
        asm volatile("bar.sync 2, 512;" ::: "memory");
    } else {
        const int c0 = (warp - 8) * NCT * 8;
        float o[MT][NCT][4];
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int j = 0; j < NCT; j++) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.0f;
        for (int i = 0; i < n; i++) {
            const int b = i % kDecodeTiles, pb = i & 1;
            wait(&p_full[pb], i / 2);
            wait(&full[b], i / kDecodeTiles);
            if (c0 < g.cp) {
#pragma unroll
                for (int m = 0; m < MT; m++) {
                    const float f0 = s_corr[pb * ROWS + 16 * m + g8], f1 = s_corr[pb * ROWS + 16 * m + g8 + 8];
#pragma unroll
                    for (int j = 0; j < NCT; j++) { o[m][j][0] *= f0; o[m][j][1] *= f0; o[m][j][2] *= f1; o[m][j][3] *= f1; }
                }
                const uint32_t vb = k_sm + (uint32_t)((b * kDecodeKeys + (lane & 15)) * row_bytes + (c0 + (lane >> 4) * 8) * 2);
#pragma unroll
                for (int ks = 0; ks < kDecodeKeys / 16; ks++) {
                    uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
                    for (int m = 0; m < MT; m++) {
                        const uint32_t at = p_sm + (uint32_t)(((2 * pb) * ROWS + 16 * m + (lane & 15)) * kPPitch + 16 * ks + (lane >> 4) * 8) * 2;
                        ldsm4(at, ph[m]);
                        ldsm4(at + ROWS * kPPitch * 2, pl[m]);
                    }
#pragma unroll
                    for (int j = 0; j < NCT; j += 2) {
                        if (c0 + 8 * j >= g.cp) break;
                        uint32_t v[4];
                        ldsm4t(vb + (uint32_t)(16 * ks * row_bytes + 16 * j), v);
#pragma unroll
                        for (int m = 0; m < MT; m++) {
                            mma_bf16(o[m][j], ph[m], v[0], v[1]);
                            mma_bf16(o[m][j + 1], ph[m], v[2], v[3]);
                            mma_bf16(o[m][j], pl[m], v[0], v[1]);
                            mma_bf16(o[m][j + 1], pl[m], v[2], v[3]);
                        }
                    }
                }
            }
            __syncwarp();
            if (lane == 0) { mbar_arrive(&empty[b]); mbar_arrive(&p_empty[pb]); }
        }
        asm volatile("bar.sync 2, 512;" ::: "memory");
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int r = 0; r < 2; r++) {
                const int row = 16 * m + g8 + 8 * r;
                if (row >= nh) continue;
                const float inv = 1.0f / s_l[row];
#pragma unroll
                for (int j = 0; j < NCT; j++) {
                    const int c = c0 + 8 * j + 2 * t4;
                    if (c >= g.cp) continue;
                    if (pieces == 1) *(uint32_t*)((bf16*)a.o + ((size_t)t * g.heads + h0 + row) * g.cp + c) = pack2(o[m][j][2 * r] * inv, o[m][j][2 * r + 1] * inv);
                    else *(float2*)(pc.o + (out_row + h0 + row) * g.cp + c) = make_float2(o[m][j][2 * r], o[m][j][2 * r + 1]);
                }
            }
    }
}

constexpr int kMaxPieces = 64;
__global__ void __launch_bounds__(128) latent_merge_kernel(LatentPieces pc, int pieces, int heads, int cp, bf16* __restrict__ out) {
    __shared__ float s_w[kMaxPieces];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, t = blockIdx.y;
    const size_t base = (size_t)t * pieces * heads + h;
    if (threadIdx.x < 32) {
        float m = -INFINITY, l = 0.0f;
        for (int i = threadIdx.x; i < pieces; i += 32) m = fmaxf(m, pc.ml[(base + (size_t)i * heads) * 2]);
        m = warp_max(m);
        for (int i = threadIdx.x; i < pieces; i += 32) {
            const float w = exp2f(pc.ml[(base + (size_t)i * heads) * 2] - m);
            s_w[i] = w;
            l += w * pc.ml[(base + (size_t)i * heads) * 2 + 1];
        }
        l = warp_sum(l);
        __syncwarp();
        for (int i = threadIdx.x; i < pieces; i += 32) s_w[i] /= l;
    }
    __syncthreads();
    for (int c = threadIdx.x * 4; c < cp; c += 512) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        const float* src = pc.o + base * cp + c;
#pragma unroll 8
        for (int i = 0; i < pieces; i++) {
            const float w = s_w[i];  // 0: an empty piece, which has written no sums
            const float4 v = w != 0.0f ? *(const float4*)(src + (size_t)i * heads * cp) : make_float4(0.f, 0.f, 0.f, 0.f);
            x.x = fmaf(w, v.x, x.x); x.y = fmaf(w, v.y, x.y); x.z = fmaf(w, v.z, x.z); x.w = fmaf(w, v.w, x.w);
        }
        *(uint2*)(out + ((size_t)t * heads + h) * cp + c) = make_uint2(pack2(x.x, x.y), pack2(x.z, x.w));
    }
}

// The cached rows of a context, in order: row row0 + i of out = position i of the sequence.
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* __restrict__ cache, int row16, int page_tokens, const int32_t* __restrict__ page_table,
                                                            int pages_per_seq, const LatentContext* __restrict__ ctx, uint4* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    const LatentContext c = ctx[blockIdx.y];
    const int n = c.len * row16;
    for (int i = blockIdx.x * 256 + threadIdx.x; i < n; i += gridDim.x * 256) {
        const int p = i / row16, w = i - p * row16;
        const int page = page_table[(size_t)c.seq * pages_per_seq + p / page_tokens];
        out[(size_t)(c.row0 + p) * row16 + w] = cache[((size_t)page * page_tokens + p % page_tokens) * row16 + w];
    }
}

// Many tokens of a sequence: keys and values of every head have been projected from the gathered latents; a CTA of four warps
// takes 64 consecutive queries of one head, tiles of 64 keys, online softmax in log2 units.
template <int NV>
__global__ void __launch_bounds__(128) latent_prefill_kernel(const LatentArgs a, const LatentPrefill p) {
    extern __shared__ __align__(128) unsigned char smem[];
    const LatentShape& g = a.g;
    const int d = g.dp + g.rp, d32 = (d + 31) & ~31, pitch = d32 + 8, rb = pitch * 2;
    constexpr int kVP = NV * 8 + 8, kVB = kVP * 2;
    bf16 *s_q = (bf16*)smem, *s_k = s_q + 64 * pitch, *s_v = s_k + 2 * kKeys * pitch;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
    pdl_launch_dependents();
    pdl_wait();
    const LatentTile tl = p.tiles[gridDim.x - 1 - blockIdx.x];  // the tiles with the longest contexts first
    const int h = blockIdx.y, ld_c = g.cp + g.rp, ldk = g.heads * g.dp, ldv = g.heads * p.ep;
    const int ctx_end = tl.pos0 + tl.n, n_kt = (ctx_end + kKeys - 1) / kKeys;
    const uint32_t q_sm = smem_u32(s_q), k_sm = smem_u32(s_k), v_sm = smem_u32(s_v);
    const bf16 *kc = (const bf16*)p.k + (size_t)tl.row0 * ldk + h * g.dp, *rc = (const bf16*)p.c + (size_t)tl.row0 * ld_c + g.cp,
               *vc = (const bf16*)p.v + (size_t)tl.row0 * ldv + h * p.ep;
    const int kch = g.dp / 8, rch = g.rp / 8, vch = p.ep / 8, per_key = kch + rch + vch;
    auto load = [&](int kt, int buf) {
        for (int i = tid; i < kKeys * per_key; i += 128) {
            const int key = i / per_key, c = i - key * per_key, kp = kt * kKeys + key;
            const bool ok = kp < ctx_end;
            const bf16* src;
            uint32_t dst;
            if (c < kch) { src = kc + (size_t)kp * ldk + c * 8; dst = k_sm + (uint32_t)((buf * kKeys + key) * rb + c * 16); }
            else if (c < kch + rch) { src = rc + (size_t)kp * ld_c + (c - kch) * 8; dst = k_sm + (uint32_t)((buf * kKeys + key) * rb + c * 16); }
            else { src = vc + (size_t)kp * ldv + (c - kch - rch) * 8; dst = v_sm + (uint32_t)((buf * kKeys + key) * kVB + (c - kch - rch) * 16); }
            cp16(dst, ok ? src : kc, ok ? 16 : 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0, 0);
    const bf16 zero = __float2bfloat16_rn(0.0f);
    for (int i = tid; i < 2 * kKeys * (pitch - d); i += 128) s_k[(i / (pitch - d)) * pitch + d + i % (pitch - d)] = zero;
    if (kVP > p.ep)
        for (int i = tid; i < 2 * kKeys * (kVP - p.ep); i += 128) s_v[(i / (kVP - p.ep)) * kVP + p.ep + i % (kVP - p.ep)] = zero;
    for (int i = tid; i < 64 * (pitch / 8); i += 128) {
        const int r = i / (pitch / 8), c = (i - r * (pitch / 8)) * 8;
        const size_t th = (size_t)(tl.tok0 + r) * g.heads + h;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < tl.n && c < d) {
            const bf16* row = (const bf16*)a.q + th * g.ld_q;
            if (c < g.dp) v = *(const uint4*)(row + c);
            else {
                const float2* tab = a.rot + (size_t)(tl.pos0 + r) * g.rot_pairs;
                uint32_t w[4];
#pragma unroll
                for (int j = 0; j < 4; j++) w[j] = pack2(rotated(row + g.dp, tab, g.rot_pairs, g.rot, c - g.dp + 2 * j), rotated(row + g.dp, tab, g.rot_pairs, g.rot, c - g.dp + 2 * j + 1));
                v = make_uint4(w[0], w[1], w[2], w[3]);
            }
        }
        *(uint4*)(s_q + r * pitch + c) = v;
    }
    float o[NV][4];
#pragma unroll
    for (int i = 0; i < NV; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
    const float sc = g.scale * 1.4426950408889634f;
    const int q0 = warp * 16, qpos[2] = {tl.pos0 + q0 + g8, tl.pos0 + q0 + g8 + 8};
    const int last_kt = min(n_kt - 1, (tl.pos0 + q0 + 15) / kKeys);
    for (int kt = 0; kt < n_kt; kt++) {
        const int buf = kt & 1;
        if (kt + 1 < n_kt) { load(kt + 1, buf ^ 1); asm volatile("cp.async.wait_group 1;" ::: "memory"); }
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (kt <= last_kt) {
            const uint32_t kb = k_sm + (uint32_t)(buf * kKeys * rb), vb = v_sm + (uint32_t)(buf * kKeys * kVB);
            float s[8][4];
#pragma unroll
            for (int i = 0; i < 8; i++) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
            const uint32_t qa = q_sm + (uint32_t)((q0 + (lane & 15)) * rb + (lane >> 4) * 16), ka = kb + (uint32_t)((lane & 7) * rb + (lane >> 3) * 16);
            for (int k = 0; k < d32; k += 32) {
                uint32_t a0[4], a1[4];
                ldsm4(qa + k * 2, a0);
                ldsm4(qa + k * 2 + 32, a1);
#pragma unroll
                for (int nt = 0; nt < 8; nt++) {
                    uint32_t b[4];
                    ldsm4(ka + (uint32_t)(8 * nt * rb + k * 2), b);
                    mma_bf16(s[nt], a0, b[0], b[1]);
                    mma_bf16(s[nt], a1, b[2], b[3]);
                }
            }
            float mx[2] = {-INFINITY, -INFINITY};
            const bool edge = kt * kKeys + kKeys - 1 > tl.pos0 + q0;
#pragma unroll
            for (int nt = 0; nt < 8; nt++)
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    float v = s[nt][i] * sc;
                    if (edge && kt * kKeys + 8 * nt + 2 * t4 + (i & 1) > qpos[i >> 1]) v = -INFINITY;
                    s[nt][i] = v;
                    mx[i >> 1] = fmaxf(mx[i >> 1], v);
                }
            float corr[2];
#pragma unroll
            for (int r = 0; r < 2; r++) {
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
                const float m = fmaxf(m_run[r], mx[r]);  // finite: key 0 is never past a query's position
                corr[r] = exp2f(m_run[r] - m);
                m_run[r] = m;
            }
            float ps[2] = {0.0f, 0.0f};
            uint32_t ph[4][4], pl[4][4];
#pragma unroll
            for (int nt = 0; nt < 8; nt++) {
                float pv[4];
#pragma unroll
                for (int i = 0; i < 4; i++) { pv[i] = exp2f(s[nt][i] - m_run[i >> 1]); ps[i >> 1] += pv[i]; }
                const int ks = nt >> 1, hs = (nt & 1) * 2;
                split2(pv[0], pv[1], ph[ks][hs], pl[ks][hs]);
                split2(pv[2], pv[3], ph[ks][hs + 1], pl[ks][hs + 1]);
            }
#pragma unroll
            for (int r = 0; r < 2; r++) {
                ps[r] += __shfl_xor_sync(0xffffffffu, ps[r], 1);
                ps[r] += __shfl_xor_sync(0xffffffffu, ps[r], 2);
                l_run[r] = l_run[r] * corr[r] + ps[r];
            }
#pragma unroll
            for (int i = 0; i < NV; i++) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
#pragma unroll
            for (int ks = 0; ks < 4; ks++)
#pragma unroll
                for (int np = 0; np < NV / 2; np++) {
                    uint32_t b[4];
                    ldsm4t(vb + (uint32_t)((16 * ks + (lane & 15)) * kVB + (16 * np + (lane >> 4) * 8) * 2), b);
                    mma_bf16(o[2 * np], ph[ks], b[0], b[1]);
                    mma_bf16(o[2 * np], pl[ks], b[0], b[1]);
                    mma_bf16(o[2 * np + 1], ph[ks], b[2], b[3]);
                    mma_bf16(o[2 * np + 1], pl[ks], b[2], b[3]);
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const int row = q0 + g8 + 8 * r;
        if (row >= tl.n) continue;
        const float inv = 1.0f / l_run[r];
        bf16* dst = (bf16*)p.out + (size_t)(tl.tok0 + row) * ldv + h * p.ep + 2 * t4;
#pragma unroll
        for (int i = 0; i < NV; i++)
            if (8 * i + 2 * t4 < p.ep) *(uint32_t*)(dst + 8 * i) = pack2(o[i][2 * r] * inv, o[i][2 * r + 1] * inv);
    }
}

size_t decode_smem(const LatentShape& g, int mt) {
    const size_t pitch = ((g.cp + g.rp + 31) & ~31) + 8, rows = 16 * (size_t)mt;
    return (rows + kDecodeTiles * kDecodeKeys) * pitch * 2 + 4 * rows * kPPitch * 2 + (4 * rows * kPartPitch + 3 * rows) * 4 + (2 * kDecodeTiles + 4) * 8;
}
size_t prefill_smem(const LatentShape& g, int nv) {
    const size_t pitch = ((g.dp + g.rp + 31) & ~31) + 8;
    return (64 + 2 * kKeys) * pitch * 2 + 2 * kKeys * ((size_t)nv * 8 + 8) * 2;
}
int value_tiles(int ep) { return ep <= 32 ? 4 : ep <= 64 ? 8 : ep <= 128 ? 16 : 32; }

int32_t launch_plain(const LatentArgs& a, cudaStream_t s) {
    const size_t smem = (size_t)(2 * a.g.cp + a.g.rp + 2 * kPlainThreads) * 4;
    LC_CHECK(smem <= kMaxSmem, LC_ERR_UNSUPPORTED, "latent attention: rank %d", a.g.rank);
    const dim3 grid((unsigned)a.g.heads, (unsigned)a.T);
    if (a.f32) {
        LC_CUDA(ensure_smem_limit((const void*)latent_attention_plain_kernel<float>, smem));
        LC_CUDA(launch_pdl(latent_attention_plain_kernel<float>, grid, dim3(kPlainThreads), smem, s, a));
    } else {
        LC_CUDA(ensure_smem_limit((const void*)latent_attention_plain_kernel<bf16>, smem));
        LC_CUDA(launch_pdl(latent_attention_plain_kernel<bf16>, grid, dim3(kPlainThreads), smem, s, a));
    }
    return LC_OK;
}

}  // namespace

size_t latent_pieces_bytes(const LatentShape& g, int tokens) {
    // pieces * tokens * row blocks stays within the SM count, so the scratch is bounded by that many row blocks
    const size_t blocks = std::max<size_t>((size_t)sm_count(), (size_t)tokens * ((g.heads + 15) / 16));
    return blocks * 32 * ((size_t)g.cp + 2) * sizeof(float) * 2;
}

int32_t launch_latent_attention(const LatentArgs& a, void* scratch, size_t scratch_bytes, int* launches, cudaStream_t s) {
    const LatentShape& g = a.g;
    const int mt = g.heads <= 16 ? 1 : 2;
    *launches = 1;
    if (a.T <= 0) return LC_OK;
    if (a.f32 || g.cp > 512 || decode_smem(g, mt) > kMaxSmem) return launch_plain(a, s);
    const int blocks = (g.heads + 16 * mt - 1) / (16 * mt);
    int pieces = std::max(1, std::min(kMaxPieces, sm_count() / (a.T * blocks)));
    pieces = std::min(pieces, (a.pages_per_seq * a.page_tokens + kDecodeKeys - 1) / kDecodeKeys);
    auto need = [&](int n) { return (size_t)a.T * n * g.heads * ((size_t)g.cp + 2) * sizeof(float); };
    while (pieces > 1 && need(pieces) > scratch_bytes) pieces--;
    LatentPieces pc;
    pc.o = (float*)scratch;
    pc.ml = pc.o + (size_t)a.T * pieces * g.heads * g.cp;
    const size_t smem = decode_smem(g, mt);
    const dim3 grid((unsigned)a.T, (unsigned)blocks, (unsigned)pieces);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3(kDecodeThreads), smem, s, a, pc, gemv_error_flag_dev()));
        return LC_OK;
    };
    const int nct = g.cp <= 128 ? 2 : g.cp <= 256 ? 4 : 8;  // latent columns of a warp, in eights
    if (mt == 1) LC_TRY(nct == 2 ? go(latent_decode_kernel<1, 2>) : nct == 4 ? go(latent_decode_kernel<1, 4>) : go(latent_decode_kernel<1, 8>));
    else LC_TRY(nct == 2 ? go(latent_decode_kernel<2, 2>) : nct == 4 ? go(latent_decode_kernel<2, 4>) : go(latent_decode_kernel<2, 8>));
    if (pieces > 1) {
        LC_CUDA(launch_pdl(latent_merge_kernel, dim3((unsigned)g.heads, (unsigned)a.T), dim3(128), 0, s, pc, pieces, g.heads, g.cp, (bf16*)a.o));
        *launches = 2;
    }
    return LC_OK;
}

bool latent_prefill_applies(const LatentShape& g, int ep, bool f32) { return !f32 && ep <= 256 && prefill_smem(g, value_tiles(ep)) <= kMaxSmem; }

int32_t launch_latent_gather(const LatentArgs& a, const LatentContext* ctx, int n_ctx, int longest, void* out, cudaStream_t s) {
    const int row16 = (a.g.cp + a.g.rp) / 8;
    const int gx = std::max(1, std::min((int)(((size_t)longest * row16 + 255) / 256), 4 * sm_count()));
    LC_CUDA(launch_pdl(latent_gather_kernel, dim3((unsigned)gx, (unsigned)n_ctx), dim3(256), 0, s, (const uint4*)a.cache, row16, a.page_tokens, a.page_table,
                       a.pages_per_seq, ctx, (uint4*)out));
    return LC_OK;
}

int32_t launch_latent_prefill(const LatentArgs& a, const LatentPrefill& p, int n_tiles, cudaStream_t s) {
    const int nv = value_tiles(p.ep);
    const size_t smem = prefill_smem(a.g, nv);
    const dim3 grid((unsigned)n_tiles, (unsigned)a.g.heads);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3(128), smem, s, a, p));
        return LC_OK;
    };
    switch (nv) {
        case 4: return go(latent_prefill_kernel<4>);
        case 8: return go(latent_prefill_kernel<8>);
        case 16: return go(latent_prefill_kernel<16>);
        default: return go(latent_prefill_kernel<32>);
    }
}

}  // namespace lc
