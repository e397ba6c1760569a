// The kernels of the checkpoint-directory layers around their products: embedding, norms and residual sums, the gated delta
// rule with its short convolutions, the preparation of latent attention.  Template parameter A = type of the activations
// (bf16, or float when a model runs in true 32-bit); norms, decays, step sizes, unit vectors, the recurrence and its state,
// rotation angles and residual sums are f32 in both.
#include <algorithm>
#include <cmath>
#include "lc_mixers.h"
#include "lc_mma.cuh"
#include "lc_tma.cuh"

namespace lc {

namespace {

__device__ __forceinline__ int mapped(const PackMap& m, int i) {
    if (m.len == 0) return i;
    const int g = i / m.len, r = i - g * m.len;
    return g * m.stride + r + (m.shift && r >= m.split ? m.shift : 0);
}
__global__ void pack_kernel(const __nv_bfloat16* __restrict__ src, int rows, int cols, __nv_bfloat16* __restrict__ dst, int ld, PackMap rm, PackMap cm, int transpose) {
    const size_t n = (size_t)rows * cols;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const int r = (int)(i / cols), c = (int)(i % cols);
        if (transpose) {
            const int g = r / rm.len, q = r - g * rm.len;
            dst[((size_t)g * rm.stride + c) * ld + q] = src[i];
        } else {
            dst[(size_t)mapped(rm, r) * ld + mapped(cm, c)] = src[i];
        }
    }
}

template <typename A> __device__ __forceinline__ float4 load4(const A* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *(const float4*)p; }
template <> __device__ __forceinline__ float4 load4<bf16>(const bf16* p) {
    const uint2 v = *(const uint2*)p;
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xFFFF0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xFFFF0000u));
}
template <typename A> __device__ __forceinline__ void store4(A* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *(float4*)p = v; }
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, float4 v) { *(uint2*)p = make_uint2(pack2(v.x, v.y), pack2(v.z, v.w)); }
__device__ __forceinline__ float sq4(float4 v, float ss) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss)))); }
__device__ __forceinline__ void add4(float4& y, float w, float4 v) { y.x = fmaf(w, v.x, y.x); y.y = fmaf(w, v.y, y.y); y.z = fmaf(w, v.z, y.z); y.w = fmaf(w, v.w, y.w); }

__global__ void __launch_bounds__(256) embed_rows_kernel(const __nv_bfloat16* __restrict__ table, int rows, int width, const int64_t* __restrict__ ids,
                                                         float* __restrict__ x, __nv_bfloat16* __restrict__ act, int ld_act) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int64_t id = ids[t];
    const bool ok = id >= 0 && id < rows;
    if (width % 8 == 0) {
        for (int c = threadIdx.x * 8; c < width; c += blockDim.x * 8) {
            const uint4 v = ok ? *(const uint4*)(table + (size_t)id * width + c) : make_uint4(0u, 0u, 0u, 0u);
            const uint32_t u[4] = {v.x, v.y, v.z, v.w};
            float4* o = (float4*)(x + (size_t)t * width + c);
            o[0] = make_float4(__uint_as_float(u[0] << 16), __uint_as_float(u[0] & 0xFFFF0000u), __uint_as_float(u[1] << 16), __uint_as_float(u[1] & 0xFFFF0000u));
            o[1] = make_float4(__uint_as_float(u[2] << 16), __uint_as_float(u[2] & 0xFFFF0000u), __uint_as_float(u[3] << 16), __uint_as_float(u[3] & 0xFFFF0000u));
            if (act) *(uint4*)(act + (size_t)t * ld_act + c) = v;
        }
        return;
    }
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const __nv_bfloat16 v = ok ? table[(size_t)id * width + c] : __float2bfloat16_rn(0.0f);
        x[(size_t)t * width + c] = __bfloat162float(v);
        if (act) act[(size_t)t * ld_act + c] = v;
    }
}

// The same with a factor on the row, the token pair's row (PAIR) and, w != null, the sum's norm as activations.
// VEC = 8: rows of a multiple of eight elements.
template <typename A, bool PAIR, int VEC>
__global__ void __launch_bounds__(512) embed_norm_kernel(const EmbedArgs a) {
    constexpr int kHeld = VEC == 8 ? 2 : 4;
    __shared__ float sh[32];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int width = a.width;
    const int64_t id = a.ids[t];
    const bool ok = id >= 0 && id < a.rows;
    const bf16 *src = a.table + (size_t)(ok ? id : 0) * width, *two = nullptr;
    if constexpr (PAIR) {
        const PairEmbed& p = a.pair;
        const int seq = p.tok_seq[t], pos = p.tok_pos[t];
        int64_t row = p.rows.buckets;
        if (pos > 0) {
            const bool here = t > 0 && p.tok_seq[t - 1] == seq && p.tok_pos[t - 1] == pos - 1;
            const int64_t prev = here ? a.ids[t - 1] : (int64_t)p.last[seq];
            row = (prev % p.rows.buckets * p.rows.mul_prev + id % p.rows.buckets * p.rows.mul_cur) % p.rows.buckets;
            if (row < 0) row += p.rows.buckets;
        }
        two = p.table + (size_t)row * width;
        if (p.one_each) {
            __syncthreads();  // every thread has read the token before
            if (threadIdx.x == 0) p.last[seq] = (int32_t)id;
        }
    }
    struct Part { float v[VEC]; };
    auto at = [&](int c) {
        Part p;
        if constexpr (VEC == 8) {
            const uint4 s = *(const uint4*)(src + c), u = PAIR ? *(const uint4*)(two + c) : make_uint4(0u, 0u, 0u, 0u);
            const uint32_t sw[4] = {s.x, s.y, s.z, s.w}, uw[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
            for (int i = 0; i < 4; i++) {
                p.v[2 * i] = fmaf(__uint_as_float(sw[i] << 16), a.scale, __uint_as_float(uw[i] << 16));
                p.v[2 * i + 1] = fmaf(__uint_as_float(sw[i] & 0xFFFF0000u), a.scale, __uint_as_float(uw[i] & 0xFFFF0000u));
            }
        } else p.v[0] = fmaf(__bfloat162float(src[c]), a.scale, PAIR ? __bfloat162float(two[c]) : 0.0f);
        if (!ok)
#pragma unroll
            for (int i = 0; i < VEC; i++) p.v[i] = 0.0f;
        return p;
    };
    float ss = 0.0f;
    auto put = [&](int c, const Part& p) {
        float* dst[2] = {a.x, a.copy};
#pragma unroll
        for (int d = 0; d < 2; d++) {
            if (!dst[d]) continue;
            float* o = dst[d] + t * width + c;
            if constexpr (VEC == 8) { *(float4*)o = make_float4(p.v[0], p.v[1], p.v[2], p.v[3]); *(float4*)(o + 4) = make_float4(p.v[4], p.v[5], p.v[6], p.v[7]); }
            else *o = p.v[0];
        }
#pragma unroll
        for (int i = 0; i < VEC; i++) ss = fmaf(p.v[i], p.v[i], ss);
    };
    const int step = blockDim.x * VEC, c0 = threadIdx.x * VEC;
    Part held[kHeld];
#pragma unroll
    for (int i = 0; i < kHeld; i++)
        if (c0 + i * step < width) held[i] = at(c0 + i * step);
#pragma unroll
    for (int i = 0; i < kHeld; i++)
        if (c0 + i * step < width) put(c0 + i * step, held[i]);
    for (int c = c0 + kHeld * step; c < width; c += step) put(c, at(c));
    if (!a.act) return;
    const float r = a.w ? 1.0f / sqrtf(block_sum_once(ss, sh) / (float)width + a.eps) : 1.0f;
    A* act = (A*)a.act + t * a.ld_act;
    auto next = [&](int c, Part p) {
#pragma unroll
        for (int i = 0; i < VEC; i++) p.v[i] = a.w ? p.v[i] * r * a.w[c + i] : p.v[i];
        if constexpr (VEC == 8) { store4<A>(act + c, make_float4(p.v[0], p.v[1], p.v[2], p.v[3])); store4<A>(act + c + 4, make_float4(p.v[4], p.v[5], p.v[6], p.v[7])); }
        else act[c] = to_act<A>(p.v[0]);
    };
#pragma unroll
    for (int i = 0; i < kHeld; i++)
        if (c0 + i * step < width) next(c0 + i * step, held[i]);
    for (int c = c0 + kHeld * step; c < width; c += step) next(c, at(c));
}

__global__ void keep_tokens_kernel(const SeqRun* __restrict__ runs, int n, const int64_t* __restrict__ ids, int32_t* __restrict__ last) {
    pdl_launch_dependents();
    pdl_wait();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) last[runs[i].seq] = (int32_t)ids[runs[i].tok0 + runs[i].n - 1];
}

__global__ void __launch_bounds__(256) act_rows_kernel(const float* __restrict__ x, int width, __nv_bfloat16* __restrict__ act, int ld_act) {
    pdl_launch_dependents();
    pdl_wait();
    for (int c = threadIdx.x; c < width; c += blockDim.x) act[(size_t)blockIdx.x * ld_act + c] = __float2bfloat16_rn(x[(size_t)blockIdx.x * width + c]);
}

// x += y, the sum over depth (DEPTH), the next sublayer's norm.  VEC as below.
template <typename A, int VEC, bool DEPTH, int THREADS>
__global__ void __launch_bounds__(THREADS) plain_residual_kernel(const ResidualArgs a) {
    constexpr int kHeld = VEC == 4 ? 4 : 8, kAhead = 8;  // results of earlier layers that are fetched together
    __shared__ float sh[32];
    pdl_launch_dependents();
    pdl_wait();
    const size_t row = (size_t)blockIdx.x * a.width;
    const int width = a.width, step = blockDim.x * VEC;
    const float* yr = a.y + row;
    float* xr = a.x + row;
    A* ar = a.act ? (A*)a.act + (size_t)blockIdx.x * a.ld_act : nullptr;
    struct Part { float v[VEC]; };
    auto get = [&](const float* p) {
        Part r;
        if constexpr (VEC == 4) { const float4 f = *(const float4*)p; r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w; }
        else r.v[0] = *p;
        return r;
    };
    auto put = [&](float* p, const Part& r) {
        if constexpr (VEC == 4) *(float4*)p = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
        else *p = r.v[0];
    };
    auto sum = [&](int c) {
        Part s = get(xr + c);
        const Part y = get(yr + c);
#pragma unroll
        for (int e = 0; e < VEC; e++) s.v[e] += y.v[e];
        if constexpr (DEPTH) {
            const DepthSum& d = a.depth;
            const Part result = s;
            const float own = __ldg(d.c + d.n);
#pragma unroll
            for (int e = 0; e < VEC; e++) s.v[e] *= own;
            const float* past = d.past + row + c;
            for (int j0 = 0; j0 < d.n; j0 += kAhead, past += kAhead * d.stride) {
                Part z[kAhead];
                float f[kAhead];
#pragma unroll
                for (int u = 0; u < kAhead; u++) {
                    const bool there = j0 + u < d.n;
                    f[u] = there ? __ldg(d.c + j0 + u) : 0.0f;
                    if (there) z[u] = get(past + u * d.stride);
                    else
#pragma unroll
                        for (int e = 0; e < VEC; e++) z[u].v[e] = 0.0f;
                }
#pragma unroll
                for (int u = 0; u < kAhead; u++)
#pragma unroll
                    for (int e = 0; e < VEC; e++) s.v[e] = fmaf(f[u], z[u].v[e], s.v[e]);
            }
            put(d.keep + row + c, result);
        }
        put(xr + c, s);
        return s;
    };
    Part held[kHeld];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < kHeld; i++) {
        const int c = threadIdx.x * VEC + i * step;
        if (c < width) {
            held[i] = sum(c);
#pragma unroll
            for (int e = 0; e < VEC; e++) ss = fmaf(held[i].v[e], held[i].v[e], ss);
        }
    }
    for (int c = threadIdx.x * VEC + kHeld * step; c < width; c += step) {
        const Part s = sum(c);
#pragma unroll
        for (int e = 0; e < VEC; e++) ss = fmaf(s.v[e], s.v[e], ss);
    }
    if (!ar) return;
    const float* wn = a.w_next;
    const float r = wn ? 1.0f / sqrtf(block_sum_once(ss, sh) / (float)width + a.eps) : 1.0f;
    auto next = [&](int c, const Part& s) {
        Part n = s;
        if (wn) {
            const Part g = get(wn + c);
#pragma unroll
            for (int e = 0; e < VEC; e++) n.v[e] = s.v[e] * r * g.v[e];
        }
        if constexpr (VEC == 4) store4<A>(ar + c, make_float4(n.v[0], n.v[1], n.v[2], n.v[3]));
        else ar[c] = to_act<A>(n.v[0]);
    };
#pragma unroll
    for (int i = 0; i < kHeld; i++) {
        const int c = threadIdx.x * VEC + i * step;
        if (c < width) next(c, held[i]);
    }
    for (int c = threadIdx.x * VEC + kHeld * step; c < width; c += step) next(c, get(xr + c));
}

// VEC = 4: rows of a multiple of four elements; a row of up to 16 elements per thread stays in registers between its passes.
// MOE, PAIR: the output is first made from a mixture's parts (MoeSum) or from two mixers' outputs (PairSum).
template <typename A, int VEC, bool MOE, bool PAIR>
__global__ void __launch_bounds__(512) residual_kernel(const ResidualArgs a) {
    constexpr int kHeld = 4;
    constexpr bool kMade = MOE || PAIR;  // the output is made here, not read
    __shared__ float sh[32], sh2[32], sh_p[2][32];
    __shared__ long long s_row[kMaxChoices];
    __shared__ float s_w[kMaxChoices], s_gate;
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int width = a.width;
    float* yr = a.y + t * width;
    float* xr = a.x + t * width;
    const float *w = a.w, *wn = a.w_next;
    A* ar = a.act ? (A*)a.act + t * a.ld_act : nullptr;
    const A* hr = MOE ? (const A*)a.moe.h + t * a.moe.ld_h : nullptr;
    float own = 0.0f, gate = 0.0f;  // weight of the input itself, of y
    if constexpr (MOE) {
        if ((int)threadIdx.x < a.moe.top) {
            const size_t i = t * a.moe.top + threadIdx.x;
            const int e = a.moe.sel[i];
            s_row[threadIdx.x] = e < a.moe.experts ? (long long)(a.moe.off[e] + a.moe.pos[i]) * a.moe.ld_rows : -1;
            s_w[threadIdx.x] = a.moe.weight[i];
        }
        if (threadIdx.x == 0) s_gate = a.moe.gate ? sigmoid_f(a.moe.gate[t * a.moe.ld_gate]) : 0.0f;
        __syncthreads();
        for (int j = 0; j < a.moe.top; j++) own += s_row[j] < 0 ? s_w[j] : 0.0f;
        gate = s_gate;
    }
    const float* y2 = PAIR ? a.pair.y2 + t * width : nullptr;
    float f0 = 0.0f, f1 = 0.0f;  // half the reciprocal roots of the pair's mean squares
    if constexpr (PAIR) {
        float s0 = 0.0f, s1 = 0.0f;
        if constexpr (VEC == 4)
            for (int c = threadIdx.x * 4; c < width; c += blockDim.x * 4) { s0 = sq4(*(const float4*)(yr + c), s0); s1 = sq4(*(const float4*)(y2 + c), s1); }
        else
            for (int c = threadIdx.x; c < width; c += blockDim.x) { s0 = fmaf(yr[c], yr[c], s0); s1 = fmaf(y2[c], y2[c], s1); }
        s0 = warp_sum(s0); s1 = warp_sum(s1);
        if ((threadIdx.x & 31) == 0) { sh_p[0][threadIdx.x >> 5] = s0; sh_p[1][threadIdx.x >> 5] = s1; }
        __syncthreads();
        s0 = s1 = 0.0f;
        for (unsigned w = 0; w < blockDim.x / 32; w++) { s0 += sh_p[0][w]; s1 += sh_p[1][w]; }
        f0 = 0.5f / sqrtf(s0 / (float)width + a.eps);
        f1 = 0.5f / sqrtf(s1 / (float)width + a.eps);
    }
    float ss = 0.0f;
    if constexpr (VEC == 4) {
        float4 yv[kHeld], xv[kHeld];
        auto out_at = [&](int c) {
            if constexpr (PAIR) {
                const float4 p = *(const float4*)(yr + c), q = *(const float4*)(y2 + c), u = *(const float4*)(a.pair.w0 + c), v = *(const float4*)(a.pair.w1 + c);
                return make_float4(p.x * f0 * u.x + q.x * f1 * v.x, p.y * f0 * u.y + q.y * f1 * v.y, p.z * f0 * u.z + q.z * f1 * v.z, p.w * f0 * u.w + q.w * f1 * v.w);
            }
            if constexpr (!MOE) return *(const float4*)(yr + c);
            float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
            if (a.moe.gate) add4(y, gate, *(const float4*)(yr + c));
            for (int j = 0; j < a.moe.top; j++)
                if (s_row[j] >= 0) add4(y, s_w[j], load4<A>((const A*)a.moe.rows + s_row[j] + c));
            if (own != 0.0f) add4(y, own, load4<A>(hr + c));
            return y;
        };
#pragma unroll
        for (int i = 0; i < kHeld; i++) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            if (c < width) {
                yv[i] = out_at(c);
                if (a.x) xv[i] = *(const float4*)(xr + c);
                else *(float4*)(yr + c) = yv[i];
            } else yv[i] = xv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            ss = sq4(yv[i], ss);
        }
        for (int c = (threadIdx.x + kHeld * blockDim.x) * 4; c < width; c += blockDim.x * 4) {
            const float4 v = out_at(c);
            if (kMade) *(float4*)(yr + c) = v;
            ss = sq4(v, ss);
        }
        if (kMade && !a.x) return;
        ss = block_sum_once(ss, sh);
        const float r = 1.0f / sqrtf(ss / (float)width + a.eps);
        float s2 = 0.0f;
        auto put = [&](int c, float4 yy, float4 xx) {
            const float4 g = *(const float4*)(w + c);
            xx.x += yy.x * r * g.x; xx.y += yy.y * r * g.y; xx.z += yy.z * r * g.z; xx.w += yy.w * r * g.w;
            *(float4*)(xr + c) = xx;
            if (ar && !wn) store4<A>(ar + c, xx);
            s2 = sq4(xx, s2);
            return xx;
        };
#pragma unroll
        for (int i = 0; i < kHeld; i++) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            if (c < width) xv[i] = put(c, yv[i], xv[i]);
        }
        for (int c = (threadIdx.x + kHeld * blockDim.x) * 4; c < width; c += blockDim.x * 4) put(c, *(const float4*)(yr + c), *(const float4*)(xr + c));
        if (!wn) return;
        const float r2 = 1.0f / sqrtf(block_sum_once(s2, sh2) / (float)width + a.eps);
        auto next = [&](int c, float4 v) {
            const float4 g = *(const float4*)(wn + c);
            store4<A>(ar + c, make_float4(v.x * r2 * g.x, v.y * r2 * g.y, v.z * r2 * g.z, v.w * r2 * g.w));
        };
#pragma unroll
        for (int i = 0; i < kHeld; i++) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            if (c < width) next(c, xv[i]);
        }
        for (int c = (threadIdx.x + kHeld * blockDim.x) * 4; c < width; c += blockDim.x * 4) next(c, *(const float4*)(xr + c));
    } else {
        for (int c = threadIdx.x; c < width; c += blockDim.x) {
            float v = 0.0f;
            if constexpr (MOE) {
                if (a.moe.gate) v = gate * yr[c];
                for (int j = 0; j < a.moe.top; j++)
                    if (s_row[j] >= 0) v = fmaf(s_w[j], act_f<A>(((const A*)a.moe.rows)[s_row[j] + c]), v);
                if (own != 0.0f) v = fmaf(own, act_f<A>(hr[c]), v);
                yr[c] = v;
            } else if constexpr (PAIR) {
                v = yr[c] * f0 * a.pair.w0[c] + y2[c] * f1 * a.pair.w1[c];
                yr[c] = v;
            } else v = yr[c];
            ss = fmaf(v, v, ss);
        }
        if (kMade && !a.x) return;
        ss = block_sum_once(ss, sh);
        const float r = 1.0f / sqrtf(ss / (float)width + a.eps);
        float s2 = 0.0f;
        for (int c = threadIdx.x; c < width; c += blockDim.x) {
            const float v = xr[c] + yr[c] * r * w[c];
            xr[c] = v;
            if (ar && !wn) ar[c] = to_act<A>(v);
            s2 = fmaf(v, v, s2);
        }
        if (!wn) return;
        const float r2 = 1.0f / sqrtf(block_sum_once(s2, sh2) / (float)width + a.eps);
        for (int c = threadIdx.x; c < width; c += blockDim.x) ar[c] = to_act<A>(xr[c] * r2 * wn[c]);
    }
}

template <typename A>
__global__ void __launch_bounds__(512) norm_rows_kernel(const float* __restrict__ x, const int32_t* __restrict__ idx, const float* __restrict__ w, float eps, int width,
                                                        A* __restrict__ out, int ldo) {
    __shared__ float sh[32];
    pdl_launch_dependents();
    pdl_wait();
    const float* xr = x + (size_t)(idx ? idx[blockIdx.x] : (int)blockIdx.x) * width;
    constexpr int kHeld = 8;  // elements of a thread that stay in registers between the passes
    float v[kHeld], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < kHeld; i++) {
        const int c = threadIdx.x + i * blockDim.x;
        v[i] = c < width ? xr[c] : 0.0f;
        ss = fmaf(v[i], v[i], ss);
    }
    for (int c = threadIdx.x + kHeld * blockDim.x; c < width; c += blockDim.x) ss = fmaf(xr[c], xr[c], ss);
    ss = block_sum_once(ss, sh);
    const float r = 1.0f / sqrtf(ss / (float)width + eps);
    A* o = out + (size_t)blockIdx.x * ldo;
#pragma unroll
    for (int i = 0; i < kHeld; i++) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < width) o[c] = to_act<A>(v[i] * r * w[c]);
    }
    for (int c = threadIdx.x + kHeld * blockDim.x; c < width; c += blockDim.x) o[c] = to_act<A>(xr[c] * r * w[c]);
}

// ---- gated delta rule ------------------------------------------------------------------------------------------------
// The convolution of one channel at token t: the inputs of earlier positions come from the call's rows as far as they belong
// to the same sequence's run, from the ring before that, and are zero before the sequence's start.
template <typename A>
__device__ __forceinline__ float conv_at(const DeltaShape& g, const A* proj, const A* ring, const float* w, const int32_t* tok_seq, const int32_t* tok_pos, int t,
                                         int seq, int pos, int channel, int column) {
    float acc = 0.0f;
    for (int j = g.taps - 1; j >= 0; j--) {  // j tokens back
        float v = 0.0f;
        if (pos - j >= 0) {
            const int tt = t - j;
            if (tt >= 0 && tok_seq[tt] == seq && tok_pos[tt] == pos - j) v = act_f<A>(proj[(size_t)tt * g.ld + column]);
            else v = act_f<A>(ring[((size_t)seq * g.taps + (pos - j) % g.taps) * g.channels + channel]);
        }
        acc = fmaf(w[channel * g.taps + (g.taps - 1 - j)], v, acc);
    }
    return acc;
}
__device__ __forceinline__ float silu32(float v) { return __fdividef(v, 1.0f + __expf(-v)); }

// One warp per (stretch of kPrepTok tokens, head unit): kv_heads units of q, kv_heads of k, heads of v; a lane owns every 32nd
// channel and keeps its last inputs in registers while it walks the stretch (TAPS of them; 0: any number, re-read).
constexpr int kPrepTok = 16;
template <typename A, int TAPS, int CPL>
__global__ void __launch_bounds__(256, CPL > 4 ? 2 : 3) delta_prep_kernel(const DeltaArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const DeltaShape& g = a.g;
    const int unit = blockIdx.y * 8 + warp_index(), lane = threadIdx.x & 31;
    if (unit >= 2 * g.kv_heads + g.heads) return;
    const A* proj = (const A*)a.proj;
    const A* ring = (const A*)a.ring;
    const bool is_v = unit >= 2 * g.kv_heads, is_k = !is_v && unit >= g.kv_heads;
    const int h = is_v ? unit - 2 * g.kv_heads : is_k ? unit - g.kv_heads : unit, n = is_v ? g.vdim : g.dim;
    const int c0 = is_v ? 2 * g.kv_heads * g.dim + h * g.vdim : unit * g.dim, col0 = is_v ? g.off_v + h * g.vdim : (is_k ? g.off_k : 0) + h * g.dim;
    const int t0 = blockIdx.x * kPrepTok, t1 = min(a.T, t0 + kPrepTok);
    float w[CPL][TAPS > 0 ? TAPS : 1], win[CPL][TAPS > 0 ? TAPS : 1];  // win[.][j]: the input j + 1 tokens back
    if constexpr (TAPS > 0)
#pragma unroll
        for (int c = 0; c < CPL; c++)
#pragma unroll
            for (int j = 0; j < TAPS; j++) w[c][j] = lane + 32 * c < n ? a.conv[(c0 + lane + 32 * c) * TAPS + j] : 0.0f;
    int prev_seq = -1, prev_pos = -1;
    const A* in = proj + col0 + lane;
    bool ok[CPL];
#pragma unroll
    for (int c = 0; c < CPL; c++) ok[c] = lane + 32 * c < n;
    float* o = (is_v ? a.v + (size_t)h * g.vdim : a.qk + (is_k ? g.kv_heads * g.dim : 0) + (size_t)h * g.dim) + lane;
    const unsigned ld_o = is_v ? g.heads * g.vdim : 2 * g.kv_heads * g.dim, ld = g.ld;
    const float q_scale = is_v || is_k ? 1.0f : 1.0f / sqrtf((float)g.dim);
    constexpr int kAhead = TAPS > 0 ? 4 : 1;  // tokens whose inputs are fetched together
    for (int tb = t0; tb < t1; tb += kAhead) {
        float ahead[kAhead][CPL];
        int seq_a[kAhead], pos_a[kAhead];
#pragma unroll
        for (int u = 0; u < kAhead; u++) {
            const unsigned t = min(tb + u, t1 - 1);
            seq_a[u] = a.tok_seq[t]; pos_a[u] = a.tok_pos[t];
            if constexpr (TAPS > 0)
#pragma unroll
                for (int c = 0; c < CPL; c++) ahead[u][c] = ok[c] ? act_f<A>(in[(size_t)(t * ld) + 32 * c]) : 0.0f;
        }
#pragma unroll
        for (int u = 0; u < kAhead; u++) {
            const int t = tb + u;
            if (t >= t1) break;
            const int seq = seq_a[u], pos = pos_a[u];
            float y[CPL], ss = 0.0f;
            if constexpr (TAPS > 0) {
                if (seq != prev_seq || pos != prev_pos + 1) {  // first token of the stretch or of a run: earlier inputs from the call's rows, the ring, or none
#pragma unroll
                    for (int j = 1; j < TAPS; j++) {
                        const int tt = t - j;
                        const bool here = tt >= 0 && pos - j >= 0 && a.tok_seq[max(tt, 0)] == seq && a.tok_pos[max(tt, 0)] == pos - j;
#pragma unroll
                        for (int c = 0; c < CPL; c++) {
                            win[c][j - 1] = 0.0f;
                            if (!ok[c] || pos - j < 0) continue;
                            win[c][j - 1] = here ? act_f<A>(in[(size_t)((unsigned)tt * ld) + 32 * c])
                                                 : act_f<A>(ring[((size_t)seq * TAPS + (pos - j) % TAPS) * g.channels + c0 + lane + 32 * c]);
                        }
                    }
                }
#pragma unroll
                for (int c = 0; c < CPL; c++) {
                    float acc = 0.0f;
#pragma unroll
                    for (int j = TAPS - 1; j > 0; j--) acc = fmaf(w[c][TAPS - 1 - j], win[c][j - 1], acc);
                    acc = fmaf(w[c][TAPS - 1], ahead[u][c], acc);
#pragma unroll
                    for (int j = TAPS - 1; j > 0; j--) win[c][j] = win[c][j - 1];
                    win[c][0] = ahead[u][c];
                    y[c] = silu32(acc);  // channels past n: zero weights, zero inputs
                    ss = fmaf(y[c], y[c], ss);
                }
                prev_seq = seq; prev_pos = pos;
            } else {
#pragma unroll
                for (int c = 0; c < CPL; c++) {
                    const int i = lane + 32 * c;
                    y[c] = ok[c] ? silu32(conv_at<A>(g, proj, ring, a.conv, a.tok_seq, a.tok_pos, t, seq, pos, c0 + i, col0 + i)) : 0.0f;
                    ss = fmaf(y[c], y[c], ss);
                }
            }
            const float r = is_v ? 1.0f : q_scale / sqrtf(warp_sum(ss) + g.unit_eps);
#pragma unroll
            for (int c = 0; c < CPL; c++)
                if (ok[c]) o[(size_t)((unsigned)t * ld_o) + 32 * c] = y[c] * r;
        }
    }
}

// The recurrence, token by token in f32.  A CTA of four warps owns 32 value columns of one head of one run; four lanes share
// a column's `dim` state entries (DPL each: float4 groups dealt round robin), eight columns per warp.
constexpr int kScanTok = 16;  // tokens staged in shared memory at a time
template <typename A, int DPL>
__global__ void __launch_bounds__(128) delta_scan_kernel(const DeltaArgs a) {
    constexpr int DP = DPL * 4;
    extern __shared__ float sm[];
    float *s_q = sm, *s_k = s_q + kScanTok * DP, *s_g = s_k + kScanTok * DP, *s_v = s_g + kScanTok * DP, *s_b = s_v + kScanTok * 32;
    pdl_launch_dependents();
    pdl_wait();
    const DeltaShape& g = a.g;
    const SeqRun run = a.runs[blockIdx.x];
    const int h = blockIdx.y, rep = g.heads / g.kv_heads, kh = h / rep;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r4 = lane & 3, col = warp * 8 + (lane >> 2), e = blockIdx.z * 32 + col;
    float* st = a.state + ((size_t)run.seq * g.heads + h) * g.dim * g.vdim;
    const A* proj = (const A*)a.proj;
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
            const size_t tok = (size_t)(run.tok0 + c0 + t);
            float q = 0.0f, k = 0.0f, gg = 0.0f;
            if (d < g.dim) {
                q = a.qk[tok * 2 * g.kv_heads * g.dim + kh * g.dim + d];
                k = a.qk[(tok * 2 + 1) * g.kv_heads * g.dim + kh * g.dim + d];
                gg = expf(a.log_decay[tok * g.heads * g.dim + h * g.dim + d]);
            }
            s_q[i] = q; s_k[i] = k; s_g[i] = gg;
        }
        for (int i = threadIdx.x; i < m * 32; i += 128) {
            const int t = i >> 5, c = blockIdx.z * 32 + (i & 31);
            s_v[i] = c < g.vdim ? a.v[(size_t)(run.tok0 + c0 + t) * g.heads * g.vdim + h * g.vdim + c] : 0.0f;
        }
        if (threadIdx.x < m) s_b[threadIdx.x] = sigmoid_f(act_f<A>(proj[(size_t)(run.tok0 + c0 + threadIdx.x) * g.ld + g.off_b + h]));
        __syncthreads();
        for (int t = 0; t < m; t++) {
            const float4 *q4 = (const float4*)(s_q + t * DP), *k4 = (const float4*)(s_k + t * DP), *g4 = (const float4*)(s_g + t * DP);
            float kk[DPL], dot = 0.0f;
#pragma unroll
            for (int i = 0; i < DPL / 4; i++) {
                const float4 kv = k4[i * 4 + r4], gv = g4[i * 4 + r4];
                kk[4 * i] = kv.x; kk[4 * i + 1] = kv.y; kk[4 * i + 2] = kv.z; kk[4 * i + 3] = kv.w;
                S[4 * i] *= gv.x; S[4 * i + 1] *= gv.y; S[4 * i + 2] *= gv.z; S[4 * i + 3] *= gv.w;
#pragma unroll
                for (int j = 0; j < 4; j++) dot = fmaf(S[4 * i + j], kk[4 * i + j], dot);
            }
            dot += __shfl_xor_sync(0xffffffffu, dot, 1);
            dot += __shfl_xor_sync(0xffffffffu, dot, 2);
            const float u = s_b[t] * (s_v[t * 32 + col] - dot);
            float o = 0.0f;
#pragma unroll
            for (int i = 0; i < DPL / 4; i++) {
                const float4 qv = q4[i * 4 + r4];
                const float qq[4] = {qv.x, qv.y, qv.z, qv.w};
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    S[4 * i + j] = fmaf(kk[4 * i + j], u, S[4 * i + j]);
                    o = fmaf(S[4 * i + j], qq[j], o);
                }
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (r4 == 0 && e < g.vdim) a.o[(size_t)(run.tok0 + c0 + t) * g.heads * g.vdim + h * g.vdim + e] = o;
        }
    }
#pragma unroll
    for (int i = 0; i < DPL; i++) {
        const int d = (i >> 2) * 16 + r4 * 4 + (i & 3);
        if (d < g.dim && e < g.vdim) st[(size_t)d * g.vdim + e] = S[i];
    }
    if (blockIdx.z == 0) delta_keep_inputs<A>(a, run, h, threadIdx.x, 128);
}

__device__ __forceinline__ int head_norm_row(const HeadNormArgs& a) {
    if (!a.runs) return blockIdx.x;
    const SeqRun r = a.runs[blockIdx.x / a.longest];
    const int i = blockIdx.x % a.longest;
    return i < r.n ? r.tok0 + i : -1;
}
// G lanes per (token, head), four elements each: heads of up to 4 G elements, a multiple of four
template <typename A, int G>
__global__ void __launch_bounds__(256) head_norm4_kernel(const HeadNormArgs a) {
    constexpr int kItems = 2, kPer = 256 / G;  // heads per group of lanes
    pdl_launch_dependents();
    pdl_wait();
    const int row = head_norm_row(a);
    if (row < 0) return;
    const size_t t = row;
    const int group = threadIdx.x / G, c = (threadIdx.x % G) * 4;
    float4 o[kItems], gate[kItems], w[kItems];
#pragma unroll
    for (int i = 0; i < kItems; i++) {
        const int h = blockIdx.y * kPer * kItems + i * kPer + group;
        o[i] = gate[i] = w[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (h < a.heads && c < a.n) {
            o[i] = *(const float4*)(a.o + (t * a.heads + h) * a.n + c);
            gate[i] = load4<A>((const A*)a.gate + t * a.ld_gate + (size_t)h * a.n + c);
            w[i] = *(const float4*)(a.w + (size_t)h * a.w_stride + c);
        }
    }
#pragma unroll
    for (int i = 0; i < kItems; i++) {
        const int h = blockIdx.y * kPer * kItems + i * kPer + group;
        float ss = sq4(o[i], 0.0f);
#pragma unroll
        for (int m = 1; m < G; m *= 2) ss += __shfl_xor_sync(0xffffffffu, ss, m);
        const float r = 1.0f / sqrtf(ss / (float)a.n + a.eps);
        if (h < a.heads && c < a.n)
            store4<A>((A*)a.out + t * a.ldo + (size_t)h * a.n + c, make_float4(o[i].x * r * w[i].x * sigmoid_f(gate[i].x), o[i].y * r * w[i].y * sigmoid_f(gate[i].y),
                                                                              o[i].z * r * w[i].z * sigmoid_f(gate[i].z), o[i].w * r * w[i].w * sigmoid_f(gate[i].w)));
    }
}
// One warp per (token, head)
template <typename A>
__global__ void __launch_bounds__(256) head_norm_kernel(const HeadNormArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = head_norm_row(a), h = blockIdx.y * 8 + warp_index(), lane = threadIdx.x & 31;
    if (t < 0 || h >= a.heads) return;
    const float *o = a.o + ((size_t)t * a.heads + h) * a.n, *w = a.w + (size_t)h * a.w_stride;
    const A* gate = (const A*)a.gate + (size_t)t * a.ld_gate + (size_t)h * a.n;
    float ss = 0.0f;
    for (int i = lane; i < a.n; i += 32) ss = fmaf(o[i], o[i], ss);
    ss = warp_sum(ss);
    const float r = 1.0f / sqrtf(ss / (float)a.n + a.eps);
    A* dst = (A*)a.out + (size_t)t * a.ldo + h * a.n;
    for (int i = lane; i < a.n; i += 32) dst[i] = to_act<A>(o[i] * r * w[i] * sigmoid_f(act_f<A>(gate[i])));
}

// One new token of every sequence: convolutions, unit vectors, recurrence, norm and gate of one head of one token per CTA.
// With G = diag(g):  dot = (G S)^T k,  u = beta (v - dot),  S' = G S + k u^T,  o = S'^T q = (G S)^T q + u (k . q), so the state
// is walked once; a thread owns VEC neighbouring value columns and every `groups`-th key row, kept in registers (ROWS of
// them; 0: re-read for the update).  The ring entry written here is not one that any head reads in this step.
template <typename A, int VEC, int ROWS, int THREADS>
__global__ void __launch_bounds__(THREADS) delta_step_kernel(const DeltaArgs a) {
    extern __shared__ float sm[];
    __shared__ float red[32], s_norm[3];
    pdl_launch_dependents();
    pdl_wait();
    const DeltaShape& g = a.g;
    const int h = blockIdx.x, t = blockIdx.y, rep = g.heads / g.kv_heads, kh = h / rep, seq = a.tok_seq[t], pos = a.tok_pos[t];
    const int cols = g.vdim / VEC, groups = THREADS / cols;
    float *s_q = sm, *s_k = s_q + g.dim, *s_g = s_k + g.dim, *s_v = s_g + g.dim, *s_dk = s_v + g.vdim, *s_dq = s_dk + groups * g.vdim;
    const A* proj = (const A*)a.proj + (size_t)t * g.ld;
    A* ring = (A*)a.ring + (size_t)seq * g.taps * g.channels;
    const int c = threadIdx.x % cols, gr = threadIdx.x / cols;
    float* st = a.state + ((size_t)seq * g.heads + h) * g.dim * g.vdim + c * VEC;
    const bool live = pos > 0, mine = gr < groups;
    float S[ROWS > 0 ? ROWS : 1][VEC];
    if (ROWS > 0 && mine) {  // the state's reads travel while the convolutions run
#pragma unroll
        for (int i = 0; i < ROWS; i++) {
            const int d = gr + i * groups;
#pragma unroll
            for (int j = 0; j < VEC; j++) S[i][j] = 0.0f;
            if (d < g.dim && live) {
                if constexpr (VEC == 4) { const float4 v = *(const float4*)(st + (size_t)d * g.vdim); S[i][0] = v.x; S[i][1] = v.y; S[i][2] = v.z; S[i][3] = v.w; }
                else S[i][0] = st[(size_t)d * g.vdim];
            }
        }
    }
    // what the later phases need travels with the state
    constexpr int kHold = 2;
    const A* gate = (const A*)a.gate + ((size_t)t * g.heads + h) * g.vdim;
    float gate_r[kHold], norm_r[kHold], decay_r[kHold];
#pragma unroll
    for (int i = 0; i < kHold; i++) {
        const int e = threadIdx.x + i * THREADS;
        gate_r[i] = e < g.vdim ? act_f<A>(gate[e]) : 0.0f;
        norm_r[i] = e < g.vdim ? a.norm_w[e] : 0.0f;
        decay_r[i] = e < g.dim ? a.log_decay[(size_t)t * g.heads * g.dim + h * g.dim + e] : 0.0f;
    }
    const float beta_in = act_f<A>(proj[g.off_b + h]);
    const int now = pos % g.taps;
    for (int i = threadIdx.x; i < 2 * g.dim + g.vdim; i += THREADS) {
        int column, channel;
        bool owner = true;
        float* dst;
        if (i < 2 * g.dim) {
            const bool is_k = i >= g.dim;
            const int d = is_k ? i - g.dim : i;
            column = (is_k ? g.off_k : 0) + kh * g.dim + d;
            channel = (is_k ? g.kv_heads * g.dim : 0) + kh * g.dim + d;
            owner = h % rep == 0;
            dst = (is_k ? s_k : s_q) + d;
        } else {
            const int d = i - 2 * g.dim;
            column = g.off_v + h * g.vdim + d;
            channel = 2 * g.kv_heads * g.dim + h * g.vdim + d;
            dst = s_v + d;
        }
        const A cur = proj[column];
        float acc = 0.0f;
        for (int j = g.taps - 1; j > 0; j--)
            if (pos - j >= 0) acc = fmaf(a.conv[channel * g.taps + g.taps - 1 - j], act_f<A>(ring[(size_t)((pos - j) % g.taps) * g.channels + channel]), acc);
        acc = fmaf(a.conv[channel * g.taps + g.taps - 1], act_f<A>(cur), acc);
        *dst = silu32(acc);
        if (owner) ring[(size_t)now * g.channels + channel] = cur;
    }
#pragma unroll
    for (int i = 0; i < kHold; i++)
        if (threadIdx.x + i * THREADS < g.dim) s_g[threadIdx.x + i * THREADS] = expf(decay_r[i]);
    __syncthreads();
    if (threadIdx.x < 96) {  // |q|^2, |k|^2, q . k
        const int w = threadIdx.x >> 5, lane = threadIdx.x & 31;
        const float *x = w == 1 ? s_k : s_q, *y = w == 0 ? s_q : s_k;
        float v = 0.0f;
        for (int d = lane; d < g.dim; d += 32) v = fmaf(x[d], y[d], v);
        v = warp_sum(v);
        if (lane == 0) s_norm[w] = v;
    }
    __syncthreads();
    const float rq = 1.0f / sqrtf(s_norm[0] + g.unit_eps) * (1.0f / sqrtf((float)g.dim)), rk = 1.0f / sqrtf(s_norm[1] + g.unit_eps), qk = s_norm[2] * rq * rk;
    const float beta = sigmoid_f(beta_in);
    float dk[VEC], dq[VEC];
#pragma unroll
    for (int j = 0; j < VEC; j++) dk[j] = dq[j] = 0.0f;
    auto load = [&](int d, float (&v)[VEC]) {
#pragma unroll
        for (int j = 0; j < VEC; j++) v[j] = live ? st[(size_t)d * g.vdim + j] : 0.0f;
    };
    if (mine) {
        if constexpr (ROWS > 0) {
#pragma unroll
            for (int i = 0; i < ROWS; i++) {
                const int d = gr + i * groups;
                if (d < g.dim) {
                    const float gg = s_g[d], k = s_k[d] * rk, q = s_q[d] * rq;
#pragma unroll
                    for (int j = 0; j < VEC; j++) { S[i][j] *= gg; dk[j] = fmaf(S[i][j], k, dk[j]); dq[j] = fmaf(S[i][j], q, dq[j]); }
                }
            }
        } else {
            for (int d = gr; d < g.dim; d += groups) {
                const float gg = s_g[d], k = s_k[d] * rk, q = s_q[d] * rq;
                float v[VEC];
                load(d, v);
#pragma unroll
                for (int j = 0; j < VEC; j++) { v[j] *= gg; dk[j] = fmaf(v[j], k, dk[j]); dq[j] = fmaf(v[j], q, dq[j]); }
            }
        }
#pragma unroll
        for (int j = 0; j < VEC; j++) { s_dk[gr * g.vdim + c * VEC + j] = dk[j]; s_dq[gr * g.vdim + c * VEC + j] = dq[j]; }
    }
    __syncthreads();
    float ss = 0.0f;
    for (int e = threadIdx.x; e < g.vdim; e += THREADS) {  // u replaces v, the read-out replaces the first partial row
        float sk = 0.0f, sq = 0.0f;
        for (int i = 0; i < groups; i++) { sk += s_dk[i * g.vdim + e]; sq += s_dq[i * g.vdim + e]; }
        const float u = beta * (s_v[e] - sk), o = fmaf(u, qk, sq);
        s_v[e] = u;
        s_dq[e] = o;
        ss = fmaf(o, o, ss);
    }
    ss = block_sum(ss, red);  // also publishes u and o
    if (mine) {
        float u[VEC];
#pragma unroll
        for (int j = 0; j < VEC; j++) u[j] = s_v[c * VEC + j];
        if constexpr (ROWS > 0) {
#pragma unroll
            for (int i = 0; i < ROWS; i++) {
                const int d = gr + i * groups;
                if (d < g.dim) {
                    const float k = s_k[d] * rk;
#pragma unroll
                    for (int j = 0; j < VEC; j++) S[i][j] = fmaf(k, u[j], S[i][j]);
                    if constexpr (VEC == 4) *(float4*)(st + (size_t)d * g.vdim) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
                    else st[(size_t)d * g.vdim] = S[i][0];
                }
            }
        } else {
            for (int d = gr; d < g.dim; d += groups) {
                float v[VEC];
                load(d, v);
#pragma unroll
                for (int j = 0; j < VEC; j++) st[(size_t)d * g.vdim + j] = fmaf(s_k[d] * rk, u[j], v[j] * s_g[d]);
            }
        }
    }
    const float r = 1.0f / sqrtf(ss / (float)g.vdim + g.eps);
    A* dst = (A*)a.out + (size_t)t * a.ldo + h * g.vdim;
#pragma unroll
    for (int i = 0; i < kHold; i++) {
        const int e = threadIdx.x + i * THREADS;
        if (e < g.vdim) dst[e] = to_act<A>(s_dq[e] * r * norm_r[i] * sigmoid_f(gate_r[i]));
    }
}

// ---- latent attention: norms of the two latents, rotation of the shared key part, cache append -------------------------------
__global__ void rot_table_kernel(const double* __restrict__ freq, int pairs, double magnitude, int positions, float2* __restrict__ out) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= positions * pairs) return;
    const int p = i / pairs;
    double s, c;
    sincos((double)p * freq[i - p * pairs], &s, &c);
    out[i] = make_float2((float)(c * magnitude), (float)(s * magnitude));
}

template <typename A>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentArgs a) {
    __shared__ float sh[32], sh2[32];
    pdl_launch_dependents();
    pdl_wait();
    const LatentShape& g = a.g;
    const int t = blockIdx.x, seq = a.tok_seq[t], pos = a.tok_pos[t];
    const float* p = a.proj + (size_t)t * a.ld_proj;
    const float* c = p + a.off_c;
    float sq = 0.0f, sc = 0.0f;
#pragma unroll 4
    for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x) sq = fmaf(p[i], p[i], sq);
#pragma unroll 4
    for (int i = threadIdx.x; i < g.rank; i += blockDim.x) sc = fmaf(c[i], c[i], sc);
    const int page = a.page_table[(size_t)seq * a.pages_per_seq + pos / a.page_tokens];
    sq = block_sum(sq, sh);
    sc = block_sum(sc, sh2);
    const float rq = 1.0f / sqrtf(sq / (float)a.q_rank + a.eps), r = 1.0f / sqrtf(sc / (float)g.rank + a.eps);
    A* cq = (A*)a.cq + (size_t)t * a.ld_cq;
#pragma unroll 4
    for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x) cq[i] = to_act<A>(p[i] * rq * a.q_norm[i]);
    A* row = (A*)a.cache + ((size_t)page * a.page_tokens + pos % a.page_tokens) * (g.cp + g.rp);
    for (int i = threadIdx.x; i < g.cp; i += blockDim.x) row[i] = to_act<A>(i < g.rank ? c[i] * r * a.c_norm[i] : 0.0f);
    const float* kr = p + a.off_r;
    for (int i = threadIdx.x; i < g.rp; i += blockDim.x) {
        float v = i < g.rot ? kr[i] : 0.0f;
        if (i < 2 * g.rot_pairs) {
            const float2 cs = a.rot[(size_t)pos * g.rot_pairs + i / 2];
            const float u = kr[i & ~1], w = kr[i | 1];
            v = (i & 1) ? w * cs.x + u * cs.y : u * cs.x - w * cs.y;
        }
        row[g.cp + i] = to_act<A>(v);
    }
}

int norm_threads(int width) { return width >= 4096 ? 512 : width >= 1024 ? 256 : 128; }

template <typename A>
int32_t prep_dispatch(const DeltaArgs& a, cudaStream_t s) {
    const dim3 grid((unsigned)((a.T + kPrepTok - 1) / kPrepTok), (unsigned)((2 * a.g.kv_heads + a.g.heads + 7) / 8));
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(launch_pdl(kern, grid, dim3(256), 0, s, a));
        return LC_OK;
    };
    const int widest = std::max(a.g.dim, a.g.vdim);
    LC_CHECK(widest <= 512, LC_ERR_UNSUPPORTED, "delta rule: %d dimensions per head", widest);
    if (widest > 128) return go(delta_prep_kernel<A, 0, 16>);
    switch (a.g.taps) {
        case 2: return go(delta_prep_kernel<A, 2, 4>);
        case 3: return go(delta_prep_kernel<A, 3, 4>);
        case 4: return go(delta_prep_kernel<A, 4, 4>);
        default: return go(delta_prep_kernel<A, 0, 4>);
    }
}

template <typename A>
int32_t scan_dispatch(const DeltaArgs& a, cudaStream_t s) {
    const dim3 grid((unsigned)a.n_runs, (unsigned)a.g.heads, (unsigned)((a.g.vdim + 31) / 32));
    const int dpl = a.g.dim <= 32 ? 8 : a.g.dim <= 64 ? 16 : a.g.dim <= 128 ? 32 : 64;
    const size_t smem = (size_t)kScanTok * (3 * 4 * dpl + 32 + 1) * sizeof(float);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3(128), smem, s, a));
        return LC_OK;
    };
    switch (dpl) {
        case 8: return go(delta_scan_kernel<A, 8>);
        case 16: return go(delta_scan_kernel<A, 16>);
        case 32: return go(delta_scan_kernel<A, 32>);
        default: return go(delta_scan_kernel<A, 64>);
    }
}

template <typename A>
int32_t step_dispatch(const DeltaArgs& a, cudaStream_t s) {
    const int vec = a.g.vdim % 4 == 0 ? 4 : 1, cols = a.g.vdim / vec, threads = vec == 4 && a.g.dim * a.g.vdim >= 8192 ? 512 : 256;
    LC_CHECK(cols <= threads && a.g.vdim <= 512, LC_ERR_UNSUPPORTED, "delta rule: %d value dimensions per head", a.g.vdim);
    const int groups = threads / cols, rows = (a.g.dim + groups - 1) / groups;
    const size_t smem = (size_t)(3 * a.g.dim + a.g.vdim + 2 * groups * a.g.vdim) * sizeof(float);
    const dim3 grid((unsigned)a.g.heads, (unsigned)a.T);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(ensure_smem_limit((const void*)kern, smem));
        LC_CUDA(launch_pdl(kern, grid, dim3((unsigned)threads), smem, s, a));
        return LC_OK;
    };
    if (threads == 512) return rows <= 4 ? go(delta_step_kernel<A, 4, 4, 512>) : rows <= 8 ? go(delta_step_kernel<A, 4, 8, 512>) : go(delta_step_kernel<A, 4, 0, 512>);
    if (vec == 4) return rows <= 4 ? go(delta_step_kernel<A, 4, 4, 256>) : rows <= 16 ? go(delta_step_kernel<A, 4, 16, 256>) : go(delta_step_kernel<A, 4, 0, 256>);
    return rows <= 16 ? go(delta_step_kernel<A, 1, 16, 256>) : go(delta_step_kernel<A, 1, 0, 256>);
}

}  // namespace

int32_t launch_pack(const __nv_bfloat16* src, int rows, int cols, __nv_bfloat16* dst, int ld, PackMap row, PackMap col, bool transpose, cudaStream_t s) {
    const size_t n = (size_t)rows * cols, blocks = (n + 255) / 256;
    pack_kernel<<<(unsigned)std::min<size_t>(blocks, (size_t)sm_count() * 16), 256, 0, s>>>(src, rows, cols, dst, ld, row, col, transpose ? 1 : 0);
    LC_CUDA(cudaGetLastError());
    return LC_OK;
}
int32_t launch_embed_rows(const EmbedArgs& a, cudaStream_t s) {
    const dim3 grid((unsigned)a.T), block(256);
    auto go = [&](auto kern) -> int32_t {
        LC_CUDA(launch_pdl(kern, grid, dim3(a.T <= sm_count() ? 512 : 256), 0, s, a));
        return LC_OK;
    };
    const bool vec = a.width % 8 == 0 && a.ld_act % 8 == 0;
    if (a.pair.table) {
        if (a.f32) return vec ? go(embed_norm_kernel<float, true, 8>) : go(embed_norm_kernel<float, true, 1>);
        return vec ? go(embed_norm_kernel<bf16, true, 8>) : go(embed_norm_kernel<bf16, true, 1>);
    }
    if (a.scale == 1.0f && !a.w && !a.copy && !(a.f32 && a.act)) {
        LC_CUDA(launch_pdl(embed_rows_kernel, grid, block, 0, s, a.table, a.rows, a.width, a.ids, a.x, (bf16*)a.act, a.ld_act));
        return LC_OK;
    }
    if (a.f32) return vec ? go(embed_norm_kernel<float, false, 8>) : go(embed_norm_kernel<float, false, 1>);
    return vec ? go(embed_norm_kernel<bf16, false, 8>) : go(embed_norm_kernel<bf16, false, 1>);
}
int32_t launch_keep_tokens(const SeqRun* runs, int n_runs, const int64_t* ids, int32_t* last, cudaStream_t s) {
    LC_CUDA(launch_pdl(keep_tokens_kernel, dim3((unsigned)((n_runs + 127) / 128)), dim3(128), 0, s, runs, n_runs, ids, last));
    return LC_OK;
}
int32_t launch_act_rows(const float* x, int width, int T, void* act, int ld_act, cudaStream_t s) {
    LC_CUDA(launch_pdl(act_rows_kernel, dim3((unsigned)T), dim3(256), 0, s, x, width, (__nv_bfloat16*)act, ld_act));
    return LC_OK;
}
int32_t launch_residual(const ResidualArgs& a, cudaStream_t s) {
    const dim3 grid((unsigned)a.T), block((unsigned)norm_threads(a.width));
    const bool moe = a.moe.rows != nullptr, pair = a.pair.y2 != nullptr;
    const bool vec = a.width % 4 == 0 && ((uintptr_t)a.pair.w0 | (uintptr_t)a.pair.w1) % 16 == 0 && (uintptr_t)a.w % 16 == 0 && (uintptr_t)a.w_next % 16 == 0 && (a.moe.ld_rows | a.moe.ld_h | a.ld_act) % 4 == 0;
    LC_CHECK(a.moe.top <= kMaxChoices && (!a.w_next || a.act), LC_ERR_INVALID, "residual sum: bad argument");
    auto go = [&](auto kern, unsigned threads = 0) -> int32_t {
        LC_CUDA(launch_pdl(kern, grid, threads ? dim3(threads) : block, 0, s, a));
        return LC_OK;
    };
    if (!a.w && a.x) {
        LC_CHECK(!moe && !pair, LC_ERR_UNSUPPORTED, "residual sum: a mixture or a pair without an output norm");
        const bool deep = a.depth.keep != nullptr;
        // few rows: a row by twice the threads
        auto plain = [&](auto act) -> int32_t {
            typedef decltype(act) A;
            const bool wide = vec && a.T <= sm_count() && a.width >= 4096;
            if (deep) return wide ? go(plain_residual_kernel<A, 4, true, 1024>, 1024) : vec ? go(plain_residual_kernel<A, 4, true, 512>) : go(plain_residual_kernel<A, 1, true, 512>);
            return wide ? go(plain_residual_kernel<A, 4, false, 1024>, 1024) : vec ? go(plain_residual_kernel<A, 4, false, 512>) : go(plain_residual_kernel<A, 1, false, 512>);
        };
        return a.f32 ? plain(0.0f) : plain(bf16());
    }
    LC_CHECK(!a.depth.keep, LC_ERR_UNSUPPORTED, "residual sum: a sum over depth behind an output norm");
    if (a.f32) {
        if (moe) return vec ? go(residual_kernel<float, 4, true, false>) : go(residual_kernel<float, 1, true, false>);
        if (pair) return vec ? go(residual_kernel<float, 4, false, true>) : go(residual_kernel<float, 1, false, true>);
        return vec ? go(residual_kernel<float, 4, false, false>) : go(residual_kernel<float, 1, false, false>);
    }
    if (moe) return vec ? go(residual_kernel<bf16, 4, true, false>) : go(residual_kernel<bf16, 1, true, false>);
    if (pair) return vec ? go(residual_kernel<bf16, 4, false, true>) : go(residual_kernel<bf16, 1, false, true>);
    return vec ? go(residual_kernel<bf16, 4, false, false>) : go(residual_kernel<bf16, 1, false, false>);
}
int32_t launch_norm_rows(const float* x, const int32_t* idx, const float* w, float eps, int width, int n, void* out, int ldo, bool f32, cudaStream_t s) {
    const dim3 grid((unsigned)n), block((unsigned)norm_threads(width));
    if (f32) LC_CUDA(launch_pdl(norm_rows_kernel<float>, grid, block, 0, s, x, idx, w, eps, width, (float*)out, ldo));
    else LC_CUDA(launch_pdl(norm_rows_kernel<__nv_bfloat16>, grid, block, 0, s, x, idx, w, eps, width, (__nv_bfloat16*)out, ldo));
    return LC_OK;
}
int32_t launch_delta_prep(const DeltaArgs& a, cudaStream_t s) {
    LC_CHECK(a.g.dim <= 256, LC_ERR_UNSUPPORTED, "delta rule: %d key dimensions per head (at most 256)", a.g.dim);
    return a.f32 ? prep_dispatch<float>(a, s) : prep_dispatch<__nv_bfloat16>(a, s);
}
int32_t launch_delta_scan(const DeltaArgs& a, cudaStream_t s) { return a.f32 ? scan_dispatch<float>(a, s) : scan_dispatch<__nv_bfloat16>(a, s); }
int32_t launch_delta_step(const DeltaArgs& a, cudaStream_t s) { return a.f32 ? step_dispatch<float>(a, s) : step_dispatch<__nv_bfloat16>(a, s); }
int32_t launch_head_norm(const HeadNormArgs& a, cudaStream_t s) {
    const bool vec = a.n % 4 == 0 && a.n <= 128 && (a.ld_gate | a.ldo | a.w_stride) % 4 == 0 && ((uintptr_t)a.w % 16) == 0 && ((uintptr_t)a.gate % 16) == 0;
    const unsigned rows = (unsigned)(a.runs ? a.n_runs * a.longest : a.T);
    if (vec) {
        const int lanes = a.n <= 32 ? 8 : a.n <= 64 ? 16 : 32, per = 256 / lanes * 2;
        auto go = [&](auto kern) -> int32_t {
            LC_CUDA(launch_pdl(kern, dim3(rows, (unsigned)((a.heads + per - 1) / per)), dim3(256), 0, s, a));
            return LC_OK;
        };
        if (a.f32) return lanes == 8 ? go(head_norm4_kernel<float, 8>) : lanes == 16 ? go(head_norm4_kernel<float, 16>) : go(head_norm4_kernel<float, 32>);
        return lanes == 8 ? go(head_norm4_kernel<bf16, 8>) : lanes == 16 ? go(head_norm4_kernel<bf16, 16>) : go(head_norm4_kernel<bf16, 32>);
    }
    const dim3 grid(rows, (unsigned)((a.heads + 7) / 8));
    if (a.f32) LC_CUDA(launch_pdl(head_norm_kernel<float>, grid, dim3(256), 0, s, a));
    else LC_CUDA(launch_pdl(head_norm_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, a));
    return LC_OK;
}
int32_t launch_latent_prep(const LatentArgs& a, cudaStream_t s) {
    if (a.f32) LC_CUDA(launch_pdl(latent_prep_kernel<float>, dim3((unsigned)a.T), dim3(256), 0, s, a));
    else LC_CUDA(launch_pdl(latent_prep_kernel<__nv_bfloat16>, dim3((unsigned)a.T), dim3(256), 0, s, a));
    return LC_OK;
}
int32_t launch_rot_table(const double* freq_dev, int pairs, double magnitude, int positions, float2* out, cudaStream_t s) {
    const size_t n = (size_t)pairs * positions;
    LC_CHECK(n < ((size_t)1 << 31), LC_ERR_UNSUPPORTED, "rotation table of %zu entries", n);
    rot_table_kernel<<<(unsigned)((n + 255) / 256), 256, 0, s>>>(freq_dev, pairs, magnitude, positions, out);
    LC_CUDA(cudaGetLastError());
    return LC_OK;
}

}  // namespace lc
