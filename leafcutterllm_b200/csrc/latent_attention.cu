// Latent attention: every head's key is the projection of ONE cached latent per token (plus a rotated part all heads share) and
// its value another projection of the same latent.  The key projection is moved onto the query and the value projection behind
// the weighted sum, so the kernels here attend with `heads` queries per token over rows [latent | rotated part] of the paged
// cache and return, per head, the weighted sum of latents.
#include <cmath>
#include "lc_mixers.h"
#include "lc_tma.cuh"

namespace lc {

namespace {

template <typename A> __device__ __forceinline__ float act_f(A v);
template <> __device__ __forceinline__ float act_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float act_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename A> __device__ __forceinline__ A to_act(float v);
template <> __device__ __forceinline__ float to_act<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 to_act<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

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

}  // namespace

int32_t launch_latent_attention(const LatentArgs& a, cudaStream_t s) {
    const size_t smem = (size_t)(2 * a.g.cp + a.g.rp + 2 * kPlainThreads) * 4;
    LC_CHECK(smem <= 100 * 1024, LC_ERR_UNSUPPORTED, "latent attention: rank %d", a.g.rank);
    const dim3 grid((unsigned)a.g.heads, (unsigned)a.T);
    if (a.f32) {
        LC_CUDA(ensure_smem_limit((const void*)latent_attention_plain_kernel<float>, smem));
        LC_CUDA(launch_pdl(latent_attention_plain_kernel<float>, grid, dim3(kPlainThreads), smem, s, a));
    } else {
        LC_CUDA(ensure_smem_limit((const void*)latent_attention_plain_kernel<__nv_bfloat16>, smem));
        LC_CUDA(launch_pdl(latent_attention_plain_kernel<__nv_bfloat16>, grid, dim3(kPlainThreads), smem, s, a));
    }
    return LC_OK;
}

}  // namespace lc
