// Routing of a mixture of experts with identity experts and group-limited choice (MoeSpec): from the router's logits to every
// token's choices and weights, the experts' token lists and the tiles of their grouped products.
//   s = softmax(z) over all outputs, or the sigmoid of each; choice score c = s + correction; the groups (equal runs of outputs)
//   are ranked by their largest c or the sum of their two largest, the outputs of the best `keep` groups by c, the first `top` of
//   them are chosen and weighted with s.
// One warp per token.  The CTA that finishes last (a ticket) turns the experts' counts into offsets and tiles.  The order of
// tokens inside a list is the order of arrival; nothing that is computed from a list depends on it.
#include <algorithm>
#include "lc_mixers.h"
#include "lc_tma.cuh"

namespace lc {

namespace {

constexpr int kWarps = 8;

// A float as an unsigned number of the same order.
__device__ __forceinline__ unsigned order_key(float v) {
    const unsigned b = __float_as_uint(v);
    return b & 0x80000000u ? ~b : b | 0x80000000u;
}

__global__ void __launch_bounds__(32 * kWarps) expert_choice_kernel(const ChoiceArgs a) {
    extern __shared__ float sm[];
    __shared__ int s_last, s_scan[2][kWarps];
    pdl_launch_dependents();
    pdl_wait();
    const MoeSpec& m = a.m;
    const bool solo = gridDim.x == 1;  // one CTA counts in shared memory and needs no ticket
    int32_t* counts = solo ? (int32_t*)(sm + kWarps * (2 * (m.experts + m.identity) + m.groups)) : a.counts;
    if (solo) {
        for (int e = threadIdx.x; e < m.experts; e += 32 * kWarps) counts[e] = 0;
        __syncthreads();
    }
    const int n = m.experts + m.identity, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * kWarps + warp, per = n / m.groups;
    float *s = sm + (size_t)warp * (2 * n + m.groups), *c = s + n, *gs = c + n;
    if (t < a.T) {
        const float* z = a.z + (size_t)t * a.ld_z;
        float mx = -INFINITY, sum = 0.0f;
        if (m.score == RouterScore::Sigmoid) {
            for (int e = lane; e < n; e += 32) { const float v = 1.0f / (1.0f + expf(-z[e])); s[e] = v; c[e] = v + a.correction[e]; }
        } else {
            for (int e = lane; e < n; e += 32) { const float v = z[e]; s[e] = v; mx = fmaxf(mx, v); }
            mx = warp_max(mx);
            for (int e = lane; e < n; e += 32) { const float v = expf(s[e] - mx); s[e] = v; sum += v; }
            sum = warp_sum(sum);
            for (int e = lane; e < n; e += 32) { const float v = s[e] / sum; s[e] = v; c[e] = v + a.correction[e]; }
        }
        __syncwarp();
        if (m.keep < m.groups) {
            for (int g = lane; g < m.groups; g += 32) {
                float best = -INFINITY, second = -INFINITY;
                for (int i = 0; i < per; i++) {
                    const float v = c[g * per + i];
                    second = fmaxf(second, fminf(best, v));
                    best = fmaxf(best, v);
                }
                gs[g] = m.group_top == 2 && per > 1 ? best + second : best;
            }
            __syncwarp();
            for (int g = lane; g < m.groups; g += 32) {
                const float mine = gs[g];
                int before = 0;  // groups ranked before this one, equal scores in index order
                for (int i = 0; i < m.groups; i++) before += gs[i] > mine || (gs[i] == mine && i < g);
                if (before >= m.keep)
                    for (int i = 0; i < per; i++) c[g * per + i] = -INFINITY;
            }
            __syncwarp();
        }
        int mine = 0;
        float w = 0.0f;
        for (int j = 0; j < m.top; j++) {
            float best = -INFINITY;
            int at = n;
            for (int e = lane; e < n; e += 32)
                if (c[e] > best) { best = c[e]; at = e; }
            const unsigned top = __reduce_max_sync(0xffffffffu, order_key(best));
            at = (int)__reduce_min_sync(0xffffffffu, order_key(best) == top ? (unsigned)at : (unsigned)n);
            if (at >= n) at = j;  // no comparable score (not a number): any valid index
            __syncwarp();
            if (lane == 0) c[at] = -INFINITY;
            if (lane == j) { mine = at; w = s[at]; }
            __syncwarp();
        }
        if (lane < m.top) {
            const size_t i = (size_t)t * m.top + lane;
            int pos = -1;
            if (mine < m.experts) {
                pos = atomicAdd(counts + mine, 1);
                if (pos < a.plan.list_stride) a.plan.lists[(size_t)mine * a.plan.list_stride + pos] = t;
            }
            a.sel[i] = mine; a.pos[i] = pos; a.weight[i] = w;
        }
    }
    if (!solo) __threadfence();
    __syncthreads();
    if (!solo) {
        if (threadIdx.x == 0) s_last = atomicAdd((unsigned*)a.counts + m.experts, 1u) == gridDim.x - 1;
        __syncthreads();
        if (!s_last) return;
        __threadfence();
    }
    int rows = 0, tiles = 0;  // of the experts before this turn's
    unsigned long long used = 0;
    for (int e0 = 0; e0 < m.experts; e0 += 32 * kWarps) {
        const int e = e0 + threadIdx.x;
        const int cnt = e >= m.experts ? 0 : solo ? counts[e] : __ldcg(a.counts + e), nt = (cnt + a.plan.tile_rows - 1) / a.plan.tile_rows;
        int r = cnt, q = nt;  // inclusive sums over the CTA
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int r2 = __shfl_up_sync(0xffffffffu, r, o), q2 = __shfl_up_sync(0xffffffffu, q, o);
            if (lane >= o) { r += r2; q += q2; }
        }
        if (lane == 31) { s_scan[0][warp] = r; s_scan[1][warp] = q; }
        __syncthreads();
        int all_r = 0, all_q = 0;
        for (int i = 0; i < kWarps; i++) {
            if (i < warp) { r += s_scan[0][i]; q += s_scan[1][i]; }
            all_r += s_scan[0][i]; all_q += s_scan[1][i];
        }
        if (e < m.experts) {
            const int row0 = rows + r - cnt, tile0 = tiles + q - nt;
            a.plan.off[e] = row0;
            const int each = nt > 0 ? ((cnt + nt - 1) / nt + 15) & ~15 : 0;
            for (int i = 0, at = 0; i < nt; i++, at += each)
                if (tile0 + i < a.plan.most_tiles) {
                    const int take = max(0, min(each, cnt - at));
                    a.plan.tiles[tile0 + i] = ExpertTile{e, at, take, row0 + at};
                }
            if (!solo) a.counts[e] = 0;
            used += cnt > 0;
        }
        rows += all_r; tiles += all_q;
        __syncthreads();
    }
    if (threadIdx.x == 0) {
        a.plan.off[m.experts] = rows;
        *a.plan.n_tiles = min(tiles, a.plan.most_tiles);
        if (!solo) a.counts[m.experts] = 0;
    }
    if (a.touched && used) atomicAdd(a.touched, used * a.touched_bytes);
}

// One CTA per token: its row is read once and written to every expert's place.
__global__ void __launch_bounds__(256) expert_gather_kernel(const MoeSum m, int chunks, uint4* __restrict__ out, int ld16) {
    __shared__ int s_row[kMaxChoices];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    if ((int)threadIdx.x < m.top) {
        const size_t i = t * m.top + threadIdx.x;
        const int e = m.sel[i];
        s_row[threadIdx.x] = e < m.experts ? m.off[e] + m.pos[i] : -1;
    }
    __syncthreads();
    const uint4* h = (const uint4*)((const __nv_bfloat16*)m.h + t * m.ld_h);
    for (int c = threadIdx.x; c < chunks; c += 256) {
        const uint4 v = h[c];
        for (int j = 0; j < m.top; j++)
            if (s_row[j] >= 0) out[(size_t)s_row[j] * ld16 + c] = v;
    }
}

}  // namespace

int32_t launch_expert_gather(const MoeSum& m, int width, int T, void* out, int ldo, cudaStream_t s) {
    LC_CHECK(m.ld_h % 8 == 0 && ldo % 8 == 0 && m.top <= kMaxChoices, LC_ERR_INVALID, "expert gather: layout");
    LC_CUDA(launch_pdl(expert_gather_kernel, dim3((unsigned)T), dim3(256), 0, s, m, (width + 7) / 8, (uint4*)out, ldo / 8));
    return LC_OK;
}

int32_t launch_expert_choice(const ChoiceArgs& a, cudaStream_t s) {
    const size_t smem = ((size_t)kWarps * (2 * a.m.outputs() + a.m.groups) + a.m.experts) * sizeof(float);
    LC_CHECK(a.m.outputs() <= kMaxRouterOutputs && a.m.top <= kMaxChoices && a.T >= 1 && a.T <= a.plan.list_stride, LC_ERR_INVALID, "expert choice: bad argument");
    LC_CUDA(ensure_smem_limit((const void*)expert_choice_kernel, smem));
    LC_CUDA(launch_pdl(expert_choice_kernel, dim3((unsigned)((a.T + kWarps - 1) / kWarps)), dim3(32 * kWarps), smem, s, a));
    return LC_OK;
}

}  // namespace lc
