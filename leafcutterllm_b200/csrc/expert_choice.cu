// Routing of a mixture of experts with identity experts and group-limited choice (MoeSpec): from the router's logits to every
// token's choices and weights, the experts' token lists and the tiles of their grouped products.
//   s = softmax(z) over all outputs; choice score c = s + correction; the groups (equal runs of outputs) are ranked by their
//   largest c, the outputs of the best `keep` groups by c, the first `top` of them are chosen and weighted with s.
// One warp per token.  The CTA that finishes last (a ticket) turns the experts' counts into offsets and tiles.  The order of
// tokens inside a list is the order of arrival; nothing that is computed from a list depends on it.
#include <algorithm>
#include "lc_mixers.h"
#include "lc_tma.cuh"

namespace lc {

namespace {

constexpr int kWarps = 8;

__global__ void __launch_bounds__(32 * kWarps) expert_choice_kernel(const ChoiceArgs a) {
    extern __shared__ float sm[];
    __shared__ int s_last, s_scan[2][kWarps];
    pdl_launch_dependents();
    pdl_wait();
    const MoeSpec& m = a.m;
    const int n = m.experts + m.identity, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * kWarps + warp, per = n / m.groups;
    float *s = sm + (size_t)warp * (2 * n + m.groups), *c = s + n, *gs = c + n;
    if (t < a.T) {
        const float* z = a.z + (size_t)t * a.ld_z;
        float mx = -INFINITY, sum = 0.0f;
        for (int e = lane; e < n; e += 32) { const float v = z[e]; s[e] = v; mx = fmaxf(mx, v); }
        mx = warp_max(mx);
        for (int e = lane; e < n; e += 32) { const float v = expf(s[e] - mx); s[e] = v; sum += v; }
        sum = warp_sum(sum);
        for (int e = lane; e < n; e += 32) { const float v = s[e] / sum; s[e] = v; c[e] = v + a.correction[e]; }
        __syncwarp();
        if (m.keep < m.groups) {
            for (int g = lane; g < m.groups; g += 32) {
                float best = -INFINITY;
                for (int i = 0; i < per; i++) best = fmaxf(best, c[g * per + i]);
                gs[g] = best;
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
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float v = __shfl_xor_sync(0xffffffffu, best, o);
                const int i = __shfl_xor_sync(0xffffffffu, at, o);
                if (v > best || (v == best && i < at)) { best = v; at = i; }
            }
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
                pos = atomicAdd(a.counts + mine, 1);
                if (pos < a.plan.list_stride) a.plan.lists[(size_t)mine * a.plan.list_stride + pos] = t;
            }
            a.sel[i] = mine; a.pos[i] = pos; a.weight[i] = w;
        }
    }
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) s_last = atomicAdd((unsigned*)a.counts + m.experts, 1u) == gridDim.x - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    int rows = 0, tiles = 0;  // of the experts before this turn's
    unsigned long long used = 0;
    for (int e0 = 0; e0 < m.experts; e0 += 32 * kWarps) {
        const int e = e0 + threadIdx.x;
        const int cnt = e < m.experts ? __ldcg(a.counts + e) : 0, nt = (cnt + a.plan.tile_rows - 1) / a.plan.tile_rows;
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
            a.counts[e] = 0;
            used += cnt > 0;
        }
        rows += all_r; tiles += all_q;
        __syncthreads();
    }
    if (threadIdx.x == 0) {
        a.plan.off[m.experts] = rows;
        *a.plan.n_tiles = min(tiles, a.plan.most_tiles);
        a.counts[m.experts] = 0;
    }
    if (a.touched && used) atomicAdd(a.touched, used * a.touched_bytes);
}

}  // namespace

int32_t launch_expert_choice(const ChoiceArgs& a, cudaStream_t s) {
    const size_t smem = (size_t)kWarps * (2 * a.m.outputs() + a.m.groups) * sizeof(float);
    LC_CHECK(a.m.outputs() <= kMaxRouterOutputs && a.m.top <= kMaxChoices && a.T >= 1 && a.T <= a.plan.list_stride, LC_ERR_INVALID, "expert choice: bad argument");
    LC_CUDA(ensure_smem_limit((const void*)expert_choice_kernel, smem));
    LC_CUDA(launch_pdl(expert_choice_kernel, dim3((unsigned)((a.T + kWarps - 1) / kWarps)), dim3(32 * kWarps), smem, s, a));
    return LC_OK;
}

}  // namespace lc
