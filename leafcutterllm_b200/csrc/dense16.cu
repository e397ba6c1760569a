// Products over bf16 weight matrices, y[t, r] = sum_k x[t, k] w[r, k], for any number of tokens.
//
// bf16 activations: dense_umma_kernel, tcgen05.mma kind::f16 with f32 accumulators in tensor memory.  The WEIGHT rows are the
// M of the instruction (128 per tile) and the tokens its N (16 .. 256), so the same kernel streams the weights of a
// one-token decode step at memory speed and multiplies prefill chunks at tensor-core speed:
//   warp 0   one thread fills a ring of stages: per 64 elements of k one bulk copy of a 128-row weight block, which lies
//            contiguous and ready swizzled in memory, and one TMA box of N tokens (128-byte swizzle); the first weight
//            blocks leave before the kernel waits for its predecessor;
//   warp 1   one thread issues the products of a stage (four K = 16 steps) and commits them to the stage's "empty" barrier;
//   warps 4-11  read finished accumulators (two sets, so the next tile's products overlap), apply the epilogue and store;
//            lane = weight row, so a warp's store of one token is contiguous.
// Few tiles: k is cut into shares over several CTAs; each leaves its partial tile in scratch and takes a ticket, the last one
// adds the shares in share order (the result does not depend on which CTA that is) and runs the epilogue.
// Grouped form (one matrix per expert): the tokens come as tiles of rows that share a matrix, found on the device.  Their
// activations come in boxes of rows, or are gathered four rows at a time (TMA gather); the instruction's N follows the tile's rows.
// Work items are dealt round robin to a grid of at most one CTA per SM.  Every wait is bounded: one that runs out raises the
// library's device error flag and the CTA winds down (copies awaited, tensor memory freed).
//
// f32 activations: dense_f32_kernel, plain f32 FMAs (64 x 64 tiles), for models that run in true 32-bit.
#include <cstdlib>
#include "lc_mixers.h"
#include "lc_tma.cuh"
#include "lc_umma.cuh"

namespace lc {

namespace {

constexpr int kM = 128;          // weight rows per tile
constexpr int kKB = 64;          // elements of k per stage
constexpr int kABytes = kM * kKB * 2;
constexpr int kEpiWarps = 8;     // warps 4 .. 11: two per quarter of the rows, each with half of the tokens
constexpr int kThreads = 128 + 32 * kEpiWarps;
__host__ __device__ constexpr int box_rows(int nt) { return nt > 16 ? nt / 2 : nt; }  // grouped form: rows of a box
constexpr int kGatherShare = 24;  // gathers of four rows per stage and issuing warp: a third of 64, rounded up

struct DenseParams {
    void* out;
    float* partial;
    unsigned* tickets;
    int* error_flag;
    const float *e0, *e1;
    size_t out_batch;
    int n, T, ldo, kblocks, mt, nt, batch, shares, items, stages, stage_tx;
    int out_f32, epi, e_div;
    float scale, cap;
    void* out2;
    int ldo2, split, act_end;
    const __nv_bfloat16* table;
    const int64_t* ids;
    int table_ld, table_rows;
    // grouped form
    const ExpertTile* tiles;
    const int32_t *n_tiles, *lists, *off;
    int list_stride;
};

// Raises the error word unless something did before; the words behind it tell which wait of which product.
__device__ void raise_wait(const DenseParams& p, int code, int tile, int grouped, int item, int at) {
    if (atomicCAS(p.error_flag, 0, code) != 0) return;
    const int words[kErrorWords - 1] = {p.n, p.kblocks, p.T, tile, grouped, item, at};
    for (int i = 0; i < kErrorWords - 1; i++) p.error_flag[1 + i] = words[i];
}
__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
// The epilogue is a template parameter of the kernels; kEpiAny stands for the rarer elementwise ones, told apart at run time.
constexpr int kEpiAny = -1;
constexpr int epi_class(int epi) { return epi == DENSE_LOG_DECAY || epi == DENSE_LOGITS ? kEpiAny : epi; }
constexpr bool epi_splits(int epi) { return epi == DENSE_SPLIT_RELU2 || epi == DENSE_SPLIT_SILU || epi == DENSE_SPLIT_TANH; }
constexpr bool epi_gated(int epi) { return epi == DENSE_GATED_SILU || epi == DENSE_GATED_GELU; }
__device__ __forceinline__ float silu_of(float g) { return g / (1.0f + expf(-g)); }
// z (1 + tanh u) / 2 = z / (1 + e^(-2u)), u = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_of(float z) { return z / (1.0f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z))); }
template <int EPI> __device__ __forceinline__ float gate_of(float g) { return EPI == DENSE_GATED_GELU ? gelu_of(g) : silu_of(g); }
// Element `row` of token t's row in the table, 0 for ids outside it.  The loads do not depend on a branch, so those of many tokens
// travel together; rows and tokens outside the product read a valid place.
__device__ __forceinline__ float table_factor(const DenseParams& p, int row, int t) {
    const int64_t id = p.ids[min(t, p.T - 1)];
    const bool ok = id >= 0 && id < p.table_rows;
    const float f = __bfloat162float(__ldg(p.table + (size_t)(ok ? id : 0) * p.table_ld + min(row, p.n - 1)));
    return ok ? f : 0.0f;
}
// ea, eb: the row's constants; `second`: behind the split of DENSE_SPLIT_*
template <int EPI>
__device__ __forceinline__ float dense_epilogue(const DenseParams& p, bool second, float ea, float eb, float y, int row) {
    const float r = fmaxf(y, 0.0f);
    if constexpr (EPI == DENSE_RELU2) return r * r;
    else if constexpr (EPI == DENSE_SPLIT_RELU2) return second ? r * r : y;
    else if constexpr (EPI == DENSE_SPLIT_SILU) return second && row < p.act_end ? silu_of(y) : y;
    else if constexpr (EPI == DENSE_SPLIT_TANH) return second && row < p.act_end ? tanhf(y) : y;
    else if constexpr (EPI == DENSE_BIAS) return y + eb;
    else if constexpr (EPI == DENSE_SIGMOID_DECAY) return __fdividef(-p.scale, 1.0f + __expf(-(y + eb)));
    else if constexpr (EPI == kEpiAny) {
        if (p.epi == DENSE_LOG_DECAY) return -ea * softplus_f(y + eb);
        const float v = y * p.scale;
        return p.cap > 0.0f ? p.cap * tanhf(v / p.cap) : v;
    } else return y;
}
__device__ __forceinline__ void dense_row_constants(const DenseParams& p, int row, float& ea, float& eb) {
    ea = eb = 0.0f;
    if (p.epi == DENSE_LOG_DECAY && row < p.n) { ea = p.e0[row / p.e_div]; eb = p.e1[row]; }
    if ((p.epi == DENSE_BIAS || p.epi == DENSE_SIGMOID_DECAY) && row < p.n) eb = p.e1[row];
}
// 16 accumulators of weight row `row`, tokens t0 .. t0 + m - 1 (m may exceed 16), for a whole warp (lane = row).  bf16: lane
// pairs swap halves, so a lane stores two rows of every other token.
template <int EPI>
__device__ __forceinline__ void dense_store16(const DenseParams& p, int b, int row, int t0, int m, const float (&v)[16], float ea, float eb) {
    if constexpr (epi_gated(EPI)) {  // even lanes hold gates, odd ones the matching values; each makes every other token's output
        const bool odd = row & 1;
        const size_t at = (size_t)b * p.out_batch + (size_t)t0 * p.ldo + (row >> 1);
#pragma unroll
        for (int j = 0; j < 16; j += 2) {
            const float other = __shfl_xor_sync(0xffffffffu, odd ? v[j] : v[j + 1], 1);
            const float y = odd ? gate_of<EPI>(other) * v[j + 1] : gate_of<EPI>(v[j]) * other;
            const int jj = j + (odd ? 1 : 0);
            if (jj >= m || row >= p.n) continue;
            if (p.out_f32) ((float*)p.out)[at + (size_t)jj * p.ldo] = y;
            else ((__nv_bfloat16*)p.out)[at + (size_t)jj * p.ldo] = __float2bfloat16_rn(y);
        }
        return;
    }
    if constexpr (EPI == DENSE_GELU_TABLE) {  // all factors ahead of the first store
        float u[16];
#pragma unroll
        for (int j = 0; j < 16; j++) u[j] = table_factor(p, row, t0 + j);
#pragma unroll
        for (int j = 0; j < 16; j++) u[j] *= gelu_of(v[j]);
        dense_store16<DENSE_STORE>(p, b, row, t0, m, u, ea, eb);
        return;
    }
    // a warp's 32 rows lie on one side of a split
    const bool second = epi_splits(EPI) && row >= p.split;
    const int ldo = second ? p.ldo2 : p.ldo, r = second ? row - p.split : row;
    void* out = second ? p.out2 : p.out;
    const size_t at = (size_t)b * p.out_batch + (size_t)t0 * ldo + r;
    if (epi_splits(EPI) ? !second : p.out_f32 != 0) {
        if (row >= p.n) return;
        float* o = (float*)out + at;
#pragma unroll
        for (int j = 0; j < 16; j++)
            if (j < m) o[(size_t)j * ldo] = dense_epilogue<EPI>(p, second, ea, eb, v[j], row);
    } else if ((p.n & 1) == 0 && (ldo & 1) == 0) {  // row pairs stay inside the matrix and 4-byte aligned
        const bool odd = row & 1;
        __nv_bfloat16* o = (__nv_bfloat16*)out + at - (odd ? 1 : 0);
#pragma unroll
        for (int j = 0; j < 16; j += 2) {
            const float x = dense_epilogue<EPI>(p, second, ea, eb, v[j], row), y = dense_epilogue<EPI>(p, second, ea, eb, v[j + 1], row);
            const float other = __shfl_xor_sync(0xffffffffu, odd ? x : y, 1);
            const __nv_bfloat162 pr = odd ? __floats2bfloat162_rn(other, y) : __floats2bfloat162_rn(x, other);
            const int jj = j + (odd ? 1 : 0);
            if (jj < m && row < p.n) *(__nv_bfloat162*)(o + (size_t)jj * ldo) = pr;
        }
    } else {
        if (row >= p.n) return;
        __nv_bfloat16* o = (__nv_bfloat16*)out + at;
#pragma unroll
        for (int j = 0; j < 16; j++)
            if (j < m) o[(size_t)j * ldo] = __float2bfloat16_rn(dense_epilogue<EPI>(p, second, ea, eb, v[j], row));
    }
}

template <int NT, bool GROUPED, int EPI>
__global__ void __launch_bounds__(kThreads, NT <= 64 ? 2 : 1)
dense_umma_kernel(const unsigned char* __restrict__ w, const __grid_constant__ CUtensorMap tx, const DenseParams p) {
    constexpr int kBBytes = NT * kKB * 2, kStage = kABytes + kBBytes;
    constexpr uint32_t kCols = NT < 32 ? 32 : NT;  // tensor-memory columns of one accumulator set
    constexpr uint32_t kAlloc = 2 * kCols;
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    uint64_t* full = (uint64_t*)(smem + (size_t)p.stages * kStage);
    uint64_t *empty = full + p.stages, *acc_full = empty + p.stages, *acc_empty = acc_full + 2;
    uint32_t* tmem_slot = (uint32_t*)(acc_empty + 2);
    volatile int* stop = (volatile int*)(tmem_slot + 1);
    unsigned* last_share = (unsigned*)(tmem_slot + 2);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int i = 0; i < p.stages; i++) { mbar_init(&full[i], GROUPED && p.lists ? 3 : 1); mbar_init(&empty[i], 1); }
        for (int i = 0; i < 2; i++) { mbar_init(&acc_full[i], 1); mbar_init(&acc_empty[i], 32 * kEpiWarps); }
        *stop = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 2) tmem_alloc(tmem_slot, kAlloc);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    pdl_launch_dependents();

    // item -> (weight tile fastest over shares, then token tiles): consecutive CTAs share a weight tile's rows
    struct Item { int b, m, n, share, k0, k1, t0, rows, first; };
    auto item_of = [&](int it) {
        Item r;
        r.share = it % p.shares; it /= p.shares;
        if constexpr (GROUPED) {  // neighbours share a tile's activations, then an expert's matrix
            r.m = it % p.mt; r.n = it / p.mt;
            const ExpertTile tl = p.tiles[r.n];
            r.b = tl.expert; r.t0 = tl.row0; r.rows = tl.rows; r.first = tl.first;
        } else {
            r.n = it % p.nt; it /= p.nt;
            r.m = it % p.mt; r.b = it / p.mt;
            r.t0 = r.n * NT; r.rows = p.T - r.t0; r.first = 0;
        }
        r.k0 = (int)((long long)p.kblocks * r.share / p.shares);
        r.k1 = (int)((long long)p.kblocks * (r.share + 1) / p.shares);
        return r;
    };
    auto block = [&](const Item& r, int kb) { return w + (((size_t)r.b * p.mt + r.m) * p.kblocks + kb) * kABytes; };
    if (GROUPED && (warp == 0 || (p.lists && (warp == 2 || warp == 3)))) {
        // rows that lie together: one thread brings one box or two (every copy costs it about a hundred cycles); rows of a list:
        // three warps deal the gathers of four among themselves, one thread of each issues them
        pdl_wait();
        constexpr int kBoxRows = box_rows(NT);
        int4* s_rows = (int4*)(tmem_slot + 4) + (warp == 0 ? 0 : warp - 1) * kGatherShare;
        const int items = *p.n_tiles * p.mt * p.shares, part = warp == 0 ? 0 : warp - 1;
        int issued = 0, st = 0;
        uint32_t phase = 1;
        bool ok = true;
        for (int it = blockIdx.x; it < items && ok; it += gridDim.x) {
            const Item r = item_of(it);
            const unsigned char* wb = block(r, r.k0);
            const int fours = (r.rows + 3) / 4, mine = fours > part ? (fours - part + 2) / 3 : 0;
            if (p.lists && lane < mine) {
                const int32_t* list = p.lists + (size_t)r.b * p.list_stride + r.first;
                const int at = (part + 3 * lane) * 4, last = r.rows - 1;
                s_rows[lane] = make_int4(list[at], list[min(at + 1, last)], list[min(at + 2, last)], list[min(at + 3, last)]);
            }
            __syncwarp();
            if (lane == 0) {
                const uint32_t tx_bytes = kABytes + (p.lists ? fours * 512 : (r.rows > kBoxRows ? 2 : 1) * (kBoxRows * 128));
                for (int kb = r.k0; kb < r.k1; kb++, wb += kABytes) {
                    unsigned char* a = smem + (size_t)st * kStage;
                    if (issued >= p.stages && !mbar_wait(&empty[st], phase)) { ok = false; break; }
                    // every issuing warp arrives, also one without a gather: a warp that fell two rounds of the ring behind would take an old phase
                    // of "empty" for the one that it waits for
                    if (warp == 0) {
                        mbar_expect_tx(&full[st], tx_bytes);
                        bulk_load(a, wb, kABytes, &full[st]);
                    } else {
                        mbar_arrive(&full[st]);
                    }
                    if (p.lists) {
#pragma unroll 4
                        for (int i = 0; i < mine; i++) tma_gather4(a + kABytes + (part + 3 * i) * 512, &tx, kb * kKB, s_rows[i], &full[st]);
                    } else {
                        tma_load_2d(a + kABytes, &tx, kb * kKB, r.t0, &full[st]);
                        if (r.rows > kBoxRows) tma_load_2d(a + kABytes + kBoxRows * 128, &tx, kb * kKB, r.t0 + kBoxRows, &full[st]);
                    }
                    issued++;
                    if (++st == p.stages) { st = 0; phase ^= 1; }
                }
            }
            ok = __shfl_sync(0xffffffffu, (int)ok, 0) != 0;
        }
        if (!ok && warp == 0 && lane == 0) {
            *stop = 1;
            raise_wait(p, 11, NT, 1, blockIdx.x, issued);
            for (int i = max(0, issued - p.stages); i < issued; i++) mbar_wait(&full[i % p.stages], (uint32_t)(i / p.stages) & 1);
        }
        __syncwarp();
    } else if (warp == 0 && lane == 0) {
        int issued = 0;
        bool ok = true;
        // weight boxes of the first stages, before the activations exist
        int pre = 0;
        {
            const Item r = item_of(blockIdx.x);
            for (; pre < p.stages && r.k0 + pre < r.k1; pre++) {
                mbar_expect_tx(&full[pre], p.stage_tx);
                bulk_load(smem + (size_t)pre * kStage, block(r, r.k0 + pre), kABytes, &full[pre]);
            }
        }
        pdl_wait();
        int st = 0;
        uint32_t phase = 1;  // parity of the "empty" phase to wait for; the first round finds every stage free
        for (int it = blockIdx.x; it < p.items && ok; it += gridDim.x) {
            const Item r = item_of(it);
            const unsigned char* wb = block(r, r.k0);
            for (int kb = r.k0; kb < r.k1; kb++, wb += kABytes) {
                unsigned char* a = smem + (size_t)st * kStage;
                if (issued >= pre) {
                    if (issued >= p.stages && !mbar_wait(&empty[st], phase)) { ok = false; break; }
                    mbar_expect_tx(&full[st], p.stage_tx);
                    bulk_load(a, wb, kABytes, &full[st]);
                }
                tma_load_3d(a + kABytes, &tx, kb * kKB, r.b, r.n * NT, &full[st]);
                issued++;
                if (++st == p.stages) { st = 0; phase ^= 1; }
            }
        }
        if (!ok) {
            *stop = 1;
            raise_wait(p, 11, NT, 0, blockIdx.x, issued);
            for (int i = max(0, issued - p.stages); i < issued; i++) mbar_wait(&full[i % p.stages], (uint32_t)(i / p.stages) & 1);
        }
    } else if (warp == 1 && lane == 0) {
        uint32_t idesc = idesc_bf16(kM, NT);
        if constexpr (GROUPED) pdl_wait();
        const int items = GROUPED ? *p.n_tiles * p.mt * p.shares : p.items;
        const uint64_t desc0 = umma_desc_sw128(smem_u32(smem));  // a start address below 256 KB: adding to the descriptor moves it
        int tile = 0, st = 0;
        uint32_t phase = 0;
        bool ok = true;
        for (int it = blockIdx.x; it < items && ok; it += gridDim.x, tile++) {
            const Item r = item_of(it);
            const int set = tile & 1;
            if constexpr (GROUPED) idesc = idesc_bf16(kM, (r.rows + 15) & ~15);
            if (tile >= 2 && !mbar_wait(&acc_empty[set], (uint32_t)(tile / 2 - 1) & 1)) { ok = false; break; }
            tc_fence_after();
            const uint32_t d = tmem + (uint32_t)set * kCols;
            for (int kb = r.k0; kb < r.k1; kb++) {
                if (!mbar_wait(&full[st], phase)) { ok = false; break; }
                tc_fence_after();
                const uint64_t da = desc0 + (uint64_t)st * (kStage / 16), db = da + kABytes / 16;
#pragma unroll
                for (int k = 0; k < 4; k++) umma_f16_ss(d, da + 2 * k, db + 2 * k, idesc, kb > r.k0 || k > 0);
                umma_commit(&empty[st]);
                if (++st == p.stages) { st = 0; phase ^= 1; }
            }
            if (ok) umma_commit(&acc_full[set]);
        }
        if (!ok) { *stop = 1; raise_wait(p, 12, NT, GROUPED, blockIdx.x, tile * 65536 + st); }
    } else if (warp >= 4) {
        pdl_wait();  // earlier kernels may still read what this one overwrites
        constexpr int kHalf = NT >= 32 ? NT / 2 : NT;  // tokens of one warp; a 16-token tile leaves the second half idle
        const int quarter = warp & 3, half = (warp - 4) >> 2, row_in = quarter * 32 + lane, c_lo = half * kHalf, c_hi = c_lo < NT ? c_lo + kHalf : c_lo;
        const int items = GROUPED ? *p.n_tiles * p.mt * p.shares : p.items;
        int tile = 0;
        for (int it = blockIdx.x; it < items; it += gridDim.x, tile++) {
            const Item r = item_of(it);
            const int set = tile & 1;
            const int row = r.m * kM + row_in, t0 = r.t0, ob = GROUPED ? 0 : r.b;
            float ea, eb;
            dense_row_constants(p, row, ea, eb);
            if constexpr (EPI == DENSE_GELU_TABLE) {  // the warp's part of its tokens' rows, a lane each, while the products run
                const int t = t0 + c_lo + lane;
                if (lane < kHalf && t < p.T && row - lane < p.n) {
                    const int64_t id = p.ids[t];
                    if (id >= 0 && id < p.table_rows) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.table + (size_t)id * p.table_ld + row - lane));
                }
            }
            if (!mbar_wait(&acc_full[set], (uint32_t)(tile / 2) & 1)) { *stop = 1; if (lane == 0) raise_wait(p, 13, NT, GROUPED, it, tile); break; }
            tc_fence_after();
            const uint32_t base = tmem + (uint32_t)set * kCols + ((uint32_t)(quarter * 32) << 16);
            const size_t plane = (size_t)NT * kM;
            const int cell = GROUPED ? r.n * p.mt + r.m : (r.b * p.mt + r.m) * p.nt + r.n;
            float* part = p.shares > 1 ? p.partial + (size_t)cell * p.shares * plane : nullptr;
#pragma unroll 1
            for (int c = c_lo; c < c_hi; c += 16) {
                if (c >= r.rows) break;
                uint32_t raw[16];
                tmem_ld16(base + c, raw);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                float v[16];
#pragma unroll
                for (int j = 0; j < 16; j++) v[j] = __uint_as_float(raw[j]);
                if (part) {
                    const int m = r.rows - c;
#pragma unroll
                    for (int j = 0; j < 16; j++)
                        if (j < m) part[(size_t)r.share * plane + (size_t)(c + j) * kM + row_in] = v[j];
                } else {
                    dense_store16<EPI>(p, ob, row, t0 + c, r.rows - c, v, ea, eb);
                }
            }
            tc_fence_before();
            mbar_arrive(&acc_empty[set]);
            if (part) {
                __threadfence();
                asm volatile("bar.sync 1, %0;" ::"n"(32 * kEpiWarps) : "memory");
                if (threadIdx.x == 128) {
                    const unsigned t = atomicAdd(&p.tickets[cell], 1u);
                    *last_share = t == (unsigned)(p.shares - 1);
                    if (*last_share) p.tickets[cell] = 0;
                    __threadfence();
                }
                asm volatile("bar.sync 1, %0;" ::"n"(32 * kEpiWarps) : "memory");
                const bool mine = *last_share != 0;
                asm volatile("bar.sync 1, %0;" ::"n"(32 * kEpiWarps) : "memory");
                if (mine) {
#pragma unroll 1
                    for (int c = c_lo; c < c_hi; c += 16) {
                        if (c >= r.rows) break;
                        float v[16];
                        const int m = r.rows - c;
#pragma unroll
                        for (int j = 0; j < 16; j++) v[j] = 0.0f;
                        const float* ps = part + (size_t)c * kM + row_in;
                        if (m >= 16) {
#pragma unroll 2
                            for (int sh = 0; sh < p.shares; sh++, ps += plane)
#pragma unroll
                                for (int j = 0; j < 16; j++) v[j] += __ldcg(ps + j * kM);
                        } else {
#pragma unroll 2
                            for (int sh = 0; sh < p.shares; sh++, ps += plane)
#pragma unroll
                                for (int j = 0; j < 16; j++)
                                    if (j < m) v[j] += __ldcg(ps + j * kM);
                        }
                        dense_store16<EPI>(p, ob, row, t0 + c, r.rows - c, v, ea, eb);
                    }
                }
            }
        }
    } else {
        pdl_wait();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (warp == 2) tmem_free(tmem, kAlloc);
}

// One 16-byte chunk (eight elements of k of one row) per thread and turn; chunk c of row r of a block sits at c ^ (r & 7).
__global__ void tile_kernel(const __nv_bfloat16* __restrict__ src, int n, int k, int ld, size_t batch_stride, size_t chunks, uint4* __restrict__ dst) {
    const int mt = (n + kM - 1) / kM, kblocks = (k + kKB - 1) / kKB;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < chunks; i += (size_t)gridDim.x * blockDim.x) {
        const int c = (int)(i & 7) ^ (int)((i >> 3) & 7), r_in = (int)(i >> 3) & (kM - 1);
        size_t b = i >> 10;
        const int kb = (int)(b % kblocks);
        b /= kblocks;
        const int row = (int)(b % mt) * kM + r_in, k0 = kb * kKB + c * 8;
        b /= mt;
        alignas(16) __nv_bfloat16 v[8];
#pragma unroll
        for (int j = 0; j < 8; j++) v[j] = row < n && k0 + j < k ? src[b * batch_stride + (size_t)row * ld + k0 + j] : __float2bfloat16_rn(0.0f);
        dst[i] = *(const uint4*)v;
    }
}

// True 32-bit: 64 weight rows x 64 tokens per CTA, 4 x 4 outputs per thread.  Grouped (p.off): blockIdx.z is the expert, the
// tokens are the rows of its list.
template <int EPI>
__global__ void __launch_bounds__(256) dense_f32_kernel(const __nv_bfloat16* __restrict__ w, int ldw, size_t w_batch, const float* __restrict__ x, int ldx,
                                                        size_t x_batch, int k, const DenseParams p) {
    constexpr int KT = 16;
    __shared__ float ws[KT][64 + 4], xs[KT][64 + 4];
    __shared__ int x_row[64];
    pdl_launch_dependents();
    pdl_wait();
    const int r0 = blockIdx.x * 64, t0 = blockIdx.y * 64, b = blockIdx.z;
    const int row0 = p.off ? p.off[b] : 0, T = p.off ? p.off[b + 1] - row0 : p.T;
    if (t0 >= T) return;
    w += (size_t)b * w_batch;
    if (!p.off) x += (size_t)b * x_batch;
    if (threadIdx.x < 64) {
        const int t = min(t0 + (int)threadIdx.x, T - 1);
        x_row[threadIdx.x] = p.lists ? p.lists[(size_t)b * p.list_stride + t] : row0 + t;
    }
    __syncthreads();
    const int tr = threadIdx.x & 15, tt = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < k; k0 += KT) {
        for (int i = threadIdx.x; i < 64 * KT; i += 256) {
            const int r = i / KT, c = i % KT, kk = k0 + c;
            ws[c][r] = (r0 + r < p.n && kk < k) ? __bfloat162float(w[(size_t)(r0 + r) * ldw + kk]) : 0.0f;
            xs[c][r] = (t0 + r < T && kk < k) ? x[(size_t)x_row[r] * ldx + kk] : 0.0f;
        }
        __syncthreads();
        float part[4][4] = {};  // sums of a tile of k join the others as one: the rounding grows with the tiles, not with k
#pragma unroll
        for (int c = 0; c < KT; c++) {
            float a[4], q[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { a[i] = ws[c][tr + 16 * i]; q[i] = xs[c][tt + 16 * i]; }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) part[i][j] = fmaf(q[i], a[j], part[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) acc[i][j] += part[i][j];
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int t = t0 + tt + 16 * i;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int row = r0 + tr + 16 * j;
            if constexpr (epi_gated(EPI)) {
                const float up = __shfl_xor_sync(0xffffffffu, acc[i][j], 1);
                if (t < T && row < p.n && (row & 1) == 0) ((float*)p.out)[(size_t)(row0 + t) * p.ldo + (row >> 1)] = gate_of<EPI>(acc[i][j]) * up;
                continue;
            }
            if (t >= T || row >= p.n) continue;
            if constexpr (EPI == DENSE_GELU_TABLE) {
                ((float*)p.out)[(size_t)t * p.ldo + row] = gelu_of(acc[i][j]) * table_factor(p, row, t);
                continue;
            }
            float ea, eb;
            dense_row_constants(p, row, ea, eb);
            if (epi_splits(EPI) && row >= p.split) ((float*)p.out2)[(size_t)t * p.ldo2 + row - p.split] = dense_epilogue<EPI>(p, true, ea, eb, acc[i][j], row);
            else ((float*)p.out)[(p.off ? 0 : (size_t)b * p.out_batch) + (size_t)(row0 + t) * p.ldo + row] = dense_epilogue<EPI>(p, false, ea, eb, acc[i][j], row);
        }
    }
}

template <int NT, bool GROUPED, int EPI>
int32_t launch_umma(const DenseArgs& a, const CUtensorMap& tx, DenseParams p, cudaStream_t s) {
    const size_t stage = kABytes + (size_t)NT * kKB * 2, fixed = 1024 + 512 + (GROUPED ? 3 * kGatherShare * 16 : 0);
    // few tokens: half of the shared memory, so that the next kernel's first weight boxes travel while this one drains
    p.stages = (int)((NT <= 64 ? kMaxSmem / 2 - 1024 : kMaxSmem) - fixed) / (int)stage;
    const size_t smem = fixed + (size_t)p.stages * stage;
    LC_CUDA(ensure_smem_limit((const void*)dense_umma_kernel<NT, GROUPED, EPI>, smem));
    const int grid = std::min(p.items, sm_count());
    LC_CUDA(launch_pdl(dense_umma_kernel<NT, GROUPED, EPI>, dim3((unsigned)grid), dim3(kThreads), smem, s, a.w->tiles, tx, p));
    return LC_OK;
}

template <bool GROUPED, int EPI>
int32_t launch_tiles(int NT, const DenseArgs& a, const CUtensorMap& tx, const DenseParams& p, cudaStream_t s) {
    switch (NT) {
        case 16: return launch_umma<16, GROUPED, EPI>(a, tx, p, s);
        case 32: return launch_umma<32, GROUPED, EPI>(a, tx, p, s);
        case 64: return launch_umma<64, GROUPED, EPI>(a, tx, p, s);
        case 128: return launch_umma<128, GROUPED, EPI>(a, tx, p, s);
        default: return launch_umma<256, GROUPED, EPI>(a, tx, p, s);
    }
}

constexpr size_t kPartialBytes = (size_t)64 << 20;
constexpr int kMaxTickets = 4096;

}  // namespace

int32_t dense_weight_init(DenseWeight* w, const __nv_bfloat16* data, int n, int k, int ld, int batch, size_t batch_stride) {
    w->data = data; w->n = n; w->k = k; w->ld = ld; w->batch = batch; w->batch_stride = batch_stride;
    LC_CHECK(n > 0 && k > 0 && ld >= k && ld % 8 == 0 && batch >= 1 && batch_stride % 8 == 0 && (uintptr_t)data % 16 == 0, LC_ERR_INVALID,
             "dense weight [%d x %d], rows %d apart: layout", n, k, ld);
    w->tiles = nullptr;
    return LC_OK;
}

size_t dense_tile_bytes(const DenseWeight& w) { return (size_t)w.batch * ((w.n + kM - 1) / kM) * ((w.k + kKB - 1) / kKB) * kABytes; }

int32_t dense_weight_tile(DenseWeight* w, void* dst, cudaStream_t s) {
    const size_t chunks = dense_tile_bytes(*w) / 16;
    tile_kernel<<<(unsigned)std::min<size_t>((chunks + 255) / 256, (size_t)sm_count() * 32), 256, 0, s>>>(w->data, w->n, w->k, w->ld, w->batch_stride, chunks, (uint4*)dst);
    LC_CUDA(cudaGetLastError());
    w->tiles = (const unsigned char*)dst;
    w->data = nullptr;
    return LC_OK;
}

int32_t dense_workspace_alloc(DenseWorkspace* ws) {
    LC_CUDA(cudaMalloc((void**)&ws->partial, kPartialBytes));
    ws->partial_bytes = kPartialBytes;
    LC_CUDA(cudaMalloc((void**)&ws->tickets, kMaxTickets * sizeof(unsigned)));
    LC_CUDA(cudaMemsetAsync(ws->tickets, 0, kMaxTickets * sizeof(unsigned), stream()));
    ws->max_tickets = kMaxTickets;
    return LC_OK;
}
void dense_workspace_free(DenseWorkspace* ws) {
    if (ws->partial) cudaFree(ws->partial);
    if (ws->tickets) cudaFree(ws->tickets);
    ws->partial = nullptr;
    ws->tickets = nullptr;
    ws->maps.clear();
}

namespace {
// Shares of k, where cutting it evens out the CTAs' work: k blocks of the busiest CTA, plus what an item and the summing of
// the shares cost.  `cells` are expected tiles, `room` the most there can be.
int choose_shares(const DenseParams& p, const DenseWorkspace& ws, int NT, int cells, int room) {
    int shares = 1;
    if (NT > 64 || room > ws.max_tickets) return shares;
    const int sms = sm_count();
    long best = -1;
    for (int c = 1; c <= std::min(16, p.kblocks / 2); c++) {
        if ((size_t)room * c * NT * kM * sizeof(float) > ws.partial_bytes) break;
        const long waves = ((long)cells * c + sms - 1) / sms;
        const long cost = waves * (((p.kblocks + c - 1) / c) + 2 + (c > 1 ? NT / 16 : 0)) + (c > 1 ? 3 + c * NT / 32 : 0);
        if (best < 0 || cost < best) { best = cost; shares = c; }
    }
    return shares;
}

// The tensor map for `key`, made by `make` when it is new.
template <typename Make>
int32_t map_of(DenseWorkspace& ws, const std::vector<uint64_t>& key, Make make, const CUtensorMap** out) {
    std::unique_ptr<DenseWorkspace::Map>& mp = ws.maps[key];
    if (!mp) {
        mp.reset(new DenseWorkspace::Map);
        const bool ok = make(mp->b);
        if (!ok) ws.maps.erase(key);
        LC_CHECK(ok, LC_ERR_CUDA, "dense product: no tensor map over the activations");
    }
    *out = (const CUtensorMap*)mp->b;
    return LC_OK;
}

int32_t launch_grouped(const DenseArgs& a, DenseWorkspace& ws, DenseParams p, cudaStream_t s) {
    const ExpertPlan& g = *a.plan;
    const DenseWeight& w = *a.w;
    const int room = p.mt * g.most_tiles;
    p.nt = 1;
    p.shares = choose_shares(p, ws, g.tile_rows, p.mt * std::min(g.most_tiles, std::min(w.batch, g.most_rows)), room);
    p.items = room * p.shares;
    const CUtensorMap* tx = nullptr;
    const uint32_t box = a.gather ? 1 : (uint32_t)box_rows(g.tile_rows);
    LC_TRY(map_of(ws, {(uint64_t)(uintptr_t)a.x, (uint64_t)w.k, (uint64_t)a.ldx, (uint64_t)a.x_rows, box},
                  [&](void* b) { return make_bf16_tmap_rows(b, a.x, (uint64_t)w.k, (uint64_t)a.x_rows, (uint64_t)a.ldx, box); }, &tx));
    LC_CHECK(a.epi == DENSE_STORE || a.epi == DENSE_RELU2 || a.epi == DENSE_GATED_SILU, LC_ERR_UNSUPPORTED, "grouped product: epilogue %d", (int)a.epi);
    if (a.epi == DENSE_GATED_SILU) return launch_tiles<true, DENSE_GATED_SILU>(g.tile_rows, a, *tx, p, s);
    return a.epi == DENSE_RELU2 ? launch_tiles<true, DENSE_RELU2>(g.tile_rows, a, *tx, p, s) : launch_tiles<true, DENSE_STORE>(g.tile_rows, a, *tx, p, s);
}
}  // namespace

int32_t launch_dense(const DenseArgs& a, DenseWorkspace& ws, cudaStream_t s) {
    if (a.T <= 0) return LC_OK;
    const DenseWeight& w = *a.w;
    DenseParams p{};
    p.out = a.out; p.e0 = a.e0; p.e1 = a.e1; p.out_batch = a.out_batch;
    p.n = w.n; p.T = a.T; p.ldo = a.ldo; p.batch = w.batch;
    p.out_f32 = a.out_f32 || a.f32; p.epi = a.epi; p.e_div = a.e_div; p.scale = a.scale; p.cap = a.cap;
    p.error_flag = gemv_error_flag_dev();
    p.out2 = a.out2; p.ldo2 = a.ldo2; p.split = a.split; p.act_end = a.act_end;
    p.table = a.table; p.table_ld = a.table_ld; p.table_rows = a.table_rows; p.ids = a.ids;
    if (a.plan) { p.tiles = a.plan->tiles; p.n_tiles = a.plan->n_tiles; p.off = a.plan->off; p.lists = a.gather ? a.plan->lists : nullptr; p.list_stride = a.plan->list_stride; }
    LC_CHECK((!epi_gated(a.epi) || w.n % 2 == 0) && (!epi_splits(a.epi) || (a.split % 32 == 0 && w.batch == 1)), LC_ERR_INVALID, "dense product: epilogue layout");
    LC_CHECK(a.f32 ? w.data != nullptr : w.tiles != nullptr, LC_ERR_STATE, "dense product: the weight is not in the form this product reads");
    if (a.f32) {
        const dim3 grid((unsigned)((w.n + 63) / 64), (unsigned)((a.T + 63) / 64), (unsigned)w.batch);
        auto go = [&](auto kern) -> int32_t {
            LC_CUDA(launch_pdl(kern, grid, dim3(256), 0, s, w.data, w.ld, w.batch_stride, (const float*)a.x, a.ldx, a.x_batch, w.k, p));
            return LC_OK;
        };
        switch (epi_class(a.epi)) {
            case DENSE_STORE: return go(dense_f32_kernel<DENSE_STORE>);
            case DENSE_RELU2: return go(dense_f32_kernel<DENSE_RELU2>);
            case DENSE_GATED_SILU: return go(dense_f32_kernel<DENSE_GATED_SILU>);
            case DENSE_SPLIT_RELU2: return go(dense_f32_kernel<DENSE_SPLIT_RELU2>);
            case DENSE_SPLIT_SILU: return go(dense_f32_kernel<DENSE_SPLIT_SILU>);
            case DENSE_GELU_TABLE: return go(dense_f32_kernel<DENSE_GELU_TABLE>);
            case DENSE_GATED_GELU: return go(dense_f32_kernel<DENSE_GATED_GELU>);
            case DENSE_BIAS: return go(dense_f32_kernel<DENSE_BIAS>);
            case DENSE_SPLIT_TANH: return go(dense_f32_kernel<DENSE_SPLIT_TANH>);
            case DENSE_SIGMOID_DECAY: return go(dense_f32_kernel<DENSE_SIGMOID_DECAY>);
            default: return go(dense_f32_kernel<kEpiAny>);
        }
    }
    const int sms = sm_count();
    p.kblocks = (w.k + kKB - 1) / kKB;
    p.mt = (w.n + kM - 1) / kM;
    p.partial = ws.partial; p.tickets = ws.tickets;
    LC_CHECK((uintptr_t)a.x % 16 == 0 && a.ldx % 8 == 0 && a.x_batch % 8 == 0 && a.x_rows >= a.T, LC_ERR_INVALID, "dense product: activation layout");
    if (a.plan) return launch_grouped(a, ws, p, s);
    // tokens per tile: what finishes first at the measured time of one block of k (in hundredths of a microsecond)
    static const struct { int nt, t; } kSizes[] = {{16, 17}, {32, 17}, {64, 19}, {128, 24}, {256, 36}};
    int NT = 16;
    long best_nt = -1;
    for (const auto& z : kSizes) {
        const long tiles = (long)p.mt * ((a.T + z.nt - 1) / z.nt) * w.batch, cost = (tiles + sms - 1) / sms * z.t;
        if (a.T <= 64 ? z.nt >= a.T && best_nt < 0 : z.nt >= 64 && (best_nt < 0 || cost <= best_nt)) { best_nt = cost; NT = z.nt; }
    }
    p.nt = (a.T + NT - 1) / NT;
    const int cells = p.mt * p.nt * w.batch;
    p.shares = choose_shares(p, ws, NT, cells, cells);
    p.items = cells * p.shares;
    // a single tile of fewer tokens than NT brings only those: what the other rows of the operand hold reaches columns that
    // are never read
    const int box = std::min(NT, a.T);
    p.stage_tx = kABytes + box * kKB * 2;
    const CUtensorMap* tx = nullptr;  // order (k, matrix, token): a token tile is one box
    LC_TRY(map_of(ws, {(uint64_t)(uintptr_t)a.x, (uint64_t)w.k, (uint64_t)a.ldx, (uint64_t)a.x_batch, (uint64_t)w.batch, (uint64_t)a.x_rows, (uint64_t)box}, [&](void* b) {
        return make_bf16_tmap_3d(b, a.x, (uint64_t)w.k, (uint64_t)w.batch, (uint64_t)a.x_rows, w.batch > 1 ? a.x_batch : (uint64_t)a.ldx, (uint64_t)a.ldx, kKB, 1, (uint32_t)box);
    }, &tx));
    switch (epi_class(a.epi)) {
        case DENSE_STORE: return launch_tiles<false, DENSE_STORE>(NT, a, *tx, p, s);
        case DENSE_RELU2: return launch_tiles<false, DENSE_RELU2>(NT, a, *tx, p, s);
        case DENSE_GATED_SILU: return launch_tiles<false, DENSE_GATED_SILU>(NT, a, *tx, p, s);
        case DENSE_SPLIT_RELU2: return launch_tiles<false, DENSE_SPLIT_RELU2>(NT, a, *tx, p, s);
        case DENSE_SPLIT_SILU: return launch_tiles<false, DENSE_SPLIT_SILU>(NT, a, *tx, p, s);
        case DENSE_GELU_TABLE: return launch_tiles<false, DENSE_GELU_TABLE>(NT, a, *tx, p, s);
        case DENSE_GATED_GELU: return launch_tiles<false, DENSE_GATED_GELU>(NT, a, *tx, p, s);
        case DENSE_BIAS: return launch_tiles<false, DENSE_BIAS>(NT, a, *tx, p, s);
        case DENSE_SPLIT_TANH: return launch_tiles<false, DENSE_SPLIT_TANH>(NT, a, *tx, p, s);
        case DENSE_SIGMOID_DECAY: return launch_tiles<false, DENSE_SIGMOID_DECAY>(NT, a, *tx, p, s);
        default: return launch_tiles<false, kEpiAny>(NT, a, *tx, p, s);
    }
}

}  // namespace lc
