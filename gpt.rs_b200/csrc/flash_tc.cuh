// tcgen05 flash attention over a paged cache, shared by latent attention (latent_attention.cu) and attention with grouped key / value
// heads (grouped_attention.cu): the kernel, the merge of key splits and the page geometry.
//
// bf16 pages are laid out so that a (page, kv head) is one contiguous block that a single bulk copy drops into shared memory ready to
// be an operand of both products: [2 groups of 8 tokens][blocks of 64 columns][8 tokens][64 columns], 16-byte chunk j of token t at
// chunk j ^ (t & 7) (the 128-byte operand swizzle). Columns past the data of a block are zero.
#pragma once
#include "umma_common.cuh"

namespace gptrs {
namespace {

constexpr int kPageTok = 16;
constexpr float kLog2e = 1.4426950408889634f;

__host__ __device__ inline int up(int v, int m) { return (v + m - 1) / m * m; }

// byte offset of 16-byte chunk `chunk` (8 columns) of token `t` inside the block of a (page, kv head)
__device__ __forceinline__ int page_chunk(int t, int chunk, int nb) {
    return (t >> 3) * nb * 1024 + (chunk >> 3) * 1024 + (t & 7) * 128 + (((chunk & 7) ^ (t & 7)) << 4);
}

// ---- tcgen05 flash attention ----------------------------------------------------------------------------------------------------
// A CTA takes a tile of up to 128 query rows = consecutive tokens of one sequence x all heads (more than 128 heads: one token
// x 128 heads), all reading the same cache rows, and walks its share of the visible keys in blocks of 64 (4 pages):
//   S[128 x 64]  = Q . K^T        A = Q tile, B = key block, both K-major in shared memory; accumulator in tensor memory,
//                                 three buffers: the scores of the next blocks are computed under the softmax of this one
//   softmax                       thread r owns row r: scaled scores, mask by position and window, running maximum with a lazy
//                                 rescale; the weights go back over the scores as two bf16 terms, P = P_hi + P_lo, so that
//                                 the weights keep 16 significant bits in the second product
//   O[128 x rank] += P . C        A = P_hi then P_lo from tensor memory, B = the latent columns of the SAME key block
//                                 (contraction index as rows: MN-major operand)
// Warps 0-3 softmax, warp 4 score MMAs and tensor memory, warp 5 page requests (one bulk copy per page), warp 6 output MMAs: a
// commit holds up its thread until the MMAs in front of it are under way, so one thread for both products would leave the
// tensor pipe idle between them. A decode step is the case of one token per tile, with the keys split over the y dimension of the grid; flash_combine_kernel merges the parts.
// Tiles of up to 64 rows (decode steps of up to 64 heads) hold every row twice: rows 64 .. 127 repeat the queries, hence the
// scores and the softmax, and put P_lo where the first copy puts P_hi, so that one product serves both terms; the two halves of
// O are added at the end. Every wait is bounded (status 3).
// Differential attention (TWO): two attentions of one head, with a query and a key part each, over the same values. A tile is 64 rows;
// rows 0 .. 63 carry the first part of the queries, rows 64 .. 127 the second one, each with zeros in the columns of the other part, so
// that one product with the whole key block gives the scores of both (an MMA of 64 rows would take as long as one of 128) and keys and
// values are read once. At the end the halves of O meet in shared memory: difference, norm over the head, gate.
// Linear distance bias and keys that are values times a number each (LINEAR): the numbers travel beside the pages and multiply the columns of
// S, so that a block holds values only and is an operand of both products. Blocks are walked from the newest to the oldest: under a steep
// bias the running maximum would otherwise move at every block.
constexpr int kRows = 128;
constexpr int kKeys = 64;
constexpr int kTcThreads = 224;
constexpr int kMaxScores = 3;        // score buffers in tensor memory: three with one CTA per SM, two with two
constexpr int kMaxStages = 6;
constexpr int kMaxBlocks = 6;        // 64-column blocks of a query
constexpr uint32_t kWaitLimit = 1u << 16;
constexpr float kRescaleStep = 8.f;

// What a kernel's keys, values and queries look like. A cache row is `blocks` blocks of 64 columns: the first value_blocks are the
// values, the query_blocks from key_block on are the key (latent attention: the key is the whole row and contains the value).
struct FlashShape {
    int heads, kv_heads, group;        // query heads; heads per kv head
    int blocks, value_blocks, key_block, query_blocks;
    int steps[kMaxBlocks];             // 16-column steps of every query block that hold data
    int mask, mask_size;               // GPTRS_MASK_*
    int out_stride;                    // output elements of a head
    int vdim;                          // of them data
    int map_blocks;                    // query blocks of one part (query_blocks without a second one)
    uint32_t block_bytes;              // (page, kv head): 16 rows
    long long page_bytes;
    int key_scales;                    // 1: 16 floats per kv head behind the blocks of a page, key = value x number
};
// What happens to the output of a head behind the softmax.
struct HeadOutput {
    float lambda, scale, eps;          // two parts: d = a1 - lambda a2, then d / sqrt(mean(d^2) + eps) scale
    const __nv_bfloat16* gate;         // times sigmoid(gate[row][head][..]), or null
    int gate_row, gate_stride;
};
// eight values times sigmoid of their gates
__device__ __forceinline__ void apply_gate(const __nv_bfloat16* g, float (&v)[8]) {
    const uint4 u = __ldg(reinterpret_cast<const uint4*>(g));
    const float z[8] = {bf16_lo(u.x), bf16_hi(u.x), bf16_lo(u.y), bf16_hi(u.y), bf16_lo(u.z), bf16_hi(u.z), bf16_lo(u.w), bf16_hi(u.w)};
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = __fdividef(v[i], 1.f + __expf(-z[i]));
}
// first key that position `pos` sees
__device__ __forceinline__ int first_visible(int mask, int size, int pos) {
    return mask == GPTRS_MASK_WINDOW ? max(pos - size + 1, 0) : mask == GPTRS_MASK_CHUNK ? pos - pos % size : 0;
}

struct TcParams {
    // queries, 128-byte swizzle. Latent: [64 columns][blocks][T x heads rows], boxes of 32 rows. Grouped: [dim][parts][heads][T], a box
    // holds the heads of a kv head for the tokens of a tile (q_map) or for one token (q_one)
    CUtensorMap q_map, q_one;
    FlashShape g;
    const unsigned char* pool;
    const int *page_table, *slot, *ctx_len;
    const int *tile_row, *tile_rows;   // first row and number of rows of every tile
    __nv_bfloat16* out;
    float* part_o;                     // splits > 1: [tile * kv heads * head blocks][split][128][64 value_blocks]
    float2* part_ml;                   // [tile * kv heads * head blocks][split][128]: running maximum (log2 units), sum
    int* status;
    int max_pages, splits, stages, head_blocks, rows_per_token;
    uint32_t tmem_cols, q_box_bytes, q_one_bytes;
    float scale_log2;                  // log2(e) scale; with a soft cap, 2 log2(e) scale / cap
    float cap_log2;                    // log2(e) cap, 0 = none
    const float *r1, *r2;              // distance penalty r1[h] ln(1 + r2[h] d), or null; LINEAR: r1[h] d
    const int* reach;                  // [kv heads] or null: keys further away than that weigh nothing
    const float* sink;                 // [heads] or null: exp(sink) in the denominator
    HeadOutput head_out;
};

__device__ __forceinline__ void tma_3d(uint32_t dst, const CUtensorMap* map, int x, int y, int z, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];\n" ::"r"(dst), "l"(map),
                 "r"(x), "r"(y), "r"(z), "r"(bar)
                 : "memory");
}
__device__ __forceinline__ void tma_4d(uint32_t dst, const CUtensorMap* map, int x, int y, int z, int w, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4, %5}], [%6];\n" ::"r"(dst), "l"(map),
                 "r"(x), "r"(y), "r"(z), "r"(w), "r"(bar)
                 : "memory");
}
__device__ __forceinline__ uint64_t desc_k_major(uint32_t addr, uint32_t group_stride) {
    uint64_t d = 0;
    d |= (uint64_t)((addr & 0x3FFFF) >> 4);
    d |= (uint64_t)1 << 16;
    d |= (uint64_t)(group_stride >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
// contraction index as rows: the next 64 columns are 1024 bytes on, the next 8 keys group_stride
__device__ __forceinline__ uint64_t desc_mn_major(uint32_t addr, uint32_t group_stride) {
    uint64_t d = 0;
    d |= (uint64_t)((addr & 0x3FFFF) >> 4);
    d |= (uint64_t)(1024 >> 4) << 16;
    d |= (uint64_t)(group_stride >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
// true in one lane of a converged warp; unlike a test of the lane number it leaves the branch known to be warp-uniform
__device__ __forceinline__ bool elect_one() {
    uint32_t p;
    asm volatile("{\n .reg .pred p;\n elect.sync _|p, 0xffffffff;\n selp.u32 %0, 1, 0, p;\n}\n" : "=r"(p));
    return p != 0;
}
__device__ __forceinline__ float ex2f(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}

// Raw products of a row -> scores in log2 units: cap tanh(scale s / cap) - r1 ln(1 + r2 d), all times log2(e). d0 is the distance of
// column 0 (a column on the far side of the row's own position is masked later; its logarithm is kept finite). The tanh is its Taylor
// series while the whole warp's arguments are at most 1/2 (7 terms, error below 2e-7), the logarithms of eight neighbouring columns
// are one logarithm in their middle and the series of ln(1 - y) around it while |y| <= 1/8 (5 terms, error below 1e-6): the
// multi-function unit, which would otherwise give four results per score, is what bounds this kernel.
__device__ __forceinline__ void score_log2(float (&s)[kKeys], float scale_log2, float cap_log2, float r1, float r2, int d0) {
    if (cap_log2 > 0.f) {
        const float cx = scale_log2 * (0.5f / kLog2e);   // scale / cap
        float mx[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < kKeys; ++j) mx[j & 3] = fmaxf(mx[j & 3], fabsf(s[j]));
        const float m = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * cx;
        if (__all_sync(0xffffffffu, m <= 0.5f)) {
            const float k0 = cap_log2;
            const uint64_t c0 = pair_of(k0, k0), c1 = pair_of(k0 * (-1.f / 3.f), k0 * (-1.f / 3.f)), c2 = pair_of(k0 * (2.f / 15.f), k0 * (2.f / 15.f)),
                           c3 = pair_of(k0 * (-17.f / 315.f), k0 * (-17.f / 315.f)), c4 = pair_of(k0 * (62.f / 2835.f), k0 * (62.f / 2835.f)),
                           c5 = pair_of(k0 * (-1382.f / 155925.f), k0 * (-1382.f / 155925.f)), c6 = pair_of(k0 * (21844.f / 6081075.f), k0 * (21844.f / 6081075.f)),
                           cc = pair_of(cx, cx);
#pragma unroll
            for (int j = 0; j < kKeys; j += 2) {
                const uint64_t x = mul2(pair_of(s[j], s[j + 1]), cc), z = mul2(x, x);
                uint64_t t = fma2(z, c6, c5);
                t = fma2(z, t, c4);
                t = fma2(z, t, c3);
                t = fma2(z, t, c2);
                t = fma2(z, t, c1);
                t = fma2(z, t, c0);
                const float2 v = split(mul2(x, t));
                s[j] = v.x; s[j + 1] = v.y;
            }
        } else {   // tanh(x) = 1 - 2 / (exp(2x) + 1)
#pragma unroll
            for (int j = 0; j < kKeys; ++j) {
                const float e = ex2f(s[j] * scale_log2) + 1.f;
                float inv;
                asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(inv) : "f"(e));
                s[j] = fmaf(-2.f * cap_log2, inv, cap_log2);
            }
        }
    } else {
#pragma unroll
        for (int j = 0; j < kKeys; ++j) s[j] *= scale_log2;
    }
    auto lg2f = [](float x) {
        float l;
        asm("lg2.approx.ftz.f32 %0, %1;\n" : "=f"(l) : "f"(x));
        return l;
    };
    if (!__any_sync(0xffffffffu, r1 != 0.f)) return;
    const float first = fmaf(r2, (float)d0, 1.f);
    if (__all_sync(0xffffffffu, fmaf(-r2, (float)(kKeys - 1), first) >= fmaxf(28.f * r2, 1e-3f))) {
#pragma unroll
        for (int j0 = 0; j0 < kKeys; j0 += 8) {
            const float a = fmaf(-r2, (float)j0 + 3.5f, first);   // 1 + r2 distance in the middle
            float w;
            asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(w) : "f"(a));
            w *= r2;
            // - r1 log2(1 - w o) at the offsets o = -3.5 .. 3.5
            const float b1 = r1 * kLog2e * w, b2 = b1 * w * 0.5f, b3 = b1 * w * w * (1.f / 3.f), b4 = b2 * w * w * 0.5f, b5 = b3 * w * w * 0.6f, b0 = -r1 * lg2f(a);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float o = 3.5f - i;
                const float even = fmaf(b4, o * o * o * o, fmaf(b2, o * o, b0)), odd = fmaf(b5, o * o * o * o * o, fmaf(b3, o * o * o, b1 * o));
                s[j0 + i] += even - odd;
                s[j0 + 7 - i] += even + odd;
            }
        }
    } else {
#pragma unroll
        for (int j = 0; j < kKeys; ++j) s[j] = fmaf(-r1, lg2f(fmaxf(fmaf(-r2, (float)j, first), 1e-30f)), s[j]);
    }
}

// column j of the scores times c[j]
__device__ __forceinline__ void scale_columns(float (&s)[kKeys], const float* c) {
#pragma unroll
    for (int j = 0; j < kKeys; j += 4) {
        const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(c + j);
        const float2 a = split(mul2(pair_of(s[j], s[j + 1]), v.x)), b = split(mul2(pair_of(s[j + 2], s[j + 3]), v.y));
        s[j] = a.x; s[j + 1] = a.y; s[j + 2] = b.x; s[j + 3] = b.y;
    }
}
// Raw products -> log2(e) (cap tanh(scale s / cap) - slope d)
__device__ __forceinline__ void score_linear(float (&s)[kKeys], float scale_log2, float cap_log2, float slope, int d0) {
    if (cap_log2 > 0.f) score_log2(s, scale_log2, cap_log2, 0.f, 0.f, 0);
    const float c = slope * kLog2e, b0 = -c * (float)d0, mul = cap_log2 > 0.f ? 1.f : scale_log2;
    const uint64_t m = pair_of(mul, mul);
#pragma unroll
    for (int j = 0; j < kKeys; j += 2) {
        const float2 v = split(fma2(pair_of(s[j], s[j + 1]), m, pair_of(fmaf(c, (float)j, b0), fmaf(c, (float)(j + 1), b0))));
        s[j] = v.x; s[j + 1] = v.y;
    }
}

// GROUPED: kv heads of their own, soft cap, distance penalty; otherwise one latent row for all heads
// kScores 2: two CTAs share an SM (tensor memory, shared memory and registers for half of one each), so that the softmax of one runs
// under the waits of the other.
// TWO: two query and key parts per head. LINEAR: linear distance bias, keys by numbers.
template <bool GROUPED, int kScores, bool TWO = false, bool LINEAR = false>
__global__ void __launch_bounds__(kTcThreads, kScores == 2 ? 2 : 1) flash_tc_kernel(const __grid_constant__ TcParams p) {
    constexpr uint32_t kOCol = kScores * kKeys;
    constexpr int kTileRows = TWO ? kRows / 2 : kRows;
    extern __shared__ unsigned char smem_raw[];
    __shared__ __align__(8) uint64_t k_full[kMaxStages], k_empty[kMaxStages], s_full[kScores], p_full[kScores], q_full;
    __shared__ __align__(16) float k_scale[LINEAR ? kMaxStages : 1][LINEAR ? kKeys : 4];
    __shared__ uint32_t tmem_holder;
    const FlashShape& g = p.g;
    const uint32_t smem = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t stage_bytes = (uint32_t)(kKeys * 128) * g.blocks, group_stride = (uint32_t)g.blocks * 1024u;
    const uint32_t sQ = smem, sK = smem + (uint32_t)g.query_blocks * (kRows * 128);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (warp == 4) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(smem_u32(&tmem_holder)), "r"(p.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    if (tid == 32 * 5) asm volatile("prefetch.tensormap [%0];\n" ::"l"(&p.q_map) : "memory");
    if constexpr (TWO) {   // zeros in the columns of the other part; the copies of the queries fill the rest
        for (int i = tid; i < g.query_blocks * (kRows / 2) * 8; i += kTcThreads) {
            const int b = i / (kRows / 2 * 8), o = i % (kRows / 2 * 8);
            st_shared_v4(sQ + (uint32_t)(b * kRows + (b < g.map_blocks ? kRows / 2 : 0)) * 128u + (uint32_t)o * 16u, 0, 0, 0, 0);
        }
        fence_proxy_async();
    }
    pdl_wait();
    const int tile = (int)gridDim.x - 1 - (int)blockIdx.x;   // long contexts come last in a token list: start them first
    const int row0 = p.tile_row[tile], n_tok = p.tile_rows[tile], hb = LINEAR ? (int)gridDim.z - 1 - (int)blockIdx.z : (int)blockIdx.z;   // later kv heads reach further
    const int kvh = GROUPED ? hb / p.head_blocks : 0, head_block = GROUPED ? hb % p.head_blocks : hb;
    const int heads_n = min(p.rows_per_token, g.group - head_block * kTileRows);   // heads of this CTA per token
    const int heads0 = kvh * g.group + head_block * kTileRows;
    const int live = n_tok * heads_n;
    const int live_warps = (live + 31) / 32;
    const bool dup = !TWO && live <= kRows / 2 && (!GROUPED || (n_tok == 1 && p.rows_per_token <= kRows / 2));   // a box of queries lands twice
    const bool halves = dup || TWO;   // rows 64 .. 127 belong to the same tokens and heads as rows 0 .. 63
    if (tid == 0) {
        for (int i = 0; i < p.stages; ++i) { mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); }
        for (int i = 0; i < kScores; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], (uint32_t)live_warps * (halves ? 64 : 32)); }
        mbar_init(&q_full, 1);
        mbar_fence_init();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_holder;
    pdl_launch_dependents();   // every CTA of this grid holds its tensor memory before a dependent grid may start

    // keys of the tile: [lo, hi), walked from a page boundary; this CTA's share of the blocks: [kb0, kb1)
    const int slot0 = p.slot[row0], cap = p.max_pages * kPageTok;
    const int hi = min(max(p.ctx_len[row0 + n_tok - 1], 0), cap);
    const int first_len = p.ctx_len[row0];
    int lo = GROUPED ? first_visible(g.mask, g.mask_size, max(first_len - 1, 0)) : max(first_len - g.mask_size, 0);
    if (LINEAR && p.reach) lo = max(lo, first_len - 1 - p.reach[kvh]);
    lo &= ~(kPageTok - 1);
    const int n_all = hi > lo ? (hi - lo + kKeys - 1) / kKeys : 0;
    const int kb0 = (int)((int64_t)n_all * blockIdx.y / p.splits), kb1 = (int)((int64_t)n_all * (blockIdx.y + 1) / p.splits);
    const int n_blocks = kb1 - kb0;
    const int key_base = lo + kb0 * kKeys;
    auto key_of = [&](int it) { return key_base + (LINEAR ? n_blocks - 1 - it : it) * kKeys; };   // first key of the block that comes as number `it`
    bool failed = false;
    auto wait = [&](uint64_t* bar, uint32_t parity) {   // whole warp
        if (!failed && !mbar_wait_parked(smem_u32(bar), parity, kWaitLimit)) failed = true;
        failed = __any_sync(0xffffffffu, failed);
        return !failed;
    };

    if (warp == 5) {
        // ================= pages and queries =======================================================================================
        const int* pt = p.page_table + (size_t)slot0 * p.max_pages;
        const uint32_t block_bytes = g.block_bytes;
        const unsigned char* pool = p.pool + (size_t)kvh * block_bytes;
        auto page_of = [&](int it) {   // lane j: the j-th page of block `it`
            const int key0 = key_of(it);
            return it < n_blocks && lane < (min(kKeys, hi - key0) + kPageTok - 1) / kPageTok ? __ldg(pt + key0 / kPageTok + lane) : 0;
        };
        int n_req = 0, page_next = page_of(0);
        auto request_queries = [&]() {   // 32 rows x 64 columns per copy; rows past the live ones are other queries, whose results nobody reads
            if (lane == 0) {
                const uint32_t bar = smem_u32(&q_full);
                if constexpr (GROUPED) {
                    const bool one = n_tok == 1;
                    mbar_expect_tx_addr(bar, (uint32_t)g.query_blocks * (one ? p.q_one_bytes * (dup ? 2u : 1u) : p.q_box_bytes));
                    for (int b = 0; b < g.query_blocks; ++b) {
                        const uint32_t dst = sQ + (uint32_t)(b * kRows) * 128u;
                        if constexpr (TWO) {
                            const int part = b >= g.map_blocks;
                            tma_4d(dst + (uint32_t)(part * (kRows / 2)) * 128u, one ? &p.q_one : &p.q_map, (b - part * g.map_blocks) * 64, part, heads0, row0, bar);
                        } else {
                            tma_4d(dst, one ? &p.q_one : &p.q_map, b * 64, 0, heads0, row0, bar);
                            if (dup) tma_4d(dst + (kRows / 2) * 128u, &p.q_one, b * 64, 0, heads0, row0, bar);
                        }
                    }
                } else {
                    mbar_expect_tx_addr(bar, (uint32_t)(live_warps * (dup ? 2 : 1) * g.query_blocks) * 4096u);
                    for (int w = 0; w < live_warps; ++w)
                        for (int b = 0; b < g.query_blocks; ++b) {
                            const uint32_t dst = sQ + (uint32_t)(b * kRows + w * 32) * 128u;
                            tma_3d(dst, &p.q_map, 0, b, row0 * g.heads + heads0 + w * 32, bar);
                            if (dup) tma_3d(dst + (kRows / 2) * 128u, &p.q_map, 0, b, row0 * g.heads + heads0 + w * 32, bar);
                        }
                }
            }
            __syncwarp();
        };
        for (int it = 0; it < n_blocks; ++it) {
            const int st = it % p.stages, lap = it / p.stages;
            const int page = page_next;
            page_next = page_of(it + 1);
            if (lap > 0 && !wait(&k_empty[st], (uint32_t)(lap - 1) & 1u)) break;
            const int key0 = key_of(it);
            const int pages = (min(kKeys, hi - key0) + kPageTok - 1) / kPageTok;
            const uint32_t bar = smem_u32(&k_full[st]);
            const bool scales = LINEAR && g.key_scales;
            if (lane == 0) mbar_expect_tx_addr(bar, (uint32_t)pages * (block_bytes + (scales ? kPageTok * 4u : 0u)));
            __syncwarp();
            if (lane < pages) {
                bulk_g2s_addr(sK + st * stage_bytes + lane * block_bytes, pool + (size_t)page * g.page_bytes, block_bytes, bar);
                if (scales)
                    bulk_g2s_addr(smem_u32(&k_scale[st][0]) + lane * kPageTok * 4u, p.pool + (size_t)page * g.page_bytes + (size_t)g.kv_heads * block_bytes + kvh * (kPageTok * 4),
                                  kPageTok * 4u, bar);
            }
            __syncwarp();
            n_req = it + 1;
            if (it == 0) request_queries();   // behind the first pages, which come from further away
        }
        // copies still in flight write this CTA's shared memory: wait for them (bounded) before leaving
        if (n_blocks > 0 && !mbar_wait_parked(smem_u32(&q_full), 0, kWaitLimit)) failed = true;
        for (int it = max(n_req - p.stages, 0); it < n_req; ++it)
            if (!mbar_wait_parked(smem_u32(&k_full[it % p.stages]), (uint32_t)(it / p.stages) & 1u, kWaitLimit)) failed = true;
        if (failed && lane == 0) atomicExch(p.status, 3);
    } else if (warp == 4) {
        // ================= scores ==================================================================================================
        const uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kKeys >> 3) << 17) | ((uint32_t)(kRows >> 4) << 24);
        // 16-column steps of every block that hold data (the columns behind them are zero). The loops are unrolled with constant
        // descriptor offsets: an MMA of 64 keys takes about 45 cycles, so its issue must not take longer.
        const uint64_t q_desc = desc_k_major(sQ, 1024);
        if (n_blocks > 0) wait(&q_full, 0);
        for (int it = 0; it < n_blocks && !failed; ++it) {
            const int st = it % p.stages;
            if (!wait(&k_full[st], (uint32_t)(it / p.stages) & 1u)) break;
            // the weights that were in this buffer have been used up; with as many stages or fewer the pages just waited for were
            // requested after that
            if (it >= kScores && p.stages > kScores && !wait(&k_empty[(it - kScores) % p.stages], (uint32_t)((it - kScores) / p.stages) & 1u)) break;
            tc_fence_after();
            const uint64_t kd = desc_k_major(sK + st * stage_bytes + (GROUPED ? (uint32_t)g.key_block * 1024u : 0u), group_stride);
            const uint32_t d = tmem + (uint32_t)(it % kScores) * kKeys;
            if (elect_one()) {
#pragma unroll
                for (int b = 0; b < kMaxBlocks; ++b)
                    if (b < g.query_blocks) {
#pragma unroll
                        for (int ks = 0; ks < 4; ++ks)
                            if (ks < g.steps[b])
                                umma_bf16(d, q_desc + (uint64_t)(b * (kRows * 128 >> 4) + 2 * ks), kd + (uint64_t)(b * (1024 >> 4) + 2 * ks), idesc_s, (b > 0 || ks > 0) ? 1u : 0u);
                    }
                umma_commit(&s_full[it % kScores]);
            }
            __syncwarp();
        }
        if (failed && lane == 0) atomicExch(p.status, 3);
    } else if (warp == 6) {
        // ================= outputs =================================================================================================
        const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(g.value_blocks * 64 >> 3) << 17) | ((uint32_t)(kRows >> 4) << 24);
        for (int it = 0; it < n_blocks; ++it) {
            const int st = it % p.stages;
            if (!wait(&p_full[it % kScores], (uint32_t)(it / kScores) & 1u)) break;
            const int keys = hi - key_of(it);
            if (keys < kKeys) {
                // cache rows past the last visible key may hold anything; their weights are 0, but 0 x NaN is not
                for (int r = keys; r < kKeys; ++r)
                    for (int c = lane; c < g.value_blocks * 8; c += 32)
                        st_shared_v4(sK + st * stage_bytes + (r >> 3) * group_stride + (c >> 3) * 1024 + (r & 7) * 128 + ((c & 7) << 4), 0, 0, 0, 0);
                fence_proxy_async();
                __syncwarp();
            }
            tc_fence_after();
            const uint64_t vd = desc_mn_major(sK + st * stage_bytes, group_stride);
            const uint32_t pa = tmem + (uint32_t)(it % kScores) * kKeys;
            if (elect_one()) {
#pragma unroll
                for (int half = 0; half < 2; ++half)
                    if (half == 0 || !dup)
#pragma unroll
                        for (int ks = 0; ks < kKeys / 16; ++ks)
                            umma_bf16_ts(tmem + kOCol, pa + (uint32_t)(half * (kKeys / 2) + 8 * ks), vd + (uint64_t)((uint32_t)ks * (group_stride >> 3)), idesc_o,
                                         (it > 0 || half > 0 || ks > 0) ? 1u : 0u);
                umma_commit(&k_empty[st]);
            }
            __syncwarp();
        }
        if (failed && lane == 0) atomicExch(p.status, 3);
    } else {
        // ================= warps 0-3: softmax, output ==============================================================================
        const int r = halves ? tid & (kRows / 2 - 1) : tid;   // row of the tile
        const bool lo_half = halves && warp >= 2;             // this copy of the row carries P_lo, or the second part
        int my_len = 0;
        if (r < live) {
            my_len = p.ctx_len[row0 + r / heads_n];
            if (my_len < 0 || my_len > cap) { atomicExch(p.status, 2); my_len = my_len < 0 ? 0 : cap; }
        }
        const int my_lo = GROUPED ? first_visible(g.mask, g.mask_size, max(my_len - 1, 0)) : max(my_len - g.mask_size, 0);
        float r1 = 0.f, r2 = 0.f;
        if (GROUPED && p.r1 && r < live) { r1 = p.r1[heads0 + r % heads_n]; if (!LINEAR) r2 = p.r2[heads0 + r % heads_n]; }
        const uint32_t t_lane = tmem + ((uint32_t)(warp * 32) << 16);
        // capped scores of up to 60 in log2 units need no running maximum: every row sees itself at no distance, so its largest weight lies
        // between 2^-60 and 2^60
        const bool fixed = GROUPED && p.cap_log2 > 0.f && p.cap_log2 <= 60.f;
        float m_run = fixed ? 0.f : -1e30f, l_run = 0.f;
        if ((halves ? warp & 1 : warp) < live_warps) {
            for (int it = 0; it < n_blocks; ++it) {
                const int buf = it % kScores;
                if (!wait(&s_full[buf], (uint32_t)(it / kScores) & 1u)) break;
                tc_fence_after();
                const uint32_t t_s = t_lane + (uint32_t)buf * kKeys;
                float s[kKeys];
                tmem_ld_32(t_s, *reinterpret_cast<float(*)[32]>(&s[0]));
                tmem_ld_32(t_s + 32u, *reinterpret_cast<float(*)[32]>(&s[32]));
                const int key0 = key_of(it);
                const int v_lo = my_lo - key0, v_hi = my_len - key0;   // visible keys of this block: [v_lo, v_hi)
                if constexpr (LINEAR) {
                    if (g.key_scales) {   // they have come with the pages; the wait is for this thread to see them
                        if (!wait(&k_full[it % p.stages], (uint32_t)(it / p.stages) & 1u)) break;
                        scale_columns(s, k_scale[it % p.stages]);
                    }
                    score_linear(s, p.scale_log2, p.cap_log2, r1, my_len - 1 - key0);
                } else if constexpr (GROUPED) {
                    score_log2(s, p.scale_log2, p.cap_log2, r1, r2, my_len - 1 - key0);
                }
                const float mul = GROUPED ? 1.f : p.scale_log2;
                if (v_lo > 0 || v_hi < kKeys) {
#pragma unroll
                    for (int j = 0; j < kKeys; ++j)
                        if (j < v_lo || j >= v_hi) s[j] = -INFINITY;
                }
                if (!fixed) {
                    float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
                    for (int j = 0; j < kKeys; ++j) mx[j & 3] = fmaxf(mx[j & 3], s[j]);
                    const float m_blk = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * mul;   // the scale is positive
                    float alpha = 1.f;
                    if (m_blk > m_run + kRescaleStep) {   // always at a row's first visible key
                        alpha = ex2f(m_run - m_blk);
                        m_run = m_blk;
                    }
                    if (it > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
                        // the product of the block before must be complete
                        if (!wait(&k_empty[(it - 1) % p.stages], (uint32_t)((it - 1) / p.stages) & 1u)) break;
                        tc_fence_after();
#pragma unroll 1
                        for (int c = 0; c < g.value_blocks * 2; ++c) {
                            float o[32];
                            tmem_ld_32(t_lane + kOCol + 32u * c, o);
#pragma unroll
                            for (int i = 0; i < 32; ++i) o[i] *= alpha;
                            tmem_st_32(t_lane + kOCol + 32u * c, *reinterpret_cast<uint32_t(*)[32]>(&o[0]));
                        }
                    }
                    l_run *= alpha;
                }
                const float neg_m = -m_run;
                float sum[4] = {0.f, 0.f, 0.f, 0.f};
                uint32_t hi_w[kKeys / 2], lo_w[kKeys / 2];
                if constexpr (GROUPED) {
                    const uint64_t nm = pair_of(neg_m, neg_m), one = pair_of(1.f, 1.f), minus = pair_of(-1.f, -1.f);
                    uint64_t acc[2] = {0, 0};
#pragma unroll
                    for (int i = 0; i < kKeys / 2; ++i) {
                        const float2 x = split(fma2(pair_of(s[2 * i], s[2 * i + 1]), one, nm));
                        const float p0 = ex2f(x.x), p1 = ex2f(x.y);
                        const uint64_t pp = pair_of(p0, p1);
                        acc[i & 1] = fma2(pp, one, acc[i & 1]);
                        hi_w[i] = pack_bf16x2(p0, p1);
                        const float2 lo = split(fma2(pair_of(bf16_lo(hi_w[i]), bf16_hi(hi_w[i])), minus, pp));
                        lo_w[i] = pack_bf16x2(lo.x, lo.y);
                    }
                    const float2 a0 = split(acc[0]), a1 = split(acc[1]);
                    sum[0] = a0.x; sum[1] = a0.y; sum[2] = a1.x; sum[3] = a1.y;
                } else {
#pragma unroll
                    for (int i = 0; i < kKeys / 2; ++i) {
                        const float p0 = ex2f(fmaf(s[2 * i], mul, neg_m)), p1 = ex2f(fmaf(s[2 * i + 1], mul, neg_m));
                        sum[i & 3] += p0 + p1;
                        hi_w[i] = pack_bf16x2(p0, p1);
                        lo_w[i] = pack_bf16x2(p0 - bf16_lo(hi_w[i]), p1 - bf16_hi(hi_w[i]));
                    }
                }
                if (!dup) {
                    tmem_st_32(t_s, hi_w);
                    tmem_st_32(t_s + 32u, lo_w);
                } else if (lo_half) {
                    tmem_st_32(t_s, lo_w);
                } else {
                    tmem_st_32(t_s, hi_w);
                }
                l_run += (sum[0] + sum[1]) + (sum[2] + sum[3]);
                asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
                tc_fence_before();
                mbar_arrive_addr(smem_u32(&p_full[buf]));
            }
            if (n_blocks > 0 && !failed) wait(&k_empty[(n_blocks - 1) % p.stages], (uint32_t)((n_blocks - 1) / p.stages) & 1u);
            tc_fence_after();
            const int cols = g.value_blocks * 64;
            const bool any = n_blocks > 0 && !failed;
            float* add = reinterpret_cast<float*>(smem_raw + (sK - smem_u32(smem_raw)));   // the other half of O, [row][cols + 4]; every page has been used
            const HeadOutput& ho = p.head_out;
            if (TWO && p.splits == 1) {
                const float inv = any && l_run > 0.f ? 1.f / l_run : 0.f;
                float4* mine = reinterpret_cast<float4*>(add + r * (cols + 4));
                if (lo_half && any) {
                    const float f = -ho.lambda * inv;
#pragma unroll 1
                    for (int c = 0; c < cols; c += 32) {
                        float o[32];
                        tmem_ld_32(t_lane + kOCol + (uint32_t)c, o);
#pragma unroll
                        for (int i = 0; i < 8; ++i) mine[c / 4 + i] = make_float4(f * o[4 * i], f * o[4 * i + 1], f * o[4 * i + 2], f * o[4 * i + 3]);
                    }
                }
                asm volatile("bar.sync 1, %0;\n" ::"r"(live_warps * 64) : "memory");
                if (!lo_half && any) {
                    float ss[4] = {0.f, 0.f, 0.f, 0.f};   // columns past vdim are zero
#pragma unroll 1
                    for (int c = 0; c < cols; c += 32) {
                        float o[32];
                        tmem_ld_32(t_lane + kOCol + (uint32_t)c, o);
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            float4 v = mine[c / 4 + i];
                            v.x = fmaf(o[4 * i], inv, v.x); v.y = fmaf(o[4 * i + 1], inv, v.y); v.z = fmaf(o[4 * i + 2], inv, v.z); v.w = fmaf(o[4 * i + 3], inv, v.w);
                            ss[0] = fmaf(v.x, v.x, ss[0]); ss[1] = fmaf(v.y, v.y, ss[1]); ss[2] = fmaf(v.z, v.z, ss[2]); ss[3] = fmaf(v.w, v.w, ss[3]);
                            mine[c / 4 + i] = v;
                        }
                    }
                    const float f = ho.scale / sqrtf(((ss[0] + ss[1]) + (ss[2] + ss[3])) / (float)g.vdim + ho.eps);
                    if (r < live) {
                        const int row = row0 + r / heads_n, head = heads0 + r % heads_n;
                        uint4* dst = reinterpret_cast<uint4*>(p.out + ((size_t)row * g.heads + head) * g.out_stride);
                        const __nv_bfloat16* gate = ho.gate ? ho.gate + (size_t)row * ho.gate_row + (size_t)head * ho.gate_stride : nullptr;
#pragma unroll 4
                        for (int c = 0; c < g.out_stride; c += 8) {
                            const float4 a = mine[c / 4], b = mine[c / 4 + 1];
                            float v[8] = {a.x * f, a.y * f, a.z * f, a.w * f, b.x * f, b.y * f, b.z * f, b.w * f};
                            if (gate) apply_gate(gate + c, v);
                            dst[c / 8] = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
                        }
                    }
                }
            }
            if (dup) {
                if (lo_half && any)
#pragma unroll 1
                    for (int c = 0; c < cols; c += 32) {
                        float o[32];
                        tmem_ld_32(t_lane + kOCol + (uint32_t)c, o);
                        float4* dst = reinterpret_cast<float4*>(add + r * (cols + 4) + c);
#pragma unroll
                        for (int i = 0; i < 8; ++i) dst[i] = make_float4(o[4 * i], o[4 * i + 1], o[4 * i + 2], o[4 * i + 3]);
                    }
                asm volatile("bar.sync 1, %0;\n" ::"r"(live_warps * 64) : "memory");
            }
            if (TWO ? p.splits > 1 : !lo_half) {
                const size_t token_head = (size_t)(row0 + r / heads_n) * g.heads + heads0 + r % heads_n;
                const size_t part = (((size_t)tile * gridDim.z + hb) * p.splits + blockIdx.y) * kRows + (TWO ? tid : r);
                if (p.splits > 1 && r < live) p.part_ml[part] = make_float2(m_run, failed ? 0.f : l_run);
                if (!TWO && p.sink && p.splits == 1) l_run += ex2f(fmaf(p.sink[heads0 + r % heads_n], kLog2e, -m_run));   // infinite: the output is 0
                const float inv = p.splits > 1 ? 1.f : l_run > 0.f ? 1.f / l_run : 0.f;
                if (any)
#pragma unroll 1
                    for (int c = 0; c < cols; c += 32) {
                        float o[32];
                        tmem_ld_32(t_lane + kOCol + (uint32_t)c, o);
                        if (dup) {
                            const float4* src = reinterpret_cast<const float4*>(add + r * (cols + 4) + c);
#pragma unroll
                            for (int i = 0; i < 8; ++i) { const float4 v = src[i]; o[4 * i] += v.x; o[4 * i + 1] += v.y; o[4 * i + 2] += v.z; o[4 * i + 3] += v.w; }
                        }
                        if (r < live && p.splits > 1) {
                            float4* dst = reinterpret_cast<float4*>(p.part_o + part * cols + c);
#pragma unroll
                            for (int i = 0; i < 8; ++i) dst[i] = make_float4(o[4 * i], o[4 * i + 1], o[4 * i + 2], o[4 * i + 3]);
                        } else if (!TWO && r < live) {
                            uint4* dst = reinterpret_cast<uint4*>(p.out + token_head * g.out_stride + c);
                            const __nv_bfloat16* gate = GROUPED && ho.gate ? ho.gate + (size_t)(row0 + r / heads_n) * ho.gate_row + (size_t)(heads0 + r % heads_n) * ho.gate_stride + c : nullptr;
#pragma unroll
                            for (int i = 0; i < 4; ++i)
                                if (c + 8 * i < g.out_stride) {
                                    float v[8];
#pragma unroll
                                    for (int e = 0; e < 8; ++e) v[e] = o[8 * i + e] * inv;
                                    if (GROUPED && gate) apply_gate(gate + 8 * i, v);
                                    dst[i] = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
                                }
                        }
                    }
            }
            if (failed && lane == 0) atomicExch(p.status, 3);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 4) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(p.tmem_cols) : "memory");
}

// One warp per (row of a tile): out = sum_s 2^(m_s - m) O_s / sum_s 2^(m_s - m) l_s, of both parts where there are two
struct CombineParams {
    const float* part_o;
    const float2* part_ml;
    const int *tile_row, *tile_rows;   // tile_rows null: one row each
    __nv_bfloat16* out;
    int heads, group, rows_per_token, head_blocks, splits, cols, out_stride, vdim;
    HeadOutput head_out;
    const float* sink;
    int part_rows;                     // rows of a part
};
template <bool TWO>
__global__ void __launch_bounds__(128) flash_combine_kernel(const CombineParams p) {
    constexpr int kTileRows = TWO ? kRows / 2 : kRows, kParts = TWO ? 2 : 1;
    pdl_launch_dependents();
    pdl_wait();
    const int tile = blockIdx.x, hb = blockIdx.z, r = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    const int kvh = hb / p.head_blocks, head_block = hb % p.head_blocks;
    const int heads_n = min(p.rows_per_token, p.group - head_block * kTileRows), heads0 = kvh * p.group + head_block * kTileRows;
    if (r >= (p.tile_rows ? p.tile_rows[tile] : 1) * heads_n) return;
    const int row = p.tile_row[tile] + r / heads_n, head = heads0 + r % heads_n;
    const HeadOutput& ho = p.head_out;
    constexpr int kSteps = 4;   // 64-column steps: values of up to 256 columns
    float2 acc[kSteps];
#pragma unroll
    for (int i = 0; i < kSteps; ++i) acc[i] = make_float2(0.f, 0.f);
#pragma unroll
    for (int q = 0; q < kParts; ++q) {
        const size_t part = ((size_t)tile * gridDim.z + hb) * p.splits * p.part_rows + q * (kRows / 2) + r;
        // a lane per split, 32 at a time
        auto part_of = [&](int s) { return s < p.splits ? p.part_ml[part + (size_t)s * p.part_rows] : make_float2(-1e30f, 0.f); };
        float m = -1e30f, l = 0.f;
        int best = 0;
        for (int s0 = 0; s0 < p.splits; s0 += 32) {
            const float2 v = part_of(s0 + lane);
            const float top = warp_max(v.y == 0.f ? -1e30f : v.x);
            if (top > m) { m = top; best = s0 + __ffs(__ballot_sync(0xffffffffu, v.y != 0.f && v.x == top)) - 1; }
        }
        for (int s0 = 0; s0 < p.splits; s0 += 32) { const float2 v = part_of(s0 + lane); l += v.y * ex2f(v.x - m); }
        l = warp_sum(l);
        if (!TWO && p.sink) l += ex2f(fmaf(p.sink[head], kLog2e, -m));
        const float inv = (l > 0.f ? 1.f / l : 0.f) * (q ? -ho.lambda : 1.f);
        for (int s0 = 0; s0 < p.splits; s0 += 32) {
            const float2 v = part_of(s0 + lane);
            const float mine = v.y == 0.f ? 0.f : ex2f(v.x - m) * inv;
            const int n = min(32, p.splits - s0);
#pragma unroll 4
            for (int k = 0; k < n; ++k) {
                const float w = __shfl_sync(0xffffffffu, mine, k);
                const int s = w != 0.f ? s0 + k : best;   // a split without a visible key left no output
                const float* src = p.part_o + (part + (size_t)s * p.part_rows) * p.cols + lane * 2;
#pragma unroll
                for (int i = 0; i < kSteps; ++i)
                    if (i * 64 < p.cols) {
                        const float2 o = *reinterpret_cast<const float2*>(src + i * 64);
                        acc[i].x = fmaf(w, o.x, acc[i].x);
                        acc[i].y = fmaf(w, o.y, acc[i].y);
                    }
            }
        }
    }
    float f = 1.f;
    if (TWO) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < kSteps; ++i) ss = fmaf(acc[i].x, acc[i].x, fmaf(acc[i].y, acc[i].y, ss));
        f = ho.scale / sqrtf(warp_sum(ss) / (float)p.vdim + ho.eps);
    }
    __nv_bfloat16* dst = p.out + ((size_t)row * p.heads + head) * p.out_stride;
    const __nv_bfloat16* gate = ho.gate ? ho.gate + (size_t)row * ho.gate_row + (size_t)head * ho.gate_stride : nullptr;
#pragma unroll
    for (int i = 0; i < kSteps; ++i) {
        const int c = i * 64 + lane * 2;
        if (c >= p.out_stride) break;
        float a = acc[i].x * f, b = acc[i].y * f;
        if (gate) {
            const uint32_t z = __ldg(reinterpret_cast<const uint32_t*>(gate + c));
            a = __fdividef(a, 1.f + __expf(-bf16_lo(z)));
            b = __fdividef(b, 1.f + __expf(-bf16_hi(z)));
        }
        *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(a, b);
    }
}

int tc_stages(int query_blocks, int blocks, int smem_kb = 220) {
    const int left = smem_kb * 1024 - 1024 - query_blocks * kRows * 128, stage = blocks * kKeys * 128;
    const int n = left > 0 ? left / stage : 0;
    return n > kMaxStages ? kMaxStages : n;
}
bool tc_fits(int query_blocks, int value_blocks, int blocks) {
    return value_blocks <= 4 && query_blocks <= kMaxBlocks && tc_stages(query_blocks, blocks) >= 2;
}
// two CTAs per SM: 256 columns of tensor memory and 112 KB of shared memory each
constexpr int kHalfSmemKb = 112;
bool tc_fits_twice(int query_blocks, int value_blocks, int blocks) { return value_blocks <= 2 && tc_stages(query_blocks, blocks, kHalfSmemKb) >= 2; }
size_t tc_scratch_bytes(int64_t n_tiles, int z_blocks, int splits, int value_blocks) {
    return (size_t)n_tiles * z_blocks * splits * kRows * ((size_t)value_blocks * 64 * 4 + 8);
}

// Launches the kernel and, with key splits, the merge. The caller has filled in everything but the fields set here.
template <bool GROUPED, int kScores, bool TWO = false, bool LINEAR = false>
int launch_flash(TcParams& p, int64_t n_tiles, void* d_scratch, cudaStream_t st) {
    constexpr int kTileRows = TWO ? kRows / 2 : kRows;
    const FlashShape& g = p.g;
    p.stages = tc_stages(g.query_blocks, g.blocks, kScores == 2 ? kHalfSmemKb : 220);
    p.head_blocks = ceil_div(g.group, kTileRows);
    p.rows_per_token = g.group < kTileRows ? g.group : kTileRows;
    p.tmem_cols = kScores * kKeys + g.value_blocks * 64 <= 256 ? 256 : 512;
    const int z = g.kv_heads * p.head_blocks;
    const size_t rows = (size_t)n_tiles * z * p.splits * kRows;
    p.part_o = static_cast<float*>(d_scratch);
    p.part_ml = reinterpret_cast<float2*>(p.part_o + rows * (g.value_blocks * 64));
    static PerDeviceOnce attr_once;
    if (attr_once.first_time()) GPTRS_CUDA_OK(cudaFuncSetAttribute(flash_tc_kernel<GROUPED, kScores, TWO, LINEAR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 221 * 1024));
    const size_t smem = (size_t)g.query_blocks * kRows * 128 + (size_t)p.stages * g.blocks * kKeys * 128 + 1024;
    int rc = launch_kernel(flash_tc_kernel<GROUPED, kScores, TWO, LINEAR>, dim3((unsigned)n_tiles, (unsigned)p.splits, (unsigned)z), dim3(kTcThreads), smem, st, 1, p);
    if (rc || p.splits == 1) return rc;
    CombineParams c = {p.part_o, p.part_ml, p.tile_row, p.tile_rows, p.out, g.heads, g.group, p.rows_per_token, p.head_blocks, p.splits, g.value_blocks * 64, g.out_stride, g.vdim, p.head_out, p.sink, kRows};
    // CTAs of four warps cover the rows of a tile
    return launch_kernel(flash_combine_kernel<TWO>, dim3((unsigned)n_tiles, kTileRows / 4, (unsigned)z), dim3(128), 0, st, 1, c);
}

}  // namespace
}  // namespace gptrs
