// Latent attention over a paged cache (no counterpart in gpt.rs): per token and layer the cache holds one normed latent
// vector c of `kv_rank` values and one rotated key part of `rot_dim` values, shared by all heads. The per-head key and value
// projections are absorbed into the query and the output,
//
//   score(i, j, h) = ((W_uk,h^T q_ih) . c_j + rot(q'_ih) . k'_j) * scale,      o_ih = W_uv,h (sum_j p_ijh c_j)
//
// so attention itself is multi-query attention with kv_rank + rot_dim key dimensions whose values are the first kv_rank of
// them, over a sliding window (position i sees i - window + 1 .. i). The two absorbed products are batched matmuls in front
// of and behind the kernels of this file:
//   latent_append_kernel        norm of the latent, rotation of the shared key part and of the queries, page write
//   latent_attention_kernel     plain CUDA-core attention, f32 or bf16 cache, any sizes (the f32 path)
//   latent_tc_kernel            tcgen05 flash attention, bf16, prompts and decode steps alike, kv_rank up to 256
//   latent_combine_kernel       merges the key splits of the former
//
// bf16 pages are laid out so that a page is one contiguous block that a single bulk copy drops into shared memory ready to
// be an operand of both products: [2 groups of 8 tokens][NB blocks of 64 columns][8 tokens][64 columns], 16-byte chunk j of
// token t at chunk j ^ (t & 7) (the 128-byte operand swizzle). The first ceil(kv_rank / 64) blocks hold c, the rest the
// rotated part; columns past either are zero. f32 pages are plain [16 tokens][kv_rank + rot_dim].
#include <cstdlib>

#include "umma_common.cuh"

namespace gptrs {
namespace {

constexpr int kPageTok = 16;
constexpr float kLog2e = 1.4426950408889634f;

__host__ __device__ inline int up(int v, int m) { return (v + m - 1) / m * m; }

struct Geometry {
    int heads, dim, rot, rank, window, rot_pairs;
    int q_head_stride, dkv_off, rot_off, q_row;
    int qa_head_stride, qa_rot_off, lat_stride;
    int nb, nbc;            // 64-column blocks of a cache row (bf16); of them latent
    long long page_bytes;
    float scale;
};
Geometry geometry(const gptrs_latent_attention& a) {
    Geometry g = {};
    g.heads = a.heads; g.dim = a.dim; g.rot = a.rot_dim; g.rank = a.kv_rank; g.window = a.window; g.rot_pairs = a.rot_dims / 2;
    g.q_head_stride = a.q_head_stride; g.dkv_off = a.dkv_offset; g.rot_off = a.rot_offset; g.q_row = a.q_row;
    g.qa_head_stride = a.qa_head_stride; g.qa_rot_off = a.qa_rot_offset; g.lat_stride = a.lat_head_stride;
    g.nbc = up(a.kv_rank, 64) / 64;
    g.nb = g.nbc + up(a.rot_dim, 64) / 64;
    g.page_bytes = a.page_bytes;
    g.scale = a.scale;
    return g;
}

// byte offset of 16-byte chunk `chunk` (8 columns) of token `t` inside a bf16 page
__device__ __forceinline__ int page_chunk(int t, int chunk, int nb) {
    return (t >> 3) * nb * 1024 + (chunk >> 3) * 1024 + (t & 7) * 128 + (((chunk & 7) ^ (t & 7)) << 4);
}

struct AppendParams {
    Geometry g;
    const void* qkv;            // [T][q_row]
    const int *pos, *slot, *page_table;
    const float* norm_w;        // [kv_rank]
    const float *cos_t, *sin_t; // [positions][rot_pairs]
    void* qa;                   // [T][heads][qa_head_stride]
    unsigned char* pool;
    int max_pages;
    float eps;
};

constexpr int kAppendThreads = 128;

template <typename TIn>
__device__ __forceinline__ float ld_val(const TIn* p) {
    if constexpr (sizeof(TIn) == 2) return __bfloat162float(*p);
    else return *p;
}

// values [8] of the rotated part starting at column 8 * chunk of `src` (rot columns), zero past the end
template <typename TIn>
__device__ __forceinline__ void rotated8(const TIn* src, int chunk, int rot, int pairs, const float* cs, const float* sn, float (&v)[8]) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int c = chunk * 8 + 2 * i;
        float a = c < rot ? ld_val(src + c) : 0.f, b = c + 1 < rot ? ld_val(src + c + 1) : 0.f;
        if ((c >> 1) < pairs) {
            const float co = cs[c >> 1], si = sn[c >> 1], u = a, w = b;
            a = u * co - w * si;
            b = w * co + u * si;
        }
        v[2 * i] = a; v[2 * i + 1] = b;
    }
}
__device__ __forceinline__ uint4 pack8(const float (&v)[8]) {
    return make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
}

template <bool BF16>
__global__ void __launch_bounds__(kAppendThreads) latent_append_kernel(const AppendParams p) {
    using T = typename std::conditional<BF16, __nv_bfloat16, float>::type;
    __shared__ float sh[kAppendThreads / 32];
    const Geometry& g = p.g;
    const int row = blockIdx.x, tid = threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    const T* q = static_cast<const T*>(p.qkv) + (size_t)row * g.q_row;
    const T* lat = q + g.dkv_off;
    const T* kr = q + g.rot_off;
    const int pos = p.pos[row];
    const float* cs = p.cos_t + (size_t)pos * g.rot_pairs;
    const float* sn = p.sin_t + (size_t)pos * g.rot_pairs;
    float ss = 0.f;
    for (int c = tid; c < g.rank; c += kAppendThreads) { const float v = ld_val(lat + c); ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) sh[tid >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < kAppendThreads / 32; ++w) ss += sh[w];
    const float inv = 1.f / sqrtf(ss / (float)g.rank + p.eps);
    unsigned char* page = p.pool + (size_t)p.page_table[(size_t)p.slot[row] * p.max_pages + pos / kPageTok] * g.page_bytes;
    const int t = pos % kPageTok;
    T* qa = static_cast<T*>(p.qa) + (size_t)row * g.heads * g.qa_head_stride;
    if constexpr (BF16) {
        const int rb = g.nb - g.nbc;   // blocks of the rotated part
        for (int j = tid; j < g.nb * 8; j += kAppendThreads) {
            float v[8];
            if (j < g.nbc * 8) {
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    const int c = j * 8 + e;
                    v[e] = c < g.rank ? ld_val(lat + c) * inv * p.norm_w[c] : 0.f;
                }
            } else {
                rotated8(kr, j - g.nbc * 8, g.rot, g.rot_pairs, cs, sn, v);
            }
            *reinterpret_cast<uint4*>(page + page_chunk(t, j, g.nb)) = pack8(v);
        }
        // queries: the rotated part, and zeros in the columns between the absorbed part and it
        const int z0 = up(g.rank, 8) / 8, zn = g.nbc * 8 - z0, per_head = zn + rb * 8;
        for (int j = tid; j < g.heads * per_head; j += kAppendThreads) {
            const int h = j / per_head, e = j % per_head;
            float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
            int chunk = z0 + e;
            if (e >= zn) {
                chunk = g.nbc * 8 + (e - zn);
                rotated8(q + h * g.q_head_stride + (g.q_head_stride - up(g.rot, 8)), e - zn, g.rot, g.rot_pairs, cs, sn, v);
            }
            *reinterpret_cast<uint4*>(qa + (size_t)h * g.qa_head_stride + chunk * 8) = pack8(v);
        }
    } else {
        float* dst = reinterpret_cast<float*>(page) + (size_t)t * (g.rank + g.rot);
        for (int c = tid; c < g.rank; c += kAppendThreads) dst[c] = ld_val(lat + c) * inv * p.norm_w[c];
        auto rotate = [&](const T* src, float* out, int c) {
            const int i = c >> 1;
            float v = ld_val(src + c);
            if (i < g.rot_pairs) v = (c & 1) ? v * cs[i] + ld_val(src + c - 1) * sn[i] : v * cs[i] - ld_val(src + c + 1) * sn[i];
            out[c] = v;
        };
        for (int c = tid; c < g.rot; c += kAppendThreads) rotate(kr, dst + g.rank, c);
        for (int j = tid; j < g.heads * g.rot; j += kAppendThreads) {
            const int h = j / g.rot, c = j % g.rot;
            rotate(q + h * g.q_head_stride + g.dim, reinterpret_cast<float*>(qa) + (size_t)h * g.qa_head_stride + g.qa_rot_off, c);
        }
    }
}

// ---- plain attention: one CTA per (head, row) ---------------------------------------------------------------------------------
struct AttnParams {
    Geometry g;
    const void* qa;
    const unsigned char* pool;
    const int *page_table, *slot, *ctx_len;
    void* out;                  // [T][heads][lat_stride]
    int* status;
    int max_pages;
};
constexpr int kPlainThreads = 128;
constexpr int kPlainCols = 8;   // latent columns per thread: kv_rank up to 1024

template <bool BF16>
__global__ void __launch_bounds__(kPlainThreads) latent_attention_kernel(const AttnParams p) {
    extern __shared__ __align__(16) float la_smem[];
    const Geometry& g = p.g;
    float* qs = la_smem;                       // [qa_head_stride]
    float* ps = la_smem + g.qa_head_stride;    // [kPlainThreads]
    __shared__ long long s_row[kPlainThreads]; // byte offset of the page of every key of the chunk
    __shared__ float sh[8];
    const int head = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    int len = p.ctx_len[row];
    if (len < 0 || len > p.max_pages * kPageTok) { if (tid == 0) atomicExch(p.status, 2); len = len < 0 ? 0 : p.max_pages * kPageTok; }
    const int lo = len > g.window ? len - g.window : 0;
    const int* pt = p.page_table + (size_t)p.slot[row] * p.max_pages;
    const size_t qo = ((size_t)row * g.heads + head) * g.qa_head_stride;
    for (int c = tid; c < g.qa_head_stride; c += kPlainThreads)
        qs[c] = BF16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.qa)[qo + c]) : static_cast<const float*>(p.qa)[qo + c];
    __syncthreads();
    float acc[kPlainCols];
#pragma unroll
    for (int i = 0; i < kPlainCols; ++i) acc[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int j0 = lo; j0 < len; j0 += kPlainThreads) {
        const int n = min(kPlainThreads, len - j0);
        float s = -INFINITY;
        if (tid < n) {
            const int j = j0 + tid;
            const long long base = (long long)pt[j / kPageTok] * g.page_bytes;
            s_row[tid] = base;
            s = 0.f;
            if constexpr (BF16) {
                const unsigned char* pg = p.pool + base;
                for (int k = 0; k < g.nb * 8; ++k) {
                    const uint4 u = __ldg(reinterpret_cast<const uint4*>(pg + page_chunk(j % kPageTok, k, g.nb)));
                    const float* qk = qs + k * 8;
                    s = fmaf(qk[0], bf16_lo(u.x), s); s = fmaf(qk[1], bf16_hi(u.x), s);
                    s = fmaf(qk[2], bf16_lo(u.y), s); s = fmaf(qk[3], bf16_hi(u.y), s);
                    s = fmaf(qk[4], bf16_lo(u.z), s); s = fmaf(qk[5], bf16_hi(u.z), s);
                    s = fmaf(qk[6], bf16_lo(u.w), s); s = fmaf(qk[7], bf16_hi(u.w), s);
                }
            } else {
                const float* kv = reinterpret_cast<const float*>(p.pool + base) + (size_t)(j % kPageTok) * (g.rank + g.rot);
                for (int c = 0; c < g.rank + g.rot; ++c) s = fmaf(qs[c], __ldg(kv + c), s);
            }
            s *= g.scale;
        }
        const float wm = warp_max(s);
        if ((tid & 31) == 0) sh[tid >> 5] = wm;
        __syncthreads();
        const float m_new = fmaxf(m, fmaxf(fmaxf(sh[0], sh[1]), fmaxf(sh[2], sh[3])));
        const float e = tid < n ? expf(s - m_new) : 0.f;
        ps[tid] = e;
        const float ws = warp_sum(e);
        if ((tid & 31) == 0) sh[4 + (tid >> 5)] = ws;
        __syncthreads();
        const float alpha = expf(m - m_new);   // 0 for the first chunk
        l = l * alpha + ((sh[4] + sh[5]) + (sh[6] + sh[7]));
        m = m_new;
#pragma unroll
        for (int i = 0; i < kPlainCols; ++i) {
            const int c = tid + i * kPlainThreads;
            if (c >= g.rank) break;
            float a = acc[i] * alpha;
            for (int k = 0; k < n; ++k) {
                const int t = (j0 + k) % kPageTok;
                float v;
                if constexpr (BF16)
                    v = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(p.pool + s_row[k] + page_chunk(t, c >> 3, g.nb) + (c & 7) * 2));
                else
                    v = __ldg(reinterpret_cast<const float*>(p.pool + s_row[k]) + (size_t)t * (g.rank + g.rot) + c);
                a = fmaf(ps[k], v, a);
            }
            acc[i] = a;
        }
        __syncthreads();
    }
    const size_t oo = ((size_t)row * g.heads + head) * g.lat_stride;
    const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
    for (int i = 0; i < kPlainCols; ++i) {
        const int c = tid + i * kPlainThreads;
        if (c >= g.lat_stride) break;
        const float v = c < g.rank ? acc[i] * inv : 0.f;
        if (BF16) static_cast<__nv_bfloat16*>(p.out)[oo + c] = __float2bfloat16_rn(v);
        else static_cast<float*>(p.out)[oo + c] = v;
    }
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
// tensor pipe idle between them. A decode step is the case of one token per tile, with the keys split over the y dimension of the grid; latent_combine_kernel merges the parts.
// Tiles of up to 64 rows (decode steps of up to 64 heads) hold every row twice: rows 64 .. 127 repeat the queries, hence the
// scores and the softmax, and put P_lo where the first copy puts P_hi, so that one product serves both terms; the two halves of
// O are added at the end. Every wait is bounded (status 3).
constexpr int kRows = 128;
constexpr int kKeys = 64;
constexpr int kTcThreads = 224;
constexpr int kScores = 3;           // score buffers in tensor memory
constexpr int kMaxStages = 6;
constexpr int kMaxBlocks = 6;        // 64-column blocks of a cache row
constexpr uint32_t kWaitLimit = 1u << 16;
constexpr float kRescaleStep = 8.f;
constexpr uint32_t kOCol = kScores * kKeys;

struct TcParams {
    CUtensorMap q_map;                 // absorbed queries: [64 columns][nb blocks][T x heads rows], 128-byte swizzle
    Geometry g;
    const unsigned char* pool;
    const int *page_table, *slot, *ctx_len;
    const int *tile_row, *tile_rows;   // first row and number of rows of every tile
    __nv_bfloat16* out;
    float* part_o;                     // splits > 1: [tile * head blocks][split][128][64 nbc]
    float2* part_ml;                   // [tile * head blocks][split][128]: running maximum (log2 units), sum
    int* status;
    int max_pages, splits, stages, head_blocks, rows_per_token;
    uint32_t tmem_cols;
    float scale_log2;
};

__device__ __forceinline__ void tma_q(uint32_t dst, const CUtensorMap* map, int block, int row, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];\n" ::"r"(dst), "l"(map),
                 "r"(0), "r"(block), "r"(row), "r"(bar)
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

__global__ void __launch_bounds__(kTcThreads, 1) latent_tc_kernel(const __grid_constant__ TcParams p) {
    extern __shared__ unsigned char smem_raw[];
    __shared__ __align__(8) uint64_t k_full[kMaxStages], k_empty[kMaxStages], s_full[kScores], p_full[kScores], q_full;
    __shared__ uint32_t tmem_holder;
    const Geometry& g = p.g;
    const uint32_t smem = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t stage_bytes = (uint32_t)(kKeys * 128) * g.nb, group_stride = (uint32_t)g.nb * 1024u;
    const uint32_t sQ = smem, sK = smem + (uint32_t)g.nb * (kRows * 128);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (warp == 4) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(smem_u32(&tmem_holder)), "r"(p.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    if (tid == 32 * 5) asm volatile("prefetch.tensormap [%0];\n" ::"l"(&p.q_map) : "memory");
    pdl_wait();
    const int tile = (int)gridDim.x - 1 - (int)blockIdx.x;   // long contexts come last in a token list: start them first
    const int row0 = p.tile_row[tile], n_tok = p.tile_rows[tile], hb = blockIdx.z;
    const int heads0 = hb * kRows, heads_n = min(p.rows_per_token, g.heads - heads0);   // heads of this CTA per token
    const int live = n_tok * heads_n;
    const int live_warps = (live + 31) / 32;
    const bool dup = live <= kRows / 2;
    if (tid == 0) {
        for (int i = 0; i < p.stages; ++i) { mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); }
        for (int i = 0; i < kScores; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], (uint32_t)live_warps * (dup ? 64 : 32)); }
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
    const int lo = max(first_len - g.window, 0) & ~(kPageTok - 1);
    const int n_all = hi > lo ? (hi - lo + kKeys - 1) / kKeys : 0;
    const int kb0 = (int)((int64_t)n_all * blockIdx.y / p.splits), kb1 = (int)((int64_t)n_all * (blockIdx.y + 1) / p.splits);
    const int n_blocks = kb1 - kb0;
    const int key_base = lo + kb0 * kKeys;
    bool failed = false;
    auto wait = [&](uint64_t* bar, uint32_t parity) {   // whole warp
        if (!failed && !mbar_wait_parked(smem_u32(bar), parity, kWaitLimit)) failed = true;
        failed = __any_sync(0xffffffffu, failed);
        return !failed;
    };

    if (warp == 5) {
        // ================= pages and queries =======================================================================================
        const int* pt = p.page_table + (size_t)slot0 * p.max_pages;
        const uint32_t page_bytes = (uint32_t)g.page_bytes;
        auto page_of = [&](int it) {   // lane j: the j-th page of block `it`
            const int key0 = key_base + it * kKeys;
            return it < n_blocks && lane < (min(kKeys, hi - key0) + kPageTok - 1) / kPageTok ? __ldg(pt + key0 / kPageTok + lane) : 0;
        };
        int n_req = 0, page_next = page_of(0);
        auto request_queries = [&]() {   // 32 rows x 64 columns per copy; rows past the live ones are other queries, whose results nobody reads
            if (lane == 0) {
                const uint32_t bar = smem_u32(&q_full);
                mbar_expect_tx_addr(bar, (uint32_t)(live_warps * (dup ? 2 : 1) * g.nb) * 4096u);
                for (int w = 0; w < live_warps; ++w)
                    for (int b = 0; b < g.nb; ++b) {
                        const uint32_t dst = sQ + (uint32_t)(b * kRows + w * 32) * 128u;
                        tma_q(dst, &p.q_map, b, row0 * g.heads + heads0 + w * 32, bar);
                        if (dup) tma_q(dst + (kRows / 2) * 128u, &p.q_map, b, row0 * g.heads + heads0 + w * 32, bar);
                    }
            }
            __syncwarp();
        };
        for (int it = 0; it < n_blocks; ++it) {
            const int st = it % p.stages, lap = it / p.stages;
            const int page = page_next;
            page_next = page_of(it + 1);
            if (lap > 0 && !wait(&k_empty[st], (uint32_t)(lap - 1) & 1u)) break;
            const int key0 = key_base + it * kKeys;
            const int pages = (min(kKeys, hi - key0) + kPageTok - 1) / kPageTok;
            const uint32_t bar = smem_u32(&k_full[st]);
            if (lane == 0) mbar_expect_tx_addr(bar, (uint32_t)pages * page_bytes);
            __syncwarp();
            if (lane < pages)
                bulk_g2s_addr(sK + st * stage_bytes + lane * page_bytes, p.pool + (size_t)page * page_bytes, page_bytes, bar);
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
        int steps[kMaxBlocks];
#pragma unroll
        for (int b = 0; b < kMaxBlocks; ++b) {
            const int cols = b < g.nbc ? g.rank - b * 64 : g.rot - (b - g.nbc) * 64;
            steps[b] = b < g.nb ? min((cols + 15) / 16, 4) : 0;
        }
        const uint64_t q_desc = desc_k_major(sQ, 1024);
        if (n_blocks > 0) wait(&q_full, 0);
        for (int it = 0; it < n_blocks && !failed; ++it) {
            const int st = it % p.stages;
            if (!wait(&k_full[st], (uint32_t)(it / p.stages) & 1u)) break;
            // the weights that were in this buffer have been used up; with three stages or fewer the pages just waited for were
            // requested after that
            if (it >= kScores && p.stages > kScores && !wait(&k_empty[(it - kScores) % p.stages], (uint32_t)((it - kScores) / p.stages) & 1u)) break;
            tc_fence_after();
            const uint64_t kd = desc_k_major(sK + st * stage_bytes, group_stride);
            const uint32_t d = tmem + (uint32_t)(it % kScores) * kKeys;
            if (elect_one()) {
#pragma unroll
                for (int b = 0; b < kMaxBlocks; ++b)
                    if (b < g.nb) {
#pragma unroll
                        for (int ks = 0; ks < 4; ++ks)
                            if (ks < steps[b])
                                umma_bf16(d, q_desc + (uint64_t)(b * (kRows * 128 >> 4) + 2 * ks), kd + (uint64_t)(b * (1024 >> 4) + 2 * ks), idesc_s, (b > 0 || ks > 0) ? 1u : 0u);
                    }
                umma_commit(&s_full[it % kScores]);
            }
            __syncwarp();
        }
        if (failed && lane == 0) atomicExch(p.status, 3);
    } else if (warp == 6) {
        // ================= outputs =================================================================================================
        const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(g.nbc * 64 >> 3) << 17) | ((uint32_t)(kRows >> 4) << 24);
        for (int it = 0; it < n_blocks; ++it) {
            const int st = it % p.stages;
            if (!wait(&p_full[it % kScores], (uint32_t)(it / kScores) & 1u)) break;
            const int keys = hi - (key_base + it * kKeys);
            if (keys < kKeys) {
                // cache rows past the last visible key may hold anything; their weights are 0, but 0 x NaN is not
                for (int r = keys; r < kKeys; ++r)
                    for (int c = lane; c < g.nbc * 8; c += 32)
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
        const int r = dup ? tid & (kRows / 2 - 1) : tid;   // row of the tile
        const bool lo_half = dup && warp >= 2;             // this copy of the row carries P_lo
        int my_len = 0;
        if (r < live) {
            my_len = p.ctx_len[row0 + r / heads_n];
            if (my_len < 0 || my_len > cap) { atomicExch(p.status, 2); my_len = my_len < 0 ? 0 : cap; }
        }
        const int my_lo = max(my_len - g.window, 0);
        const uint32_t t_lane = tmem + ((uint32_t)(warp * 32) << 16);
        float m_run = -1e30f, l_run = 0.f;
        if ((dup ? warp & 1 : warp) < live_warps) {
            for (int it = 0; it < n_blocks; ++it) {
                const int buf = it % kScores;
                if (!wait(&s_full[buf], (uint32_t)(it / kScores) & 1u)) break;
                tc_fence_after();
                const uint32_t t_s = t_lane + (uint32_t)buf * kKeys;
                float s[kKeys];
                tmem_ld_32(t_s, *reinterpret_cast<float(*)[32]>(&s[0]));
                tmem_ld_32(t_s + 32u, *reinterpret_cast<float(*)[32]>(&s[32]));
                const int key0 = key_base + it * kKeys;
                const int v_lo = my_lo - key0, v_hi = my_len - key0;   // visible keys of this block: [v_lo, v_hi)
                if (v_lo > 0 || v_hi < kKeys) {
#pragma unroll
                    for (int j = 0; j < kKeys; ++j)
                        if (j < v_lo || j >= v_hi) s[j] = -INFINITY;
                }
                float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
                for (int j = 0; j < kKeys; ++j) mx[j & 3] = fmaxf(mx[j & 3], s[j]);
                const float m_blk = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * p.scale_log2;   // the scale is positive
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
                    for (int c = 0; c < g.nbc * 2; ++c) {
                        float o[32];
                        tmem_ld_32(t_lane + kOCol + 32u * c, o);
#pragma unroll
                        for (int i = 0; i < 32; ++i) o[i] *= alpha;
                        tmem_st_32(t_lane + kOCol + 32u * c, *reinterpret_cast<uint32_t(*)[32]>(&o[0]));
                    }
                }
                l_run *= alpha;
                const float neg_m = -m_run;
                float sum[4] = {0.f, 0.f, 0.f, 0.f};
                uint32_t hi_w[kKeys / 2], lo_w[kKeys / 2];
#pragma unroll
                for (int i = 0; i < kKeys / 2; ++i) {
                    const float p0 = ex2f(fmaf(s[2 * i], p.scale_log2, neg_m)), p1 = ex2f(fmaf(s[2 * i + 1], p.scale_log2, neg_m));
                    sum[i & 3] += p0 + p1;
                    hi_w[i] = pack_bf16x2(p0, p1);
                    lo_w[i] = pack_bf16x2(p0 - bf16_lo(hi_w[i]), p1 - bf16_hi(hi_w[i]));
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
            const int cols = g.nbc * 64;
            const bool any = n_blocks > 0 && !failed;
            float* add = reinterpret_cast<float*>(smem_raw + (sK - smem_u32(smem_raw)));   // dup: the P_lo half of O, [row][cols + 4]; every page has been used
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
            if (!lo_half) {
                const size_t token_head = (size_t)(row0 + r / heads_n) * g.heads + heads0 + r % heads_n;
                const size_t part = (((size_t)tile * p.head_blocks + hb) * p.splits + blockIdx.y) * kRows + r;
                if (p.splits > 1 && r < live) p.part_ml[part] = make_float2(m_run, failed ? 0.f : l_run);
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
                        } else if (r < live) {
                            uint4* dst = reinterpret_cast<uint4*>(p.out + token_head * g.lat_stride + c);
#pragma unroll
                            for (int i = 0; i < 4; ++i)
                                if (c + 8 * i < g.lat_stride)
                                    dst[i] = make_uint4(pack_bf16x2(o[8 * i] * inv, o[8 * i + 1] * inv), pack_bf16x2(o[8 * i + 2] * inv, o[8 * i + 3] * inv),
                                                        pack_bf16x2(o[8 * i + 4] * inv, o[8 * i + 5] * inv), pack_bf16x2(o[8 * i + 6] * inv, o[8 * i + 7] * inv));
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

// One warp per (row of a tile): out = sum_s 2^(m_s - m) O_s / sum_s 2^(m_s - m) l_s
struct CombineParams {
    const float* part_o;
    const float2* part_ml;
    const int *tile_row, *tile_rows;
    __nv_bfloat16* out;
    int heads, rows_per_token, head_blocks, splits, cols, lat_stride;
};
__global__ void __launch_bounds__(128) latent_combine_kernel(const CombineParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int tile = blockIdx.x, hb = blockIdx.z, r = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    const int heads0 = hb * kRows, heads_n = min(p.rows_per_token, p.heads - heads0);
    if (r >= p.tile_rows[tile] * heads_n) return;
    const size_t part = ((size_t)tile * p.head_blocks + hb) * p.splits * kRows + r;
    float m = -1e30f;
    for (int s = 0; s < p.splits; ++s) m = fmaxf(m, p.part_ml[part + (size_t)s * kRows].x);
    float l = 0.f;
    for (int s = 0; s < p.splits; ++s) { const float2 v = p.part_ml[part + (size_t)s * kRows]; l += v.y * ex2f(v.x - m); }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    __nv_bfloat16* dst = p.out + ((size_t)(p.tile_row[tile] + r / heads_n) * p.heads + heads0 + r % heads_n) * p.lat_stride;
    for (int c = lane * 2; c < p.lat_stride; c += 64) {
        float a = 0.f, b = 0.f;
        for (int s = 0; s < p.splits; ++s) {
            const float2 v = p.part_ml[part + (size_t)s * kRows];
            if (v.y == 0.f) continue;   // a split without a visible key left no output
            const float w = ex2f(v.x - m);
            const float2 o = *reinterpret_cast<const float2*>(p.part_o + (part + (size_t)s * kRows) * p.cols + c);
            a = fmaf(w, o.x, a);
            b = fmaf(w, o.y, b);
        }
        *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(a * inv, b * inv);
    }
}

int encode_queries(const void* qa, const Geometry& g, int64_t n_tokens, CUtensorMap* map) {
    EncodeTiledFn enc = encode_fn();
    if (!enc) return fail(GPTRS_EXECUTION, "cuTensorMapEncodeTiled is not available");
    cuuint64_t dims[3] = {64, (cuuint64_t)g.nb, (cuuint64_t)(n_tokens * g.heads)};
    cuuint64_t strides[2] = {128, (cuuint64_t)g.qa_head_stride * 2};
    cuuint32_t box[3] = {64, 1, 32};
    cuuint32_t estr[3] = {1, 1, 1};
    CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(qa), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                     CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(GPTRS_EXECUTION, "cuTensorMapEncodeTiled failed for latent attention (" + std::to_string((int)r) + ")");
    return GPTRS_OK;
}

int tc_stages(int nb) {
    const int left = 220 * 1024 - 1024 - nb * kRows * 128, stage = nb * kKeys * 128;
    const int n = left > 0 ? left / stage : 0;
    return n > kMaxStages ? kMaxStages : n;
}
bool tc_fits(const Geometry& g) { return g.nbc <= 4 && g.nb <= kMaxBlocks && tc_stages(g.nb) >= 2; }

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" {

int gptrs_cuda_latent_layout(gptrs_latent_attention* a) {
    GPTRS_REQUIRE(a, "null pointer");
    GPTRS_REQUIRE(a->heads > 0 && a->dim > 0 && a->rot_dim > 0 && a->vdim > 0 && a->kv_rank > 0 && a->window > 0, "latent attention: sizes must be positive");
    GPTRS_REQUIRE(a->rot_dims >= 0 && a->rot_dims <= a->rot_dim && a->rot_dims % 2 == 0, "latent attention: rotated dimensions");
    GPTRS_REQUIRE(a->scale > 0.f, "latent attention: the scale must be positive");
    GPTRS_REQUIRE(a->dtype == GPTRS_F32 || a->dtype == GPTRS_BF16, "latent attention: f32 or bf16");
    if (a->kv_rank > kPlainThreads * kPlainCols) return fail(GPTRS_UNIMPLEMENTED, "latent attention: kv_rank above 1024");
    if (a->dtype == GPTRS_F32) {
        a->q_head_stride = a->dim + a->rot_dim;
        a->dkv_offset = a->heads * a->q_head_stride;
        a->rot_offset = a->dkv_offset + a->kv_rank;
        a->q_row = a->rot_offset + a->rot_dim;
        a->q_rot_offset = a->dim;
        a->qa_head_stride = a->kv_rank + a->rot_dim;
        a->qa_rot_offset = a->kv_rank;
        a->lat_head_stride = a->kv_rank;
        a->out_head_stride = a->vdim;
        a->page_bytes = (int64_t)kPageTok * (a->kv_rank + a->rot_dim) * 4;
    } else {
        a->q_rot_offset = up(a->dim, 8);
        a->q_head_stride = a->q_rot_offset + up(a->rot_dim, 8);
        a->dkv_offset = a->heads * a->q_head_stride;
        a->rot_offset = a->dkv_offset + up(a->kv_rank, 8);
        a->q_row = a->rot_offset + up(a->rot_dim, 8);
        a->qa_rot_offset = up(a->kv_rank, 64);
        a->qa_head_stride = a->qa_rot_offset + up(a->rot_dim, 64);
        a->lat_head_stride = up(a->kv_rank, 8);
        a->out_head_stride = up(a->vdim, 8);
        a->page_bytes = (int64_t)kPageTok * a->qa_head_stride * 2;
    }
    return GPTRS_OK;
}

int gptrs_cuda_latent_append(const gptrs_latent_attention* a, const void* d_qkv, const int32_t* d_positions, const int32_t* d_slot,
                             const int32_t* d_page_table, int64_t max_pages, const float* d_norm_w, float eps, const float* d_cos, const float* d_sin,
                             void* d_qa, void* d_pool, int64_t n_tokens, void* stream) {
    GPTRS_REQUIRE(a && d_qkv && d_positions && d_slot && d_page_table && d_norm_w && d_qa && d_pool, "null pointer");
    GPTRS_REQUIRE(a->q_row > 0 && max_pages > 0 && (a->rot_dims == 0 || (d_cos && d_sin)), "latent attention: layout not filled in, or no rotation tables");
    if (n_tokens == 0) return GPTRS_OK;
    AppendParams p = {geometry(*a), d_qkv, d_positions, d_slot, d_page_table, d_norm_w, d_cos, d_sin, d_qa, static_cast<unsigned char*>(d_pool), (int)max_pages, eps};
    const dim3 grid((unsigned)n_tokens);
    return a->dtype == GPTRS_BF16 ? launch_kernel(latent_append_kernel<true>, grid, dim3(kAppendThreads), 0, as_stream(stream), 1, p)
                                  : launch_kernel(latent_append_kernel<false>, grid, dim3(kAppendThreads), 0, as_stream(stream), 1, p);
}

int gptrs_cuda_latent_tile_tokens(const gptrs_latent_attention* a) {
    if (!a || a->dtype != GPTRS_BF16 || a->heads < 1 || !tc_fits(geometry(*a))) return 0;
    return a->heads >= kRows ? 1 : kRows / a->heads;
}

int gptrs_cuda_latent_splits(const gptrs_latent_attention* a, int64_t n_tiles, int64_t max_ctx_len) {
    if (!a || n_tiles <= 0 || gptrs_cuda_latent_tile_tokens(a) == 0) return 1;
    const int64_t span = (max_ctx_len < (int64_t)a->window + gptrs_cuda_latent_tile_tokens(a) ? max_ctx_len : (int64_t)a->window + gptrs_cuda_latent_tile_tokens(a));
    const int64_t blocks = (span + kPageTok - 1 + kKeys - 1) / kKeys;
    int64_t s = sm_count() / (n_tiles * ceil_div(a->heads, kRows));
    if (s > blocks) s = blocks;
    return (int)(s < 1 ? 1 : s);
}

size_t gptrs_cuda_latent_scratch_bytes(const gptrs_latent_attention* a, int64_t n_tiles, int splits) {
    if (!a || splits <= 1) return 0;
    return (size_t)n_tiles * ceil_div(a->heads, kRows) * splits * kRows * ((size_t)up(a->kv_rank, 64) * 4 + 8);
}

int gptrs_cuda_latent_attention(const gptrs_latent_attention* a, const void* d_qa, const void* d_pool, const int32_t* d_page_table, int64_t max_pages,
                                const int32_t* d_slot, const int32_t* d_ctx_len, const int32_t* d_tile_row, const int32_t* d_tile_rows, int64_t n_tiles,
                                int splits, void* d_out, void* d_scratch, size_t scratch_bytes, int32_t* d_status, int64_t n_tokens, void* stream) {
    GPTRS_REQUIRE(a && d_qa && d_pool && d_page_table && d_slot && d_ctx_len && d_out && d_status, "null pointer");
    GPTRS_REQUIRE(a->q_row > 0 && max_pages > 0 && max_pages * kPageTok < ((int64_t)1 << 30), "latent attention: layout not filled in, or a bad page table");
    if (n_tokens == 0) return GPTRS_OK;
    const Geometry g = geometry(*a);
    cudaStream_t st = as_stream(stream);
    if (n_tiles <= 0) {   // plain kernel: every row by itself
        GPTRS_REQUIRE(n_tokens <= 65535 && a->heads <= 0x7fffffff, "latent attention: too many rows in one launch");
        AttnParams p = {g, d_qa, static_cast<const unsigned char*>(d_pool), d_page_table, d_slot, d_ctx_len, d_out, d_status, (int)max_pages};
        const size_t smem = ((size_t)g.qa_head_stride + kPlainThreads) * 4;
        const dim3 grid((unsigned)g.heads, (unsigned)n_tokens);
        return a->dtype == GPTRS_BF16 ? launch_kernel(latent_attention_kernel<true>, grid, dim3(kPlainThreads), smem, st, 1, p)
                                      : launch_kernel(latent_attention_kernel<false>, grid, dim3(kPlainThreads), smem, st, 1, p);
    }
    if (gptrs_cuda_latent_tile_tokens(a) == 0) return fail(GPTRS_UNIMPLEMENTED, "latent attention: these sizes do not fit the tensor-core kernel (pass n_tiles = 0)");
    GPTRS_REQUIRE(d_tile_row && d_tile_rows && splits >= 1 && splits <= 65535, "latent attention: tile list");
    GPTRS_REQUIRE((reinterpret_cast<uintptr_t>(d_pool) & 15) == 0 && (reinterpret_cast<uintptr_t>(d_qa) & 15) == 0 && (reinterpret_cast<uintptr_t>(d_out) & 15) == 0,
                  "latent attention: 16-byte alignment");
    const size_t need = gptrs_cuda_latent_scratch_bytes(a, n_tiles, splits);
    GPTRS_REQUIRE(need == 0 || (d_scratch && scratch_bytes >= need), "latent attention: scratch too small");
    TcParams p = {};
    p.g = g;
    int erc = encode_queries(d_qa, g, n_tokens, &p.q_map);
    if (erc) return erc;
    p.pool = static_cast<const unsigned char*>(d_pool);
    p.page_table = d_page_table; p.slot = d_slot; p.ctx_len = d_ctx_len; p.tile_row = d_tile_row; p.tile_rows = d_tile_rows;
    p.out = static_cast<__nv_bfloat16*>(d_out);
    p.status = d_status;
    p.max_pages = (int)max_pages; p.splits = splits; p.stages = tc_stages(g.nb);
    p.head_blocks = ceil_div(g.heads, kRows);
    p.rows_per_token = g.heads < kRows ? g.heads : kRows;
    p.tmem_cols = kOCol + g.nbc * 64 <= 256 ? 256 : 512;
    p.scale_log2 = kLog2e * g.scale;
    const size_t rows = (size_t)n_tiles * p.head_blocks * splits * kRows;
    p.part_o = static_cast<float*>(d_scratch);
    p.part_ml = reinterpret_cast<float2*>(p.part_o + rows * (g.nbc * 64));
    static PerDeviceOnce attr_once;
    if (attr_once.first_time()) GPTRS_CUDA_OK(cudaFuncSetAttribute(latent_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 221 * 1024));
    const size_t smem = (size_t)g.nb * kRows * 128 + (size_t)p.stages * g.nb * kKeys * 128 + 1024;
    int rc = launch_kernel(latent_tc_kernel, dim3((unsigned)n_tiles, (unsigned)splits, (unsigned)p.head_blocks), dim3(kTcThreads), smem, st, 1, p);
    if (rc || splits == 1) return rc;
    CombineParams c = {p.part_o, p.part_ml, d_tile_row, d_tile_rows, p.out, g.heads, p.rows_per_token, p.head_blocks, splits, g.nbc * 64, g.lat_stride};
    // with splits every tile has at most rows_per_token * tokens live rows; 32 CTAs of four warps cover the 128 rows
    return launch_kernel(latent_combine_kernel, dim3((unsigned)n_tiles, kRows / 4, (unsigned)p.head_blocks), dim3(128), 0, st, 1, c);
}

}  // extern "C"
