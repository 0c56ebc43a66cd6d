// Latent attention over a paged cache (no counterpart in gpt.rs): per token and layer the cache holds one normed latent
// vector c of `kv_rank` values and one rotated key part of `rot_dim` values, shared by all heads. The per-head key and value
// projections are absorbed into the query and the output,
//
//   score(i, j, h) = ((W_uk,h^T q_ih) . c_j + rot(q'_ih) . k'_j) * scale,      o_ih = W_uv,h (sum_j p_ijh c_j)
//
// so attention itself is multi-query attention with kv_rank + rot_dim key dimensions whose values are the first kv_rank of
// them, over a sliding window (position i sees i - window + 1 .. i) or all of 0 .. i; a sink per head adds exp(sink) to the denominator
// of the softmax. The two absorbed products are batched matmuls in front of and behind the kernels of this file. Where queries come through a latent of their own, the first projection gives both
// latents, and the kernel that writes the page also norms the query latent for the second projection:
//   latent_append_kernel        norm of the latent(s), rotation of the shared key part and of the queries, page write
//   latent_keys_kernel          its first half for bf16 rows with a query latent
//   latent_attention_kernel     plain CUDA-core attention, f32 or bf16 cache, any sizes (the f32 path)
//   flash_tc_kernel             tcgen05 flash attention (flash_tc.cuh), bf16, prompts and decode steps alike, kv_rank up to 256
//
// The first ceil(kv_rank / 64) blocks of a bf16 cache row (layout in flash_tc.cuh) hold c, the rest the rotated part; columns past
// either are zero. f32 pages are plain [16 tokens][kv_rank + rot_dim].
#include <cstdlib>

#include "flash_tc.cuh"

namespace gptrs {
namespace {

struct Geometry {
    int heads, dim, rot, rank, window, rot_pairs;
    int q_head_stride, dkv_off, rot_off, q_row, kv_row, q_rank, q_latent_row;
    int qa_head_stride, qa_rot_off, lat_stride;
    int nb, nbc;            // 64-column blocks of a cache row (bf16); of them latent
    long long page_bytes;
    float scale;
};
int window_of(const gptrs_latent_attention& a) { return a.window > 0 ? a.window : 1 << 30; }
Geometry geometry(const gptrs_latent_attention& a) {
    Geometry g = {};
    g.heads = a.heads; g.dim = a.dim; g.rot = a.rot_dim; g.rank = a.kv_rank; g.window = window_of(a); g.rot_pairs = a.rot_dims / 2;
    g.kv_row = a.kv_row; g.q_rank = a.q_rank; g.q_latent_row = a.q_latent_row;
    g.q_head_stride = a.q_head_stride; g.dkv_off = a.dkv_offset; g.rot_off = a.rot_offset; g.q_row = a.q_row;
    g.qa_head_stride = a.qa_head_stride; g.qa_rot_off = a.qa_rot_offset; g.lat_stride = a.lat_head_stride;
    g.nbc = up(a.kv_rank, 64) / 64;
    g.nb = g.nbc + up(a.rot_dim, 64) / 64;
    g.page_bytes = a.page_bytes;
    g.scale = a.scale;
    return g;
}

struct AppendParams {
    Geometry g;
    const void* kv;             // [T][kv_row]
    const void* q;              // [T][q_row]
    const int *pos, *slot, *page_table;
    const float *norm_w, *q_norm_w;   // [kv_rank], [q_rank]
    void* q_latent;             // [T][q_latent_row]
    const float *cos_t, *sin_t; // [positions][rot_pairs]
    void* qa;                   // [T][heads][qa_head_stride]
    unsigned char* pool;
    int max_pages;
    float eps;
    int rows;
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

// KEYS: the page (and the query latent, where there is one); QUERIES: the rotated query parts. Both at once where one projection gives
// everything.
template <bool BF16, bool KEYS, bool QUERIES>
__global__ void __launch_bounds__(kAppendThreads) latent_append_kernel(const AppendParams p) {
    using T = typename std::conditional<BF16, __nv_bfloat16, float>::type;
    __shared__ float2 sh[kAppendThreads / 32];
    const Geometry& g = p.g;
    const int row = blockIdx.x, tid = threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    const T* kv = static_cast<const T*>(p.kv) + (size_t)row * g.kv_row;
    const T* q = static_cast<const T*>(p.q) + (size_t)row * g.q_row;
    const T* lat = kv + g.dkv_off;
    const T* kr = kv + g.rot_off;
    const int pos = p.pos[row];
    const float* cs = p.cos_t + (size_t)pos * g.rot_pairs;
    const float* sn = p.sin_t + (size_t)pos * g.rot_pairs;
    unsigned char* page = nullptr;
    float inv = 0.f;
    const int t = pos % kPageTok;
    if constexpr (KEYS) {
        page = p.pool + (size_t)p.page_table[(size_t)p.slot[row] * p.max_pages + pos / kPageTok] * g.page_bytes;
        const int q_rank = QUERIES ? 0 : g.q_rank;   // the query latent is at the start of the row
        float ss = 0.f, qs = 0.f;
        for (int c = tid; c < g.rank; c += kAppendThreads) { const float v = ld_val(lat + c); ss = fmaf(v, v, ss); }
        for (int c = tid; c < q_rank; c += kAppendThreads) { const float v = ld_val(kv + c); qs = fmaf(v, v, qs); }
        ss = warp_sum(ss);
        if (!QUERIES) qs = warp_sum(qs);
        if ((tid & 31) == 0) sh[tid >> 5] = make_float2(ss, qs);
        __syncthreads();
        ss = qs = 0.f;
#pragma unroll
        for (int w = 0; w < kAppendThreads / 32; ++w) { ss += sh[w].x; qs += sh[w].y; }
        inv = 1.f / sqrtf(ss / (float)g.rank + p.eps);
        if constexpr (!QUERIES) {
            const float q_inv = 1.f / sqrtf(qs / (float)q_rank + p.eps);
            T* ql = static_cast<T*>(p.q_latent) + (size_t)row * g.q_latent_row;
            if constexpr (BF16) {
                for (int c0 = tid * 8; c0 < g.q_latent_row; c0 += kAppendThreads * 8) {
                    float v[8];
#pragma unroll
                    for (int e = 0; e < 8; ++e) v[e] = c0 + e < q_rank ? ld_val(kv + c0 + e) * q_inv * p.q_norm_w[c0 + e] : 0.f;
                    *reinterpret_cast<uint4*>(ql + c0) = pack8(v);
                }
            } else {
                for (int c = tid; c < q_rank; c += kAppendThreads) ql[c] = ld_val(kv + c) * q_inv * p.q_norm_w[c];
            }
        }
    }
    T* qa = static_cast<T*>(p.qa) + (size_t)row * g.heads * g.qa_head_stride;
    if constexpr (BF16) {
        const int rb = g.nb - g.nbc;   // blocks of the rotated part
        if constexpr (KEYS)
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
        for (int j = tid; QUERIES && j < g.heads * per_head; j += kAppendThreads) {
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
        auto rotate = [&](const T* src, float* out, int c) {
            const int i = c >> 1;
            float v = ld_val(src + c);
            if (i < g.rot_pairs) v = (c & 1) ? v * cs[i] + ld_val(src + c - 1) * sn[i] : v * cs[i] - ld_val(src + c + 1) * sn[i];
            out[c] = v;
        };
        if constexpr (KEYS) {
            float* dst = reinterpret_cast<float*>(page) + (size_t)t * (g.rank + g.rot);
            for (int c = tid; c < g.rank; c += kAppendThreads) dst[c] = ld_val(lat + c) * inv * p.norm_w[c];
            for (int c = tid; c < g.rot; c += kAppendThreads) rotate(kr, dst + g.rank, c);
        }
        for (int j = tid; QUERIES && j < g.heads * g.rot; j += kAppendThreads) {
            const int h = j / g.rot, c = j % g.rot;
            rotate(q + h * g.q_head_stride + g.dim, reinterpret_cast<float*>(qa) + (size_t)h * g.qa_head_stride + g.qa_rot_off, c);
        }
    }
}

// KEYS of a bf16 model alone, a warp per row with the row in registers: all loads are under way before the first one is needed (the norms'
// gains before the kernel in front has ended), and no barrier is.
constexpr int kKeyRows = 4;          // rows of a CTA
constexpr int kLatChunks = 4;        // 16-byte chunks per lane: kv_rank up to 1024
constexpr int kQueryChunks = 8;      // query latents of up to 2048 values
__device__ __forceinline__ void unpack8(const uint4& u, float (&v)[8]) {
    v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y);
    v[4] = bf16_lo(u.z); v[5] = bf16_hi(u.z); v[6] = bf16_lo(u.w); v[7] = bf16_hi(u.w);
}
// eight values from column c0 on, of which those before n count: the sum of their squares; the normed values, zeros from n on
__device__ __forceinline__ float squares8(const uint4& u, int c0, int n) {
    float v[8], s = 0.f;
    unpack8(u, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) s = c0 + e < n ? fmaf(v[e], v[e], s) : s;
    return s;
}
__device__ __forceinline__ uint4 normed8(const uint4& u, int c0, int n, float inv, const float (&w)[8]) {
    float v[8];
    unpack8(u, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = c0 + e < n ? v[e] * inv * w[e] : 0.f;
    return pack8(v);
}
// eight gains from column c0 on (zeros from n on)
__device__ __forceinline__ void gains8(const float* w, int c0, int n, float (&v)[8]) {
    if (c0 + 8 <= n) {
        const float4 a = __ldg(reinterpret_cast<const float4*>(w + c0)), b = __ldg(reinterpret_cast<const float4*>(w + c0) + 1);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = c0 + e < n ? __ldg(w + c0 + e) : 0.f;
    }
}

// LC, QC: chunks per lane of the latent and of the query latent
template <int LC, int QC>
__global__ void __launch_bounds__(kKeyRows * 32) latent_keys_kernel(const AppendParams p) {
    const Geometry& g = p.g;
    const int lane = threadIdx.x & 31, row = blockIdx.x * kKeyRows + (threadIdx.x >> 5);
    pdl_launch_dependents();
    float wl[LC][8], wq[QC][8];
#pragma unroll
    for (int i = 0; i < LC; ++i) gains8(p.norm_w, (i * 32 + lane) * 8, g.rank, wl[i]);
#pragma unroll
    for (int i = 0; i < QC; ++i) gains8(p.q_norm_w, (i * 32 + lane) * 8, g.q_rank, wq[i]);
    pdl_wait();
    if (row >= p.rows) return;
    const int pos = p.pos[row], slot = p.slot[row];
    const __nv_bfloat16* kv = static_cast<const __nv_bfloat16*>(p.kv) + (size_t)row * g.kv_row;
    const uint4* lat = reinterpret_cast<const uint4*>(kv + g.dkv_off);
    const int n_q = g.q_latent_row / 8, n_lat = up(g.rank, 8) / 8;
    uint4 q[QC], l[LC];
#pragma unroll
    for (int i = 0; i < LC; ++i) l[i] = i * 32 + lane < n_lat ? lat[i * 32 + lane] : make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int i = 0; i < QC; ++i) q[i] = i * 32 + lane < n_q ? reinterpret_cast<const uint4*>(kv)[i * 32 + lane] : make_uint4(0, 0, 0, 0);
    unsigned char* page = p.pool + (size_t)p.page_table[(size_t)slot * p.max_pages + pos / kPageTok] * g.page_bytes;
    const int t = pos % kPageTok;
    for (int j = lane; j < (g.nb - g.nbc) * 8; j += 32) {
        float v[8];
        rotated8(kv + g.rot_off, j, g.rot, g.rot_pairs, p.cos_t + (size_t)pos * g.rot_pairs, p.sin_t + (size_t)pos * g.rot_pairs, v);
        *reinterpret_cast<uint4*>(page + page_chunk(t, g.nbc * 8 + j, g.nb)) = pack8(v);
    }
    float sl = 0.f, sq = 0.f;
#pragma unroll
    for (int i = 0; i < LC; ++i) sl += squares8(l[i], (i * 32 + lane) * 8, g.rank);
#pragma unroll
    for (int i = 0; i < QC; ++i) sq += squares8(q[i], (i * 32 + lane) * 8, g.q_rank);
    const float inv_l = 1.f / sqrtf(warp_sum(sl) / (float)g.rank + p.eps), inv_q = 1.f / sqrtf(warp_sum(sq) / (float)g.q_rank + p.eps);
#pragma unroll
    for (int i = 0; i < LC; ++i) {
        const int j = i * 32 + lane;
        if (j < g.nbc * 8) *reinterpret_cast<uint4*>(page + page_chunk(t, j, g.nb)) = normed8(l[i], j * 8, g.rank, inv_l, wl[i]);
    }
    uint4* ql = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.q_latent) + (size_t)row * g.q_latent_row);
#pragma unroll
    for (int i = 0; i < QC; ++i) {
        const int j = i * 32 + lane;
        if (j < n_q) ql[j] = normed8(q[i], j * 8, g.q_rank, inv_q, wq[i]);
    }
}

// ---- plain attention: one CTA per (head, row) ---------------------------------------------------------------------------------
struct AttnParams {
    Geometry g;
    const void* qa;
    const unsigned char* pool;
    const int *page_table, *slot, *ctx_len;
    const float* sink;          // [heads] or null
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
    if (p.sink) l += expf(p.sink[head] - m);   // infinite where the sink outweighs everything: the output is 0
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

template <bool KEYS, bool QUERIES>
int launch_append(const gptrs_latent_attention* a, const AppendParams& p, int64_t n_tokens, void* stream) {
    const dim3 grid((unsigned)n_tokens);
    return a->dtype == GPTRS_BF16 ? launch_kernel(latent_append_kernel<true, KEYS, QUERIES>, grid, dim3(kAppendThreads), 0, as_stream(stream), 1, p)
                                  : launch_kernel(latent_append_kernel<false, KEYS, QUERIES>, grid, dim3(kAppendThreads), 0, as_stream(stream), 1, p);
}

bool fits(const Geometry& g) { return tc_fits(g.nb, g.nbc, g.nb); }

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" {

int gptrs_cuda_latent_layout(gptrs_latent_attention* a) {
    GPTRS_REQUIRE(a, "null pointer");
    GPTRS_REQUIRE(a->heads > 0 && a->dim > 0 && a->rot_dim > 0 && a->vdim > 0 && a->kv_rank > 0 && a->window >= 0 && a->q_rank >= 0, "latent attention: sizes must be positive");
    GPTRS_REQUIRE(a->rot_dims >= 0 && a->rot_dims <= a->rot_dim && a->rot_dims % 2 == 0, "latent attention: rotated dimensions");
    GPTRS_REQUIRE(a->scale > 0.f, "latent attention: the scale must be positive");
    GPTRS_REQUIRE(a->dtype == GPTRS_F32 || a->dtype == GPTRS_BF16, "latent attention: f32 or bf16");
    if (a->kv_rank > kPlainThreads * kPlainCols) return fail(GPTRS_UNIMPLEMENTED, "latent attention: kv_rank above 1024");
    if (a->dtype == GPTRS_F32) {
        a->q_head_stride = a->dim + a->rot_dim;
        a->q_latent_row = a->q_rank;
        a->dkv_offset = a->q_rank > 0 ? a->q_latent_row : a->heads * a->q_head_stride;
        a->rot_offset = a->dkv_offset + a->kv_rank;
        a->kv_row = a->rot_offset + a->rot_dim;
        a->q_rot_offset = a->dim;
        a->qa_head_stride = a->kv_rank + a->rot_dim;
        a->qa_rot_offset = a->kv_rank;
        a->lat_head_stride = a->kv_rank;
        a->out_head_stride = a->vdim;
        a->page_bytes = (int64_t)kPageTok * (a->kv_rank + a->rot_dim) * 4;
    } else {
        a->q_rot_offset = up(a->dim, 8);
        a->q_head_stride = a->q_rot_offset + up(a->rot_dim, 8);
        a->q_latent_row = up(a->q_rank, 8);
        a->dkv_offset = a->q_rank > 0 ? a->q_latent_row : a->heads * a->q_head_stride;
        a->rot_offset = a->dkv_offset + up(a->kv_rank, 8);
        a->kv_row = a->rot_offset + up(a->rot_dim, 8);
        a->qa_rot_offset = up(a->kv_rank, 64);
        a->qa_head_stride = a->qa_rot_offset + up(a->rot_dim, 64);
        a->lat_head_stride = up(a->kv_rank, 8);
        a->out_head_stride = up(a->vdim, 8);
        a->page_bytes = (int64_t)kPageTok * a->qa_head_stride * 2;
    }
    a->q_row = a->q_rank > 0 ? a->heads * a->q_head_stride : a->kv_row;
    return GPTRS_OK;
}

int gptrs_cuda_latent_append(const gptrs_latent_attention* a, const void* d_qkv, const int32_t* d_positions, const int32_t* d_slot,
                             const int32_t* d_page_table, int64_t max_pages, const float* d_norm_w, float eps, const float* d_cos, const float* d_sin,
                             void* d_qa, void* d_pool, int64_t n_tokens, void* stream) {
    GPTRS_REQUIRE(a && d_qkv && d_positions && d_slot && d_page_table && d_norm_w && d_qa && d_pool, "null pointer");
    GPTRS_REQUIRE(a->q_row > 0 && max_pages > 0 && (a->rot_dims == 0 || (d_cos && d_sin)), "latent attention: layout not filled in, or no rotation tables");
    GPTRS_REQUIRE(a->q_rank == 0, "latent attention: queries with a latent of their own are appended in two steps");
    if (n_tokens == 0) return GPTRS_OK;
    AppendParams p = {};
    p.g = geometry(*a); p.kv = p.q = d_qkv; p.pos = d_positions; p.slot = d_slot; p.page_table = d_page_table; p.norm_w = d_norm_w; p.cos_t = d_cos; p.sin_t = d_sin;
    p.qa = d_qa; p.pool = static_cast<unsigned char*>(d_pool); p.max_pages = (int)max_pages; p.eps = eps;
    return launch_append<true, true>(a, p, n_tokens, stream);
}

int gptrs_cuda_latent_append_keys(const gptrs_latent_attention* a, const void* d_kv, const int32_t* d_positions, const int32_t* d_slot, const int32_t* d_page_table,
                                  int64_t max_pages, const float* d_norm_w, const float* d_q_norm_w, float eps, const float* d_cos, const float* d_sin,
                                  void* d_q_latent, void* d_pool, int64_t n_tokens, void* stream) {
    GPTRS_REQUIRE(a && d_kv && d_positions && d_slot && d_page_table && d_norm_w && d_q_norm_w && d_q_latent && d_pool, "null pointer");
    GPTRS_REQUIRE(a->q_rank > 0 && a->q_row > 0 && max_pages > 0 && (a->rot_dims == 0 || (d_cos && d_sin)), "latent attention: layout not filled in, or no rotation tables");
    if (n_tokens == 0) return GPTRS_OK;
    AppendParams p = {};
    p.g = geometry(*a); p.kv = d_kv; p.pos = d_positions; p.slot = d_slot; p.page_table = d_page_table; p.norm_w = d_norm_w; p.q_norm_w = d_q_norm_w;
    p.cos_t = d_cos; p.sin_t = d_sin; p.q_latent = d_q_latent; p.pool = static_cast<unsigned char*>(d_pool); p.max_pages = (int)max_pages; p.eps = eps;
    const bool aligned = ((reinterpret_cast<uintptr_t>(d_norm_w) | reinterpret_cast<uintptr_t>(d_q_norm_w) | reinterpret_cast<uintptr_t>(d_kv) | reinterpret_cast<uintptr_t>(d_q_latent)) & 15) == 0;
    p.rows = (int)n_tokens;
    if (a->dtype == GPTRS_BF16 && aligned && a->q_rank <= kQueryChunks * 256) {
        const dim3 grid((unsigned)ceil_div((int)n_tokens, kKeyRows));
        void (*kern)(AppendParams) = a->kv_rank > 256 ? latent_keys_kernel<kLatChunks, kQueryChunks> : a->q_rank <= 512 ? latent_keys_kernel<1, 2>
                                   : a->q_rank <= 1024 ? latent_keys_kernel<1, 4> : latent_keys_kernel<1, kQueryChunks>;
        return launch_kernel(kern, grid, dim3(kKeyRows * 32), 0, as_stream(stream), 1, p);
    }
    return launch_append<true, false>(a, p, n_tokens, stream);
}

int gptrs_cuda_latent_rotate_queries(const gptrs_latent_attention* a, const void* d_q, const int32_t* d_positions, const float* d_cos, const float* d_sin, void* d_qa,
                                     int64_t n_tokens, void* stream) {
    GPTRS_REQUIRE(a && d_q && d_positions && d_qa, "null pointer");
    GPTRS_REQUIRE(a->q_row > 0 && (a->rot_dims == 0 || (d_cos && d_sin)), "latent attention: layout not filled in, or no rotation tables");
    if (n_tokens == 0) return GPTRS_OK;
    AppendParams p = {};
    p.g = geometry(*a); p.q = d_q; p.pos = d_positions; p.cos_t = d_cos; p.sin_t = d_sin; p.qa = d_qa;
    return launch_append<false, true>(a, p, n_tokens, stream);
}

int gptrs_cuda_latent_tile_tokens(const gptrs_latent_attention* a) {
    if (!a || a->dtype != GPTRS_BF16 || a->heads < 1 || !fits(geometry(*a))) return 0;
    return a->heads >= kRows ? 1 : kRows / a->heads;
}

int gptrs_cuda_latent_splits(const gptrs_latent_attention* a, int64_t n_tiles, int64_t max_ctx_len) {
    if (!a || n_tiles <= 0 || gptrs_cuda_latent_tile_tokens(a) == 0) return 1;
    const int64_t widest = (int64_t)window_of(*a) + gptrs_cuda_latent_tile_tokens(a), span = max_ctx_len < widest ? max_ctx_len : widest;
    const int64_t blocks = (span + kPageTok - 1 + kKeys - 1) / kKeys;
    int64_t s = sm_count() / (n_tiles * ceil_div(a->heads, kRows));
    if (s > blocks) s = blocks;
    return (int)(s < 1 ? 1 : s);
}

size_t gptrs_cuda_latent_scratch_bytes(const gptrs_latent_attention* a, int64_t n_tiles, int splits) {
    if (!a || splits <= 1) return 0;
    return tc_scratch_bytes(n_tiles, ceil_div(a->heads, kRows), splits, up(a->kv_rank, 64) / 64);
}

int gptrs_cuda_latent_attention(const gptrs_latent_attention* a, const void* d_qa, const void* d_pool, const int32_t* d_page_table, int64_t max_pages,
                                const int32_t* d_slot, const int32_t* d_ctx_len, const float* d_sink, const int32_t* d_tile_row, const int32_t* d_tile_rows, int64_t n_tiles,
                                int splits, void* d_out, void* d_scratch, size_t scratch_bytes, int32_t* d_status, int64_t n_tokens, void* stream) {
    GPTRS_REQUIRE(a && d_qa && d_pool && d_page_table && d_slot && d_ctx_len && d_out && d_status, "null pointer");
    GPTRS_REQUIRE(a->q_row > 0 && max_pages > 0 && max_pages * kPageTok < ((int64_t)1 << 30), "latent attention: layout not filled in, or a bad page table");
    if (n_tokens == 0) return GPTRS_OK;
    const Geometry g = geometry(*a);
    cudaStream_t st = as_stream(stream);
    if (n_tiles <= 0) {   // plain kernel: every row by itself
        GPTRS_REQUIRE(n_tokens <= 65535 && a->heads <= 0x7fffffff, "latent attention: too many rows in one launch");
        AttnParams p = {g, d_qa, static_cast<const unsigned char*>(d_pool), d_page_table, d_slot, d_ctx_len, d_sink, d_out, d_status, (int)max_pages};
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
    int erc = encode_queries(d_qa, g, n_tokens, &p.q_map);
    if (erc) return erc;
    FlashShape& f = p.g;
    f.heads = f.group = g.heads; f.kv_heads = 1;
    f.blocks = f.query_blocks = g.nb; f.value_blocks = g.nbc; f.key_block = 0;
    for (int b = 0; b < g.nb; ++b) {
        const int cols = b < g.nbc ? g.rank - b * 64 : g.rot - (b - g.nbc) * 64;
        f.steps[b] = cols >= 64 ? 4 : (cols + 15) / 16;
    }
    f.mask = GPTRS_MASK_WINDOW; f.mask_size = g.window;
    f.out_stride = g.lat_stride;
    f.page_bytes = g.page_bytes; f.block_bytes = (uint32_t)g.page_bytes;
    p.pool = static_cast<const unsigned char*>(d_pool);
    p.page_table = d_page_table; p.slot = d_slot; p.ctx_len = d_ctx_len; p.tile_row = d_tile_row; p.tile_rows = d_tile_rows;
    p.out = static_cast<__nv_bfloat16*>(d_out);
    p.status = d_status;
    p.max_pages = (int)max_pages; p.splits = splits;
    p.scale_log2 = kLog2e * g.scale;
    p.sink = d_sink;
    return launch_flash<false, 3>(p, n_tiles, d_scratch, st);
}

}  // extern "C"
