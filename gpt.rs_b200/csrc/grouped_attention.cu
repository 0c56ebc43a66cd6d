// Attention with grouped key / value heads of any size over a paged cache (no counterpart in gpt.rs, whose own attention has
// heads of one size and neither a soft cap nor a distance penalty):
//
//   score(i, j, h) = cap tanh(scale q_ih . k_jg / cap) - r1_h ln(1 + r2_h (i - j)),   g = h / (heads / kv_heads)
//   o_ih = softmax over the visible j . v_jg
//
// A mask says where the keys of position i begin: at 0, at i - size + 1 (window) or at the last multiple of size (chunks).
// Differential attention gives every query and key head two parts, each a softmax attention of its own over the same values; the output
// of a head is their difference a1 - lambda a2, brought to unit root mean square. An output gate multiplies by sigmoid(gate). A layer may
// read keys and values that another layer has put into the cache. The penalty may be linear in the distance instead, r1_h (i - j). Queries and
// keys may pass a short causal convolution over time and a norm per head, and the values may be the keys in front of that norm: then the
// cache holds a vector and a number per key, and a key is their product.
//   grouped_append_kernel       key / value part of a projection row -> the token's page
//   grouped_prepare_kernel      convolutions with their state, norms, queries, page write: a warp per head and up to eight rows (bf16)
//   grouped_prepare_any_kernel  the same for f32 and for sizes that the former does not take, a warp per head and row
//   grouped_attention_kernel    plain CUDA-core attention, f32 or bf16 cache, any sizes (the f32 path)
//   flash_tc_kernel<true>       tcgen05 flash attention (flash_tc.cuh), bf16, prompts and decode steps alike
//   grouped_decode_kernel       decode steps with few heads per kv head, bf16 (grouped_decode.cuh; GPTRS_GROUPED_DECODE=0 keeps the former)
// A page holds, kv head by kv head, 16 rows of [value | key] or [value | key part 1 | key part 2]; in bf16 all are padded to whole
// 64-column blocks in the layout of flash_tc.cuh, in f32 the rows are plain.
#include "grouped_decode.cuh"

namespace gptrs {
namespace {

struct Shape {
    int heads, kv_heads, group, dim, vdim, mask, mask_size;
    int q_head_stride, k_off, k_head_stride, v_off, v_head_stride, q_row, out_stride;
    int maps, map_stride, g_off, g_head_stride;   // parts of a head; gate (g_head_stride 0: none)
    int query_row, tied, width;   // row of queries; the cache holds values and numbers; columns of a cache row (f32)
    int nb, nbv, nbk;       // 64-column blocks of a cache row (bf16); of them values; of one key part
    long long page_bytes, block_bytes;
    float scale, softcap, lambda, head_scale, head_eps;
};
Shape shape_of(const gptrs_grouped_attention& a) {
    Shape g = {};
    g.heads = a.heads; g.kv_heads = a.kv_heads; g.group = a.heads / a.kv_heads; g.dim = a.dim; g.vdim = a.vdim;
    g.mask = a.mask; g.mask_size = a.mask_size;
    g.q_head_stride = a.q_head_stride; g.k_off = a.k_offset; g.k_head_stride = a.k_head_stride; g.v_off = a.v_offset; g.v_head_stride = a.v_head_stride;
    g.q_row = a.q_row; g.out_stride = a.out_head_stride;
    g.maps = a.maps > 1 ? a.maps : 1; g.map_stride = a.map_stride; g.g_off = a.g_offset; g.g_head_stride = a.g_head_stride;
    g.nbv = up(a.vdim, 64) / 64;
    g.tied = a.tied;
    g.nbk = a.tied ? 0 : up(a.dim, 64) / 64;
    g.nb = g.nbv + g.maps * g.nbk;
    g.query_row = a.query_row; g.width = a.tied ? a.vdim : a.vdim + g.maps * a.dim;
    g.page_bytes = a.page_bytes; g.block_bytes = (long long)kPageTok * (a.dtype == GPTRS_BF16 ? g.nb * 128 : g.width * 4);
    g.scale = a.scale; g.softcap = a.softcap;
    g.lambda = a.lambda_; g.head_scale = a.head_scale; g.head_eps = a.head_eps;
    return g;
}

// behind the blocks of a page: the numbers of its keys, [kv heads][16]
__device__ __forceinline__ float* key_scale(const Shape& g, unsigned char* page, int kv_head, int t) {
    return reinterpret_cast<float*>(page + g.kv_heads * g.block_bytes) + kv_head * kPageTok + t;
}

struct AppendParams {
    Shape g;
    const void* qkv;
    const int *pos, *slot, *page_table;
    unsigned char* pool;
    int max_pages;
};
constexpr int kAppendThreads = 128;

template <bool BF16>
__global__ void __launch_bounds__(kAppendThreads) grouped_append_kernel(const AppendParams p) {
    const Shape& g = p.g;
    const int row = blockIdx.x, tid = threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    const int pos = p.pos[row];
    unsigned char* page = p.pool + (size_t)p.page_table[(size_t)p.slot[row] * p.max_pages + pos / kPageTok] * g.page_bytes;
    const int t = pos % kPageTok;
    if constexpr (BF16) {
        const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.qkv) + (size_t)row * g.q_row;
        const int per_head = g.nb * 8;
        for (int j = tid; j < g.kv_heads * per_head; j += kAppendThreads) {
            const int h = j / per_head, c = j % per_head;
            const bool val = c < g.nbv * 8;
            const int kc = c - g.nbv * 8, part = val ? 0 : kc / (g.nbk * 8);
            const int col = (val ? c : kc - part * g.nbk * 8) * 8, n = val ? g.vdim : g.dim;
            const __nv_bfloat16* s = src + (val ? g.v_off + h * g.v_head_stride : g.k_off + h * g.k_head_stride + part * g.map_stride) + col;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (col + 8 <= n) {
                v = *reinterpret_cast<const uint4*>(s);
            } else if (col < n) {   // the last, partly filled chunk
                __nv_bfloat16 e[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) e[i] = col + i < n ? s[i] : __float2bfloat16_rn(0.f);
                v = *reinterpret_cast<const uint4*>(e);
            }
            *reinterpret_cast<uint4*>(page + h * g.block_bytes + page_chunk(t, c, g.nb)) = v;
        }
    } else {
        const float* src = static_cast<const float*>(p.qkv) + (size_t)row * g.q_row;
        const int width = g.vdim + g.maps * g.dim;   // the parts of a key lie next to one another
        for (int j = tid; j < g.kv_heads * width; j += kAppendThreads) {
            const int h = j / width, c = j % width;
            reinterpret_cast<float*>(page + h * g.block_bytes)[(size_t)t * width + c] =
                c < g.vdim ? src[g.v_off + h * g.v_head_stride + c] : src[g.k_off + h * g.k_head_stride + c - g.vdim];
        }
    }
}

// ---- convolutions, norms, queries, page write -----------------------------------------------------------------------------------
struct PrepareParams {
    Shape g;
    gptrs_grouped_step s;
    int taps, channels, norm;
    float eps;
};
constexpr int kPrepareWarps = 4;

// What a row needs of its sequence. Inputs in front of its run come from the half `old`, where the input of position q lies at q % (taps - 1).
struct PrepareRow { int pos, first, last; const float* old; float* fresh; unsigned char* page; };
__device__ __forceinline__ PrepareRow prepare_row(const PrepareParams& p, int pos, int slot, int first, int last, int parity) {
    PrepareRow r;
    r.pos = pos; r.first = first; r.last = last;
    const size_t half = (size_t)(p.taps - 1) * p.channels;
    float* state = p.s.d_conv_state + (size_t)slot * 2 * half;
    r.old = state + (parity & 1) * half; r.fresh = state + ((parity & 1) ^ 1) * half;
    r.page = static_cast<unsigned char*>(p.s.d_pool) + (size_t)p.s.d_page_table[(size_t)slot * p.s.max_pages + pos / kPageTok] * p.g.page_bytes;
    return r;
}

// Sums of R values over the warp, R a power of two up to 32: lane i gets the sum of v[i mod R].
template <int R>
__device__ __forceinline__ float transpose_sum(float (&v)[R]) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int h = R / 2; h >= 1; h >>= 1)
#pragma unroll
        for (int i = 0; i < h; ++i) {
            const float give = (lane & h) ? v[i] : v[i + h], keep = (lane & h) ? v[i + h] : v[i];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, give, h);
        }
#pragma unroll
    for (int h = R; h < 32; h <<= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], h);
    return v[0];
}
__device__ __forceinline__ void unpack4(const uint2& u, float (&v)[4]) { v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y); }

// A lane holds the channels (i * 32 + lane) * 4 + e, i < NI, of a head for R rows, with the inputs in front of them. Rows away from the ends of
// their run (nearly all of a prompt's) need nothing but rows of this pass.
template <int TAPS, int NI, int R>
__global__ void __launch_bounds__(kPrepareWarps * 32) grouped_prepare_kernel(const PrepareParams p) {
    constexpr int KEEP = TAPS - 1, HIST = KEEP > 0 ? KEEP : 1;
    const Shape& g = p.g;
    const int lane = threadIdx.x & 31, job = blockIdx.y * kPrepareWarps + (threadIdx.x >> 5);
    pdl_launch_dependents();
    const bool is_q = job < g.heads;
    const int head = is_q ? job : job - g.heads, col0 = is_q ? head * g.q_head_stride : g.k_off + head * g.k_head_stride;
    const bool live = job < g.heads + g.kv_heads, has_gain = p.norm && (is_q || !g.tied);
    float w[TAPS][NI][4];
#pragma unroll
    for (int i = 0; i < NI; ++i) {   // constants: on their way before the kernel in front has ended
        const int c = (i * 32 + lane) * 4;
        const bool in = live && c < g.map_stride;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const float4 v = in ? (p.s.d_conv ? __ldg(reinterpret_cast<const float4*>(p.s.d_conv + (size_t)j * p.channels + col0 + c)) : make_float4(1.f, 1.f, 1.f, 1.f))
                                : make_float4(0.f, 0.f, 0.f, 0.f);
            w[j][i][0] = v.x; w[j][i][1] = v.y; w[j][i][2] = v.z; w[j][i][3] = v.w;
        }
    }
    pdl_wait();
    if (!live) return;
    const int row0 = blockIdx.x * R, rows = min(R, (int)p.s.rows - row0);
    int v_pos = 0, v_slot = 0, v_first = 0, v_last = 0, v_par = 0;
    if (lane < rows) {
        v_pos = p.s.d_pos[row0 + lane]; v_slot = p.s.d_slot[row0 + lane];
        v_first = p.s.d_run_first[row0 + lane]; v_last = p.s.d_run_last[row0 + lane]; v_par = p.s.d_parity[row0 + lane];
    }
    const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(p.s.d_qkv) + (size_t)row0 * g.q_row + col0;
    uint2 raw[KEEP + R][NI];   // rows row0 - KEEP .. row0 + R - 1
#pragma unroll
    for (int r = 0; r < KEEP + R; ++r)
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int c = (i * 32 + lane) * 4;
            raw[r][i] = r < KEEP + rows && row0 + r >= KEEP && c < g.map_stride ? *reinterpret_cast<const uint2*>(x + (int64_t)(r - KEEP) * g.q_row + c) : make_uint2(0, 0);
        }
    const int first = __shfl_sync(0xffffffffu, v_first, 0), last = __shfl_sync(0xffffffffu, v_last, 0);
    const bool inner = R > 1 && rows == R && row0 - KEEP >= first && row0 + R - 1 + KEEP <= last;
    float y[R][NI][4], ss[R];
#pragma unroll
    for (int r = 0; r < R; ++r) ss[r] = 0.f;
    if (inner || KEEP == 0) {
#pragma unroll
        for (int r = 0; r < R; ++r)
#pragma unroll
            for (int i = 0; i < NI; ++i) {
#pragma unroll
                for (int e = 0; e < 4; ++e) y[r][i][e] = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {
                    float v[4];
                    unpack4(raw[r + j][i], v);
#pragma unroll
                    for (int e = 0; e < 4; ++e) y[r][i][e] = fmaf(w[j][i][e], v[e], y[r][i][e]);
                }
            }
    } else {
        float hist[HIST][NI][4];   // hist[k]: the input k + 1 positions back
#pragma unroll
        for (int r = 0; r < R; ++r) {
            if (r >= rows) break;
            const int row = row0 + r, pos = __shfl_sync(0xffffffffu, v_pos, r), r_first = __shfl_sync(0xffffffffu, v_first, r), r_last = __shfl_sync(0xffffffffu, v_last, r);
            const size_t half = (size_t)KEEP * p.channels;
            const int par = __shfl_sync(0xffffffffu, v_par, r) & 1;
            float* state = p.s.d_conv_state + (size_t)__shfl_sync(0xffffffffu, v_slot, r) * 2 * half + col0;
            const float* old = state + par * half;
            float* fresh = state + (par ^ 1) * half;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int c = (i * 32 + lane) * 4;
                const bool in = c < g.map_stride;
                if (r == 0 || row == r_first) {
#pragma unroll
                    for (int k = 0; k < KEEP; ++k) {
                        const int at = pos - 1 - k;
#pragma unroll
                        for (int e = 0; e < 4; ++e) hist[k][i][e] = 0.f;
                        if (row - 1 - k >= r_first) {
                            unpack4(raw[r + KEEP - 1 - k][i], hist[k][i]);
                        } else if (at >= 0 && in) {
                            const float4 v = *reinterpret_cast<const float4*>(old + (size_t)(at % HIST) * p.channels + c);
                            hist[k][i][0] = v.x; hist[k][i][1] = v.y; hist[k][i][2] = v.z; hist[k][i][3] = v.w;
                        }
                    }
                }
                float now[4];
                unpack4(raw[r + KEEP][i], now);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    float a = 0.f;
#pragma unroll
                    for (int k = KEEP - 1; k >= 0; --k) a = fmaf(w[KEEP - 1 - k][i][e], hist[k][i][e], a);
                    y[r][i][e] = fmaf(w[KEEP][i][e], now[e], a);
                }
                if (r_last - row < KEEP && in) {   // the inputs that the sequence's next step needs
                    *reinterpret_cast<float4*>(fresh + (size_t)(pos % HIST) * p.channels + c) = make_float4(now[0], now[1], now[2], now[3]);
                    if (row == r_first)   // a run shorter than the state: what it does not push out stays
#pragma unroll
                        for (int k = 0; k < KEEP - 1; ++k)
                            if (pos - 1 - k >= 0 && k + 1 + r_last - row < KEEP)
                                *reinterpret_cast<float4*>(fresh + (size_t)((pos - 1 - k) % HIST) * p.channels + c) = make_float4(hist[k][i][0], hist[k][i][1], hist[k][i][2], hist[k][i][3]);
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
#pragma unroll
                    for (int k = KEEP - 1; k > 0; --k) hist[k][i][e] = hist[k - 1][i][e];
                    hist[0][i][e] = now[e];
                }
            }
        }
    }
    float my_inv = 1.f;   // of row lane mod R
    if (p.norm) {
#pragma unroll
        for (int r = 0; r < R; ++r)
            if (r < rows)
#pragma unroll
                for (int i = 0; i < NI; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) ss[r] = fmaf(y[r][i][e], y[r][i][e], ss[r]);
        my_inv = 1.f / sqrtf(transpose_sum(ss) / (float)g.dim + p.eps);
    }
    float gain[NI][4];
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = (i * 32 + lane) * 4 + e;
            gain[i][e] = has_gain && c < g.dim ? __ldg((is_q ? p.s.d_q_gain : p.s.d_k_gain) + c) : 1.f;
        }
    if (is_q) {
        __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.s.d_q) + (size_t)row0 * g.query_row + col0;
#pragma unroll
        for (int r = 0; r < R; ++r) {
            if (r >= rows) break;
            const float inv = __shfl_sync(0xffffffffu, my_inv, r);
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int c = (i * 32 + lane) * 4;
                if (c < g.map_stride)
                    *reinterpret_cast<uint2*>(dst + (size_t)r * g.query_row + c) = make_uint2(pack_bf16x2(y[r][i][0] * inv * gain[i][0], y[r][i][1] * inv * gain[i][1]),
                                                                                              pack_bf16x2(y[r][i][2] * inv * gain[i][2], y[r][i][3] * inv * gain[i][3]));
            }
        }
        return;
    }
    long long v_page = 0;
    if (lane < rows) v_page = (long long)p.s.d_page_table[(size_t)v_slot * p.s.max_pages + v_pos / kPageTok] * g.page_bytes;
    if (g.tied && lane < rows) *key_scale(g, static_cast<unsigned char*>(p.s.d_pool) + v_page, head, v_pos % kPageTok) = my_inv;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        if (r >= rows) break;
        const int t = __shfl_sync(0xffffffffu, v_pos, r) % kPageTok;
        unsigned char* block = static_cast<unsigned char*>(p.s.d_pool) + __shfl_sync(0xffffffffu, v_page, r) + head * g.block_bytes;
        const float f = g.tied ? 1.f : __shfl_sync(0xffffffffu, my_inv, r);
#pragma unroll
        for (int i = 0; i < NI; ++i) {   // the columns of the last block that hold no data get zeros
            const int c = (i * 32 + lane) * 4, at = c + (g.tied ? 0 : g.nbv * 64);
            if (c < up(g.dim, 64))
                *reinterpret_cast<uint2*>(block + page_chunk(t, at >> 3, g.nb) + (at & 7) * 2) =
                    make_uint2(pack_bf16x2(y[r][i][0] * f * gain[i][0], y[r][i][1] * f * gain[i][1]), pack_bf16x2(y[r][i][2] * f * gain[i][2], y[r][i][3] * f * gain[i][3]));
        }
        if (!g.tied) {
            const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(p.s.d_qkv) + (size_t)(row0 + r) * g.q_row + g.v_off + head * g.v_head_stride;
            for (int c = lane * 4; c < g.nbv * 64; c += 128)
                *reinterpret_cast<uint2*>(block + page_chunk(t, c >> 3, g.nb) + (c & 7) * 2) = c < g.v_head_stride ? *reinterpret_cast<const uint2*>(v + c) : make_uint2(0, 0);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(kPrepareWarps * 32) grouped_prepare_any_kernel(const PrepareParams p) {
    constexpr bool BF16 = sizeof(T) == 2;
    const Shape& g = p.g;
    const int lane = threadIdx.x & 31, job = blockIdx.y * kPrepareWarps + (threadIdx.x >> 5), row = blockIdx.x, keep = p.taps - 1;
    pdl_launch_dependents();
    pdl_wait();
    if (job >= g.heads + g.kv_heads) return;
    const bool is_q = job < g.heads;
    const int head = is_q ? job : job - g.heads, col0 = is_q ? head * g.q_head_stride : g.k_off + head * g.k_head_stride;
    const PrepareRow q = prepare_row(p, p.s.d_pos[row], p.s.d_slot[row], p.s.d_run_first[row], p.s.d_run_last[row], p.s.d_parity[row]);
    auto value = [](T v) -> float { if constexpr (sizeof(T) == 2) return __bfloat162float(v); else return v; };
    auto put = [](T* dst, float v) { if constexpr (sizeof(T) == 2) *dst = __float2bfloat16_rn(v); else *dst = v; };
    const T* x = static_cast<const T*>(p.s.d_qkv) + (size_t)row * g.q_row;
    auto input = [&](int k, int c) -> float {   // k positions back
        if (row - k >= q.first) return value(x[col0 + c - (int64_t)k * g.q_row]);
        const int at = q.pos - k;
        return at >= 0 ? q.old[(size_t)(at % keep) * p.channels + col0 + c] : 0.f;
    };
    auto conv = [&](int c) -> float {
        if (!p.s.d_conv) return input(0, c);
        float a = 0.f;
        for (int k = keep; k >= 0; --k) a = fmaf(p.s.d_conv[(size_t)(keep - k) * p.channels + col0 + c], input(k, c), a);
        return a;
    };
    float inv = 1.f;
    if (p.norm) {
        float ss = 0.f;
        for (int c = lane; c < g.dim; c += 32) { const float v = conv(c); ss = fmaf(v, v, ss); }
        inv = 1.f / sqrtf(warp_sum(ss) / (float)g.dim + p.eps);
    }
    const float* gp = p.norm && (is_q || !g.tied) ? (is_q ? p.s.d_q_gain : p.s.d_k_gain) : nullptr;
    const int t = q.pos % kPageTok;
    unsigned char* block = q.page + head * g.block_bytes;
    auto cell = [&](int c) -> T* {   // column c of the token's cache row, values first
        if constexpr (BF16) return reinterpret_cast<T*>(block + page_chunk(t, c >> 3, g.nb) + (c & 7) * 2);
        else return reinterpret_cast<T*>(block) + (size_t)t * g.width + c;
    };
    const int key0 = g.tied ? 0 : BF16 ? g.nbv * 64 : g.vdim, key_cols = BF16 ? up(g.dim, 64) : g.dim, val_cols = BF16 ? g.nbv * 64 : g.vdim;
    for (int c = lane; c < (is_q ? g.map_stride : key_cols); c += 32) {
        const float f = !is_q && g.tied ? 1.f : inv;
        const float v = c < g.dim ? conv(c) * f * (gp ? gp[c] : 1.f) : 0.f;
        put(is_q ? static_cast<T*>(p.s.d_q) + (size_t)row * g.query_row + col0 + c : cell(key0 + c), v);
    }
    if (!is_q && g.tied && lane == 0) *key_scale(g, q.page, head, t) = inv;
    if (!is_q && !g.tied)
        for (int c = lane; c < val_cols; c += 32) put(cell(c), c < g.vdim ? value(x[g.v_off + head * g.v_head_stride + c]) : 0.f);
    if (keep > 0 && q.last - row < keep)
        for (int c = lane; c < g.map_stride; c += 32) {
            float* f = q.fresh + col0 + c;
            f[(size_t)(q.pos % keep) * p.channels] = input(0, c);
            if (row == q.first)
                for (int k = 1; k < keep; ++k)
                    if (q.pos - k >= 0 && k + q.last - row < keep) f[(size_t)((q.pos - k) % keep) * p.channels] = input(k, c);
        }
}

template <int TAPS, int NI>
int launch_prepare_rows(const PrepareParams& p, cudaStream_t st) {
    const unsigned jobs = (unsigned)ceil_div(p.g.heads + p.g.kv_heads, kPrepareWarps);
    if (p.s.rows <= 256) return launch_kernel(grouped_prepare_kernel<TAPS, NI, 1>, dim3((unsigned)p.s.rows, jobs), dim3(kPrepareWarps * 32), 0, st, 1, p);
    return launch_kernel(grouped_prepare_kernel<TAPS, NI, 8>, dim3((unsigned)ceil_div((int)p.s.rows, 8), jobs), dim3(kPrepareWarps * 32), 0, st, 1, p);
}
template <int NI>
int launch_prepare(const PrepareParams& p, cudaStream_t st) {
    return p.taps == 1 ? launch_prepare_rows<1, NI>(p, st) : p.taps == 2 ? launch_prepare_rows<2, NI>(p, st) : p.taps == 3 ? launch_prepare_rows<3, NI>(p, st) : launch_prepare_rows<4, NI>(p, st);
}

// ---- plain attention: one CTA per (head, row) ---------------------------------------------------------------------------------
struct AttnParams {
    Shape g;
    const void* qkv;
    const unsigned char* pool;
    const int *page_table, *slot, *ctx_len;
    const float *r1, *r2;
    const int* reach;
    void* out;
    int* status;
    int max_pages;
};
constexpr int kPlainThreads = 128;
constexpr int kPlainCols = 8;   // value columns per thread: vdim up to 1024

template <bool BF16>
__global__ void __launch_bounds__(kPlainThreads) grouped_attention_kernel(const AttnParams p) {
    extern __shared__ __align__(16) float ga_smem[];
    const Shape& g = p.g;
    const int dim_pad = up(g.dim, 8);
    float* qs = ga_smem;              // [dim_pad]
    float* ps = ga_smem + dim_pad;    // [kPlainThreads]
    __shared__ long long s_row[kPlainThreads];   // byte offset of the block of every key of the round
    __shared__ float sh[8];
    const int head = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    int len = p.ctx_len[row];
    if (len < 0 || len > p.max_pages * kPageTok) { if (tid == 0) atomicExch(p.status, 2); len = len < 0 ? 0 : p.max_pages * kPageTok; }
    const int kvh = head / g.group, width = g.width;
    int lo = first_visible(g.mask, g.mask_size, max(len - 1, 0));
    if (p.reach) lo = max(lo, len - 1 - p.reach[kvh]);
    const int* pt = p.page_table + (size_t)p.slot[row] * p.max_pages;
    const float r1 = p.r1 ? p.r1[head] : 0.f, r2 = p.r2 ? p.r2[head] : 0.f;
    float o[kPlainCols], acc[kPlainCols];
    float m, l;
    for (int part = 0; part < g.maps; ++part) {
        const size_t qo = (size_t)row * g.query_row + (size_t)head * g.q_head_stride + (size_t)part * g.map_stride;
        for (int c = tid; c < dim_pad; c += kPlainThreads) {
            float v = 0.f;
            if (c < g.dim) v = BF16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.qkv)[qo + c]) : static_cast<const float*>(p.qkv)[qo + c];
            qs[c] = v;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kPlainCols; ++i) acc[i] = 0.f;
        m = -INFINITY; l = 0.f;
        for (int j0 = lo; j0 < len; j0 += kPlainThreads) {
            const int n = min(kPlainThreads, len - j0);
            float s = -INFINITY;
            if (tid < n) {
                const int j = j0 + tid;
                const long long page = (long long)pt[j / kPageTok] * g.page_bytes, base = page + kvh * g.block_bytes;
                s_row[tid] = base;
                s = 0.f;
                if constexpr (BF16) {
                    const unsigned char* pg = p.pool + base;
                    for (int k = 0; k < dim_pad / 8; ++k) {
                        const uint4 u = __ldg(reinterpret_cast<const uint4*>(pg + page_chunk(j % kPageTok, (g.tied ? 0 : g.nbv + part * g.nbk) * 8 + k, g.nb)));
                        const float* qk = qs + k * 8;
                        s = fmaf(qk[0], bf16_lo(u.x), s); s = fmaf(qk[1], bf16_hi(u.x), s);
                        s = fmaf(qk[2], bf16_lo(u.y), s); s = fmaf(qk[3], bf16_hi(u.y), s);
                        s = fmaf(qk[4], bf16_lo(u.z), s); s = fmaf(qk[5], bf16_hi(u.z), s);
                        s = fmaf(qk[6], bf16_lo(u.w), s); s = fmaf(qk[7], bf16_hi(u.w), s);
                    }
                } else {
                    const float* kv = reinterpret_cast<const float*>(p.pool + base) + (size_t)(j % kPageTok) * width + (g.tied ? 0 : g.vdim + part * g.dim);
                    for (int c = 0; c < g.dim; ++c) s = fmaf(qs[c], __ldg(kv + c), s);
                }
                if (g.tied) s *= __ldg(reinterpret_cast<const float*>(p.pool + page + g.kv_heads * g.block_bytes) + kvh * kPageTok + j % kPageTok);
                s *= g.scale;
                if (g.softcap > 0.f) s = g.softcap * tanhf(s / g.softcap);
                if (p.r1) s -= r1 * (p.r2 ? log1pf(r2 * (float)(len - 1 - j)) : (float)(len - 1 - j));
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
            const float alpha = expf(m - m_new);   // 0 for the first round
            l = l * alpha + ((sh[4] + sh[5]) + (sh[6] + sh[7]));
            m = m_new;
#pragma unroll
            for (int i = 0; i < kPlainCols; ++i) {
                const int c = tid + i * kPlainThreads;
                if (c >= g.vdim) break;
                float a = acc[i] * alpha;
                for (int k = 0; k < n; ++k) {
                    const int t = (j0 + k) % kPageTok;
                    float v;
                    if constexpr (BF16)
                        v = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(p.pool + s_row[k] + page_chunk(t, c >> 3, g.nb) + (c & 7) * 2));
                    else
                        v = __ldg(reinterpret_cast<const float*>(p.pool + s_row[k]) + (size_t)t * width + c);
                    a = fmaf(ps[k], v, a);
                }
                acc[i] = a;
            }
            __syncthreads();
        }
        const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
        for (int i = 0; i < kPlainCols; ++i) {
            const float v = tid + i * kPlainThreads < g.vdim ? acc[i] * inv : 0.f;
            o[i] = part == 0 ? v : fmaf(-g.lambda, v, o[i]);
        }
    }
    float f = 1.f;
    if (g.maps > 1) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < kPlainCols; ++i) ss = fmaf(o[i], o[i], ss);
        ss = warp_sum(ss);
        __syncthreads();
        if ((tid & 31) == 0) sh[tid >> 5] = ss;
        __syncthreads();
        f = g.head_scale / sqrtf(((sh[0] + sh[1]) + (sh[2] + sh[3])) / (float)g.vdim + g.head_eps);
    }
    const size_t oo = ((size_t)row * g.heads + head) * g.out_stride, go = (size_t)row * g.q_row + g.g_off + (size_t)head * g.g_head_stride;
#pragma unroll
    for (int i = 0; i < kPlainCols; ++i) {
        const int c = tid + i * kPlainThreads;
        if (c >= g.out_stride) break;
        float v = o[i] * f;
        if (g.g_head_stride > 0 && c < g.vdim) {
            const float z = BF16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(p.qkv)[go + c]) : static_cast<const float*>(p.qkv)[go + c];
            v /= 1.f + expf(-z);
        }
        if (BF16) static_cast<__nv_bfloat16*>(p.out)[oo + c] = __float2bfloat16_rn(v);
        else static_cast<float*>(p.out)[oo + c] = v;
    }
}

// queries [dim][parts][heads][T] of projection rows; a box is 64 columns of one part of `heads` heads of `tokens` tokens
int encode_queries(const void* qkv, const Shape& g, int64_t n_tokens, int heads, int tokens, CUtensorMap* map) {
    EncodeTiledFn enc = encode_fn();
    if (!enc) return fail(GPTRS_EXECUTION, "cuTensorMapEncodeTiled is not available");
    cuuint64_t dims[4] = {(cuuint64_t)g.map_stride, (cuuint64_t)g.maps, (cuuint64_t)g.heads, (cuuint64_t)n_tokens};
    cuuint64_t strides[3] = {(cuuint64_t)g.map_stride * 2, (cuuint64_t)g.q_head_stride * 2, (cuuint64_t)g.query_row * 2};
    cuuint32_t box[4] = {64, 1, (cuuint32_t)heads, (cuuint32_t)tokens};
    cuuint32_t estr[4] = {1, 1, 1, 1};
    CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(qkv), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                     CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(GPTRS_EXECUTION, "cuTensorMapEncodeTiled failed for grouped attention (" + std::to_string((int)r) + ")");
    return GPTRS_OK;
}

int tile_rows(const Shape& g) { return g.maps > 1 ? kRows / 2 : kRows; }   // rows of a tile that are (token, head) pairs of their own
int query_blocks(const Shape& g) { return g.tied ? g.nbv : g.nb - g.nbv; }
uint32_t decode_stage_bytes(const Shape& g) { return (uint32_t)g.block_bytes + (g.tied ? kPageTok * 4u : 0u); }
bool decode_fits(const Shape& g) {
    static const bool on = [] { const char* e = getenv("GPTRS_GROUPED_DECODE"); return !e || atoi(e) != 0; }();
    return on && g.maps == 1 && g.g_head_stride == 0 && g.group <= kDecHeads && g.nbv <= 2 && query_blocks(g) <= 2 && decode_stages(decode_stage_bytes(g)) >= 2;
}
int tile_tokens(const Shape& g) { return g.group >= tile_rows(g) ? 1 : tile_rows(g) / g.group; }

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" {

int gptrs_cuda_grouped_layout(gptrs_grouped_attention* a) {
    GPTRS_REQUIRE(a, "null pointer");
    GPTRS_REQUIRE(a->heads > 0 && a->kv_heads > 0 && a->dim > 0 && a->vdim > 0, "grouped attention: sizes must be positive");
    GPTRS_REQUIRE(a->heads % a->kv_heads == 0, "grouped attention: query heads must be a multiple of kv heads");
    GPTRS_REQUIRE(a->mask == GPTRS_MASK_CAUSAL || ((a->mask == GPTRS_MASK_WINDOW || a->mask == GPTRS_MASK_CHUNK) && a->mask_size > 0), "grouped attention: mask");
    GPTRS_REQUIRE(a->scale > 0.f && a->softcap >= 0.f, "grouped attention: the scale must be positive, the soft cap not negative");
    GPTRS_REQUIRE(a->dtype == GPTRS_F32 || a->dtype == GPTRS_BF16, "grouped attention: f32 or bf16");
    GPTRS_REQUIRE(a->maps >= 0 && a->maps <= 2, "grouped attention: one or two parts of a head");
    if (a->vdim > kPlainThreads * kPlainCols || a->dim > 8192) return fail(GPTRS_UNIMPLEMENTED, "grouped attention: vdim above 1024 or dim above 8192");
    const bool bf16 = a->dtype == GPTRS_BF16;
    const int maps = a->maps > 1 ? a->maps : 1;
    const bool prepared = a->taps > 0 || a->qk_norm || a->tied;
    GPTRS_REQUIRE(a->distance_bias >= GPTRS_DISTANCE_NONE && a->distance_bias <= GPTRS_DISTANCE_LINEAR && a->taps >= 0, "grouped attention: distance penalty or taps");
    GPTRS_REQUIRE(!a->tied || (a->dim == a->vdim && a->distance_bias != GPTRS_DISTANCE_LOG), "grouped attention: values that are keys have the keys' size and no logarithmic penalty");
    if (maps > 1 && (prepared || a->distance_bias == GPTRS_DISTANCE_LINEAR)) return fail(GPTRS_UNIMPLEMENTED, "grouped attention: two parts with convolutions, norms or a linear penalty");
    if (prepared && (a->gate || a->shared_kv)) return fail(GPTRS_UNIMPLEMENTED, "grouped attention: convolutions or norms with a gate or shared keys");
    a->map_stride = bf16 ? up(a->dim, 8) : a->dim;
    a->q_head_stride = a->k_head_stride = maps * a->map_stride;
    a->v_head_stride = a->out_head_stride = bf16 ? up(a->vdim, 8) : a->vdim;
    a->k_offset = a->heads * a->q_head_stride;
    a->v_offset = a->k_offset + (a->shared_kv ? 0 : a->kv_heads * a->k_head_stride);
    a->g_offset = a->v_offset + (a->shared_kv || a->tied ? 0 : a->kv_heads * a->v_head_stride);
    a->g_head_stride = a->gate ? a->out_head_stride : 0;
    a->q_row = a->g_offset + a->heads * a->g_head_stride;
    a->query_row = prepared ? a->heads * a->q_head_stride : a->q_row;
    a->conv_channels = a->v_offset;
    a->conv_floats = a->taps > 1 ? (int64_t)2 * (a->taps - 1) * a->conv_channels : 0;
    const int key_parts = a->tied ? 0 : maps;
    a->page_bytes = (int64_t)a->kv_heads * kPageTok * (bf16 ? (key_parts * up(a->dim, 64) + up(a->vdim, 64)) * 2 : (key_parts * a->dim + a->vdim) * 4);
    if (a->tied) a->page_bytes = (a->page_bytes + (int64_t)a->kv_heads * kPageTok * 4 + 127) / 128 * 128;
    return GPTRS_OK;
}

int gptrs_cuda_grouped_append(const gptrs_grouped_attention* a, const void* d_qkv, const int32_t* d_positions, const int32_t* d_slot,
                              const int32_t* d_page_table, int64_t max_pages, void* d_pool, int64_t n_tokens, void* stream) {
    GPTRS_REQUIRE(a && d_qkv && d_positions && d_slot && d_page_table && d_pool, "null pointer");
    GPTRS_REQUIRE(a->q_row > 0 && max_pages > 0, "grouped attention: layout not filled in");
    GPTRS_REQUIRE(!a->shared_kv, "grouped attention: these rows hold no keys and values");
    GPTRS_REQUIRE(a->taps == 0 && !a->qk_norm && !a->tied, "grouped attention: these rows go through gptrs_cuda_grouped_prepare");
    if (n_tokens == 0) return GPTRS_OK;
    AppendParams p = {shape_of(*a), d_qkv, d_positions, d_slot, d_page_table, static_cast<unsigned char*>(d_pool), (int)max_pages};
    const dim3 grid((unsigned)n_tokens);
    return a->dtype == GPTRS_BF16 ? launch_kernel(grouped_append_kernel<true>, grid, dim3(kAppendThreads), 0, as_stream(stream), 1, p)
                                  : launch_kernel(grouped_append_kernel<false>, grid, dim3(kAppendThreads), 0, as_stream(stream), 1, p);
}

int gptrs_cuda_grouped_prepare(const gptrs_grouped_attention* a, const gptrs_grouped_step* step, void* stream) {
    GPTRS_REQUIRE(a && step && a->q_row > 0, "null pointer, or layout not filled in");
    const gptrs_grouped_step& s = *step;
    GPTRS_REQUIRE(a->taps > 0 || a->qk_norm || a->tied, "grouped attention: these rows go through gptrs_cuda_grouped_append");
    GPTRS_REQUIRE(s.d_qkv && s.d_slot && s.d_pos && s.d_run_first && s.d_run_last && s.d_parity && s.d_page_table && s.d_pool && s.d_q && s.max_pages > 0, "null pointer");
    GPTRS_REQUIRE((a->taps == 0 || s.d_conv) && (a->taps <= 1 || s.d_conv_state) && (!a->qk_norm || (s.d_q_gain && (a->tied || s.d_k_gain))), "null pointer");
    GPTRS_REQUIRE(s.rows >= 0 && s.rows < (1ll << 31) && a->heads + a->kv_heads <= 65535 * kPrepareWarps, "bad shape");
    if (s.rows == 0) return GPTRS_OK;
    PrepareParams p = {shape_of(*a), s, a->taps > 0 ? a->taps : 1, a->conv_channels, a->qk_norm, a->head_eps};
    if (a->taps == 0) p.s.d_conv = nullptr;
    cudaStream_t st = as_stream(stream);
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(s.d_qkv) | reinterpret_cast<uintptr_t>(s.d_conv) | reinterpret_cast<uintptr_t>(s.d_conv_state) |
                           reinterpret_cast<uintptr_t>(s.d_pool) | reinterpret_cast<uintptr_t>(s.d_q);
    if (a->dtype == GPTRS_BF16 && p.taps <= 4 && a->dim <= 256 && (ptrs & 15) == 0) return a->dim <= 128 ? launch_prepare<1>(p, st) : launch_prepare<2>(p, st);
    const dim3 grid((unsigned)s.rows, (unsigned)ceil_div(a->heads + a->kv_heads, kPrepareWarps));
    return a->dtype == GPTRS_BF16 ? launch_kernel(grouped_prepare_any_kernel<__nv_bfloat16>, grid, dim3(kPrepareWarps * 32), 0, st, 1, p)
                                  : launch_kernel(grouped_prepare_any_kernel<float>, grid, dim3(kPrepareWarps * 32), 0, st, 1, p);
}

int gptrs_cuda_grouped_tile_tokens(const gptrs_grouped_attention* a) {
    if (!a || a->dtype != GPTRS_BF16 || a->heads < 1) return 0;
    const Shape g = shape_of(*a);
    return tc_fits(query_blocks(g), g.nbv, g.nb) ? tile_tokens(g) : 0;
}

int gptrs_cuda_grouped_splits(const gptrs_grouped_attention* a, int64_t n_tokens, int64_t n_tiles, int64_t max_ctx_len) {
    const int tokens = gptrs_cuda_grouped_tile_tokens(a);
    if (n_tiles <= 0 || tokens == 0) return 1;
    const int64_t limit = a->mask == GPTRS_MASK_CAUSAL ? max_ctx_len : (int64_t)a->mask_size + tokens - 1;
    const int64_t span = max_ctx_len < limit ? max_ctx_len : limit;
    const int64_t blocks = (span + kPageTok - 1 + kKeys - 1) / kKeys;
    const Shape g = shape_of(*a);
    if (n_tiles == n_tokens && decode_fits(g)) return decode_splits(n_tiles * a->kv_heads, span);
    int64_t s = (tc_fits_twice(query_blocks(g), g.nbv, g.nb) ? 2 : 1) * sm_count() / (n_tiles * a->kv_heads * ceil_div(g.group, tile_rows(g)));
    if (s > blocks) s = blocks;
    return (int)(s < 1 ? 1 : s);
}

size_t gptrs_cuda_grouped_scratch_bytes(const gptrs_grouped_attention* a, int64_t n_tiles, int splits) {
    if (!a || splits <= 1) return 0;
    const Shape g = shape_of(*a);
    return tc_scratch_bytes(n_tiles, g.kv_heads * ceil_div(g.group, tile_rows(g)), splits, g.nbv);
}

int gptrs_cuda_grouped_attention(const gptrs_grouped_attention* a, const void* d_qkv, const void* d_pool, const int32_t* d_page_table, int64_t max_pages,
                                 const int32_t* d_slot, const int32_t* d_ctx_len, const float* d_r1, const float* d_r2, const int32_t* d_reach, const int32_t* d_tile_row,
                                 const int32_t* d_tile_rows, int64_t n_tiles, int splits, void* d_out, void* d_scratch, size_t scratch_bytes,
                                 int32_t* d_status, int64_t n_tokens, void* stream) {
    GPTRS_REQUIRE(a && d_qkv && d_pool && d_page_table && d_slot && d_ctx_len && d_out && d_status, "null pointer");
    GPTRS_REQUIRE(a->distance_bias == GPTRS_DISTANCE_NONE || (d_r1 && (d_r2 || a->distance_bias == GPTRS_DISTANCE_LINEAR)), "grouped attention: distance penalty without its numbers");
    GPTRS_REQUIRE(a->q_row > 0 && max_pages > 0 && max_pages * kPageTok < ((int64_t)1 << 30), "grouped attention: layout not filled in, or a bad page table");
    if (n_tokens == 0) return GPTRS_OK;
    const Shape g = shape_of(*a);
    cudaStream_t st = as_stream(stream);
    const float *r1 = a->distance_bias != GPTRS_DISTANCE_NONE ? d_r1 : nullptr, *r2 = a->distance_bias == GPTRS_DISTANCE_LOG ? d_r2 : nullptr;
    if (n_tiles <= 0) {   // plain kernel: every row by itself
        GPTRS_REQUIRE(n_tokens <= 65535, "grouped attention: too many rows in one launch");
        AttnParams p = {g, d_qkv, static_cast<const unsigned char*>(d_pool), d_page_table, d_slot, d_ctx_len, r1, r2, d_reach, d_out, d_status, (int)max_pages};
        const size_t smem = ((size_t)up(g.dim, 8) + kPlainThreads) * 4;
        const dim3 grid((unsigned)g.heads, (unsigned)n_tokens);
        return a->dtype == GPTRS_BF16 ? launch_kernel(grouped_attention_kernel<true>, grid, dim3(kPlainThreads), smem, st, 1, p)
                                      : launch_kernel(grouped_attention_kernel<false>, grid, dim3(kPlainThreads), smem, st, 1, p);
    }
    const int tokens = gptrs_cuda_grouped_tile_tokens(a);
    if (tokens == 0) return fail(GPTRS_UNIMPLEMENTED, "grouped attention: these sizes do not fit the tensor-core kernel (pass n_tiles = 0)");
    GPTRS_REQUIRE(d_tile_row && d_tile_rows && splits >= 1 && splits <= 65535, "grouped attention: tile list");
    GPTRS_REQUIRE((reinterpret_cast<uintptr_t>(d_pool) & 15) == 0 && (reinterpret_cast<uintptr_t>(d_qkv) & 15) == 0 && (reinterpret_cast<uintptr_t>(d_out) & 15) == 0,
                  "grouped attention: 16-byte alignment");
    const bool decode = n_tiles == n_tokens && decode_fits(g);   // every row is a tile
    const size_t need = decode ? (splits > 1 ? (size_t)n_tiles * g.kv_heads * splits * kDecHeads * (g.nbv * 256 + 8) : 0) : gptrs_cuda_grouped_scratch_bytes(a, n_tiles, splits);
    GPTRS_REQUIRE(need == 0 || (d_scratch && scratch_bytes >= need), "grouped attention: scratch too small");
    if (decode) {
        DecodeParams p = {};
        FlashShape& f = p.g;
        f.heads = g.heads; f.kv_heads = g.kv_heads; f.group = g.group; f.blocks = g.nb; f.key_block = g.tied ? 0 : g.nbv; f.mask = g.mask; f.mask_size = g.mask_size;
        f.out_stride = g.out_stride; f.vdim = g.vdim; f.key_scales = g.tied; f.page_bytes = g.page_bytes; f.block_bytes = (uint32_t)g.block_bytes;
        p.q = static_cast<const __nv_bfloat16*>(d_qkv); p.q_row = g.query_row; p.q_head_stride = g.q_head_stride; p.q_cols = g.map_stride;
        p.pool = static_cast<const unsigned char*>(d_pool);
        p.page_table = d_page_table; p.slot = d_slot; p.ctx_len = d_ctx_len; p.tile_row = d_tile_row;
        p.out = static_cast<__nv_bfloat16*>(d_out); p.status = d_status;
        p.max_pages = (int)max_pages; p.splits = splits; p.stage_bytes = (int)decode_stage_bytes(g); p.stages = decode_stages(decode_stage_bytes(g));
        p.scale = g.scale; p.cap = g.softcap; p.r1 = r1; p.r2 = r2; p.reach = d_reach;
        const bool k2 = query_blocks(g) == 2, v2 = g.nbv == 2;
        return k2 ? (v2 ? launch_decode<2, 2>(p, n_tiles, d_scratch, st) : launch_decode<2, 1>(p, n_tiles, d_scratch, st))
                  : (v2 ? launch_decode<1, 2>(p, n_tiles, d_scratch, st) : launch_decode<1, 1>(p, n_tiles, d_scratch, st));
    }
    TcParams p = {};
    const int box_heads = g.group < tile_rows(g) ? g.group : tile_rows(g);
    int rc = encode_queries(d_qkv, g, n_tokens, box_heads, tokens, &p.q_map);
    if (!rc) rc = encode_queries(d_qkv, g, n_tokens, box_heads, 1, &p.q_one);
    if (rc) return rc;
    p.q_box_bytes = (uint32_t)(box_heads * tokens) * 128u;
    p.q_one_bytes = (uint32_t)box_heads * 128u;
    FlashShape& f = p.g;
    f.heads = g.heads; f.kv_heads = g.kv_heads; f.group = g.group;
    f.blocks = g.nb; f.value_blocks = g.nbv; f.key_block = g.tied ? 0 : g.nbv; f.query_blocks = query_blocks(g);
    f.map_blocks = f.query_blocks / g.maps;
    f.key_scales = g.tied;
    for (int b = 0; b < f.query_blocks; ++b) {
        const int left = g.dim - b % f.map_blocks * 64;
        f.steps[b] = left >= 64 ? 4 : (left + 15) / 16;
    }
    f.mask = g.mask; f.mask_size = g.mask_size;
    f.out_stride = g.out_stride; f.vdim = g.vdim;
    f.page_bytes = g.page_bytes; f.block_bytes = (uint32_t)g.block_bytes;
    p.pool = static_cast<const unsigned char*>(d_pool);
    p.page_table = d_page_table; p.slot = d_slot; p.ctx_len = d_ctx_len; p.tile_row = d_tile_row; p.tile_rows = d_tile_rows;
    p.out = static_cast<__nv_bfloat16*>(d_out);
    p.status = d_status;
    p.max_pages = (int)max_pages; p.splits = splits;
    p.r1 = r1; p.r2 = r2; p.reach = d_reach;
    p.scale_log2 = g.softcap > 0.f ? 2.f * kLog2e * g.scale / g.softcap : kLog2e * g.scale;
    p.cap_log2 = g.softcap > 0.f ? kLog2e * g.softcap : 0.f;
    p.head_out = {g.lambda, g.head_scale, g.head_eps, g.g_head_stride > 0 ? static_cast<const __nv_bfloat16*>(d_qkv) + g.g_off : nullptr, g.q_row, g.g_head_stride};
    const bool twice = tc_fits_twice(f.query_blocks, f.value_blocks, f.blocks);
    if (g.maps > 1) return twice ? launch_flash<true, 2, true>(p, n_tiles, d_scratch, st) : launch_flash<true, 3, true>(p, n_tiles, d_scratch, st);
    if (g.tied || a->distance_bias == GPTRS_DISTANCE_LINEAR) return twice ? launch_flash<true, 2, false, true>(p, n_tiles, d_scratch, st) : launch_flash<true, 3, false, true>(p, n_tiles, d_scratch, st);
    return twice ? launch_flash<true, 2>(p, n_tiles, d_scratch, st) : launch_flash<true, 3>(p, n_tiles, d_scratch, st);
}

}  // extern "C"
