// Decode steps of attention with up to eight query heads per key / value head (grouped_attention.cu): every row is a token of its own, so
// the whole cache is read for a handful of rows and the kernel is a matter of bytes. One CTA per (row, key split, kv head); each of its four
// warps has a ring of pages of its own, filled by bulk copies, and walks every fourth page from the newest to the oldest with a running maximum,
// sum and output; the warps' parts meet in shared memory at the end, those of the splits in flash_combine_kernel.
//
// A page is 16 keys: S is two m16n8k16 products per 16 columns, with the heads as rows 0 .. 7 of the 16. The weights enter the second product as
// two bf16 terms, P_hi in rows 0 .. 7 and P_lo in rows 8 .. 15 of ONE operand, which costs no instruction more than rounded weights would. Scores and
// sums are f32, as in the tcgen05 kernel, whose rows of a tile would be all but empty here.
#pragma once
#include "flash_tc.cuh"

namespace gptrs {
namespace {

constexpr int kDecWarps = 4;
constexpr int kDecHeads = 8;      // most heads per kv head
constexpr int kDecMaxStages = 6;
constexpr int kDecCtas = 3;       // per SM

struct DecodeParams {
    FlashShape g;
    const __nv_bfloat16* q;
    int q_row, q_head_stride, q_cols;   // q_cols: columns of a head that exist
    const unsigned char* pool;
    const int *page_table, *slot, *ctx_len, *tile_row;
    __nv_bfloat16* out;
    float* part_o;                      // splits > 1: [row][kv head][split][8][64 value_blocks]
    float2* part_ml;
    int* status;
    int max_pages, splits, stages, stage_bytes;
    float scale, cap;                   // cap 0: none
    const float *r1, *r2;               // distance penalty: r1 ln(1 + r2 d), or r1 d without r2, or none
    const int* reach;
};

template <int KB, int VB>   // 64-column blocks of a key and of a value
__global__ void __launch_bounds__(kDecWarps * 32, kDecCtas) grouped_decode_kernel(const DecodeParams p) {
    extern __shared__ __align__(128) unsigned char gd_smem[];
    __shared__ __align__(8) uint64_t full[kDecWarps][kDecMaxStages];
    __shared__ float2 s_ml[kDecWarps][kDecHeads];
    const FlashShape& g = p.g;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gi = lane >> 2, t = lane & 3;
    const int kvh = (int)gridDim.z - 1 - (int)blockIdx.z, group = g.group;   // later kv heads reach further: start them first
    unsigned char* ring = gd_smem + warp * p.stages * p.stage_bytes;
    if (lane == 0) {
        for (int i = 0; i < p.stages; ++i) mbar_init(&full[warp][i], 1);
        mbar_fence_init();
    }
    __syncwarp();
    pdl_launch_dependents();
    pdl_wait();
    const int row = p.tile_row[blockIdx.x], cap_len = p.max_pages * kPageTok;
    int len = p.ctx_len[row];
    if (len < 0 || len > cap_len) { if (tid == 0) atomicExch(p.status, 2); len = len < 0 ? 0 : cap_len; }
    int lo = first_visible(g.mask, g.mask_size, max(len - 1, 0));
    if (p.reach) lo = max(lo, len - 1 - p.reach[kvh]);
    const int p_lo = lo / kPageTok, n_all = len > lo ? (len + kPageTok - 1) / kPageTok - p_lo : 0;
    const int b0 = (int)((int64_t)n_all * blockIdx.y / p.splits), b1 = (int)((int64_t)n_all * (blockIdx.y + 1) / p.splits);
    const int n_my = b1 - b0 > warp ? (b1 - b0 - warp + kDecWarps - 1) / kDecWarps : 0, newest = p_lo + b1 - 1 - warp;
    const int* pt = p.page_table + (size_t)p.slot[row] * p.max_pages;
    auto page_of = [&](int j) { return j < n_my ? __ldg(pt + newest - j * kDecWarps) : 0; };
    const uint32_t page_bytes = g.block_bytes + (g.key_scales ? kPageTok * 4u : 0u);
    auto issue = [&](int j, int st, int page) {
        if (lane == 0 && j < n_my) {
            uint64_t* bar = &full[warp][st];
            mbar_expect_tx(bar, page_bytes);
            const unsigned char* src = p.pool + (size_t)page * g.page_bytes;
            bulk_g2s(ring + st * p.stage_bytes, src + (size_t)kvh * g.block_bytes, g.block_bytes, bar);
            if (g.key_scales) bulk_g2s(ring + st * p.stage_bytes + g.block_bytes, src + (size_t)g.kv_heads * g.block_bytes + kvh * (kPageTok * 4), kPageTok * 4, bar);
        }
    };
    for (int j = 0; j < p.stages; ++j) issue(j, j, page_of(j));
    int page_next = page_of(p.stages);

    const bool valid = gi < group;
    const int head = kvh * group + (valid ? gi : 0);
    uint32_t qf[KB * 4][2];
    {
        const __nv_bfloat16* q = p.q + (size_t)row * p.q_row + (size_t)head * p.q_head_stride;
#pragma unroll
        for (int ks = 0; ks < KB * 4; ++ks)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int c = ks * 16 + i * 8 + 2 * t;
                qf[ks][i] = valid && c < p.q_cols ? __ldg(reinterpret_cast<const uint32_t*>(q + c)) : 0u;
            }
    }
    const float r1 = valid && p.r1 ? p.r1[head] : 0.f, r2 = valid && p.r2 ? p.r2[head] : 0.f;
    float o[VB * 8][4];
#pragma unroll
    for (int i = 0; i < VB * 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
    float m_run = -1e30f, l_run = 0.f;
    bool failed = false;
    const uint32_t ring_addr = smem_u32(ring), nb = (uint32_t)g.blocks;
    const int k_tok = ((lane >> 4) << 3) + (lane & 7), k_half = (lane >> 3) & 1;     // rows and chunk of the K operand
    const int v_tok = (((lane >> 3) & 1) << 3) + (lane & 7), v_chunk = lane >> 4;    // and of the transposed V operand
    const uint32_t k_row = (uint32_t)(k_tok >> 3) * nb * 1024u + (uint32_t)(k_tok & 7) * 128u + (uint32_t)g.key_block * 1024u;
    const uint32_t v_row = (uint32_t)(v_tok >> 3) * nb * 1024u + (uint32_t)(v_tok & 7) * 128u;
    const float scale_log2 = p.cap > 0.f ? p.scale / p.cap : p.scale * kLog2e;

    int st = 0;
    uint32_t phase = 0;
    for (int j = 0; j < n_my; ++j) {
        if (!mbar_wait_bounded(&full[warp][st], phase)) failed = true;
        if (__any_sync(0xffffffffu, failed)) { failed = true; break; }
        const uint32_t page = ring_addr + (uint32_t)(st * p.stage_bytes);
        const int tok0 = (newest - j * kDecWarps) * kPageTok;
        if (tok0 + kPageTok > len) {   // cache rows past the last key may hold anything; their weights are 0, but 0 x NaN is not
            for (int i = lane; i < (tok0 + kPageTok - len) * VB * 8; i += 32) {
                const int r = len - tok0 + i / (VB * 8), c = i % (VB * 8);
                st_shared_v4(page + (uint32_t)(r >> 3) * nb * 1024u + (uint32_t)(c >> 3) * 1024u + (uint32_t)(r & 7) * 128u + (uint32_t)((c & 7) << 4), 0, 0, 0, 0);
            }
            __syncwarp();
        }
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
        for (int ks = 0; ks < KB * 4; ++ks) {
            uint32_t b[4];
            const int c = 2 * ks + k_half;
            ldmatrix_x4(b, page + k_row + (uint32_t)(c >> 3) * 1024u + (uint32_t)(((c & 7) ^ (k_tok & 7)) << 4));
            const uint32_t a[4] = {qf[ks][0], 0u, qf[ks][1], 0u};
            mma_bf16_16816(s[0], a, b[0], b[1]);
            mma_bf16_16816(s[1], a, b[2], b[3]);
        }
        float x[4], mx = -INFINITY;
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            float2 f = make_float2(1.f, 1.f);
            if (g.key_scales) f = *reinterpret_cast<const float2*>(ring + st * p.stage_bytes + g.block_bytes + (n * 8 + 2 * t) * 4);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int key = tok0 + n * 8 + 2 * t + e;
                float v = s[n][e] * (e ? f.y : f.x) * scale_log2;
                if (p.cap > 0.f) v = p.cap * kLog2e * tanhf(v);
                if (p.r1) {
                    const float dist = (float)(len - 1 - key);
                    float l = dist * kLog2e;
                    if (p.r2) asm("lg2.approx.ftz.f32 %0, %1;\n" : "=f"(l) : "f"(fmaf(r2, fmaxf(dist, 0.f), 1.f)));
                    v = fmaf(-r1, l, v);
                }
                v = key >= lo && key < len ? v : -INFINITY;
                x[2 * n + e] = v;
                mx = fmaxf(mx, v);
            }
        }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        if (__any_sync(0xffffffffu, mx > m_run)) {   // every page has a visible key, so the maximum is finite from the first one on
            const float m_new = fmaxf(m_run, mx), alpha = ex2f(m_run - m_new);
            m_run = m_new;
            l_run *= alpha;
#pragma unroll
            for (int i = 0; i < VB * 8; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[i][e] *= alpha;
        }
        uint32_t w[4];
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const float p0 = ex2f(x[2 * n] - m_run), p1 = ex2f(x[2 * n + 1] - m_run);
            l_run += p0 + p1;
            w[2 * n] = pack_bf16x2(p0, p1);
            w[2 * n + 1] = pack_bf16x2(p0 - bf16_lo(w[2 * n]), p1 - bf16_hi(w[2 * n]));
        }
#pragma unroll
        for (int i = 0; i < VB * 4; ++i) {
            uint32_t b[4];
            const int c = 2 * i + v_chunk;
            ldmatrix_x4_trans(b, page + v_row + (uint32_t)(c >> 3) * 1024u + (uint32_t)(((c & 7) ^ (v_tok & 7)) << 4));
            mma_bf16_16816(o[2 * i], w, b[0], b[1]);
            mma_bf16_16816(o[2 * i + 1], w, b[2], b[3]);
        }
        __syncwarp();
        if (j + p.stages < n_my) {
            fence_proxy_async();
            issue(j + p.stages, st, page_next);
            page_next = page_of(j + p.stages + 1);
        }
        if (++st == p.stages) { st = 0; phase ^= 1u; }
    }
    if (failed) {   // copies in flight write this CTA's shared memory: wait for them (bounded) before going on
        if (lane == 0) atomicExch(p.status, 3);
        for (int i = 0; i < p.stages; ++i) {
            mbar_wait_bounded(&full[warp][st], phase);
            if (++st == p.stages) { st = 0; phase ^= 1u; }
        }
        l_run = 0.f;
    }
    l_run += __shfl_xor_sync(0xffffffffu, l_run, 1);
    l_run += __shfl_xor_sync(0xffffffffu, l_run, 2);
    __syncthreads();   // every page has been used: the rings hold the warps' outputs from here on
    constexpr int COLS = VB * 64;
    float* mine = reinterpret_cast<float*>(gd_smem);   // [warp][8][COLS]
    if (valid) {
#pragma unroll
        for (int i = 0; i < VB * 8; ++i)
            *reinterpret_cast<float2*>(mine + (size_t)(warp * kDecHeads + gi) * COLS + i * 8 + 2 * t) = make_float2(o[i][0] + o[i][2], o[i][1] + o[i][3]);
        if (t == 0) s_ml[warp][gi] = make_float2(m_run, l_run);
    }
    __syncthreads();
    const size_t part = (((size_t)blockIdx.x * g.kv_heads + kvh) * p.splits + blockIdx.y) * kDecHeads;
    for (int i = tid; i < group * (COLS / 4); i += kDecWarps * 32) {
        const int r = i / (COLS / 4), c = i % (COLS / 4) * 4;
        float m = -1e30f, l = 0.f;
#pragma unroll
        for (int k = 0; k < kDecWarps; ++k) m = fmaxf(m, s_ml[k][r].x);
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int k = 0; k < kDecWarps; ++k) {
            const float f = ex2f(s_ml[k][r].x - m);
            l = fmaf(f, s_ml[k][r].y, l);
            const float4 v = *reinterpret_cast<const float4*>(mine + (size_t)(k * kDecHeads + r) * COLS + c);
            a.x = fmaf(f, v.x, a.x); a.y = fmaf(f, v.y, a.y); a.z = fmaf(f, v.z, a.z); a.w = fmaf(f, v.w, a.w);
        }
        if (p.splits > 1) {
            *reinterpret_cast<float4*>(p.part_o + (part + r) * COLS + c) = a;
            if (c == 0) p.part_ml[part + r] = make_float2(m, l);
        } else if (c < g.out_stride) {
            const float inv = l > 0.f ? 1.f / l : 0.f;
            *reinterpret_cast<uint2*>(p.out + ((size_t)row * g.heads + kvh * group + r) * g.out_stride + c) = make_uint2(pack_bf16x2(a.x * inv, a.y * inv), pack_bf16x2(a.z * inv, a.w * inv));
        }
    }
}

// Key splits of a decode step: a wave of CTAs (three where sequences are long, since heads with a reach end early), but not so many that the
// merge, which takes their parts one after another, weighs more than the pages a warp then does not have to walk.
inline int decode_splits(int64_t ctas, int64_t span) {
    const int64_t pages = span / kPageTok + 1, slots = (int64_t)kDecCtas * sm_count() * (pages >= 512 ? 3 : 1);
    int64_t s = (2 * slots + ctas) / (2 * ctas), most = (int64_t)(0.7 * sqrt((double)pages));
    if (most > pages / 16) most = pages / 16;
    if (s > most) s = most;
    return (int)(s < 1 ? 1 : s);
}

// stages of a warp's ring (0: these sizes do not fit)
inline int decode_stages(uint32_t stage_bytes) {
    const int n = (int)((uint32_t)(72 * 1024) / (kDecWarps * stage_bytes));
    return n > kDecMaxStages ? kDecMaxStages : n;
}

template <int KB, int VB>
int launch_decode(DecodeParams& p, int64_t n_rows, void* d_scratch, cudaStream_t st) {
    const FlashShape& g = p.g;
    const size_t ring = (size_t)kDecWarps * p.stages * p.stage_bytes, merge = (size_t)kDecWarps * kDecHeads * VB * 64 * 4, smem = ring > merge ? ring : merge;
    const size_t parts = (size_t)n_rows * g.kv_heads * p.splits * kDecHeads;
    p.part_o = static_cast<float*>(d_scratch);
    p.part_ml = reinterpret_cast<float2*>(p.part_o + parts * (VB * 64));
    static PerDeviceOnce once;
    if (once.first_time()) GPTRS_CUDA_OK(cudaFuncSetAttribute(grouped_decode_kernel<KB, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, 73 * 1024));
    int rc = launch_kernel(grouped_decode_kernel<KB, VB>, dim3((unsigned)n_rows, (unsigned)p.splits, (unsigned)g.kv_heads), dim3(kDecWarps * 32), smem, st, 1, p);
    if (rc || p.splits == 1) return rc;
    CombineParams c = {p.part_o, p.part_ml, p.tile_row, nullptr, p.out, g.heads, g.group, g.group, 1, p.splits, VB * 64, g.out_stride, g.vdim, {}, nullptr, kDecHeads};
    return launch_kernel(flash_combine_kernel<false>, dim3((unsigned)n_rows, (unsigned)ceil_div(g.group, 4), (unsigned)g.kv_heads), dim3(128), 0, st, 1, c);
}

}  // namespace
}  // namespace gptrs
