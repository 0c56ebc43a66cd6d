// Gated delta rule with a decay per key channel, or one per head (no counterpart in gpt.rs). Per head and token
//
//   S <- g S (rows of S are key channels);   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
// with q, k, v behind short causal convolutions and silu, q and k of unit length, and o normed and gated. The columns of S are
// independent of one another. Prompts take the recurrence in blocks of four tokens, which is exact algebra, not an approximation:
// with p_t the product of the block's decays up to token t (per key channel) and S0 the state in front of the block,
//
//   r_t = S0^T (p_t k_t)      u_t = beta_t (v_t - r_t - sum_{s<t} A_ts u_s)        A_ts = sum_d k_t k_s (decays of s+1 .. t)
//   w_t = S0^T (p_t q_t)      o_t = w_t + sum_{s<=t} B_ts u_s                      B_ts = sum_d q_t k_s (decays of s+1 .. t)
//   S4  = p_3 S0 + sum_t c_t u_t^T,   c_t = k_t (decays of t+1 .. 3)
//
// so that a block costs 13 multiply-adds per element of S instead of 16 and one reduction over the key channels instead of four.
// Every factor is a product of decays, at most 1. With one decay per head (HEAD) the decays leave the sums: r_t = p_t (S0^T k_t), c_t u_t^T =
// k_t (decay u_t)^T, so a block is the vectors k_t and q_t and eight numbers more.
//   delta_prepare_kernel   (delta_prepare.cu) prompts: a CTA per block, a warp per head: convolutions with their state, unit norms, decays, the vectors
//                          p_t k_t, p_t q_t, c_t, p_3 and the numbers A, B of the block
//   delta_scan_kernel      prompts: a warp keeps a few columns of a head's S in registers over a whole run (packed pairs of key channels,
//                          fma.rn.f32x2); blocks arrive by bulk copies in a ring of shared-memory stages (bounded waits, status 3); the sums meet in a transposing reduction
//   delta_output_kernel    prompts: norm and gate of the read-outs
//   delta_decode_kernel    rows that are runs of their own: all of the above in one launch, a CTA per (head, row), S is read and
//                          written once
// Everything that enters the recurrence, and S itself, is f32. S is updated in place (one CTA owns a column of a slot's state);
// the convolution state has two halves like the one of post_norm_conv.cu.
#include "delta_rule.cuh"

namespace gptrs {
namespace delta {
namespace {

constexpr int kMaxDim = 512;

// The convolution state that a single-token run reads and writes; place: where in the ring of taps - 1 inputs the last one lies.
struct RowState { int pos, place; const float* old; float* fresh; };
__device__ __forceinline__ RowState row_state(const Params& p, int row) {
    RowState r;
    const int keep = p.g.taps - 1;
    r.pos = p.s.d_pos[row];
    r.place = keep > 0 && r.pos > 0 ? (r.pos - 1) % keep : 0;
    const size_t half = (size_t)keep * p.g.channels;
    float* state = p.s.d_conv_state + (size_t)p.s.d_slot[row] * 2 * half;
    const int par = p.s.d_parity[row] & 1;
    r.old = state + par * half; r.fresh = state + (par ^ 1) * half;
    return r;
}
// silu(convolution) of channel `ch` (column `col` of the projection row) where the row is a run of its own; `keep_state`: this thread
// also passes the channel's inputs on to the next step. The loads of four taps or fewer are all under way at once.
template <typename T>
__device__ __forceinline__ float conv_channel(const Params& p, const RowState& r, int row, int ch, int col, bool keep_state) {
    const int keep = p.g.taps - 1;
    const float now = ld(static_cast<const T*>(p.s.d_proj) + (size_t)row * p.g.row + col);
    const float* w = p.s.d_conv + (size_t)ch * p.g.taps;
    float acc = 0.f;
    if (keep <= 3) {
        float v[3] = {0.f, 0.f, 0.f}, wt[3] = {0.f, 0.f, 0.f};
        int at[3];
#pragma unroll
        for (int k = 0; k < 3; ++k) {   // the input k + 1 positions back lies at r.place - k of the ring
            at[k] = r.place - k < 0 ? r.place - k + keep : r.place - k;
            if (k < keep) {
                wt[k] = __ldg(w + keep - 1 - k);
                if (r.pos - 1 - k >= 0) v[k] = r.old[(size_t)at[k] * p.g.channels + ch];
            }
        }
        const float w_now = __ldg(w + keep);
#pragma unroll
        for (int k = 2; k >= 0; --k) acc = fmaf(wt[k], v[k], acc);
        if (keep_state && keep > 0) {
#pragma unroll
            for (int k = 0; k < 2; ++k)   // the oldest one leaves
                if (k < keep - 1 && r.pos - 1 - k >= 0) r.fresh[(size_t)at[k] * p.g.channels + ch] = v[k];
            r.fresh[(size_t)(r.pos % keep) * p.g.channels + ch] = now;
        }
        return silu(fmaf(w_now, now, acc));
    }
    for (int k = keep; k >= 1; --k) {
        const int q = r.pos - k;
        if (q < 0) continue;
        const float v = r.old[(size_t)(q % keep) * p.g.channels + ch];
        acc = fmaf(w[keep - k], v, acc);
        if (keep_state && k < keep) r.fresh[(size_t)(q % keep) * p.g.channels + ch] = v;
    }
    if (keep_state) r.fresh[(size_t)(r.pos % keep) * p.g.channels + ch] = now;
    return silu(fmaf(w[keep], now, acc));
}

// ---- the scan ------------------------------------------------------------------------------------------------------------------
constexpr int kScanWarps = 8;

// LPC lanes share a column: lane l holds the channels (LPC i + l) 4 + e, i < NI, of CPL neighbouring columns; 32 / LPC such groups
// make a warp. dim <= 4 LPC NI. 
template <int NI, int CPL, int LPC, int STAGES, bool HEAD>
__global__ void __launch_bounds__(kScanWarps * 32) delta_scan_kernel(const Params p) {
    constexpr int kVecs = vecs_of(HEAD), kNums = nums_of(HEAD);
    constexpr int W = 4 * LPC * NI;                                 // channels with padding
    constexpr int GROUPS = 32 / LPC, COLS = kScanWarps * GROUPS * CPL;
    constexpr int kStage = kVecs * W + kBlock * COLS + kNums;       // floats
    constexpr int SH = (LPC == 16 ? 4 : 3) - (CPL == 4 ? 2 : CPL == 2 ? 1 : 0) - 1;   // lane bits that are left after (column, k or q)
    extern __shared__ __align__(16) float ds_smem[];
    __shared__ __align__(8) uint64_t full[STAGES];
    const Geo& g = p.g;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = lane & (LPC - 1), cg = lane / LPC;
    const int head = blockIdx.y;
    const int c_blk = blockIdx.x * COLS, col0 = c_blk + (warp * GROUPS + cg) * CPL;
    for (int i = tid; i < STAGES * kStage; i += kScanWarps * 32) ds_smem[i] = 0.f;   // the padding stays zero
    if (tid == 0) {
        for (int i = 0; i < STAGES; ++i) mbar_init(&full[i], 1);
        mbar_fence_init();
    }
    fence_proxy_async();
    pdl_launch_dependents();
    pdl_wait();
    const int run = blockIdx.z, r0 = p.s.d_runs[run], r1 = p.s.d_run_last[r0] + 1;
    const int blk0 = r0 / kBlock + run, n_blk = (r1 - r0 + kBlock - 1) / kBlock;
    float* state = p.s.d_state + ((size_t)p.s.d_slot[r0] * g.heads + head) * g.dim * g.vdim;
    const bool fresh = p.s.d_pos[r0] == 0;
    uint64_t S[NI][2][CPL];
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
            for (int j = 0; j < CPL; ++j) {
                const int d = (LPC * i + l) * 4 + 2 * e;
                const bool in = !fresh && col0 + j < g.vdim;
                S[i][e][j] = pair_of(in && d < g.dim ? state[(size_t)d * g.vdim + col0 + j] : 0.f, in && d + 1 < g.dim ? state[(size_t)(d + 1) * g.vdim + col0 + j] : 0.f);
            }
    __syncthreads();
    // the copies of a block, one per lane of warp 0: 13 vectors (a single one where they need no padding), 4 rows of values, the numbers
    const bool packed = g.dp == W;
    const uint32_t vec_bytes = (uint32_t)(packed ? kVecs : 1) * g.dp * 4, v_bytes = (uint32_t)min(COLS, g.vp - c_blk) * 4;
    const float* src = nullptr;   // of block 0
    uint32_t dst = 0, bytes = 0;
    size_t step = 0;
    if (warp == 0) {
        const size_t at = (size_t)blk0 * g.heads + head;
        if (lane < kVecs && (lane == 0 || !packed)) { src = p.w.vec + (at * kVecs + lane) * g.dp; dst = lane * W; bytes = vec_bytes; step = (size_t)g.heads * kVecs * g.dp; }
        else if (lane >= 16 && lane < 16 + kBlock) { src = p.w.v + (at * kBlock + lane - 16) * g.vp + c_blk; dst = kVecs * W + (lane - 16) * COLS; bytes = v_bytes; step = (size_t)g.heads * kBlock * g.vp; }
        else if (lane == 20) { src = p.w.num + at * kNums; dst = kVecs * W + kBlock * COLS; bytes = kNums * 4; step = (size_t)g.heads * kNums; }
    }
    const uint32_t total = (uint32_t)kVecs * g.dp * 4 + kBlock * v_bytes + kNums * 4, smem0 = smem_u32(ds_smem);
    auto request = [&](int b) {   // warp 0: block b of the run
        if (b >= n_blk) return;
        const uint32_t bar = smem_u32(&full[b % STAGES]);
        if (lane == 0) mbar_expect_tx_addr(bar, total);
        __syncwarp();
        if (bytes) bulk_g2s_addr(smem0 + ((b % STAGES) * kStage + dst) * 4, src + b * step, bytes, bar);
    };
    if (warp == 0)
#pragma unroll
        for (int b = 0; b < STAGES - 1; ++b) request(b);
    bool failed = false;
#pragma unroll 1
    for (int b = 0; b < n_blk; ++b) {
        __syncthreads();          // everyone is done with block b - 1
        if (warp == 0) request(b + STAGES - 1);
        if (!failed && !mbar_wait_relaxed(&full[b % STAGES], (uint32_t)(b / STAGES) & 1u)) failed = true;   // bounded: reported below
        const float* sm = ds_smem + (b % STAGES) * kStage;
        const float* lanes = sm + l * 4;
        uint64_t acc[8][CPL];     // p_t k_t, then p_t q_t (HEAD: without p_t)
        uint64_t kv[HEAD ? NI : 1][kBlock][2];
#pragma unroll
        for (int x = 0; x < 8; ++x)
#pragma unroll
            for (int j = 0; j < CPL; ++j) acc[x][j] = 0;
#pragma unroll
        for (int i = 0; i < NI; ++i)
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(lanes + x * W + 4 * LPC * i);
                if (HEAD && x < kBlock) { kv[HEAD ? i : 0][x & 3][0] = v.x; kv[HEAD ? i : 0][x & 3][1] = v.y; }
#pragma unroll
                for (int j = 0; j < CPL; ++j) acc[x][j] = fma2(S[i][1][j], v.y, fma2(S[i][0][j], v.x, acc[x][j]));
            }
        // transposing reduction over the lanes of a column: this lane ends up with the four sums of (column j_mine, k or q)
        float r[CPL][2][kBlock];
#pragma unroll
        for (int j = 0; j < CPL; ++j)
#pragma unroll
            for (int x = 0; x < 8; ++x) { const float2 h = split(acc[x][j]); r[j][x >> 2][x & 3] = h.x + h.y; }
        if constexpr (CPL == 4) {
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int x = 0; x < 8; ++x) {
                    float &a = r[j][x >> 2][x & 3], &c = r[j + 2][x >> 2][x & 3];
                    constexpr int bit = LPC / 2;
                    const float give = (l & bit) ? a : c, keep = (l & bit) ? c : a;
                    a = keep + __shfl_xor_sync(0xffffffffu, give, bit);
                }
        }
        if constexpr (CPL >= 2) {
            constexpr int bit = CPL == 4 ? LPC / 4 : LPC / 2;
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                float &a = r[0][x >> 2][x & 3], &c = r[1][x >> 2][x & 3];
                const float give = (l & bit) ? a : c, keep = (l & bit) ? c : a;
                a = keep + __shfl_xor_sync(0xffffffffu, give, bit);
            }
        }
        float y[kBlock];
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
            constexpr int bit = 1 << SH;
            const float a = r[0][0][t], c = r[0][1][t];
            const float give = (l & bit) ? a : c, keep = (l & bit) ? c : a;
            y[t] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
#pragma unroll
            for (int o = (1 << SH) >> 1; o > 0; o >>= 1) y[t] += __shfl_xor_sync(0xffffffffu, y[t], o);
        }
        const int m = l >> SH, j_mine = m >> 1;
        const float* num = sm + kVecs * W + kBlock * COLS;
        const float4 beta = *reinterpret_cast<const float4*>(num), a0 = *reinterpret_cast<const float4*>(num + 4), a1 = *reinterpret_cast<const float4*>(num + 8);
        const float* vs = sm + kVecs * W + col0 - c_blk + j_mine;
        float4 tail = make_float4(1.f, 1.f, 1.f, 1.f);
        uint64_t whole = 0;       // the decay of the block
        if constexpr (HEAD) {
            const float4 pt = *reinterpret_cast<const float4*>(num + 24);
            tail = *reinterpret_cast<const float4*>(num + 28);
            y[0] *= pt.x; y[1] *= pt.y; y[2] *= pt.z; y[3] *= pt.w;
            whole = pair_of(pt.w, pt.w);
        }
        float u[kBlock];          // meaningful in the lanes of the k sums
        u[0] = beta.x * (vs[0] - y[0]);
        u[1] = beta.y * (vs[COLS] - fmaf(a0.x, u[0], y[1]));
        u[2] = beta.z * (vs[2 * COLS] - fmaf(a0.z, u[1], fmaf(a0.y, u[0], y[2])));
        u[3] = beta.w * (vs[3 * COLS] - fmaf(a1.y, u[2], fmaf(a1.x, u[1], fmaf(a0.w, u[0], y[3]))));
        uint64_t uu[CPL][kBlock];
#pragma unroll
        for (int j = 0; j < CPL; ++j)
#pragma unroll
            for (int t = 0; t < kBlock; ++t) {
                float x = __shfl_sync(0xffffffffu, u[t], (lane & ~(LPC - 1)) + ((2 * j) << SH));
                if (HEAD) x *= t == 0 ? tail.x : t == 1 ? tail.y : t == 2 ? tail.z : 1.f;
                uu[j][t] = pair_of(x, x);
            }
        float uo[kBlock];
#pragma unroll
        for (int t = 0; t < kBlock; ++t) uo[t] = __shfl_xor_sync(0xffffffffu, u[t], 1 << SH);
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            ulonglong2 gv;
            if constexpr (HEAD) gv = make_ulonglong2(whole, whole);
            else gv = *reinterpret_cast<const ulonglong2*>(lanes + 12 * W + 4 * LPC * i);
#pragma unroll
            for (int j = 0; j < CPL; ++j) { S[i][0][j] = mul2(S[i][0][j], gv.x); S[i][1][j] = mul2(S[i][1][j], gv.y); }
#pragma unroll
            for (int t = 0; t < kBlock; ++t) {
                ulonglong2 c;
                if constexpr (HEAD) c = make_ulonglong2(kv[i][t][0], kv[i][t][1]);
                else c = *reinterpret_cast<const ulonglong2*>(lanes + (8 + t) * W + 4 * LPC * i);
#pragma unroll
                for (int j = 0; j < CPL; ++j) { S[i][0][j] = fma2(c.x, uu[j][t], S[i][0][j]); S[i][1][j] = fma2(c.y, uu[j][t], S[i][1][j]); }
            }
        }
        if ((m & 1) && (l & ((1 << SH) - 1)) == 0 && col0 + j_mine < g.vdim) {
            const float4 b0 = *reinterpret_cast<const float4*>(num + 12), b1 = *reinterpret_cast<const float4*>(num + 16), b2 = *reinterpret_cast<const float4*>(num + 20);
            const int row = r0 + b * kBlock;
            float* o = p.w.o + ((size_t)row * g.heads + head) * g.vp + col0 + j_mine;
            const size_t step = (size_t)g.heads * g.vp;
            o[0] = fmaf(b0.x, uo[0], y[0]);
            if (row + 1 < r1) o[step] = fmaf(b0.z, uo[1], fmaf(b0.y, uo[0], y[1]));
            if (row + 2 < r1) o[2 * step] = fmaf(b1.y, uo[2], fmaf(b1.x, uo[1], fmaf(b0.w, uo[0], y[2])));
            if (row + 3 < r1) o[3 * step] = fmaf(b2.y, uo[3], fmaf(b2.x, uo[2], fmaf(b1.w, uo[1], fmaf(b1.z, uo[0], y[3]))));
        }
    }
    if (failed) {
        for (int b = max(n_blk - STAGES, 0); b < n_blk; ++b) mbar_wait_relaxed(&full[b % STAGES], (uint32_t)(b / STAGES) & 1u);   // copies in flight land in this CTA
        atomicExch(p.s.d_status, 3);
    }
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
            for (int j = 0; j < CPL; ++j) {
                const int d = (LPC * i + l) * 4 + 2 * e;
                const float2 x = split(S[i][e][j]);
                if (col0 + j < g.vdim && d < g.dim) state[(size_t)d * g.vdim + col0 + j] = x.x;
                if (col0 + j < g.vdim && d + 1 < g.dim) state[(size_t)(d + 1) * g.vdim + col0 + j] = x.y;
            }
}

// a warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) delta_output_kernel(const Params p) {
    const Geo& g = p.g;
    const int64_t job = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    pdl_launch_dependents();
    pdl_wait();
    if (job >= (int64_t)p.s.rows * g.heads) return;
    const int row = (int)(job / g.heads), head = (int)(job % g.heads);
    const float* o = p.w.o + job * g.vp;
    const T* gate = static_cast<const T*>(p.s.d_gate) + (size_t)row * g.gate_row + head * g.vdim;
    T* out = static_cast<T*>(p.s.d_out) + job * g.out_stride;
    if constexpr (sizeof(T) == 2) {
        if (g.vdim % 4 == 0 && g.vdim <= 128) {   // the row in one register each
            const int c = lane * 4;
            const bool in = c < g.vdim;
            const float4 v = in ? *reinterpret_cast<const float4*>(o + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            const float inv = 1.f / sqrtf(warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w) / (float)g.vdim + g.eps);
            if (in) {
                const uint2 gu = *reinterpret_cast<const uint2*>(gate + c);
                const float4 w = *reinterpret_cast<const float4*>(p.s.d_norm + c);
                *reinterpret_cast<uint2*>(out + c) = make_uint2(pack_bf16x2(v.x * inv * w.x * gate_of(g, bf16_lo(gu.x)), v.y * inv * w.y * gate_of(g, bf16_hi(gu.x))),
                                                                pack_bf16x2(v.z * inv * w.z * gate_of(g, bf16_lo(gu.y)), v.w * inv * w.w * gate_of(g, bf16_hi(gu.y))));
            } else if (c < g.out_stride) {
                *reinterpret_cast<uint2*>(out + c) = make_uint2(0, 0);
            }
            return;
        }
    }
    float ss = 0.f;
    for (int c = lane; c < g.vdim; c += 32) ss = fmaf(o[c], o[c], ss);
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)g.vdim + g.eps);
    for (int c = lane; c < g.out_stride; c += 32) st(out + c, c < g.vdim ? o[c] * inv * p.s.d_norm[c] * gate_of(g, ld(gate + c)) : 0.f);
}

// ---- decode: one token per sequence ----------------------------------------------------------------------------------------------
constexpr int kDecThreads = 256, kDecWarps = 8;

// Warp w holds the key channels w, w + 8, .. of 32 VEC columns at a time. dim <= 8 NR.
template <typename T, int NR, int VEC>
__global__ void __launch_bounds__(kDecThreads, NR * VEC <= 64 ? 2 : 1) delta_decode_kernel(const Params p) {
    extern __shared__ __align__(16) float dd_smem[];
    __shared__ float sh_sum[3], sh_ss[kDecWarps];
    const Geo& g = p.g;
    float *q = dd_smem, *k = q + g.dp, *gd = k + g.dp, *v = gd + g.dp, *o = v + g.vp;   // [dp] x 3, [vp] x 2
    float* red = o + g.vp;                                                             // [warps][2][32 VEC]
    const int head = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kvh = head / g.group;
    pdl_launch_dependents();
    pdl_wait();
    const RowState r = row_state(p, row);
    float* state = p.s.d_state + ((size_t)p.s.d_slot[row] * g.heads + head) * g.dim * g.vdim;
    const bool fresh = r.pos == 0;
    constexpr int CB = 32 * VEC;
    float S[NR][VEC];
    auto load_state = [&](int cb) {
        const int c = cb + lane * VEC;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = warp + kDecWarps * i;
#pragma unroll
            for (int e = 0; e < VEC; ++e) S[i][e] = 0.f;
            if (!fresh && d < g.dim && c < g.vdim) {
                if constexpr (VEC == 4) {
                    const float4 x = *reinterpret_cast<const float4*>(state + (size_t)d * g.vdim + c);
                    S[i][0] = x.x; S[i][1] = x.y; S[i][2] = x.z; S[i][3] = x.w;
                } else {
                    S[i][0] = state[(size_t)d * g.vdim + c];
                }
            }
        }
    };
    load_state(0);   // travels while the vectors are prepared
    const float beta_raw = ld(static_cast<const T*>(p.s.d_proj) + (size_t)row * g.row + g.beta_off + head);
    for (int d = tid; d < g.dim; d += kDecThreads) gd[d] = decay_of<T>(p, row, head, d);
    const bool own = head % g.group == 0;   // heads that share q and k: the first passes their convolution state on
    for (int i = tid; i < 2 * g.dim + g.vdim; i += kDecThreads) {
        if (i < g.dim) q[i] = conv_channel<T>(p, r, row, kvh * g.dim + i, g.q_off + kvh * g.dim + i, own);
        else if (i < 2 * g.dim) k[i - g.dim] = conv_channel<T>(p, r, row, g.kv_heads * g.dim + kvh * g.dim + i - g.dim, g.k_off + kvh * g.dim + i - g.dim, own);
        else v[i - 2 * g.dim] = conv_channel<T>(p, r, row, 2 * g.kv_heads * g.dim + head * g.vdim + i - 2 * g.dim, g.v_off + head * g.vdim + i - 2 * g.dim, true);
    }
    __syncthreads();
    if (warp < 3) {
        const float *a = warp == 1 ? k : q, *b = warp == 0 ? q : k;   // q.q, k.k, q.k
        float s = 0.f;
        for (int d = lane; d < g.dim; d += 32) s = fmaf(a[d], b[d], s);
        s = warp_sum(s);
        if (lane == 0) sh_sum[warp] = s;
    }
    __syncthreads();
    const float qs = g.q_scale / sqrtf(sh_sum[0] + 1e-6f), ks = 1.f / sqrtf(sh_sum[1] + 1e-6f), qk = sh_sum[2] * qs * ks;
    const float beta = sigmoid(beta_raw);
    for (int cb = 0; cb < g.vdim; cb += CB) {
        if (cb > 0) load_state(cb);
        const int c = cb + lane * VEC;
        float t1[VEC], t2[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) t1[e] = t2[e] = 0.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = warp + kDecWarps * i;
            if (d >= g.dim) break;
            const float gv = gd[d], kv = k[d] * ks, qv = q[d] * qs;
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                S[i][e] *= gv;
                t1[e] = fmaf(S[i][e], kv, t1[e]);
                t2[e] = fmaf(S[i][e], qv, t2[e]);
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) { red[(warp * 2) * CB + lane * VEC + e] = t1[e]; red[(warp * 2 + 1) * CB + lane * VEC + e] = t2[e]; }
        __syncthreads();
        float u[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float a = 0.f;
#pragma unroll
            for (int w = 0; w < kDecWarps; ++w) a += red[w * 2 * CB + lane * VEC + e];
            u[e] = c + e < g.vdim ? beta * (v[c + e] - a) : 0.f;
        }
        if (warp == 0)
#pragma unroll
            for (int e = 0; e < VEC; ++e)
                if (c + e < g.vdim) {
                    float b = 0.f;
#pragma unroll
                    for (int w = 0; w < kDecWarps; ++w) b += red[(w * 2 + 1) * CB + lane * VEC + e];
                    o[c + e] = fmaf(qk, u[e], b);
                }
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = warp + kDecWarps * i;
            if (d >= g.dim || c >= g.vdim) break;
            const float kv = k[d] * ks;
            if constexpr (VEC == 4)
                *reinterpret_cast<float4*>(state + (size_t)d * g.vdim + c) =
                    make_float4(fmaf(kv, u[0], S[i][0]), fmaf(kv, u[1], S[i][1]), fmaf(kv, u[2], S[i][2]), fmaf(kv, u[3], S[i][3]));
            else
                state[(size_t)d * g.vdim + c] = fmaf(kv, u[0], S[i][0]);
        }
        __syncthreads();
    }
    float ss = 0.f;
    for (int c = tid; c < g.vdim; c += kDecThreads) ss = fmaf(o[c], o[c], ss);
    ss = warp_sum(ss);
    if (lane == 0) sh_ss[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) ss += sh_ss[w];
    const float inv = 1.f / sqrtf(ss / (float)g.vdim + g.eps);
    const T* gate = static_cast<const T*>(p.s.d_gate) + (size_t)row * g.gate_row + head * g.vdim;
    T* out = static_cast<T*>(p.s.d_out) + ((size_t)row * g.heads + head) * g.out_stride;
    for (int c = tid; c < g.out_stride; c += kDecThreads) st(out + c, c < g.vdim ? o[c] * inv * p.s.d_norm[c] * gate_of(g, ld(gate + c)) : 0.f);
}

template <int NI, int CPL, int LPC, int STAGES, bool HEAD>
int launch_scan_of(const Params& p, cudaStream_t s) {
    constexpr int cols = kScanWarps * 32 / LPC * CPL;
    constexpr size_t smem = (size_t)STAGES * (vecs_of(HEAD) * 4 * LPC * NI + kBlock * cols + nums_of(HEAD)) * 4;
    static PerDeviceOnce once;
    if (once.first_time()) GPTRS_CUDA_OK(cudaFuncSetAttribute(delta_scan_kernel<NI, CPL, LPC, STAGES, HEAD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return launch_kernel(delta_scan_kernel<NI, CPL, LPC, STAGES, HEAD>, dim3((unsigned)ceil_div(p.g.vdim, cols), (unsigned)p.g.heads, (unsigned)p.s.n_runs), dim3(kScanWarps * 32), smem,
                         s, 1, p);
}
template <int NI, int CPL, int LPC, int STAGES>
int launch_scan(const Params& p, cudaStream_t s) {
    // a run is a chain of blocks: while there are SMs to spare, fewer columns per warp make its links shorter
    if constexpr (CPL > 1 && LPC == 16) {
        constexpr int cols = kScanWarps * 32 / LPC * CPL;
        if ((int64_t)ceil_div(p.g.vdim, cols) * p.g.heads * p.s.n_runs * 2 <= sm_count()) return launch_scan<NI, CPL / 2, LPC, STAGES>(p, s);
    }
    return p.g.head_decay ? launch_scan_of<NI, CPL, LPC, STAGES, true>(p, s) : launch_scan_of<NI, CPL, LPC, STAGES, false>(p, s);
}
template <typename T, int NR, int VEC>
int launch_decode(const Params& p, cudaStream_t s) {
    const size_t smem = ((size_t)3 * p.g.dp + 2 * p.g.vp + kDecWarps * 2 * 32 * VEC) * 4;
    static PerDeviceOnce once;
    if (once.first_time()) GPTRS_CUDA_OK(cudaFuncSetAttribute(delta_decode_kernel<T, NR, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024));
    return launch_kernel(delta_decode_kernel<T, NR, VEC>, dim3((unsigned)p.g.heads, (unsigned)p.s.rows), dim3(kDecThreads), smem, s, 1, p);
}
template <typename T>
int run(const Params& p, cudaStream_t s) {
    const Geo& g = p.g;
    if (p.s.n_runs == p.s.rows) {
        if (g.vdim % 4 == 0) {
            if (g.dim <= 64) return launch_decode<T, 8, 4>(p, s);
            if (g.dim <= 128) return launch_decode<T, 16, 4>(p, s);
            if (g.dim <= 256) return launch_decode<T, 32, 4>(p, s);
        }
        if (g.dim <= 128) return launch_decode<T, 16, 1>(p, s);
        return launch_decode<T, 64, 1>(p, s);
    }
    int rc = launch_prepare(p, sizeof(T) == 2, s);
    if (rc) return rc;
    if (g.dim <= 32) rc = launch_scan<1, 2, 8, 4>(p, s);
    else if (g.dim <= 64) rc = launch_scan<1, 4, 16, 4>(p, s);
    else if (g.dim <= 128) rc = launch_scan<2, 4, 16, 4>(p, s);
    else if (g.dim <= 256) rc = launch_scan<4, 4, 16, 4>(p, s);
    else rc = launch_scan<8, 2, 16, 4>(p, s);
    if (rc) return rc;
    return launch_kernel(delta_output_kernel<T>, dim3((unsigned)ceil_div(p.s.rows * g.heads, 8)), dim3(256), 0, s, 1, p);
}

}  // namespace
}  // namespace delta
}  // namespace gptrs

using namespace gptrs;
using namespace gptrs::delta;

extern "C" {

int gptrs_cuda_delta_layout(gptrs_delta_rule* a) {
    GPTRS_REQUIRE(a, "null pointer");
    GPTRS_REQUIRE(a->heads > 0 && a->kv_heads > 0 && a->dim > 0 && a->vdim > 0 && a->taps > 0 && a->decay_rank >= 0 && a->gate_rank >= 0, "delta rule: sizes must be positive");
    GPTRS_REQUIRE(a->heads % a->kv_heads == 0, "delta rule: heads must be a multiple of the q/k heads");
    GPTRS_REQUIRE(a->dtype == GPTRS_F32 || a->dtype == GPTRS_BF16, "delta rule: f32 or bf16");
    if (a->dim > kMaxDim || a->vdim > 4096 || a->heads > 65535) return fail(GPTRS_UNIMPLEMENTED, "delta rule: dim above 512, vdim above 4096 or more than 65535 heads");
    auto pad = [&](int v) { return a->dtype == GPTRS_BF16 ? (v + 7) / 8 * 8 : v; };
    a->q_offset = 0;
    a->k_offset = a->q_offset + pad(a->kv_heads * a->dim);
    a->v_offset = a->k_offset + pad(a->kv_heads * a->dim);
    a->beta_offset = a->v_offset + pad(a->heads * a->vdim);
    a->a_offset = a->beta_offset + pad(a->heads);
    a->g_offset = a->a_offset + pad(a->decay_rank > 0 ? a->decay_rank : a->heads);
    a->row = a->g_offset + pad(a->gate_rank > 0 ? a->gate_rank : a->heads * a->vdim);
    a->decay_row = a->decay_rank > 0 ? pad(a->heads * a->dim) : 0;
    a->gate_row = a->gate_rank > 0 ? pad(a->heads * a->vdim) : a->row;
    a->out_head_stride = pad(a->vdim);
    a->conv_channels = 2 * a->kv_heads * a->dim + a->heads * a->vdim;
    a->state_floats = (int64_t)a->heads * a->dim * a->vdim;
    a->conv_floats = (int64_t)2 * (a->taps - 1) * a->conv_channels;
    return GPTRS_OK;
}

int64_t gptrs_cuda_delta_scratch_floats(const gptrs_delta_rule* a, int64_t rows, int64_t n_runs) {
    if (!a || n_runs == rows) return 0;
    const Geo g = geo(*a);
    return max_blocks(rows, n_runs) * block_floats(g) + rows * g.heads * g.vp;
}

int gptrs_cuda_delta_rule(const gptrs_delta_rule* a, const gptrs_delta_step* step, void* stream) {
    GPTRS_REQUIRE(a && step && a->row > 0, "null pointer, or layout not filled in");
    const gptrs_delta_step& s = *step;
    GPTRS_REQUIRE((s.d_decay || a->decay_rank == 0) && (s.d_gate || a->gate_rank == 0), "null pointer");
    GPTRS_REQUIRE(s.d_proj && s.d_conv && s.d_a_log && s.d_dt_bias && s.d_norm && s.d_state && (s.d_conv_state || a->taps == 1) && s.d_out, "null pointer");
    GPTRS_REQUIRE(s.d_slot && s.d_pos && s.d_run_first && s.d_run_last && s.d_parity, "null pointer");
    GPTRS_REQUIRE(s.rows >= 0 && s.rows < (1ll << 31) && s.n_runs >= 0 && s.n_runs <= s.rows && s.n_runs <= 65535, "delta rule: rows and runs");
    if (s.rows == 0) return GPTRS_OK;
    GPTRS_REQUIRE(s.n_runs == s.rows || (s.n_runs > 0 && s.d_runs && s.d_status && s.d_scratch && (reinterpret_cast<uintptr_t>(s.d_scratch) & 15) == 0), "delta rule: run list and scratch");
    Params p = {s, geo(*a), {}};
    if (a->gate_rank == 0) p.s.d_gate = static_cast<const unsigned char*>(s.d_proj) + (size_t)a->g_offset * (a->dtype == GPTRS_BF16 ? 2 : 4);
    if (s.n_runs != s.rows) p.w = planes(p.g, s.d_scratch, s.rows, s.n_runs);
    return a->dtype == GPTRS_BF16 ? run<__nv_bfloat16>(p, as_stream(stream)) : run<float>(p, as_stream(stream));
}

}  // extern "C"
