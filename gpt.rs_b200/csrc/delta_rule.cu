// Gated delta rule with a decay per key channel (no counterpart in gpt.rs). Per head and token
//
//   S <- g S (rows of S are key channels);   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
// with q, k, v behind short causal convolutions and silu, q and k of unit length, and o normed and gated. The columns of S are
// independent of one another. With S' = g S one pass over S' gives S'^T k and S'^T q, hence u, and o = S'^T q + (q . k) u.
//   delta_prepare_kernel   prompts: convolutions with their state, unit norms, decays, step sizes -> f32 planes, a CTA per row
//   delta_scan_kernel      prompts: a warp keeps 16 columns of a head's S in registers over a whole run; tokens arrive in stages of
//                          shared memory; the two sums over the key channels meet in one transposing warp reduction
//   delta_output_kernel    prompts: norm and gate of the read-outs
//   delta_decode_kernel    rows that are runs of their own: all of the above in one launch, a CTA per (head, row), S is read and
//                          written once
// Everything that enters the recurrence, and S itself, is f32. S is updated in place (one CTA owns a column of a slot's state);
// the convolution state has two halves like the one of post_norm_conv.cu.
#include "common.cuh"

namespace gptrs {
namespace {

struct Geo {
    int heads, kv_heads, group, dim, vdim, taps;
    int q_off, k_off, v_off, beta_off, row, decay_row, gate_row, out_stride, channels;
    int dp, vp;              // dim and vdim of the f32 planes, multiples of 4
    float eps, q_scale;
};
__host__ __device__ inline int pad4(int v) { return (v + 3) / 4 * 4; }
Geo geo(const gptrs_delta_rule& a) {
    Geo g = {a.heads, a.kv_heads, a.heads / a.kv_heads, a.dim, a.vdim, a.taps, a.q_offset, a.k_offset, a.v_offset, a.beta_offset, a.row, a.decay_row, a.gate_row,
             a.out_head_stride, a.conv_channels, pad4(a.dim), pad4(a.vdim), a.eps, 1.f / sqrtf((float)a.dim)};
    return g;
}
// f32 planes of a prompt's rows behind one another in the scratch: q, k, v, decay, step size, q . k, read-out
struct Planes { float *q, *k, *v, *g, *beta, *qk, *o; };
int64_t plane_floats(const Geo& g) { return (int64_t)2 * g.kv_heads * g.dp + (int64_t)g.heads * (2 * g.vp + g.dp) + pad4(g.heads) + pad4(g.kv_heads); }
Planes planes(const Geo& g, float* s, int64_t rows) {
    Planes p;
    p.q = s; s += rows * g.kv_heads * g.dp;
    p.k = s; s += rows * g.kv_heads * g.dp;
    p.v = s; s += rows * g.heads * g.vp;
    p.g = s; s += rows * g.heads * g.dp;
    p.o = s; s += rows * g.heads * g.vp;
    p.beta = s; s += rows * pad4(g.heads);
    p.qk = s;
    return p;
}

struct Params {
    gptrs_delta_step s;
    Geo g;
    Planes w;
};

__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
template <typename T>
__device__ __forceinline__ float ld(const T* p) {
    if constexpr (sizeof(T) == 2) return __bfloat162float(*p);
    else return *p;
}
template <typename T>
__device__ __forceinline__ void st(T* p, float v) {
    if constexpr (sizeof(T) == 2) *p = __float2bfloat16_rn(v);
    else *p = v;
}
__device__ __forceinline__ float decay_of(const Params& p, int row, int head, int d) {
    const int c = head * p.g.dim + d;
    return expf(-expf(p.s.d_a_log[head]) * softplus(p.s.d_decay[(size_t)row * p.g.decay_row + c] + p.s.d_dt_bias[c]));
}

// A row's place in its run, and the convolution state it reads and writes.
struct RowState { int pos, first, len_before, last; const float* old; float* fresh; };
__device__ __forceinline__ RowState row_state(const Params& p, int row) {
    RowState r;
    r.pos = p.s.d_pos[row]; r.first = p.s.d_run_first[row]; r.last = p.s.d_run_last[row];
    r.len_before = row - r.first;
    const size_t half = (size_t)(p.g.taps - 1) * p.g.channels;
    float* state = p.s.d_conv_state + (size_t)p.s.d_slot[row] * 2 * half;
    const int par = p.s.d_parity[row] & 1;
    r.old = state + par * half; r.fresh = state + (par ^ 1) * half;
    return r;
}
// silu(convolution) of channel `ch` (column `col` of the projection row); `keep_state`: this thread also passes the channel's
// inputs on to the next step
template <typename T>
__device__ __forceinline__ float conv_channel(const Params& p, const RowState& r, int row, int ch, int col, bool keep_state) {
    const int keep = p.g.taps - 1;
    const T* x = static_cast<const T*>(p.s.d_proj) + (size_t)row * p.g.row + col;
    const float* w = p.s.d_conv + (size_t)ch * p.g.taps;
    float acc = 0.f;
    for (int k = keep; k >= 1; --k) {   // the input k positions back
        const int at = r.pos - k;
        float v = 0.f;
        if (k <= r.len_before) v = ld(x - (size_t)k * p.g.row);
        else if (at >= 0) v = r.old[(size_t)(at % keep) * p.g.channels + ch];
        acc = fmaf(w[keep - k], v, acc);
        // first row of a run shorter than the state: what the run does not push out stays
        if (keep_state && row == r.first && at >= 0 && at > r.pos + (r.last - row) - keep) r.fresh[(size_t)(at % keep) * p.g.channels + ch] = v;
    }
    const float now = ld(x);
    if (keep_state && keep > 0 && r.last - row < keep) r.fresh[(size_t)(r.pos % keep) * p.g.channels + ch] = now;
    return silu(fmaf(w[keep], now, acc));
}

constexpr int kPrepThreads = 256;
constexpr int kMaxDim = 512;

template <typename T>
__global__ void __launch_bounds__(kPrepThreads) delta_prepare_kernel(const Params p) {
    const Geo& g = p.g;
    const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_launch_dependents();
    pdl_wait();
    const RowState r = row_state(p, row);
    const int v_jobs = (g.heads * g.vp + 127) / 128, g_jobs = (g.heads * g.dp + 127) / 128;
    const int jobs = g.kv_heads + v_jobs + g_jobs + 1;
    for (int job = warp; job < jobs; job += kPrepThreads / 32) {
        if (job < g.kv_heads) {   // q and k of one head
            float q[kMaxDim / 32], k[kMaxDim / 32], qq = 0.f, kk = 0.f, qk = 0.f;
            const int c0 = job * g.dim;
#pragma unroll
            for (int i = 0; i < kMaxDim / 32; ++i) {
                const int d = i * 32 + lane;
                q[i] = k[i] = 0.f;
                if (d < g.dim) {
                    q[i] = conv_channel<T>(p, r, row, c0 + d, g.q_off + c0 + d, true);
                    k[i] = conv_channel<T>(p, r, row, g.kv_heads * g.dim + c0 + d, g.k_off + c0 + d, true);
                }
                qq = fmaf(q[i], q[i], qq); kk = fmaf(k[i], k[i], kk); qk = fmaf(q[i], k[i], qk);
            }
            const float qs = g.q_scale / sqrtf(warp_sum(qq) + 1e-6f), ks = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
            qk = warp_sum(qk);
            float *dq = p.w.q + ((size_t)row * g.kv_heads + job) * g.dp, *dk = p.w.k + ((size_t)row * g.kv_heads + job) * g.dp;
#pragma unroll
            for (int i = 0; i < kMaxDim / 32; ++i) {
                const int d = i * 32 + lane;
                if (d < g.dp) { dq[d] = q[i] * qs; dk[d] = k[i] * ks; }
            }
            if (lane == 0) p.w.qk[(size_t)row * g.kv_heads + job] = qk * qs * ks;
        } else if (job < g.kv_heads + v_jobs) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int e = (job - g.kv_heads) * 128 + i * 32 + lane, h = e / g.vp, c = e % g.vp;
                if (h >= g.heads) continue;
                float v = 0.f;
                if (c < g.vdim) v = conv_channel<T>(p, r, row, 2 * g.kv_heads * g.dim + h * g.vdim + c, g.v_off + h * g.vdim + c, true);
                p.w.v[(size_t)row * g.heads * g.vp + e] = v;
            }
        } else if (job < jobs - 1) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int e = (job - g.kv_heads - v_jobs) * 128 + i * 32 + lane, h = e / g.dp, d = e % g.dp;
                if (h >= g.heads) continue;
                p.w.g[(size_t)row * g.heads * g.dp + e] = d < g.dim ? decay_of(p, row, h, d) : 0.f;
            }
        } else {
            for (int h = lane; h < g.heads; h += 32)
                p.w.beta[(size_t)row * g.heads + h] = sigmoid(ld(static_cast<const T*>(p.s.d_proj) + (size_t)row * g.row + g.beta_off + h));
        }
    }
}

// ---- the scan ------------------------------------------------------------------------------------------------------------------
constexpr int kScanWarps = 4;
__device__ __forceinline__ void cp_async_4(uint32_t dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(dst), "l"(src));
}

// Eight lanes share a column: lane l holds the channels (8 i + l) 4 + e, i < NI, of CPL neighbouring columns; four such groups
// make a warp. dim <= 32 NI.
template <int NI, int CPL, int TB>
__global__ void __launch_bounds__(kScanWarps * 32) delta_scan_kernel(const Params p) {
    constexpr int W = 32 * NI;                       // channels with padding
    constexpr int COLS = kScanWarps * 4 * CPL;       // columns of the CTA
    constexpr int kStage = TB * (3 * W + COLS + 2);  // floats: k, q, g, v, beta, qk
    constexpr int M = 2 * CPL, SH = M == 8 ? 0 : M == 4 ? 1 : 2;
    extern __shared__ __align__(16) float ds_smem[];
    const Geo& g = p.g;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = lane & 7, cg = lane >> 3;
    const int head = blockIdx.y, kvh = head / g.group;
    const int c_blk = blockIdx.x * COLS, col0 = c_blk + (warp * 4 + cg) * CPL;
    pdl_launch_dependents();
    pdl_wait();
    const int r0 = p.s.d_runs[blockIdx.z], r1 = p.s.d_run_last[r0] + 1;
    float* state = p.s.d_state + ((size_t)p.s.d_slot[r0] * g.heads + head) * g.dim * g.vdim;
    const bool fresh = p.s.d_pos[r0] == 0;
    float S[NI][4][CPL];
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int j = 0; j < CPL; ++j) {
                const int d = (8 * i + l) * 4 + e;
                S[i][e][j] = (!fresh && d < g.dim && col0 + j < g.vdim) ? state[(size_t)d * g.vdim + col0 + j] : 0.f;
            }
    for (int i = tid; i < 2 * kStage; i += kScanWarps * 32) ds_smem[i] = 0.f;   // the padding stays zero
    __syncthreads();
    const int kq4 = g.dp / 4, v4 = min(COLS, g.vp - c_blk) / 4;
    auto request = [&](int t0, int buf) {   // rows t0 .. t0 + TB of the run
        float* sm = ds_smem + buf * kStage;
        const int n = min(TB, r1 - t0);
        for (int i = tid; i < n * kq4; i += kScanWarps * 32) {
            const int t = i / kq4, c = (i % kq4) * 4;
            const size_t kv = ((size_t)(t0 + t) * g.kv_heads + kvh) * g.dp + c, hd = ((size_t)(t0 + t) * g.heads + head) * g.dp + c;
            cp_async_16(sm + t * W + c, p.w.k + kv, true);
            cp_async_16(sm + (TB + t) * W + c, p.w.q + kv, true);
            cp_async_16(sm + (2 * TB + t) * W + c, p.w.g + hd, true);
        }
        for (int i = tid; i < n * v4; i += kScanWarps * 32) {
            const int t = i / v4, c = (i % v4) * 4;
            cp_async_16(sm + 3 * TB * W + t * COLS + c, p.w.v + ((size_t)(t0 + t) * g.heads + head) * g.vp + c_blk + c, true);
        }
        for (int t = tid; t < n; t += kScanWarps * 32) {
            cp_async_4(smem_u32(sm + TB * (3 * W + COLS) + t), p.w.beta + (size_t)(t0 + t) * g.heads + head);
            cp_async_4(smem_u32(sm + TB * (3 * W + COLS + 1) + t), p.w.qk + (size_t)(t0 + t) * g.kv_heads + kvh);
        }
        cp_async_commit();
    };
    request(r0, 0);
    int buf = 0;
    for (int t0 = r0; t0 < r1; t0 += TB, buf ^= 1) {
        if (t0 + TB < r1) { request(t0 + TB, buf ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const float* sm = ds_smem + buf * kStage;
        const int n = min(TB, r1 - t0);
#pragma unroll 1
        for (int t = 0; t < n; ++t) {
            float r[M];
#pragma unroll
            for (int j = 0; j < M; ++j) r[j] = 0.f;
            float4 kk[NI];
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                kk[i] = *reinterpret_cast<const float4*>(sm + t * W + (8 * i + l) * 4);
                const float4 qv = *reinterpret_cast<const float4*>(sm + (TB + t) * W + (8 * i + l) * 4);
                const float4 gv = *reinterpret_cast<const float4*>(sm + (2 * TB + t) * W + (8 * i + l) * 4);
                const float ka[4] = {kk[i].x, kk[i].y, kk[i].z, kk[i].w}, qa[4] = {qv.x, qv.y, qv.z, qv.w}, ga[4] = {gv.x, gv.y, gv.z, gv.w};
#pragma unroll
                for (int e = 0; e < 4; ++e)
#pragma unroll
                    for (int j = 0; j < CPL; ++j) {
                        const float s = S[i][e][j] * ga[e];
                        S[i][e][j] = s;
                        r[2 * j] = fmaf(s, ka[e], r[2 * j]);
                        r[2 * j + 1] = fmaf(s, qa[e], r[2 * j + 1]);
                    }
            }
            // transposing reduction over the eight lanes: afterwards this lane holds the sum number l >> SH
            if constexpr (M == 8) {
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float give = (l & 4) ? r[j] : r[j + 4], keep = (l & 4) ? r[j + 4] : r[j];
                    r[j] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
                }
            }
            if constexpr (M >= 4) {
                constexpr int bit = M == 8 ? 2 : 4;
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const float give = (l & bit) ? r[j] : r[j + 2], keep = (l & bit) ? r[j + 2] : r[j];
                    r[j] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
                }
            }
            {
                constexpr int bit = 1 << SH;
                const float give = (l & bit) ? r[0] : r[1], keep = (l & bit) ? r[1] : r[0];
                r[0] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
            }
#pragma unroll
            for (int b = (1 << SH) >> 1; b > 0; b >>= 1) r[0] += __shfl_xor_sync(0xffffffffu, r[0], b);
            const int m = l >> SH, j_mine = m >> 1;
            const float beta = sm[TB * (3 * W + COLS) + t], qk = sm[TB * (3 * W + COLS + 1) + t];
            const float v = sm[3 * TB * W + t * COLS + col0 - c_blk + j_mine];
            const float u_mine = beta * (v - r[0]);   // meaningful where m is even
            float u[CPL];
#pragma unroll
            for (int j = 0; j < CPL; ++j) u[j] = __shfl_sync(0xffffffffu, u_mine, (lane & 24) + ((2 * j) << SH));
            float uo = u[0];
#pragma unroll
            for (int j = 1; j < CPL; ++j) uo = j_mine == j ? u[j] : uo;
            if ((m & 1) && (l & ((1 << SH) - 1)) == 0 && col0 + j_mine < g.vdim)
                p.w.o[((size_t)(t0 + t) * g.heads + head) * g.vp + col0 + j_mine] = fmaf(qk, uo, r[0]);
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const float ka[4] = {kk[i].x, kk[i].y, kk[i].z, kk[i].w};
#pragma unroll
                for (int e = 0; e < 4; ++e)
#pragma unroll
                    for (int j = 0; j < CPL; ++j) S[i][e][j] = fmaf(ka[e], u[j], S[i][e][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int j = 0; j < CPL; ++j) {
                const int d = (8 * i + l) * 4 + e;
                if (d < g.dim && col0 + j < g.vdim) state[(size_t)d * g.vdim + col0 + j] = S[i][e][j];
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
    float ss = 0.f;
    for (int c = lane; c < g.vdim; c += 32) ss = fmaf(o[c], o[c], ss);
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)g.vdim + g.eps);
    const T* gate = static_cast<const T*>(p.s.d_gate) + (size_t)row * g.gate_row + head * g.vdim;
    T* out = static_cast<T*>(p.s.d_out) + job * g.out_stride;
    for (int c = lane; c < g.out_stride; c += 32) st(out + c, c < g.vdim ? o[c] * inv * p.s.d_norm[c] * sigmoid(ld(gate + c)) : 0.f);
}

// ---- decode: one token per sequence ----------------------------------------------------------------------------------------------
constexpr int kDecThreads = 256, kDecWarps = 8;

// Warp w holds the key channels w, w + 8, .. of 32 VEC columns at a time. dim <= 8 NR.
template <typename T, int NR, int VEC>
__global__ void __launch_bounds__(kDecThreads) delta_decode_kernel(const Params p) {
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
            const int d = warp + 8 * i;
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
    const bool own = head % g.group == 0;   // heads that share q and k: the first passes their convolution state on
    for (int i = tid; i < 2 * g.dim + g.vdim; i += kDecThreads) {
        if (i < g.dim) q[i] = conv_channel<T>(p, r, row, kvh * g.dim + i, g.q_off + kvh * g.dim + i, own);
        else if (i < 2 * g.dim) k[i - g.dim] = conv_channel<T>(p, r, row, g.kv_heads * g.dim + kvh * g.dim + i - g.dim, g.k_off + kvh * g.dim + i - g.dim, own);
        else v[i - 2 * g.dim] = conv_channel<T>(p, r, row, 2 * g.kv_heads * g.dim + head * g.vdim + i - 2 * g.dim, g.v_off + head * g.vdim + i - 2 * g.dim, true);
    }
    for (int d = tid; d < g.dim; d += kDecThreads) gd[d] = decay_of(p, row, head, d);
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
    const float beta = sigmoid(ld(static_cast<const T*>(p.s.d_proj) + (size_t)row * g.row + g.beta_off + head));
    for (int cb = 0; cb < g.vdim; cb += CB) {
        if (cb > 0) load_state(cb);
        const int c = cb + lane * VEC;
        float t1[VEC], t2[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) t1[e] = t2[e] = 0.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = warp + 8 * i;
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
            const int d = warp + 8 * i;
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
    for (int c = tid; c < g.out_stride; c += kDecThreads) st(out + c, c < g.vdim ? o[c] * inv * p.s.d_norm[c] * sigmoid(ld(gate + c)) : 0.f);
}

template <int NI, int CPL, int TB>
int launch_scan(const Params& p, cudaStream_t s) {
    constexpr int cols = kScanWarps * 4 * CPL;
    constexpr size_t smem = (size_t)2 * TB * (3 * 32 * NI + cols + 2) * 4;
    static PerDeviceOnce once;
    if (once.first_time()) GPTRS_CUDA_OK(cudaFuncSetAttribute(delta_scan_kernel<NI, CPL, TB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return launch_kernel(delta_scan_kernel<NI, CPL, TB>, dim3((unsigned)ceil_div(p.g.vdim, cols), (unsigned)p.g.heads, (unsigned)p.s.n_runs), dim3(kScanWarps * 32), smem, s, 1, p);
}
template <typename T, int NR, int VEC>
int launch_decode(const Params& p, cudaStream_t s) {
    const size_t smem = ((size_t)3 * p.g.dp + 2 * p.g.vp + kDecWarps * 2 * 32 * VEC) * 4;
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
    int rc = launch_kernel(delta_prepare_kernel<T>, dim3((unsigned)p.s.rows), dim3(kPrepThreads), 0, s, 1, p);
    if (rc) return rc;
    if (g.dim <= 32) rc = launch_scan<1, 4, 16>(p, s);
    else if (g.dim <= 64) rc = launch_scan<2, 4, 16>(p, s);
    else if (g.dim <= 128) rc = launch_scan<4, 4, 16>(p, s);
    else if (g.dim <= 256) rc = launch_scan<8, 2, 8>(p, s);
    else rc = launch_scan<16, 1, 8>(p, s);
    if (rc) return rc;
    return launch_kernel(delta_output_kernel<T>, dim3((unsigned)ceil_div(p.s.rows * g.heads, 8)), dim3(256), 0, s, 1, p);
}

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" {

int gptrs_cuda_delta_layout(gptrs_delta_rule* a) {
    GPTRS_REQUIRE(a, "null pointer");
    GPTRS_REQUIRE(a->heads > 0 && a->kv_heads > 0 && a->dim > 0 && a->vdim > 0 && a->taps > 0 && a->decay_rank > 0 && a->gate_rank > 0, "delta rule: sizes must be positive");
    GPTRS_REQUIRE(a->heads % a->kv_heads == 0, "delta rule: heads must be a multiple of the q/k heads");
    GPTRS_REQUIRE(a->dtype == GPTRS_F32 || a->dtype == GPTRS_BF16, "delta rule: f32 or bf16");
    if (a->dim > kMaxDim || a->vdim > 4096 || a->heads > 65535) return fail(GPTRS_UNIMPLEMENTED, "delta rule: dim above 512, vdim above 4096 or more than 65535 heads");
    auto pad = [&](int v) { return a->dtype == GPTRS_BF16 ? (v + 7) / 8 * 8 : v; };
    a->q_offset = 0;
    a->k_offset = a->q_offset + pad(a->kv_heads * a->dim);
    a->v_offset = a->k_offset + pad(a->kv_heads * a->dim);
    a->beta_offset = a->v_offset + pad(a->heads * a->vdim);
    a->a_offset = a->beta_offset + pad(a->heads);
    a->g_offset = a->a_offset + pad(a->decay_rank);
    a->row = a->g_offset + pad(a->gate_rank);
    a->decay_row = pad(a->heads * a->dim);
    a->gate_row = pad(a->heads * a->vdim);
    a->out_head_stride = pad(a->vdim);
    a->conv_channels = 2 * a->kv_heads * a->dim + a->heads * a->vdim;
    a->state_floats = (int64_t)a->heads * a->dim * a->vdim;
    a->conv_floats = (int64_t)2 * (a->taps - 1) * a->conv_channels;
    a->scratch_floats = plane_floats(geo(*a));
    return GPTRS_OK;
}

int gptrs_cuda_delta_rule(const gptrs_delta_rule* a, const gptrs_delta_step* step, void* stream) {
    GPTRS_REQUIRE(a && step && a->row > 0, "null pointer, or layout not filled in");
    const gptrs_delta_step& s = *step;
    GPTRS_REQUIRE(s.d_proj && s.d_decay && s.d_gate && s.d_conv && s.d_a_log && s.d_dt_bias && s.d_norm && s.d_state && (s.d_conv_state || a->taps == 1) && s.d_out, "null pointer");
    GPTRS_REQUIRE(s.d_slot && s.d_pos && s.d_run_first && s.d_run_last && s.d_parity, "null pointer");
    GPTRS_REQUIRE(s.rows >= 0 && s.rows < (1ll << 31) && s.n_runs >= 0 && s.n_runs <= s.rows && s.n_runs <= 65535, "delta rule: rows and runs");
    if (s.rows == 0) return GPTRS_OK;
    GPTRS_REQUIRE(s.n_runs == s.rows || (s.n_runs > 0 && s.d_runs && s.d_scratch && (reinterpret_cast<uintptr_t>(s.d_scratch) & 15) == 0), "delta rule: run list and scratch");
    Params p = {s, geo(*a), {}};
    if (s.n_runs != s.rows) p.w = planes(p.g, s.d_scratch, s.rows);
    return a->dtype == GPTRS_BF16 ? run<__nv_bfloat16>(p, as_stream(stream)) : run<float>(p, as_stream(stream));
}

}  // extern "C"
