// Prompts of the gated delta rule, first step (delta_rule.cu has the algebra): convolutions with their state, unit norms, decays, and from them
// the vectors, values and numbers of every block of four tokens.
#include "delta_rule.cuh"

namespace gptrs {
namespace delta {
namespace {

constexpr int kPrepThreads = 256;

// What a block's channels need: the first row of the block, its live tokens, the convolution state of the sequence.
struct BlockState { bool inner; int row, n, first, last, pos; const float* old; float* fresh; };
// silu(convolution) of channel `ch` (column `col` of the projection rows) for the tokens of a block; tokens that are not there give 0.
// TAPS 0: any number. `keep_state`: this thread also passes the channel's inputs on to the next step.
template <typename T, int TAPS>
__device__ __forceinline__ void conv_block(const Params& p, const BlockState& b, int ch, int col, bool keep_state, float (&out)[kBlock]) {
    const int taps = TAPS ? TAPS : p.g.taps, keep = taps - 1;
    const T* x = static_cast<const T*>(p.s.d_proj) + (size_t)b.row * p.g.row + col;
    const float* w = p.s.d_conv + (size_t)ch * taps;
    auto input = [&](int k) -> float {   // k rows after the block's first one (k < 0: before it)
        if (b.row + k >= b.first) return ld(x + (int64_t)k * p.g.row);
        const int at = b.pos + k;
        return at >= 0 ? b.old[(size_t)(at % keep) * p.g.channels + ch] : 0.f;
    };
    if constexpr (TAPS > 0) {
        float in[TAPS - 1 + kBlock], wt[TAPS];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) wt[j] = __ldg(w + j);
        if (b.inner) {   // a whole block away from the start of its run: all inputs are rows of this pass
#pragma unroll
            for (int k = 0; k < TAPS - 1 + kBlock; ++k) in[k] = ld(x + (int64_t)(k - (TAPS - 1)) * p.g.row);
        } else {
#pragma unroll
            for (int k = 0; k < TAPS - 1 + kBlock; ++k) in[k] = k - (TAPS - 1) < b.n ? input(k - (TAPS - 1)) : 0.f;
        }
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) acc = fmaf(wt[j], in[t + j], acc);
            out[t] = t < b.n ? (sizeof(T) == 2 ? silu_fast(acc) : silu(acc)) : 0.f;
        }
    } else {
        for (int t = 0; t < kBlock; ++t) {
            float acc = 0.f;
            if (t < b.n)
                for (int j = 0; j < taps; ++j) acc = fmaf(w[j], input(t + j - keep), acc);
            out[t] = t < b.n ? silu(acc) : 0.f;
        }
    }
    if (!keep_state || keep == 0 || (b.inner && b.last - (b.row + kBlock - 1) >= keep)) return;
    if (b.row == b.first)   // a run shorter than the state: what it does not push out stays
        for (int k = 1; k <= keep; ++k) {
            const int at = b.pos - k;
            if (at >= 0 && at > b.pos + (b.last - b.row) - keep) b.fresh[(size_t)(at % keep) * p.g.channels + ch] = b.old[(size_t)(at % keep) * p.g.channels + ch];
        }
    for (int t = 0; t < b.n; ++t)
        if (b.last - (b.row + t) < keep) b.fresh[(size_t)((b.pos + t) % keep) * p.g.channels + ch] = ld(x + (int64_t)t * p.g.row);
}

// the same out of line, for kernels that would hold many copies of it
template <typename T>
__device__ __noinline__ void conv_block_far(const Params& p, const BlockState& b, int ch, int col, bool keep_state, float (&out)[kBlock]) {
    conv_block<T, 0>(p, b, ch, col, keep_state, out);
}

// sums of N values over the warp: lane i gets the sum of v[i mod N]
template <int N>
__device__ __forceinline__ float transpose_sum(float (&v)[N]) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int h = N / 2; h >= 1; h >>= 1)
#pragma unroll
        for (int i = 0; i < h; ++i) {
            const float give = (lane & h) ? v[i] : v[i + h], keep = (lane & h) ? v[i + h] : v[i];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, give, h);
        }
#pragma unroll
    for (int h = N; h < 32; h <<= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], h);
    return v[0];
}

// NI: groups of 32 key channels
template <typename T, int NI, int TAPS, bool HEAD>
__global__ void __launch_bounds__(kPrepThreads, NI <= 4 ? 4 : 1) delta_prepare_kernel(const Params p) {
    constexpr int kVecs = vecs_of(HEAD), kNums = nums_of(HEAD), ND = HEAD ? 1 : NI;
    const Geo& g = p.g;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, blk = blockIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    int run = 0;   // the last run whose blocks start at or before this one
    for (int lo = 0, hi = (int)p.s.n_runs; lo < hi;) {
        const int mid = (lo + hi) / 2;
        if (p.s.d_runs[mid] / kBlock + mid <= blk) { run = mid; lo = mid + 1; }
        else hi = mid;
    }
    BlockState b;
    b.first = p.s.d_runs[run];
    b.last = p.s.d_run_last[b.first];
    b.row = b.first + (blk - (b.first / kBlock + run)) * kBlock;
    if (b.row > b.last) return;
    b.n = min(kBlock, b.last - b.row + 1);
    b.pos = p.s.d_pos[b.row];
    b.inner = b.n == kBlock && b.row - b.first >= g.taps - 1;
    {
        const size_t half = (size_t)(g.taps - 1) * g.channels;
        float* state = p.s.d_conv_state + (size_t)p.s.d_slot[b.row] * 2 * half;
        const int par = p.s.d_parity[b.row] & 1;
        b.old = state + par * half; b.fresh = state + (par ^ 1) * half;
    }
    auto conv = [&](int ch, int col, bool keep_state, float (&out)[kBlock]) {
        if constexpr (TAPS == 0 && NI >= 8) conv_block_far<T>(p, b, ch, col, keep_state, out);
        else conv_block<T, TAPS>(p, b, ch, col, keep_state, out);
    };
    const int v_groups = (g.vp + 127) / 128;   // of 128 value columns of a head
    for (int job = warp; job < g.heads * (1 + v_groups); job += kPrepThreads / 32) {
        if (job >= g.heads) {
            const int h = (job - g.heads) / v_groups, c0 = (job - g.heads) % v_groups * 128 + lane;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int c = c0 + i * 32;
                if (c >= g.vp) break;
                float v[kBlock] = {0.f, 0.f, 0.f, 0.f};
                if (c < g.vdim) conv(2 * g.kv_heads * g.dim + h * g.vdim + c, g.v_off + h * g.vdim + c, true, v);
                float* dst = p.w.v + ((size_t)blk * g.heads + h) * kBlock * g.vp + c;
#pragma unroll
                for (int t = 0; t < kBlock; ++t) dst[(size_t)t * g.vp] = v[t];
            }
            continue;
        }
        const int head = job, kvh = head / g.group;
        const bool own = head % g.group == 0;   // heads that share q and k: the first passes their convolution state on
        float q[NI][kBlock], k[NI][kBlock], dec[ND][kBlock];
#pragma unroll
        for (int i = 0; i < ND; ++i)   // travels while the convolutions are computed
#pragma unroll
            for (int t = 0; t < kBlock; ++t) {
                const int d = HEAD ? 0 : i * 32 + lane;
                dec[i][t] = t < b.n && d < g.dim ? decay_input<T>(p, b.row + t, head, d) : 0.f;
            }
        float sums[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) sums[i] = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int d = i * 32 + lane;
#pragma unroll
            for (int t = 0; t < kBlock; ++t) q[i][t] = k[i][t] = 0.f;
            if (d < g.dim) {
                conv(kvh * g.dim + d, g.q_off + kvh * g.dim + d, own, q[i]);
                conv((g.kv_heads + kvh) * g.dim + d, g.k_off + kvh * g.dim + d, own, k[i]);
            }
#pragma unroll
            for (int t = 0; t < kBlock; ++t) { sums[t] = fmaf(q[i][t], q[i][t], sums[t]); sums[4 + t] = fmaf(k[i][t], k[i][t], sums[4 + t]); }
        }
        float norm = 1.f / sqrtf(transpose_sum(sums) + 1e-6f);
        if (lane < 4) norm *= g.q_scale;
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
            const float qs = __shfl_sync(0xffffffffu, norm, t), ks = __shfl_sync(0xffffffffu, norm, 4 + t);
#pragma unroll
            for (int i = 0; i < NI; ++i) { q[i][t] *= qs; k[i][t] *= ks; }
        }
        const float rate = -expf(p.s.d_a_log[head]);
        float* vec = p.w.vec + ((size_t)blk * g.heads + head) * kVecs * g.dp;
        float num[16];   // A in 0 .. 5, B in 6 .. 15
#pragma unroll
        for (int i = 0; i < 16; ++i) num[i] = 0.f;
        float gd[kBlock];
        auto decays = [&](int i, int d) {
#pragma unroll
            for (int t = 0; t < kBlock; ++t) gd[t] = 1.f;
            if (d < g.dim) {
                const float bias = decay_bias(p, head, d);
#pragma unroll
                for (int t = 0; t < kBlock; ++t)
                    if (t < b.n) {
                        const float x = dec[i][t] + bias;
                        gd[t] = sizeof(T) == 2 ? decay_fast(x, rate) : expf(rate * softplus(x));
                    }
            }
        };
        if (HEAD) decays(0, 0);
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int d = i * 32 + lane;
            if (!HEAD) decays(HEAD ? 0 : i, d);
            const float g10 = gd[1], g21 = gd[2], g32 = gd[3], g20 = g21 * g10, g31 = g32 * g21, g30 = g31 * g10;   // decays of s+1 .. t
            const float* kk = k[i];
            const float* qq = q[i];
            num[0] = fmaf(kk[1] * kk[0], g10, num[0]);
            num[1] = fmaf(kk[2] * kk[0], g20, num[1]);
            num[2] = fmaf(kk[2] * kk[1], g21, num[2]);
            num[3] = fmaf(kk[3] * kk[0], g30, num[3]);
            num[4] = fmaf(kk[3] * kk[1], g31, num[4]);
            num[5] = fmaf(kk[3] * kk[2], g32, num[5]);
            num[6] = fmaf(qq[0], kk[0], num[6]);
            num[7] = fmaf(qq[1] * kk[0], g10, num[7]);
            num[8] = fmaf(qq[1], kk[1], num[8]);
            num[9] = fmaf(qq[2] * kk[0], g20, num[9]);
            num[10] = fmaf(qq[2] * kk[1], g21, num[10]);
            num[11] = fmaf(qq[2], kk[2], num[11]);
            num[12] = fmaf(qq[3] * kk[0], g30, num[12]);
            num[13] = fmaf(qq[3] * kk[1], g31, num[13]);
            num[14] = fmaf(qq[3] * kk[2], g32, num[14]);
            num[15] = fmaf(qq[3], kk[3], num[15]);
            if (d < g.dp) {
                float* o = vec + d;
                if constexpr (HEAD) {
#pragma unroll
                    for (int t = 0; t < kBlock; ++t) { o[t * g.dp] = kk[t]; o[(kBlock + t) * g.dp] = qq[t]; }
                    continue;
                }
                const float p0 = gd[0], p1 = p0 * gd[1], p2 = p1 * gd[2], p3 = p2 * gd[3];
                o[0] = p0 * kk[0]; o[g.dp] = p1 * kk[1]; o[2 * g.dp] = p2 * kk[2]; o[3 * g.dp] = p3 * kk[3];
                o[4 * g.dp] = p0 * qq[0]; o[5 * g.dp] = p1 * qq[1]; o[6 * g.dp] = p2 * qq[2]; o[7 * g.dp] = p3 * qq[3];
                o[8 * g.dp] = kk[0] * g30; o[9 * g.dp] = kk[1] * g31; o[10 * g.dp] = kk[2] * g32; o[11 * g.dp] = kk[3];
                o[12 * g.dp] = p3;
            }
        }
        const float mine = transpose_sum(num);
        float* dst = p.w.num + ((size_t)blk * g.heads + head) * kNums;
        if (lane < 16) dst[lane < 6 ? 4 + lane : 6 + lane] = mine;
        if (HEAD && lane == 0) {
            const float p1 = gd[0] * gd[1], p2 = p1 * gd[2];
            *reinterpret_cast<float4*>(dst + 24) = make_float4(gd[0], p1, p2, p2 * gd[3]);
            *reinterpret_cast<float4*>(dst + 28) = make_float4(gd[1] * gd[2] * gd[3], gd[2] * gd[3], gd[3], 1.f);
        }
        if (lane < kBlock)
            dst[lane] = lane < b.n ? sigmoid(ld(static_cast<const T*>(p.s.d_proj) + (size_t)(b.row + lane) * g.row + g.beta_off + head)) : 0.f;
    }
}

template <typename T, int NI>
int launch_groups(const Params& p, cudaStream_t s) {
    const dim3 grid((unsigned)max_blocks(p.s.rows, p.s.n_runs));
    constexpr int kTaps = NI <= 8 ? 4 : 0;   // convolutions of four taps are unrolled
    void (*kern)(Params) = p.g.head_decay ? (p.g.taps == kTaps ? delta_prepare_kernel<T, NI, kTaps, true> : delta_prepare_kernel<T, NI, 0, true>)
                                          : (p.g.taps == kTaps ? delta_prepare_kernel<T, NI, kTaps, false> : delta_prepare_kernel<T, NI, 0, false>);
    return launch_kernel(kern, grid, dim3(kPrepThreads), 0, s, 1, p);
}
template <typename T>
int launch_of(const Params& p, cudaStream_t s) {
    const int dim = p.g.dim;
    return dim <= 32 ? launch_groups<T, 1>(p, s) : dim <= 64 ? launch_groups<T, 2>(p, s) : dim <= 128 ? launch_groups<T, 4>(p, s) : dim <= 256 ? launch_groups<T, 8>(p, s)
                                                                                                                                : launch_groups<T, 16>(p, s);
}

}  // namespace

int launch_prepare(const Params& p, bool bf16, cudaStream_t s) { return bf16 ? launch_of<__nv_bfloat16>(p, s) : launch_of<float>(p, s); }

}  // namespace delta
}  // namespace gptrs
