// The step between two sublayers of a model whose norms sit on the sublayers' OUTPUTS and whose sublayers read the residual
// stream through a short causal convolution (no counterpart in gpt.rs):
//
//   x_t  <- x_t + y_t / sqrt(mean(y_t^2) + eps) * gamma           (or the normed embedding row at the start of the model)
//   h_t   = x_t + sum_j w[:, j] * x_(t - taps + 1 + j)            what the next sublayer reads
//
// in ONE kernel. The convolution looks back over rows of the same sequence: inside the launch those are the rows in front
// (a CTA recomputes the taps - 1 rows ahead of its tile, so nothing is exchanged between CTAs; the residual is read from one
// buffer and written to another), before it they are the sequence's state, the last taps - 1 values of x per channel. The
// state of a slot has two halves: a launch reads one and writes the other (`parity` says which), so no CTA can read what
// another one of the same launch has replaced. Everything is f32; y and h may be bf16.
#include "common.cuh"

namespace gptrs {
namespace {

constexpr int kThreads = 256;
constexpr int kMaxTaps = 16;
constexpr int kMaxTile = 16;
constexpr int kMaxRows = kMaxTile + kMaxTaps - 1;

__device__ __forceinline__ float cta_sum(float v, float* sh) {
    v = warp_sum(v);
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
    __syncthreads();
    if (l == 0) sh[w] = v;
    __syncthreads();
    return warp_sum(l < kThreads / 32 ? sh[l] : 0.f);
}

struct StepParams {
    gptrs_conv_step s;
    int tile;   // rows of a CTA
};

template <int VEC>
struct Vals { float v[VEC]; };

template <int VEC>
__device__ __forceinline__ Vals<VEC> load_f32(const float* p) {
    Vals<VEC> r;
    if constexpr (VEC == 4) {
        const float4 a = __ldg(reinterpret_cast<const float4*>(p));
        r.v[0] = a.x; r.v[1] = a.y; r.v[2] = a.z; r.v[3] = a.w;
    } else {
        r.v[0] = __ldg(p);
    }
    return r;
}
template <int VEC>
__device__ __forceinline__ void store_f32(float* p, const Vals<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int VEC>
__device__ __forceinline__ void store_any(void* base, size_t i, bool bf16, const Vals<VEC>& r) {
    if (!bf16) { store_f32<VEC>(static_cast<float*>(base) + i, r); return; }
    __nv_bfloat16* p = static_cast<__nv_bfloat16*>(base) + i;
    if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(r.v[0], r.v[1]), pack_bf16x2(r.v[2], r.v[3]));
    else *p = __float2bfloat16_rn(r.v[0]);
}
// the row that is normed: a sublayer's output (f32 or bf16) or an embedding row (f32)
struct Source { const void* base; bool bf16; };
template <int VEC>
__device__ __forceinline__ Vals<VEC> load_any(const Source& s, size_t i) {
    if (!s.bf16) return load_f32<VEC>(static_cast<const float*>(s.base) + i);
    Vals<VEC> r;
    const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(s.base) + i;
    if constexpr (VEC == 4) {
        const uint2 u = __ldg(reinterpret_cast<const uint2*>(p));
        r.v[0] = bf16_lo(u.x); r.v[1] = bf16_hi(u.x); r.v[2] = bf16_lo(u.y); r.v[3] = bf16_hi(u.y);
    } else {
        r.v[0] = __bfloat162float(__ldg(p));
    }
    return r;
}

template <int TAPS, int VEC>
__global__ void __launch_bounds__(kThreads) post_norm_conv_kernel(const StepParams p) {
    __shared__ float inv[kMaxRows], sh[32];
    __shared__ int s_slot[kMaxRows], s_pos[kMaxRows], s_first[kMaxRows], s_last[kMaxRows], s_par[kMaxRows];
    __shared__ long long s_src[kMaxRows];   // element offset of the row in the normed source
    const gptrs_conv_step& a = p.s;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int T = (int)a.rows, D = (int)a.dim;
    const int r0 = blockIdx.x * p.tile, r1 = min(r0 + p.tile, T);
    const bool conv = a.d_conv != nullptr;
    const int keep = conv ? (int)a.taps - 1 : 0;   // values of state per channel
    pdl_launch_dependents();
    pdl_wait();
    const int first0 = conv ? a.d_run_first[r0] : r0;
    const int i0 = max(r0 - keep, first0);  // the first row whose x this CTA needs
    const int n = r1 - i0;
    if (tid < n) {
        const int r = i0 + tid;
        if (conv) {
            s_slot[tid] = a.d_slot[r]; s_pos[tid] = a.d_pos[r]; s_first[tid] = a.d_run_first[r]; s_last[tid] = a.d_run_last[r];
            s_par[tid] = a.d_parity[r] & 1;
        }
        if (a.d_embed) {
            int id = a.d_tokens[r];
            if (id < 0 || id >= a.vocab) { atomicExch(a.d_status, 2); id = 0; }
            s_src[tid] = (long long)id * D;
        } else {
            s_src[tid] = (long long)r * a.ldy;
        }
    }
    __syncthreads();
    const Source src = {a.d_embed ? static_cast<const void*>(a.d_embed) : a.d_y, !a.d_embed && a.y_dtype == GPTRS_BF16};
    // ---- 1 / rms of the rows ------------------------------------------------------------------------------------------------
    if (n < 4) {   // few rows: the whole CTA on each
        for (int i = 0; i < n; ++i) {
            float ss = 0.f;
            for (int c = tid * VEC; c < D; c += kThreads * VEC) {
                const Vals<VEC> v = load_any<VEC>(src, (size_t)s_src[i] + c);
#pragma unroll
                for (int e = 0; e < VEC; ++e) ss = fmaf(v.v[e], v.v[e], ss);
            }
            ss = cta_sum(ss, sh);
            if (tid == 0) inv[i] = 1.f / sqrtf(ss / (float)D + a.eps);
        }
    } else {
        for (int i = warp; i < n; i += kThreads / 32) {
            float ss = 0.f;
#pragma unroll 4
            for (int c = lane * VEC; c < D; c += 32 * VEC) {
                const Vals<VEC> v = load_any<VEC>(src, (size_t)s_src[i] + c);
#pragma unroll
                for (int e = 0; e < VEC; ++e) ss = fmaf(v.v[e], v.v[e], ss);
            }
            ss = warp_sum(ss);
            if (lane == 0) inv[i] = 1.f / sqrtf(ss / (float)D + a.eps);
        }
    }
    __syncthreads();
    // ---- columns: a thread walks down the rows with the last taps - 1 values of its channels in registers ----------------------
    const bool h_bf16 = a.h_dtype == GPTRS_BF16;
    for (int c = tid * VEC; c < D; c += kThreads * VEC) {
        const Vals<VEC> gamma = load_f32<VEC>(a.d_gamma + c);
        float w[TAPS][VEC];          // w[k] multiplies x_(t - k)
        float hist[TAPS > 1 ? TAPS - 1 : 1][VEC];
#pragma unroll
        for (int k = 0; k < TAPS; ++k)
#pragma unroll
            for (int e = 0; e < VEC; ++e) w[k][e] = (conv && k < (int)a.taps) ? __ldg(a.d_conv + (size_t)(c + e) * a.taps + (a.taps - 1 - k)) : 0.f;
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
            for (int e = 0; e < VEC; ++e) hist[k][e] = 0.f;
        Vals<VEC> y_next = load_any<VEC>(src, (size_t)s_src[0] + c), x_next;
        if (a.d_x) x_next = load_f32<VEC>(a.d_x + (size_t)i0 * D + c);
        for (int i = 0; i < n; ++i) {
            const int r = i0 + i;
            const Vals<VEC> y = y_next, xin = x_next;
            if (i + 1 < n) {
                y_next = load_any<VEC>(src, (size_t)s_src[i + 1] + c);
                if (a.d_x) x_next = load_f32<VEC>(a.d_x + (size_t)(r + 1) * D + c);
            }
            Vals<VEC> x;
#pragma unroll
            for (int e = 0; e < VEC; ++e) x.v[e] = y.v[e] * inv[i] * gamma.v[e] + (a.d_x ? xin.v[e] : 0.f);
            if (conv) {
                const int pos = s_pos[i];
                float* state = a.d_state + (size_t)s_slot[i] * 2 * keep * D + c;
                if (s_first[i] == r && keep > 0) {   // start of a run: what the sequence left behind
                    const float* old = state + (size_t)s_par[i] * keep * D;
                    float* fresh = state + (size_t)(s_par[i] ^ 1) * keep * D;
                    const int len = s_last[i] - r + 1;
#pragma unroll
                    for (int k = 0; k < TAPS - 1; ++k) {
                        Vals<VEC> o;
#pragma unroll
                        for (int e = 0; e < VEC; ++e) o.v[e] = 0.f;
                        const int at = pos - 1 - k;
                        if (k < keep && at >= 0) {
#pragma unroll
                            for (int e = 0; e < VEC; ++e) o.v[e] = old[(size_t)(at % keep) * D + e];
                            // a run shorter than the state: the values it does not push out stay
                            if (at > pos + len - 1 - keep) store_f32<VEC>(fresh + (size_t)(at % keep) * D, o);
                        }
#pragma unroll
                        for (int e = 0; e < VEC; ++e) hist[k][e] = o.v[e];
                    }
                }
                if (r >= r0) {
                    if (s_last[i] - r < keep) store_f32<VEC>(state + ((size_t)(s_par[i] ^ 1) * keep + pos % keep) * D, x);
                    Vals<VEC> h;
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        float s = 0.f;
#pragma unroll
                        for (int k = TAPS - 1; k >= 1; --k) s = fmaf(w[k][e], hist[k - 1][e], s);
                        h.v[e] = x.v[e] + fmaf(w[0][e], x.v[e], s);
                    }
                    store_any<VEC>(a.d_h, (size_t)r * a.ldh + c, h_bf16, h);
                }
#pragma unroll
                for (int k = TAPS - 2; k >= 1; --k)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) hist[k][e] = hist[k - 1][e];
                if (TAPS > 1)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) hist[0][e] = x.v[e];
            }
            if (r >= r0 && a.d_x_out) store_f32<VEC>(a.d_x_out + (size_t)r * D + c, x);
        }
    }
    if (conv && h_bf16)   // padding columns of the bf16 rows
        for (int r = r0; r < r1; ++r)
            for (int c = D + tid; c < (int)a.ldh; c += kThreads) static_cast<__nv_bfloat16*>(a.d_h)[(size_t)r * a.ldh + c] = __float2bfloat16_rn(0.f);
}

template <int VEC>
int launch_taps(const StepParams& p, dim3 grid, cudaStream_t st) {
    const int taps = p.s.d_conv ? (int)p.s.taps : 1;
    if (taps <= 1) return launch_kernel(post_norm_conv_kernel<1, VEC>, grid, dim3(kThreads), 0, st, 1, p);
    if (taps == 2) return launch_kernel(post_norm_conv_kernel<2, VEC>, grid, dim3(kThreads), 0, st, 1, p);
    if (taps == 3) return launch_kernel(post_norm_conv_kernel<3, VEC>, grid, dim3(kThreads), 0, st, 1, p);
    if (taps == 4) return launch_kernel(post_norm_conv_kernel<4, VEC>, grid, dim3(kThreads), 0, st, 1, p);
    if (taps <= 8) return launch_kernel(post_norm_conv_kernel<8, VEC>, grid, dim3(kThreads), 0, st, 1, p);
    return launch_kernel(post_norm_conv_kernel<kMaxTaps, VEC>, grid, dim3(kThreads), 0, st, 1, p);
}

// End of the model: the last sublayer's output joins the residual stream and the sum is normed again, for the listed rows.
struct FinalParams {
    const float* x;
    const void* y;
    const float* gamma;
    const float* final_gamma;
    const int* rows;
    void* out;
    int y_bf16, out_bf16, D;
    long long ldy, ldo;
    float eps;
};
__global__ void __launch_bounds__(kThreads) post_norm_final_kernel(const FinalParams p) {
    __shared__ float sh[32];
    const int tid = threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    const int r = p.rows ? p.rows[blockIdx.x] : (int)blockIdx.x;
    const Source src = {p.y, p.y_bf16 != 0};
    float ss = 0.f;
    for (int c = tid; c < p.D; c += kThreads) { const float v = load_any<1>(src, (size_t)r * p.ldy + c).v[0]; ss = fmaf(v, v, ss); }
    const float inv = 1.f / sqrtf(cta_sum(ss, sh) / (float)p.D + p.eps);
    auto value = [&](int c) {
        return load_any<1>(src, (size_t)r * p.ldy + c).v[0] * inv * p.gamma[c] + p.x[(size_t)r * p.D + c];
    };
    ss = 0.f;
    for (int c = tid; c < p.D; c += kThreads) { const float v = value(c); ss = fmaf(v, v, ss); }
    const float inv2 = 1.f / sqrtf(cta_sum(ss, sh) / (float)p.D + p.eps);
    for (int c = tid; c < (int)p.ldo; c += kThreads) {
        const float v = c < p.D ? value(c) * inv2 * p.final_gamma[c] : 0.f;
        if (p.out_bf16) static_cast<__nv_bfloat16*>(p.out)[(size_t)blockIdx.x * p.ldo + c] = __float2bfloat16_rn(v);
        else static_cast<float*>(p.out)[(size_t)blockIdx.x * p.ldo + c] = v;
    }
}

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" {

int gptrs_cuda_post_norm_conv(const gptrs_conv_step* step, void* stream) {
    GPTRS_REQUIRE(step, "null pointer");
    const gptrs_conv_step& a = *step;
    GPTRS_REQUIRE(a.d_gamma && (a.d_embed ? a.d_tokens != nullptr && a.d_status != nullptr : a.d_y != nullptr), "null pointer");
    GPTRS_REQUIRE(a.rows >= 0 && a.rows < (1ll << 31) && a.dim > 0 && a.dim < (1ll << 31), "bad shape");
    GPTRS_REQUIRE(a.d_x == nullptr || a.d_x != a.d_x_out, "the residual is read from one buffer and written to another");
    GPTRS_REQUIRE((a.y_dtype == GPTRS_F32 || a.y_dtype == GPTRS_BF16) && (a.h_dtype == GPTRS_F32 || a.h_dtype == GPTRS_BF16), "f32 or bf16");
    if (a.d_conv) {
        GPTRS_REQUIRE(a.taps >= 1, "a convolution needs at least one tap");
        if (a.taps > kMaxTaps) return fail(GPTRS_UNIMPLEMENTED, "short convolutions of more than 16 taps");
        GPTRS_REQUIRE(a.d_h && a.ldh >= a.dim && a.d_slot && a.d_pos && a.d_run_first && a.d_run_last && a.d_parity && (a.taps == 1 || a.d_state), "null pointer");
    }
    if (a.rows == 0) return GPTRS_OK;
    StepParams p;
    p.s = a;
    // few rows: one per CTA; many: tiles of up to 14 rows (with two rows of halo two rounds of the eight warps)
    const int64_t fill = a.rows / (2 * sm_count());
    p.tile = (int)(fill < 1 ? 1 : fill > 14 ? 14 : fill);
    const bool vec = a.dim % 4 == 0 && (a.d_embed || a.ldy % 4 == 0) && (!a.d_conv || a.ldh % 4 == 0);
    const dim3 grid((unsigned)ceil_div(a.rows, p.tile));
    return vec ? launch_taps<4>(p, grid, as_stream(stream)) : launch_taps<1>(p, grid, as_stream(stream));
}

int gptrs_cuda_post_norm_final(const float* d_x, const void* d_y, int y_dtype, int64_t ldy, const float* d_gamma, const float* d_final_gamma,
                               float eps, const int32_t* d_rows, void* d_out, int out_dtype, int64_t ldo, int64_t n_rows, int64_t dim, void* stream) {
    GPTRS_REQUIRE(d_x && d_y && d_gamma && d_final_gamma && d_out, "null pointer");
    GPTRS_REQUIRE(n_rows >= 0 && dim > 0 && dim < (1ll << 31) && ldy >= dim && ldo >= dim, "bad shape");
    if (n_rows == 0) return GPTRS_OK;
    FinalParams p = {d_x, d_y, d_gamma, d_final_gamma, d_rows, d_out, y_dtype == GPTRS_BF16, out_dtype == GPTRS_BF16, (int)dim, ldy, ldo, eps};
    return launch_kernel(post_norm_final_kernel, dim3((unsigned)n_rows), dim3(kThreads), 0, as_stream(stream), 1, p);
}

}  // extern "C"
