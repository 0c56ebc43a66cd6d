// The step between two sublayers of a model with a norm in front of every sublayer and several copies ("streams") of the residual that
// are mixed with one another at every sublayer (no counterpart in gpt.rs):
//
//   x_t <- sum_s mix[s][t] x_s + out[t] y        all streams at once from the old ones (or the scaled embedding in every stream)
//   h    = rms(sum_s in[s] x_s) gamma_in         what the next sublayer reads
//
// in ONE kernel, a CTA per row: a thread reads its columns of all streams, mixes them in registers and writes them back, and only the
// combination that the norm needs stays in registers over the row's sum. y may be the weighted sum of the rows that a token's experts
// put out, plus a shared expert's. Everything is f32; y and h may be bf16.
#include "row_step.cuh"

namespace gptrs {
namespace {

struct Params { gptrs_stream_step s; };

// y of VEC columns from `c` on
template <int VEC>
__device__ __forceinline__ void load_y(const gptrs_stream_step& a, int row, int c, float (&y)[VEC]) {
    const bool bf16 = a.y_dtype == GPTRS_BF16;
    if (a.d_pair) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = 0.f;
#pragma unroll 4
        for (int k = 0; k < (int)a.top; ++k) {
            const float w = __ldg(a.d_pair_weight + (size_t)row * a.top + k);
            float v[VEC];
            load_act<VEC>(a.d_y, (size_t)__ldg(a.d_pair + (size_t)row * a.top + k) * a.ldy + c, bf16, v);
#pragma unroll
            for (int e = 0; e < VEC; ++e) y[e] = fmaf(w, v[e], y[e]);
        }
    } else {
        load_act<VEC>(a.d_y, (size_t)row * a.ldy + c, bf16, y);
    }
    if (a.d_add) {
        float v[VEC];
        load_act<VEC>(a.d_add, (size_t)row * a.ld_add + c, bf16, v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] += v[e];
    }
}

// Up to four streams of widths that are multiples of 4: a thread holds the columns (i * THREADS + tid) * VEC + e, i < N, of up to S streams.
template <int THREADS, int N, int VEC, int S>
__global__ void __launch_bounds__(THREADS) stream_step_kernel(const Params p) {
    __shared__ float sh[32], s_mix[S * S], s_out[S], s_in[S];
    const gptrs_stream_step& a = p.s;
    const int tid = threadIdx.x, D = (int)a.dim, n = a.streams;
    pdl_launch_dependents();
    // constants; rows and columns past the streams in use are zero
    for (int i = tid; i < S * S; i += THREADS) {
        const int from = i / S, to = i % S;
        s_mix[i] = from < n && to < n ? (a.d_mix ? a.d_mix[from * n + to] : from == to ? 1.f : 0.f) : 0.f;
    }
    if (tid < S) {
        s_out[tid] = tid < n ? (a.d_out ? a.d_out[tid] : 1.f) : 0.f;
        s_in[tid] = tid < n ? (a.d_in ? a.d_in[tid] : 1.f) : 0.f;
    }
    pdl_wait();
    __syncthreads();
    const int row = a.d_rows ? a.d_rows[blockIdx.x] : (int)blockIdx.x;
    float* x_row = a.d_x + (size_t)row * n * D;
    int id = 0;
    if (a.d_embed) {
        id = a.d_tokens[row];
        if (id < 0 || id >= a.vocab) { if (tid == 0) atomicExch(a.d_status, 2); id = 0; }
    }
    const bool write = !a.d_rows && (a.d_embed || a.d_y);
    float u[N][VEC];
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int c = (i * THREADS + tid) * VEC;
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[i][e] = 0.f;
        if (c >= D) continue;
        float old[S][VEC], y[VEC], sum[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = sum[e] = 0.f;
        if (a.d_embed) {
            load_act<VEC>(a.d_embed, (size_t)id * D + c, false, y);
#pragma unroll
            for (int e = 0; e < VEC; ++e) y[e] *= a.embed_scale;
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s)
                if (s < n) load_act<VEC>(x_row, (size_t)s * D + c, false, old[s]);
            if (a.d_y) load_y<VEC>(a, row, c, y);
        }
#pragma unroll
        for (int t = 0; t < S; ++t) {
            if (t >= n) break;
            float v[VEC];
            if (a.d_embed) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[e] = y[e];
            } else if (a.d_y) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[e] = s_out[t] * y[e];
#pragma unroll
                for (int s = 0; s < S; ++s)
                    if (s < n)
#pragma unroll
                        for (int e = 0; e < VEC; ++e) v[e] = fmaf(s_mix[s * S + t], old[s][e], v[e]);
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[e] = old[t][e];
            }
            if (write) store_act<VEC>(x_row, (size_t)t * D + c, false, v);
#pragma unroll
            for (int e = 0; e < VEC; ++e) { u[i][e] = fmaf(s_in[t], v[e], u[i][e]); sum[e] += v[e]; }
        }
        if (a.d_sum) store_act<VEC>(a.d_sum, (size_t)row * D + c, false, sum);
    }
    if (!a.d_gamma_in) return;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(u[i][e], u[i][e], ss);
    const float inv = 1.f / sqrtf(row_sum<THREADS>(ss, sh) / (float)D + a.eps);
    const bool h_bf16 = a.h_dtype == GPTRS_BF16;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int c = (i * THREADS + tid) * VEC;
        if (c >= D) continue;
        float g[VEC];
        load_act<VEC>(a.d_gamma_in, c, false, g);
#pragma unroll
        for (int e = 0; e < VEC; ++e) g[e] *= u[i][e] * inv;
        store_act<VEC>(a.d_h, (size_t)blockIdx.x * a.ldh + c, h_bf16, g);
    }
    for (int c = D + tid; c < (int)a.ldh; c += THREADS) {
        const float z[1] = {0.f};
        store_act<1>(a.d_h, (size_t)blockIdx.x * a.ldh + c, h_bf16, z);
    }
}

// Any width and up to 16 streams: the combination lies in shared memory, nothing is unrolled over columns or new streams.
constexpr int kAnyThreads = 256;
__global__ void __launch_bounds__(kAnyThreads) stream_step_any_kernel(const Params p) {
    constexpr int S = GPTRS_MAX_STREAMS;
    extern __shared__ float ss_u[];   // [dim]
    __shared__ float sh[32];
    const gptrs_stream_step& a = p.s;
    const int tid = threadIdx.x, D = (int)a.dim, n = a.streams;
    pdl_launch_dependents();
    pdl_wait();
    const int row = a.d_rows ? a.d_rows[blockIdx.x] : (int)blockIdx.x;
    float* x_row = a.d_x + (size_t)row * n * D;
    int id = 0;
    if (a.d_embed) {
        id = a.d_tokens[row];
        if (id < 0 || id >= a.vocab) { if (tid == 0) atomicExch(a.d_status, 2); id = 0; }
    }
    float ss = 0.f;
    for (int c = tid; c < D; c += kAnyThreads) {
        float y[1] = {0.f}, old[S], u = 0.f, sum = 0.f;
        if (a.d_embed) y[0] = a.d_embed[(size_t)id * D + c] * a.embed_scale;
        else if (a.d_y) load_y<1>(a, row, c, y);
#pragma unroll
        for (int s = 0; s < S; ++s) old[s] = !a.d_embed && s < n ? x_row[(size_t)s * D + c] : 0.f;
#pragma unroll 1
        for (int t = 0; t < n; ++t) {
            float v = a.d_embed ? y[0] : a.d_y ? (a.d_out ? __ldg(a.d_out + t) : 1.f) * y[0] : 0.f;
#pragma unroll
            for (int s = 0; s < S; ++s)
                if (s < n) v = fmaf(a.d_y && a.d_mix ? __ldg(a.d_mix + s * n + t) : s == t ? 1.f : 0.f, old[s], v);
            if (!a.d_rows && (a.d_embed || a.d_y)) x_row[(size_t)t * D + c] = v;
            u = fmaf(a.d_in ? __ldg(a.d_in + t) : 1.f, v, u);
            sum += v;
        }
        if (a.d_sum) a.d_sum[(size_t)row * D + c] = sum;
        ss_u[c] = u;
        ss = fmaf(u, u, ss);
    }
    if (!a.d_gamma_in) return;
    const float inv = 1.f / sqrtf(row_sum<kAnyThreads>(ss, sh) / (float)D + a.eps);
    for (int c = tid; c < (int)a.ldh; c += kAnyThreads) {
        const float h[1] = {c < D ? ss_u[c] * inv * a.d_gamma_in[c] : 0.f};
        store_act<1>(a.d_h, (size_t)blockIdx.x * a.ldh + c, a.h_dtype == GPTRS_BF16, h);
    }
}

template <int THREADS, int N>
int launch(const Params& p, cudaStream_t st) {
    const dim3 grid((unsigned)p.s.rows), block(THREADS);
    const int n = p.s.streams;
    if (n == 1) return launch_kernel(stream_step_kernel<THREADS, N, 4, 1>, grid, block, 0, st, 1, p);
    if (n == 2) return launch_kernel(stream_step_kernel<THREADS, N, 4, 2>, grid, block, 0, st, 1, p);
    return launch_kernel(stream_step_kernel<THREADS, N, 4, 4>, grid, block, 0, st, 1, p);
}

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" int gptrs_cuda_stream_step(const gptrs_stream_step* step, void* stream) {
    GPTRS_REQUIRE(step && step->d_x, "null pointer");
    const gptrs_stream_step& a = *step;
    GPTRS_REQUIRE(a.rows >= 0 && a.rows < (1ll << 31) && a.dim > 0 && a.streams >= 1, "bad shape");
    GPTRS_REQUIRE(!a.d_embed || (a.d_tokens && a.d_status && !a.d_rows && !a.d_y), "embedding: token ids, status, no sublayer output");
    GPTRS_REQUIRE(!a.d_y || !a.d_pair || (a.d_pair_weight && a.top > 0), "null pointer");
    GPTRS_REQUIRE(!a.d_add || a.d_y, "a second output belongs to a first one");
    GPTRS_REQUIRE(!a.d_gamma_in || (a.d_h && a.ldh >= a.dim), "norm of the next sublayer's input: output");
    GPTRS_REQUIRE((!a.d_y || a.y_dtype == GPTRS_F32 || a.y_dtype == GPTRS_BF16) && (!a.d_gamma_in || a.h_dtype == GPTRS_F32 || a.h_dtype == GPTRS_BF16), "f32 or bf16");
    if (a.streams > GPTRS_MAX_STREAMS) return fail(GPTRS_UNIMPLEMENTED, "more than 16 residual streams");
    if (a.rows == 0) return GPTRS_OK;
    const Params p = {a};
    const bool vec = a.dim % 4 == 0 && (!a.d_y || a.ldy % 4 == 0) && (!a.d_add || a.ld_add % 4 == 0) && (!a.d_gamma_in || a.ldh % 4 == 0);
    cudaStream_t st = as_stream(stream);
    if (vec && a.streams <= 4) {
        if (a.dim <= 512) return launch<128, 1>(p, st);
        if (a.dim <= 1024) return launch<256, 1>(p, st);
        if (a.dim <= 2048) return launch<512, 1>(p, st);
        if (a.dim <= 4096) return launch<512, 2>(p, st);
    }
    const size_t smem = (size_t)a.dim * 4;
    if (smem > 200 * 1024) return fail(GPTRS_UNIMPLEMENTED, "stream step: rows of more than 51200 values");
    if (smem > 40 * 1024) GPTRS_CUDA_OK(cudaFuncSetAttribute(stream_step_any_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return launch_kernel(stream_step_any_kernel, dim3((unsigned)a.rows), dim3(kAnyThreads), smem, st, 1, p);
}
