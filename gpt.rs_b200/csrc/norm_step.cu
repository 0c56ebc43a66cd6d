// The step between two sublayers of a model with a norm in front of and behind every sublayer (no counterpart in gpt.rs):
//
//   x_t  <- x_t + y_t / sqrt(mean(y_t^2) + eps) * gamma_out     (or token embedding + position vector at the start of the model)
//   h_t   = x_t / sqrt(mean(x_t^2) + eps) * gamma_in            what the next sublayer reads
//
// in ONE kernel, a CTA per row with the row in registers: two sums over the row, one pass over memory. y may be the weighted sum
// of the rows that a token's experts put out, so that the combination needs no kernel of its own. Everything is f32; y and h may
// be bf16.
#include "row_step.cuh"

namespace gptrs {
namespace {

struct Params { gptrs_norm_step s; };

// A thread holds the elements (i * THREADS + tid) * VEC + e, i < N.
template <int THREADS, int N, int VEC>
__global__ void __launch_bounds__(THREADS) norm_step_kernel(const Params p) {
    __shared__ float sh[32];
    const gptrs_norm_step& a = p.s;
    const int tid = threadIdx.x, D = (int)a.dim;
    pdl_launch_dependents();
    pdl_wait();
    const int row = a.d_rows ? a.d_rows[blockIdx.x] : (int)blockIdx.x;
    float x[N][VEC];
    bool in[N];
#pragma unroll
    for (int i = 0; i < N; ++i) in[i] = (i * THREADS + tid) * VEC < D;
    if (a.d_embed) {
        int id = a.d_tokens[row], pos = a.d_pos_embed ? a.d_pos[row] : 0;
        if (id < 0 || id >= a.vocab) { if (tid == 0) atomicExch(a.d_status, 2); id = 0; }
        if (a.d_pos_embed && (pos < 0 || pos >= a.positions)) { if (tid == 0) atomicExch(a.d_status, 2); pos = 0; }
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (in[i]) {
                const int c = (i * THREADS + tid) * VEC;
                load_act<VEC>(a.d_embed, (size_t)id * D + c, false, x[i]);
                if (a.d_pos_embed) {
                    float q[VEC];
                    load_act<VEC>(a.d_pos_embed, (size_t)pos * D + c, false, q);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) x[i][e] += q[e];
                }
                store_act<VEC>(a.d_x, (size_t)row * D + c, false, x[i]);
            }
    } else if (a.d_y) {
        const bool y_bf16 = a.y_dtype == GPTRS_BF16;
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (in[i]) {
                const int c = (i * THREADS + tid) * VEC;
                if (a.d_pair) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) x[i][e] = 0.f;
                    for (int k = 0; k < (int)a.top; ++k) {
                        const float w = __ldg(a.d_pair_weight + (size_t)row * a.top + k);
                        float v[VEC];
                        load_act<VEC>(a.d_y, (size_t)__ldg(a.d_pair + (size_t)row * a.top + k) * a.ldy + c, y_bf16, v);
#pragma unroll
                        for (int e = 0; e < VEC; ++e) x[i][e] = fmaf(w, v[e], x[i][e]);
                    }
                } else {
                    load_act<VEC>(a.d_y, (size_t)row * a.ldy + c, y_bf16, x[i]);
                }
#pragma unroll
                for (int e = 0; e < VEC; ++e) ss = fmaf(x[i][e], x[i][e], ss);
            }
        const float inv = 1.f / sqrtf(row_sum<THREADS>(ss, sh) / (float)D + a.eps);
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (in[i]) {
                const int c = (i * THREADS + tid) * VEC;
                float g[VEC], o[VEC];
                load_act<VEC>(a.d_gamma_out, c, false, g);
                load_act<VEC>(a.d_x, (size_t)row * D + c, false, o);
#pragma unroll
                for (int e = 0; e < VEC; ++e) x[i][e] = o[e] + x[i][e] * inv * g[e];
                if (!a.d_rows) store_act<VEC>(a.d_x, (size_t)row * D + c, false, x[i]);
            }
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (in[i]) load_act<VEC>(a.d_x, (size_t)row * D + (i * THREADS + tid) * VEC, false, x[i]);
    }
    if (!a.d_gamma_in) return;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i)
        if (in[i])
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss = fmaf(x[i][e], x[i][e], ss);
    const float inv = 1.f / sqrtf(row_sum<THREADS>(ss, sh) / (float)D + a.eps);
    const bool h_bf16 = a.h_dtype == GPTRS_BF16;
#pragma unroll
    for (int i = 0; i < N; ++i)
        if (in[i]) {
            const int c = (i * THREADS + tid) * VEC;
            float g[VEC];
            load_act<VEC>(a.d_gamma_in, c, false, g);
#pragma unroll
            for (int e = 0; e < VEC; ++e) g[e] *= x[i][e] * inv;
            store_act<VEC>(a.d_h, (size_t)blockIdx.x * a.ldh + c, h_bf16, g);
        }
    for (int c = D + tid; c < (int)a.ldh; c += THREADS) {
        const float z[1] = {0.f};
        store_act<1>(a.d_h, (size_t)blockIdx.x * a.ldh + c, h_bf16, z);
    }
}

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" int gptrs_cuda_norm_step(const gptrs_norm_step* step, void* stream) {
    GPTRS_REQUIRE(step && step->d_x, "null pointer");
    const gptrs_norm_step& a = *step;
    GPTRS_REQUIRE(a.rows >= 0 && a.rows < (1ll << 31) && a.dim > 0, "bad shape");
    GPTRS_REQUIRE(!a.d_embed || (a.d_tokens && a.d_status && !a.d_rows && (!a.d_pos_embed || (a.d_pos && a.positions > 0))), "embedding: token ids, positions, status");
    GPTRS_REQUIRE(a.d_embed || !a.d_y || (a.d_gamma_out && (a.d_pair ? a.d_pair_weight && a.top > 0 : true)), "null pointer");
    GPTRS_REQUIRE(!a.d_gamma_in || (a.d_h && a.ldh >= a.dim), "norm of the next sublayer's input: output");
    GPTRS_REQUIRE((!a.d_y || a.y_dtype == GPTRS_F32 || a.y_dtype == GPTRS_BF16) && (!a.d_gamma_in || a.h_dtype == GPTRS_F32 || a.h_dtype == GPTRS_BF16), "f32 or bf16");
    if (a.rows == 0) return GPTRS_OK;
    const Params p = {a};
    const bool vec = a.dim % 4 == 0 && (!a.d_y || a.ldy % 4 == 0) && (!a.d_gamma_in || a.ldh % 4 == 0);
    const dim3 grid((unsigned)a.rows);
    cudaStream_t st = as_stream(stream);
    if (vec) {
        if (a.dim <= 512) return launch_kernel(norm_step_kernel<128, 1, 4>, grid, dim3(128), 0, st, 1, p);
        if (a.dim <= 1024) return launch_kernel(norm_step_kernel<256, 1, 4>, grid, dim3(256), 0, st, 1, p);
        if (a.dim <= 2048) return launch_kernel(norm_step_kernel<256, 2, 4>, grid, dim3(256), 0, st, 1, p);
        if (a.dim <= 4096) return launch_kernel(norm_step_kernel<256, 4, 4>, grid, dim3(256), 0, st, 1, p);
        if (a.dim <= 16384) return launch_kernel(norm_step_kernel<512, 8, 4>, grid, dim3(512), 0, st, 1, p);
    } else {
        if (a.dim <= 512) return launch_kernel(norm_step_kernel<256, 2, 1>, grid, dim3(256), 0, st, 1, p);
        if (a.dim <= 4096) return launch_kernel(norm_step_kernel<512, 8, 1>, grid, dim3(512), 0, st, 1, p);
        if (a.dim <= 16384) return launch_kernel(norm_step_kernel<512, 32, 1>, grid, dim3(512), 0, st, 1, p);
    }
    return fail(GPTRS_UNIMPLEMENTED, "norm step: rows of more than 16384 values");
}
