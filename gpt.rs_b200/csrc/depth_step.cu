// The step between two sublayers of a model with norms on the sublayers' outputs only, taken over equal groups of channels, and a weighted
// average over depth behind every layer (no counterpart in gpt.rs):
//
//   r  = x + mult N(y) gamma_out             N: every group of channels divided by its own root mean square
//   x' = sum_j weights[j] state_j + w r      the embedding and the results of the layers so far; r becomes the next state
//   h  = x', or N(x') gamma at the end       what the next sublayer reads
//
// in ONE kernel, a CTA per row with the row in registers: a middle step is one pass over memory, the end of layer l reads l + 1 states
// beside it. y may be the weighted sum of the rows that a token's experts put out, plus a gated shared expert's. Everything is f32; y and h
// may be bf16.
// Second kernel of this file: a feed-forward's activation that is a polynomial of normed powers, a CTA per row.
#include "row_step.cuh"

namespace gptrs {
namespace {

struct Params { gptrs_depth_step s; };

// y of VEC columns from `c` on
template <int VEC>
__device__ __forceinline__ void load_y(const gptrs_depth_step& a, int row, int c, float gate, float (&y)[VEC]) {
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
        for (int e = 0; e < VEC; ++e) y[e] = fmaf(gate, v[e], y[e]);
    }
}

__device__ __forceinline__ float add_gate(const gptrs_depth_step& a, int row) {
    return a.d_add_gate ? 1.f / (1.f + expf(-a.d_add_gate[(size_t)row * a.ld_add_gate])) : 1.f;
}

// A thread holds the columns (i * THREADS + tid) * 4 + e, i < N. Groups are whole multiples of 128 channels, so that the columns a warp holds for
// one i lie in one group: a sum per (i, warp), added up per group from shared memory in a fixed order.
template <int THREADS, int N>
__global__ void __launch_bounds__(THREADS) depth_step_kernel(const Params p) {
    constexpr int kSlots = N * THREADS / 32;
    __shared__ float part[2][kSlots];
    const gptrs_depth_step& a = p.s;
    const int tid = threadIdx.x, D = (int)a.dim, size = D / a.groups, per_group = size / 128;
    pdl_launch_dependents();
    pdl_wait();
    const int row = a.d_rows ? a.d_rows[blockIdx.x] : (int)blockIdx.x;
    float r[N][4];
    bool in[N];
    int group[N];
#pragma unroll
    for (int i = 0; i < N; ++i) { const int c = (i * THREADS + tid) * 4; in[i] = c < D; group[i] = c / size; }
    // 1 / root mean square of the group of every column held
    auto group_norm = [&](int buf, float (&inv)[N]) {
#pragma unroll
        for (int i = 0; i < N; ++i) {
            float ss = 0.f;
            if (in[i])
#pragma unroll
                for (int e = 0; e < 4; ++e) ss = fmaf(r[i][e], r[i][e], ss);
            ss = warp_sum(ss);
            if ((tid & 31) == 0) part[buf][i * (THREADS / 32) + (tid >> 5)] = ss;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < N; ++i) {
            if (!in[i]) continue;
            float s = 0.f;
            for (int k = 0; k < per_group; ++k) s += part[buf][group[i] * per_group + k];
            inv[i] = 1.f / sqrtf(s / (float)size + a.eps);
        }
    };
    if (a.d_embed) {
        int id = a.d_tokens[row];
        if (id < 0 || id >= a.vocab) { if (tid == 0) atomicExch(a.d_status, 2); id = 0; }
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (in[i]) load_act<4>(a.d_embed, (size_t)id * D + (i * THREADS + tid) * 4, false, r[i]);
    } else {
        float x[N][4];
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (in[i]) load_act<4>(a.d_x, (size_t)row * D + (i * THREADS + tid) * 4, false, x[i]);
        if (a.d_y) {
            const float gate = add_gate(a, row);
#pragma unroll
            for (int i = 0; i < N; ++i)
                if (in[i]) load_y<4>(a, row, (i * THREADS + tid) * 4, gate, r[i]);
            float inv[N];
            group_norm(0, inv);
#pragma unroll
            for (int i = 0; i < N; ++i)
                if (in[i]) {
                    float g[4];
                    load_act<4>(a.d_gamma_out, (i * THREADS + tid) * 4, false, g);
#pragma unroll
                    for (int e = 0; e < 4; ++e) r[i][e] = fmaf(a.mult, r[i][e] * inv[i] * g[e], x[i][e]);
                }
        } else {
#pragma unroll
            for (int i = 0; i < N; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) r[i][e] = x[i][e];
        }
    }
    if (a.d_weights) {
        const float w_own = __ldg(a.d_weights + a.n_states);
#pragma unroll
        for (int i = 0; i < N; ++i) {
            if (!in[i]) continue;
            const size_t at = (size_t)row * D + (i * THREADS + tid) * 4;
            if (!a.d_rows) store_act<4>(a.d_states, (size_t)a.n_states * a.state_stride + at, false, r[i]);
#pragma unroll
            for (int e = 0; e < 4; ++e) r[i][e] *= w_own;
        }
#pragma unroll 4
        for (int j = 0; j < (int)a.n_states; ++j) {
            const float w = __ldg(a.d_weights + j);
#pragma unroll
            for (int i = 0; i < N; ++i) {
                if (!in[i]) continue;
                float v[4];
                load_act<4>(a.d_states, (size_t)j * a.state_stride + (size_t)row * D + (i * THREADS + tid) * 4, false, v);
#pragma unroll
                for (int e = 0; e < 4; ++e) r[i][e] = fmaf(w, v[e], r[i][e]);
            }
        }
    }
    if (a.d_x_out && !a.d_rows)
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (in[i]) store_act<4>(a.d_x_out, (size_t)row * D + (i * THREADS + tid) * 4, false, r[i]);
    if (!a.d_h) return;
    const bool h_bf16 = a.h_dtype == GPTRS_BF16;
    if (a.d_gamma_in) {
        float inv[N];
        group_norm(1, inv);
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (in[i]) {
                float g[4];
                load_act<4>(a.d_gamma_in, (i * THREADS + tid) * 4, false, g);
#pragma unroll
                for (int e = 0; e < 4; ++e) r[i][e] *= inv[i] * g[e];
            }
    }
#pragma unroll
    for (int i = 0; i < N; ++i)
        if (in[i]) store_act<4>(a.d_h, (size_t)blockIdx.x * a.ldh + (i * THREADS + tid) * 4, h_bf16, r[i]);
    for (int c = D + tid; c < (int)a.ldh; c += THREADS) {
        const float z[1] = {0.f};
        store_act<1>(a.d_h, (size_t)blockIdx.x * a.ldh + c, h_bf16, z);
    }
}

// Any width and any groups: the row lies in shared memory.
constexpr int kAnyThreads = 256;
__global__ void __launch_bounds__(kAnyThreads) depth_step_any_kernel(const Params p) {
    extern __shared__ float ds_row[];   // [dim], then [groups]
    const gptrs_depth_step& a = p.s;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, D = (int)a.dim, size = D / a.groups;
    float* inv = ds_row + D;
    pdl_launch_dependents();
    pdl_wait();
    const int row = a.d_rows ? a.d_rows[blockIdx.x] : (int)blockIdx.x;
    auto group_norm = [&]() {   // a warp per group
        __syncthreads();
        for (int g = warp; g < a.groups; g += kAnyThreads / 32) {
            float ss = 0.f;
            for (int c = lane; c < size; c += 32) { const float v = ds_row[g * size + c]; ss = fmaf(v, v, ss); }
            ss = warp_sum(ss);
            if (lane == 0) inv[g] = 1.f / sqrtf(ss / (float)size + a.eps);
        }
        __syncthreads();
    };
    int id = 0;
    if (a.d_embed) {
        id = a.d_tokens[row];
        if (id < 0 || id >= a.vocab) { if (tid == 0) atomicExch(a.d_status, 2); id = 0; }
    }
    const bool add = !a.d_embed && a.d_y;
    const float gate = add ? add_gate(a, row) : 1.f;
    for (int c = tid; c < D; c += kAnyThreads) {
        float v[1];
        if (a.d_embed) v[0] = a.d_embed[(size_t)id * D + c];
        else if (add) load_y<1>(a, row, c, gate, v);
        else v[0] = a.d_x[(size_t)row * D + c];
        ds_row[c] = v[0];
    }
    if (add) group_norm();
    for (int c = tid; c < D; c += kAnyThreads) {   // every thread goes on with the columns that it has written
        const size_t at = (size_t)row * D + c;
        float r = ds_row[c];
        if (add) r = fmaf(a.mult, r * inv[c / size] * a.d_gamma_out[c], a.d_x[at]);
        if (a.d_weights) {
            if (!a.d_rows) a.d_states[(size_t)a.n_states * a.state_stride + at] = r;
            r *= __ldg(a.d_weights + a.n_states);
            for (int j = 0; j < (int)a.n_states; ++j) r = fmaf(__ldg(a.d_weights + j), a.d_states[(size_t)j * a.state_stride + at], r);
        }
        if (a.d_x_out && !a.d_rows) a.d_x_out[at] = r;
        ds_row[c] = r;
    }
    if (!a.d_h) return;
    if (a.d_gamma_in) group_norm();
    for (int c = tid; c < (int)a.ldh; c += kAnyThreads) {
        const float h[1] = {c < D ? (a.d_gamma_in ? ds_row[c] * inv[c / size] * a.d_gamma_in[c] : ds_row[c]) : 0.f};
        store_act<1>(a.d_h, (size_t)blockIdx.x * a.ldh + c, a.h_dtype == GPTRS_BF16, h);
    }
}

// ---- polynomial of normed powers -------------------------------------------------------------------------------------------------
struct PolyParams {
    const void* z;
    const float* act;
    void* y;
    float eps;
    int bf16, n, ld;
};
// Sums of z^2, z^4, z^6 over the CTA -> act[i] / sqrt(mean + eps); the first warp adds up what the warps have.
template <int THREADS>
__device__ __forceinline__ float3 power_scales(const PolyParams& p, float s2, float s4, float s6, float (*sh)[3], float* scale) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    s2 = warp_sum(s2); s4 = warp_sum(s4); s6 = warp_sum(s6);
    if (lane == 0) { sh[warp][0] = s2; sh[warp][1] = s4; sh[warp][2] = s6; }
    __syncthreads();
    if (threadIdx.x < 3) {
        float t = 0.f;
#pragma unroll
        for (int w = 0; w < THREADS / 32; ++w) t += sh[w][lane];
        scale[lane] = p.act[lane] / sqrtf(t / (float)p.n + p.eps);
    }
    __syncthreads();
    return make_float3(scale[0], scale[1], scale[2]);
}

// A thread holds the columns (i * THREADS + tid) * 8 + e, i < N, of a row whose length in memory is a multiple of 8.
template <bool BF16>
__device__ __forceinline__ void load8(const void* base, size_t i, float (&v)[8]) {
    if constexpr (BF16) {
        const uint4 u = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(base) + i);
        v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y);
        v[4] = bf16_lo(u.z); v[5] = bf16_hi(u.z); v[6] = bf16_lo(u.w); v[7] = bf16_hi(u.w);
    } else {
        const float4* q = reinterpret_cast<const float4*>(static_cast<const float*>(base) + i);
        const float4 a = q[0], b = q[1];
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
}
template <int THREADS, int N, bool BF16>
__global__ void __launch_bounds__(THREADS) poly_norm_kernel(const PolyParams p) {
    __shared__ float sh[THREADS / 32][3], scale[3];
    const int tid = threadIdx.x;
    const size_t base = (size_t)blockIdx.x * p.ld;
    pdl_launch_dependents();
    const float shift = __ldg(p.act + 3);
    pdl_wait();
    float z[N][8], s2 = 0.f, s4 = 0.f, s6 = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int c = (i * THREADS + tid) * 8;
        if (c < p.n) load8<BF16>(p.z, base + c, z[i]);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int left = p.n - (i * THREADS + tid) * 8;
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            if (e >= left) z[i][e] = 0.f;
            const float q = z[i][e] * z[i][e], f = q * q;
            s2 += q; s4 = fmaf(q, q, s4); s6 = fmaf(f, q, s6);
        }
    }
    const float3 k = power_scales<THREADS>(p, s2, s4, s6, sh, scale);
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int c = (i * THREADS + tid) * 8, left = p.n - c;
        if (c >= p.ld) continue;
        float y[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] = e < left ? fmaf(z[i][e], fmaf(z[i][e], fmaf(z[i][e], k.z, k.y), k.x), shift) : 0.f;
        if constexpr (BF16) {
            *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.y) + base + c) = make_uint4(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]), pack_bf16x2(y[4], y[5]), pack_bf16x2(y[6], y[7]));
        } else {
            float4* d = reinterpret_cast<float4*>(static_cast<float*>(p.y) + base + c);
            d[0] = make_float4(y[0], y[1], y[2], y[3]); d[1] = make_float4(y[4], y[5], y[6], y[7]);
        }
    }
}
template <int THREADS, int N>
int launch_poly(const PolyParams& p, dim3 grid, cudaStream_t st) {
    return p.bf16 ? launch_kernel(poly_norm_kernel<THREADS, N, true>, grid, dim3(THREADS), 0, st, 1, p) : launch_kernel(poly_norm_kernel<THREADS, N, false>, grid, dim3(THREADS), 0, st, 1, p);
}

__global__ void __launch_bounds__(kAnyThreads) poly_norm_any_kernel(const PolyParams p) {
    __shared__ float sh[kAnyThreads / 32][3], scale[3];
    const int tid = threadIdx.x;
    const size_t base = (size_t)blockIdx.x * p.ld;
    pdl_launch_dependents();
    pdl_wait();
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    for (int c = tid; c < p.n; c += kAnyThreads) {
        float z[1];
        load_act<1>(p.z, base + c, p.bf16, z);
        const float q = z[0] * z[0], f = q * q;
        s2 += q; s4 += f; s6 = fmaf(f, q, s6);
    }
    const float3 k = power_scales<kAnyThreads>(p, s2, s4, s6, sh, scale);
    for (int c = tid; c < p.ld; c += kAnyThreads) {   // the columns that this thread has read
        float z[1] = {0.f}, y[1] = {0.f};
        if (c < p.n) {
            load_act<1>(p.z, base + c, p.bf16, z);
            y[0] = fmaf(z[0], fmaf(z[0], fmaf(z[0], k.z, k.y), k.x), p.act[3]);
        }
        store_act<1>(p.y, base + c, p.bf16, y);
    }
}

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" {

int gptrs_cuda_depth_step(const gptrs_depth_step* step, void* stream) {
    GPTRS_REQUIRE(step, "null pointer");
    const gptrs_depth_step& a = *step;
    GPTRS_REQUIRE(a.rows >= 0 && a.rows < (1ll << 31) && a.dim > 0 && a.groups > 0 && a.dim % a.groups == 0, "bad shape: a row must hold a whole number of equal groups");
    GPTRS_REQUIRE(a.d_embed ? a.d_tokens && a.d_status && !a.d_rows && !a.d_y : a.d_x != nullptr, "embedding: token ids, status, no sublayer output; otherwise a stream");
    GPTRS_REQUIRE(!a.d_y || (a.d_gamma_out && (!a.d_pair || (a.d_pair_weight && a.top > 0))), "null pointer");
    GPTRS_REQUIRE(!a.d_add || a.d_y, "a second output belongs to a first one");
    GPTRS_REQUIRE(!a.d_weights || (a.d_states && a.n_states >= 0 && a.state_stride >= 0), "average over depth: states");
    GPTRS_REQUIRE(!a.d_h || a.ldh >= a.dim, "rows of the next input are too short");
    GPTRS_REQUIRE(!a.d_gamma_in || a.d_h, "norm of the next input: output");
    GPTRS_REQUIRE((!a.d_y || a.y_dtype == GPTRS_F32 || a.y_dtype == GPTRS_BF16) && (!a.d_h || a.h_dtype == GPTRS_F32 || a.h_dtype == GPTRS_BF16), "f32 or bf16");
    if (a.rows == 0) return GPTRS_OK;
    const Params p = {a};
    const bool vec = (a.dim / a.groups) % 128 == 0 && (!a.d_y || a.ldy % 4 == 0) && (!a.d_add || a.ld_add % 4 == 0) && (!a.d_h || a.ldh % 4 == 0) && a.state_stride % 4 == 0;
    const dim3 grid((unsigned)a.rows);
    cudaStream_t st = as_stream(stream);
    if (vec) {
        if (a.dim <= 512) return launch_kernel(depth_step_kernel<128, 1>, grid, dim3(128), 0, st, 1, p);
        if (a.dim <= 1024) return launch_kernel(depth_step_kernel<256, 1>, grid, dim3(256), 0, st, 1, p);
        if (a.dim <= 2048) return launch_kernel(depth_step_kernel<512, 1>, grid, dim3(512), 0, st, 1, p);
        if (a.dim <= 4096) return launch_kernel(depth_step_kernel<512, 2>, grid, dim3(512), 0, st, 1, p);
        if (a.dim <= 8192) return launch_kernel(depth_step_kernel<512, 4>, grid, dim3(512), 0, st, 1, p);
    }
    const size_t smem = (size_t)(a.dim + a.groups) * 4;
    if (smem > 200 * 1024) return fail(GPTRS_UNIMPLEMENTED, "depth step: rows of more than 51200 values and groups");
    if (smem > 40 * 1024) GPTRS_CUDA_OK(cudaFuncSetAttribute(depth_step_any_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return launch_kernel(depth_step_any_kernel, grid, dim3(kAnyThreads), smem, st, 1, p);
}

int gptrs_cuda_poly_norm(const void* d_z, const float* d_act, float eps, void* d_y, int dtype, int64_t rows, int64_t n, int64_t ld, void* stream) {
    GPTRS_REQUIRE(d_z && d_act && d_y, "null pointer");
    GPTRS_REQUIRE(rows >= 0 && rows < (1ll << 31) && n > 0 && ld >= n && ld < (1ll << 31), "bad shape");
    GPTRS_REQUIRE(dtype == GPTRS_F32 || dtype == GPTRS_BF16, "f32 or bf16");
    if (rows == 0) return GPTRS_OK;
    const PolyParams p = {d_z, d_act, d_y, eps, dtype == GPTRS_BF16, (int)n, (int)ld};
    const dim3 grid((unsigned)rows);
    cudaStream_t st = as_stream(stream);
    if (ld % 8 == 0) {
        if (ld <= 1024) return launch_poly<128, 1>(p, grid, st);
        if (ld <= 2048) return launch_poly<128, 2>(p, grid, st);
        if (ld <= 3072) return launch_poly<128, 3>(p, grid, st);
        if (ld <= 4096) return launch_poly<256, 2>(p, grid, st);
        if (ld <= 6144) return launch_poly<256, 3>(p, grid, st);
        if (ld <= 9216) return launch_poly<384, 3>(p, grid, st);
        if (ld <= 12288) return launch_poly<512, 3>(p, grid, st);
        if (ld <= 16384) return launch_poly<512, 4>(p, grid, st);
    }
    return launch_kernel(poly_norm_any_kernel, grid, dim3(kAnyThreads), 0, st, 1, p);
}

}  // extern "C"
