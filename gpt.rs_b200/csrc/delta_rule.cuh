// Shared by the two files of the gated delta rule (delta_rule.cu, delta_prepare.cu): geometry, the scratch of a prompt's blocks, and what turns a
// projection into decays and gates.
#pragma once
#include "umma_common.cuh"

namespace gptrs {
namespace delta {

struct Geo {
    int heads, kv_heads, group, dim, vdim, taps;
    int q_off, k_off, v_off, beta_off, row, decay_row, gate_row, out_stride, channels;
    int dp, vp;              // dim and vdim of the f32 planes, multiples of 4
    float eps, q_scale;
    int head_decay, a_off, gate_silu;   // one decay per head: column a_off + head of the projection row
};
__host__ __device__ inline int pad4(int v) { return (v + 3) / 4 * 4; }
inline Geo geo(const gptrs_delta_rule& a) {
    Geo g = {a.heads, a.kv_heads, a.heads / a.kv_heads, a.dim, a.vdim, a.taps, a.q_offset, a.k_offset, a.v_offset, a.beta_offset, a.row, a.decay_row, a.gate_row,
             a.out_head_stride, a.conv_channels, pad4(a.dim), pad4(a.vdim), a.eps, 1.f / sqrtf((float)a.dim), a.decay_rank == 0, a.a_offset, a.gate_silu};
    return g;
}
constexpr int kBlock = 4;        // tokens of a block
// per block, head and key channel: p_t k_t (4), p_t q_t (4), c_t (4), p_3; HEAD: k_t (4), q_t (4)
__host__ __device__ constexpr int vecs_of(bool head_decay) { return head_decay ? 8 : 13; }
// per block and head: beta (4), A10 A20 A21 A30 A31 A32 (+ 2), B00 B10 B11 B20 B21 B22 B30 .. B33 (+ 2); HEAD: p_t (4), decays of t+1 .. 3 (4)
__host__ __device__ constexpr int nums_of(bool head_decay) { return head_decay ? 32 : 24; }
// Scratch of a prompt's blocks: vectors [block][head][vecs][dp], values [block][head][4][vp], numbers [block][head][nums]; then the
// read-outs [row][head][vp]. Run i with first row r keeps its blocks from number r / 4 + i on.
struct Planes { float *vec, *v, *num, *o; };
inline int64_t block_floats(const Geo& g) { return (int64_t)g.heads * (vecs_of(g.head_decay) * g.dp + kBlock * g.vp + nums_of(g.head_decay)); }
inline int64_t max_blocks(int64_t rows, int64_t runs) { return rows / kBlock + runs; }
inline Planes planes(const Geo& g, float* s, int64_t rows, int64_t runs) {
    const int64_t n = max_blocks(rows, runs);
    Planes p;
    p.vec = s; s += n * g.heads * vecs_of(g.head_decay) * g.dp;
    p.v = s; s += n * g.heads * kBlock * g.vp;
    p.num = s; s += n * g.heads * nums_of(g.head_decay);
    p.o = s;
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
// silu of a convolution that is rounded to bf16 anyway; exp(rate softplus(x)) with the hardware's exponential and logarithm, the latter
// as the series of ln(1 + e) where 1 + e would lose e
__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.f + __expf(-x)); }
__device__ __forceinline__ float decay_fast(float x, float rate) {
    const float e = __expf(-fabsf(x));
    const float series = e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 1.f / 3.f), -0.5f), 1.f);
    return __expf(rate * (fmaxf(x, 0.f) + (e < 0.02f ? series : __logf(1.f + e))));
}
// what the softplus of a decay takes, without its bias; the bias
template <typename T>
__device__ __forceinline__ float decay_input(const Params& p, int row, int head, int d) {
    return p.g.head_decay ? ld(static_cast<const T*>(p.s.d_proj) + (size_t)row * p.g.row + p.g.a_off + head) : p.s.d_decay[(size_t)row * p.g.decay_row + head * p.g.dim + d];
}
__device__ __forceinline__ float decay_bias(const Params& p, int head, int d) { return p.s.d_dt_bias[p.g.head_decay ? head : head * p.g.dim + d]; }
template <typename T>
__device__ __forceinline__ float decay_of(const Params& p, int row, int head, int d) {
    return expf(-expf(p.s.d_a_log[head]) * softplus(decay_input<T>(p, row, head, d) + decay_bias(p, head, d)));
}
__device__ __forceinline__ float gate_of(const Geo& g, float z) { return g.gate_silu ? silu(z) : sigmoid(z); }

// delta_prepare.cu: the vectors, values and numbers of all blocks of a prompt's rows
int launch_prepare(const Params& p, bool bf16, cudaStream_t s);

}  // namespace delta
}  // namespace gptrs
