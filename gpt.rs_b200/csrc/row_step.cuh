// Pieces of the kernels that run between two sublayers with a CTA per row (norm_step.cu, stream_step.cu): the sum over a row and the
// loads and stores of f32 or bf16 rows.
#pragma once
#include "common.cuh"

namespace gptrs {
namespace {

template <int THREADS>
__device__ __forceinline__ float row_sum(float v, float* sh) {
    v = warp_sum(v);
    if constexpr (THREADS == 32) return v;
    __syncthreads();
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) s += sh[w];
    return s;
}

template <int VEC>
__device__ __forceinline__ void load_act(const void* base, size_t i, bool bf16, float (&v)[VEC]) {
    if (bf16) {
        const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(base) + i;
        if constexpr (VEC == 4) {
            const uint2 u = *reinterpret_cast<const uint2*>(p);
            v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y);
        } else {
            v[0] = __bfloat162float(*p);
        }
    } else {
        const float* p = static_cast<const float*>(base) + i;
        if constexpr (VEC == 4) {
            const float4 a = *reinterpret_cast<const float4*>(p);
            v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
        } else {
            v[0] = *p;
        }
    }
}
template <int VEC>
__device__ __forceinline__ void store_act(void* base, size_t i, bool bf16, const float (&v)[VEC]) {
    if (bf16) {
        __nv_bfloat16* p = static_cast<__nv_bfloat16*>(base) + i;
        if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
        else *p = __float2bfloat16_rn(v[0]);
    } else {
        float* p = static_cast<float*>(base) + i;
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        else *p = v[0];
    }
}

}  // namespace
}  // namespace gptrs
