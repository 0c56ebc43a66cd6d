// Mixture of experts: which experts a row goes to, and the order of rows in which the grouped matmuls (dense_bf16.cu, dense_f32.cu)
// find every expert's rows next to one another (no counterpart in gpt.rs).
//   moe_choose_kernel   a warp per row: softmax or sigmoid scores, best groups, best experts of those; counts per expert
//   moe_plan            row offsets of the experts and the tile list of the grouped matmuls; with few rows the tail of the kernel above,
//                       otherwise a kernel of its own
//   moe_gather_kernel   copies every row to its places
// Where a row lies among its expert's rows depends on the order of atomic additions; no value depends on it.
#include "common.cuh"

namespace gptrs {
namespace {

struct Params {
    gptrs_moe a;
    const float* logits;
    const float* correction;              // added to the scores that choose, or null
    int64_t ld;
    const unsigned char* h;
    unsigned char* sorted;
    int row_bytes;
    int* pair;
    float* weight;
    gptrs_row_tile* tiles;
    int* n_tiles;
    int *counts, *offsets, *id, *place;   // [kMaxExperts] each, [rows][top] each
    int rows, per_cta;
};
constexpr int kMaxExperts = 1024;
constexpr int kWarps = 32;

// order-preserving map of floats to signed integers
__device__ __forceinline__ int order_of(float v) {
    const int b = __float_as_int(v);
    return b ^ ((b >> 31) & 0x7fffffff);
}

__device__ __forceinline__ float value_of(int order) { return __int_as_float(order ^ ((order >> 31) & 0x7fffffff)); }

// inclusive sum over the 1024 threads of a CTA
__device__ __forceinline__ int cta_scan(int v, int* sh) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const int u = __shfl_up_sync(0xffffffffu, v, o); if (lane >= o) v += u; }
    __syncthreads();
    if (lane == 31) sh[warp] = v;
    __syncthreads();
    if (warp == 0) {
        int w = sh[lane];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const int u = __shfl_up_sync(0xffffffffu, w, o); if (lane >= o) w += u; }
        sh[lane] = w;
    }
    __syncthreads();
    return v + (warp > 0 ? sh[warp - 1] : 0);
}

__device__ __forceinline__ void moe_plan(const Params& p, int* sh) {
    const int e = threadIdx.x;
    const int n = e < p.a.experts ? p.counts[e] : 0, nt = (n + p.a.tile_rows - 1) / p.a.tile_rows;
    const int end = cta_scan(n, sh), t_end = cta_scan(nt, sh);
    if (e < p.a.experts) {
        const int r0 = end - n;
        p.offsets[e] = r0;
        p.counts[e] = 0;   // for the next call
        for (int t = 0; t < nt; ++t) {
            const gptrs_row_tile tile = {e, r0 + t * p.a.tile_rows, min(p.a.tile_rows, n - t * p.a.tile_rows), 0};
            p.tiles[t_end - nt + t] = tile;
        }
    }
    if (e == kWarps * 32 - 1) *p.n_tiles = t_end;
}

template <int VPL, bool SIGMOID>
__global__ void __launch_bounds__(kWarps * 32) moe_choose_kernel(const Params p) {
    __shared__ int hist[kMaxExperts], sh[32];
    extern __shared__ int mc_groups[];   // [warps][groups]: best score of every group, then whether it takes part
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int E = p.a.experts, G = p.a.groups, size = E / G;
    int* gm = mc_groups + warp * G;
    pdl_launch_dependents();
    pdl_wait();
    for (int e = tid; e < E; e += kWarps * 32) hist[e] = 0;
    __syncthreads();
    const int r_lo = blockIdx.x * p.per_cta, r_hi = min(r_lo + p.per_cta, p.rows);
    for (int row = r_lo + warp; row < r_hi; row += kWarps) {
        constexpr int kNone = (int)0x80000000;
        float z[VPL];
        int key[VPL];   // order of what chooses; kNone: not to be chosen (any more)
        float mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < VPL; ++i) {
            const int e = i * 32 + lane;
            z[i] = e < E ? p.logits[(size_t)row * p.ld + e] : -INFINITY;
            mx = fmaxf(mx, z[i]);
        }
        mx = warp_max(mx);
        float sum = 0.f;
        if (SIGMOID) {
#pragma unroll
            for (int i = 0; i < VPL; ++i) z[i] = 1.f / (1.f + expf(-z[i]));
        } else {
#pragma unroll
            for (int i = 0; i < VPL; ++i) {
                const float w = i * 32 + lane < E ? expf(z[i] - mx) : 0.f;
                sum += w;
                if (p.correction) z[i] = w;   // scores choose in the same order as logits; a correction needs the scores themselves
            }
            sum = warp_sum(sum);
            if (p.correction)
#pragma unroll
                for (int i = 0; i < VPL; ++i) z[i] /= sum;
        }
#pragma unroll
        for (int i = 0; i < VPL; ++i) {
            const int e = i * 32 + lane;
            if (p.correction && e < E) z[i] += __ldg(p.correction + e);
            key[i] = e < E ? max(order_of(z[i]), kNone + 1) : kNone;
        }
        // largest key of `v` and the lowest index that has it
        auto best_of = [&](int v, int index, int* at) {
            const int best = __reduce_max_sync(0xffffffffu, v);
            *at = __reduce_min_sync(0xffffffffu, v == best ? index : 0x7fffffff);
            return best;
        };
        if (p.a.keep < G) {
            if (p.a.group_best == 2) {   // the sum of a group's two best
                for (int g = 0; g < G; ++g) {
                    const int e0 = g * size;
                    int best = kNone, index = 0x7fffffff, second = kNone, at, at2;
#pragma unroll
                    for (int i = 0; i < VPL; ++i) {
                        const int e = i * 32 + lane;
                        if (e < e0 || e >= e0 + size) continue;
                        if (key[i] > best) { second = best; best = key[i]; index = e; }
                        else if (key[i] > second) second = key[i];
                    }
                    const int first = best_of(best, index, &at);
                    const int next = best_of(index == at ? second : best, lane, &at2);
                    if (lane == 0) gm[g] = min(order_of(value_of(first) + (size > 1 ? value_of(next) : 0.f)), 0x7ffffffe);
                }
            } else {
                for (int g = lane; g < G; g += 32) gm[g] = kNone;
                __syncwarp();
#pragma unroll
                for (int i = 0; i < VPL; ++i)
                    if (i * 32 + lane < E) atomicMax(gm + (i * 32 + lane) / size, key[i]);
            }
            __syncwarp();
            for (int n = 0; n < p.a.keep; ++n) {
                int best = kNone, index = 0x7fffffff, at;
                for (int g = lane; g < G; g += 32)
                    if (gm[g] != 0x7fffffff && gm[g] > best) { best = gm[g]; index = g; }
                best_of(best, index, &at);
                __syncwarp();
                if (lane == 0 && at < G) gm[at] = 0x7fffffff;   // taken
                __syncwarp();
            }
#pragma unroll
            for (int i = 0; i < VPL; ++i)
                if (i * 32 + lane < E && gm[(i * 32 + lane) / size] != 0x7fffffff) key[i] = kNone;
            __syncwarp();
        }
        int mine = 0, chosen = 0;   // lane k: the k-th choice (of the current 32)
        float total = 0.f;          // this lane's scores
        for (int k = 0; k < p.a.top; ++k) {
            int best = kNone, index = 0x7fffffff, at;
#pragma unroll
            for (int i = 0; i < VPL; ++i)
                if (key[i] > best) { best = key[i]; index = i * 32 + lane; }
            best = best_of(best, index, &at);
            if (at >= E) at = 0;   // only where logits are not numbers
#pragma unroll
            for (int i = 0; i < VPL; ++i)
                if (i * 32 + lane == at) key[i] = kNone;
            if (lane == (k & 31)) { mine = best; chosen = at; }
            if ((k & 31) == 31 || k + 1 == p.a.top) {
                const int k0 = k & ~31;
                if (lane <= k - k0) {
                    const size_t o = (size_t)row * p.a.top + k0 + lane;
                    float w;
                    if (SIGMOID) w = 1.f / (1.f + expf(-p.logits[(size_t)row * p.ld + chosen]));
                    else w = expf((p.correction ? p.logits[(size_t)row * p.ld + chosen] : value_of(mine)) - mx) / sum;
                    total += w;
                    p.weight[o] = w;
                    p.id[o] = chosen;
                    p.place[o] = atomicAdd(hist + chosen, 1);
                }
            }
        }
        if (p.a.weight_scale > 0.f) {   // in proportion; every lane changes what it has written itself
            const float f = p.a.weight_scale / (warp_sum(total) + 1e-20f);
            for (int k = lane; k < p.a.top; k += 32) p.weight[(size_t)row * p.a.top + k] *= f;
        }
    }
    __syncthreads();
    if (gridDim.x == 1) {   // few rows: this CTA has seen them all
        for (int e = tid; e < E; e += kWarps * 32) p.counts[e] = hist[e];
        __syncthreads();
        moe_plan(p, sh);
        return;
    }
    for (int e = tid; e < E; e += kWarps * 32) hist[e] = hist[e] > 0 ? atomicAdd(p.counts + e, hist[e]) : 0;   // first place of this CTA's rows
    __syncthreads();
    for (int i = r_lo * p.a.top + tid; i < r_hi * p.a.top; i += kWarps * 32) p.place[i] += hist[p.id[i]];
}

__global__ void __launch_bounds__(kWarps * 32) moe_plan_kernel(const Params p) {
    __shared__ int sh[32];
    pdl_launch_dependents();
    pdl_wait();
    moe_plan(p, sh);
}

// a CTA per (row, k)
__global__ void __launch_bounds__(128) moe_gather_kernel(const Params p) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x, k = blockIdx.y;
    const size_t o = (size_t)row * p.a.top + k;
    const int dst = p.offsets[p.id[o]] + p.place[o];
    if (threadIdx.x == 0) p.pair[o] = dst;
    const unsigned char* s = p.h + (size_t)row * p.row_bytes;
    unsigned char* d = p.sorted + (size_t)dst * p.row_bytes;
    if (p.row_bytes % 16 == 0)
        for (int i = threadIdx.x * 16; i < p.row_bytes; i += 128 * 16) *reinterpret_cast<uint4*>(d + i) = *reinterpret_cast<const uint4*>(s + i);
    else
        for (int i = threadIdx.x * 4; i < p.row_bytes; i += 128 * 4) *reinterpret_cast<uint32_t*>(d + i) = *reinterpret_cast<const uint32_t*>(s + i);
}

struct PairParams { const float* x; float* y; int n, gate; };
__global__ void __launch_bounds__(128) gated_pairs_kernel(const PairParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const float* x = p.x + (size_t)blockIdx.x * 2 * p.n;
    for (int i = threadIdx.x; i < p.n; i += 128) {
        const int c = (i >> 3) * 16 + (i & 7);
        const float g = x[c];
        const float a = p.gate == GPTRS_GATE_GELU_TANH ? 0.5f * g * (1.f + tanhf(0.7978845608028654f * fmaf(0.044715f * g * g, g, g))) : g / (1.f + expf(-g));
        p.y[(size_t)blockIdx.x * p.n + i] = a * x[c + 8];
    }
}

template <int VPL>
int launch_choose(const Params& p, int ctas, size_t smem, cudaStream_t st) {
    const auto kern = p.a.scores == GPTRS_ROUTE_SIGMOID ? moe_choose_kernel<VPL, true> : moe_choose_kernel<VPL, false>;
    if (smem > 40 * 1024) GPTRS_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return launch_kernel(kern, dim3((unsigned)ctas), dim3(kWarps * 32), smem, st, 1, p);
}

int check(const gptrs_moe* a) {
    GPTRS_REQUIRE(a && a->experts > 0 && a->top > 0 && a->groups > 0 && a->keep > 0 && a->tile_rows > 0, "experts: sizes must be positive");
    GPTRS_REQUIRE(a->experts % a->groups == 0 && a->keep <= a->groups && a->top <= a->keep * (a->experts / a->groups), "experts: groups must be equal and hold enough experts");
    GPTRS_REQUIRE((a->scores == GPTRS_ROUTE_SOFTMAX || a->scores == GPTRS_ROUTE_SIGMOID) && a->group_best >= 0 && a->group_best <= 2 && a->weight_scale >= 0.f,
                  "experts: scores, group score or weight scale");
    if (a->experts > kMaxExperts) return fail(GPTRS_UNIMPLEMENTED, "experts: more than 1024");
    return GPTRS_OK;
}

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" {

int64_t gptrs_cuda_moe_max_tiles(const gptrs_moe* a, int64_t rows) {
    if (!a || a->tile_rows < 1 || rows < 0) return 0;
    const int64_t pairs = rows * a->top;
    return (pairs < a->experts ? pairs : a->experts) + pairs / a->tile_rows;
}

int64_t gptrs_cuda_moe_work_ints(const gptrs_moe* a, int64_t rows) { return a ? 2 * (int64_t)kMaxExperts + 2 * rows * a->top : 0; }

int gptrs_cuda_moe_route(const gptrs_moe* a, const float* d_logits, int64_t ld, const float* d_correction, const void* d_h, int h_dtype, int64_t ldh, int32_t* d_pair, float* d_weight,
                         gptrs_row_tile* d_tiles, int32_t* d_n_tiles, void* d_sorted, int32_t* d_work, int64_t rows, void* stream) {
    int rc = check(a);
    if (rc) return rc;
    GPTRS_REQUIRE(d_logits && d_h && d_pair && d_weight && d_tiles && d_n_tiles && d_sorted && d_work, "null pointer");
    GPTRS_REQUIRE(ld >= a->experts && ldh > 0 && rows >= 0 && rows * a->top < (1ll << 30), "bad shape");
    GPTRS_REQUIRE(h_dtype == GPTRS_F32 || (h_dtype == GPTRS_BF16 && ldh % 2 == 0), "rows of f32, or of an even number of bf16");
    if (rows == 0) return GPTRS_OK;
    Params p = {};
    p.a = *a; p.logits = d_logits; p.ld = ld; p.correction = d_correction;
    p.h = static_cast<const unsigned char*>(d_h); p.sorted = static_cast<unsigned char*>(d_sorted);
    p.row_bytes = (int)(ldh * (h_dtype == GPTRS_F32 ? 4 : 2));
    p.pair = d_pair; p.weight = d_weight; p.tiles = d_tiles; p.n_tiles = d_n_tiles;
    // the same places for every number of experts: the counts stay zero in between
    p.counts = d_work; p.offsets = d_work + kMaxExperts; p.id = p.offsets + kMaxExperts; p.place = p.id + rows * a->top;
    p.rows = (int)rows;
    p.per_cta = rows <= 128 ? (int)rows : 64;
    const int ctas = ceil_div(rows, p.per_cta);
    cudaStream_t st = as_stream(stream);
    const size_t smem = (size_t)kWarps * a->groups * 4;
    const int vpl = ceil_div(a->experts, 32);
    if (vpl <= 1) rc = launch_choose<1>(p, ctas, smem, st);
    else if (vpl <= 2) rc = launch_choose<2>(p, ctas, smem, st);
    else if (vpl <= 4) rc = launch_choose<4>(p, ctas, smem, st);
    else if (vpl <= 8) rc = launch_choose<8>(p, ctas, smem, st);
    else rc = launch_choose<32>(p, ctas, smem, st);
    if (!rc && ctas > 1) rc = launch_kernel(moe_plan_kernel, dim3(1), dim3(kWarps * 32), 0, st, 1, p);
    if (rc) return rc;
    return launch_kernel(moe_gather_kernel, dim3((unsigned)rows, (unsigned)a->top), dim3(128), 0, st, 1, p);
}

int gptrs_cuda_gated_pairs_f32(const float* d_gate_up, float* d_y, int64_t rows, int64_t n, int gate, void* stream) {
    GPTRS_REQUIRE(d_gate_up && d_y, "null pointer");
    GPTRS_REQUIRE(rows >= 0 && rows < (1ll << 31) && n > 0 && n % 8 == 0 && n < (1ll << 30), "bad shape");
    if (rows == 0) return GPTRS_OK;
    GPTRS_REQUIRE(gate == GPTRS_GATE_SILU || gate == GPTRS_GATE_GELU_TANH, "unknown gate activation");
    const PairParams p = {d_gate_up, d_y, (int)n, gate};
    return launch_kernel(gated_pairs_kernel, dim3((unsigned)rows), dim3(128), 0, as_stream(stream), 1, p);
}

}  // extern "C"
