// Dense bf16 matmuls on the tcgen05 tensor cores: y[M][N] = act(x[M][K] . w[N][K]^T + bias), optionally batched over the
// heads of an attention layer (functional::matmul, crates/gpt-rs/src/ops/functional/linalg.rs:109-127, on bf16 weights).
// Both operands are K-major in memory and reach shared memory by TMA tensor copies with the 128-byte swizzle, K tails and rows
// past the end zero-filled by the copy engine. Two kernels share that plan:
//   dense_rows_kernel      more than 128 rows (prompts): persistent CTAs walk over 128 x BN output tiles, x rows are the M side
//                          of the MMA. Warp 5 requests stages, warp 4 issues the MMAs into one of two accumulators in tensor
//                          memory while warps 0-3 and 8-11 (thread = row, half of the columns) turn the other one into bias + activation + stores.
//   dense_channels_kernel  up to 128 rows (decode steps): 128 output channels are the M side, the rows the N side (16 .. 128);
//                          the weights of the first stages are requested before griddepcontrol.wait; K is split over a thread
//                          block cluster and the partial tiles meet in the owner's shared memory (matmul_common.cuh).
// Every wait is bounded: a timeout records code 3 in the caller's status word, tensor memory is freed, the kernel returns.
#include <cuda.h>

#include "matmul_common.cuh"
#include "umma_common.cuh"

namespace gptrs {
namespace {

constexpr int kBK = 64;              // bf16 per 128-byte swizzle span
constexpr int kTileM = 128;
constexpr int kATile = kTileM * 128; // bytes of a 128 x 64 operand tile

__device__ __forceinline__ void tmem_alloc(uint32_t* holder, uint32_t cols) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(smem_u32(holder)), "r"(cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
}
__device__ __forceinline__ void tmem_free(uint32_t tmem, uint32_t cols) {
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(cols) : "memory");
}

// ---- prompts -------------------------------------------------------------------------------------------------------------------
struct RowsParams {
    CUtensorMap x_map, w_map;
    void* y;
    const float* bias;
    int* status;
    DenseAct act;
    int gate;                    // GPTRS_GATE_*
    int M, N, K, batch, out_f32;
    int m_tiles, n_tiles;
    int x_step, w_rows;          // x columns between batches; weight rows between batches
    int64_t ldy, y_step;
    const gptrs_row_tile* tiles; // grouped form
    const int* n_row_tiles;
};

constexpr int kRowsThreads = 384;    // warps 0-3 and 8-11 epilogue, 4 MMA + tensor memory, 5 loader
// ACT: 0 none, 1 xIELU, 2 whatever p.act says (with a soft cap), 3 act(gate) partner (8 gates, then their 8 partners), 4 squared relu.
// GROUPED: the row tiles come from a list in device memory, each with the weight matrix that it meets.
template <int BN, int STAGES, int ACT, bool GROUPED = false>
__global__ void __launch_bounds__(kRowsThreads, 1) dense_rows_kernel(const __grid_constant__ RowsParams p) {
    constexpr int kStageBytes = kATile + BN * 128;
    constexpr uint32_t kCols = 2 * BN < 32 ? 32 : 2 * BN;
    constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kTileM >> 4) << 24);
    extern __shared__ unsigned char smem_raw[];
    __shared__ __align__(8) uint64_t full[STAGES], empty[STAGES], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_holder;
    unsigned char* smem = smem_raw + ((1024 - (smem_u32(smem_raw) & 1023)) & 1023);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (int s = 0; s < STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(&acc_full[i], 1); mbar_init(&acc_empty[i], 256); }
        mbar_fence_init();
    }
    if (warp == 4) tmem_alloc(&tmem_holder, kCols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_holder;
    pdl_launch_dependents();
    pdl_wait();
    const int n_k = (p.K + kBK - 1) / kBK;
    const int tiles = GROUPED ? *p.n_row_tiles * p.n_tiles : p.m_tiles * p.n_tiles * p.batch;
    bool failed = false;
    struct Tile { int m0, m_end, n0, b; };
    auto tile_of = [&](int t) {
        Tile r;
        if constexpr (GROUPED) {   // column tile fastest: the rows are read once, an expert's weights stay in L2 for its row tiles
            const gptrs_row_tile g = p.tiles[t / p.n_tiles];
            r = {g.row0, g.row0 + g.rows, (t % p.n_tiles) * BN, g.group};
        } else {                   // row tile fastest, so that the CTAs running at one time share weight tiles
            const int rest = t / p.m_tiles;
            r = {(t % p.m_tiles) * kTileM, p.M, (rest % p.n_tiles) * BN, rest / p.n_tiles};
        }
        return r;
    };
    auto wait = [&](uint64_t* bar, uint32_t parity) {
        if (!failed && !mbar_wait_relaxed(bar, parity)) failed = true;
        failed = __any_sync(0xffffffffu, failed);
        return !failed;
    };
    if (warp == 5) {
        int it = 0, last_it = 0;
        for (int t = blockIdx.x; t < tiles && !failed; t += gridDim.x) {
            const Tile tl = tile_of(t);
            const int m0 = tl.m0, n0 = tl.n0, b = tl.b;
            for (int k = 0; k < n_k; ++k, ++it) {
                const int s = it % STAGES;
                if (it >= STAGES && !wait(&empty[s], (uint32_t)(it / STAGES - 1) & 1u)) break;
                if (lane == 0) {
                    const uint32_t bar = smem_u32(&full[s]);
                    mbar_expect_tx_addr(bar, kStageBytes);
                    tma_load_2d(smem + s * kStageBytes, &p.x_map, (GROUPED ? 0 : b * p.x_step) + k * kBK, m0, bar);
                    tma_load_2d(smem + s * kStageBytes + kATile, &p.w_map, k * kBK, b * p.w_rows + n0, bar);
                }
                __syncwarp();
                last_it = it + 1;
            }
        }
        // stages in flight write this CTA's shared memory (only after a timeout are there any left unread)
        for (int i = max(last_it - STAGES, 0); i < last_it; ++i) mbar_wait_relaxed(&full[i % STAGES], (uint32_t)(i / STAGES) & 1u);
    } else if (warp == 4) {
        int it = 0, n = 0;
        for (int t = blockIdx.x; t < tiles && !failed; t += gridDim.x, ++n) {
            const int buf = n & 1;
            if (n >= 2 && !wait(&acc_empty[buf], (uint32_t)(n / 2 - 1) & 1u)) break;
            tc_fence_after();
            for (int k = 0; k < n_k; ++k, ++it) {
                const int s = it % STAGES;
                if (!wait(&full[s], (uint32_t)(it / STAGES) & 1u)) break;
                tc_fence_after();
                if (lane == 0) {
                    const uint64_t ad = make_smem_desc(smem_u32(smem + s * kStageBytes)), bd = make_smem_desc(smem_u32(smem + s * kStageBytes + kATile));
#pragma unroll
                    for (int k4 = 0; k4 < 4; ++k4) umma_bf16(tmem + (uint32_t)(buf * BN), ad + 2 * k4, bd + 2 * k4, kIdesc, (k > 0 || k4 > 0) ? 1u : 0u);
                    umma_commit(&empty[s]);
                    if (k == n_k - 1) umma_commit(&acc_full[buf]);
                }
                __syncwarp();
            }
        }
    } else if (warp < 4 || warp >= 8) {
        const int quarter = warp & 3, c_lo = warp < 4 ? 0 : BN / 2;   // lane quarter and half of the columns
        int n = 0;
        for (int t = blockIdx.x; t < tiles && !failed; t += gridDim.x, ++n) {
            const int buf = n & 1;
            const Tile tl = tile_of(t);
            const int m0 = tl.m0, n0 = tl.n0;
            if (!wait(&acc_full[buf], (uint32_t)(n / 2) & 1u)) break;
            tc_fence_after();
            const int m = m0 + quarter * 32 + lane;
            const int64_t row = (GROUPED ? 0 : tl.b * p.y_step) + (int64_t)m * p.ldy;
#pragma unroll 1
            for (int c0 = c_lo; c0 < c_lo + BN / 2 && n0 + c0 < p.N; c0 += 32) {
                float v[32];
                tmem_ld_32(tmem + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(buf * BN + c0), v);
                const int left = p.N - (n0 + c0);   // a multiple of 8
                if (p.bias) {
#pragma unroll
                    for (int i = 0; i < 8; ++i)
                        if (4 * i < left) {
                            const float4 bb = __ldg(reinterpret_cast<const float4*>(p.bias + n0 + c0) + i);
                            v[4 * i] += bb.x; v[4 * i + 1] += bb.y; v[4 * i + 2] += bb.z; v[4 * i + 3] += bb.w;
                        }
                }
                if constexpr (ACT == 1) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = dense_act<true>({1, p.act.pos, p.act.neg, 0.f}, v[i]);
                } else if constexpr (ACT == 2) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = dense_act<true>(p.act, v[i]);
                } else if constexpr (ACT == 4) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = dense_act<true>({2, 0.f, 0.f, 0.f}, v[i]);
                }
                if constexpr (ACT == 3) {
                    if (m < tl.m_end) {
                        float o[16];
                        if (p.gate == GPTRS_GATE_GELU_TANH) {
#pragma unroll
                            for (int i = 0; i < 16; ++i) o[i] = gelu_tanh_fast(v[(i >> 3) * 16 + (i & 7)]) * v[(i >> 3) * 16 + (i & 7) + 8];
                        } else {
#pragma unroll
                            for (int i = 0; i < 16; ++i) o[i] = silu_fast(v[(i >> 3) * 16 + (i & 7)]) * v[(i >> 3) * 16 + (i & 7) + 8];
                        }
                        uint4* dst = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.y) + row + ((n0 + c0) >> 1));
#pragma unroll
                        for (int i = 0; i < 2; ++i)
                            if (16 * i < left)
                                dst[i] = make_uint4(pack_bf16x2(o[8 * i], o[8 * i + 1]), pack_bf16x2(o[8 * i + 2], o[8 * i + 3]),
                                                    pack_bf16x2(o[8 * i + 4], o[8 * i + 5]), pack_bf16x2(o[8 * i + 6], o[8 * i + 7]));
                    }
                } else if (m < tl.m_end) {
                    if (p.out_f32) {
                        float4* dst = reinterpret_cast<float4*>(static_cast<float*>(p.y) + row + n0 + c0);
#pragma unroll
                        for (int i = 0; i < 8; ++i)
                            if (4 * i < left) dst[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
                    } else {
                        uint4* dst = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.y) + row + n0 + c0);
#pragma unroll
                        for (int i = 0; i < 4; ++i)
                            if (8 * i < left)
                                dst[i] = make_uint4(pack_bf16x2(v[8 * i], v[8 * i + 1]), pack_bf16x2(v[8 * i + 2], v[8 * i + 3]),
                                                    pack_bf16x2(v[8 * i + 4], v[8 * i + 5]), pack_bf16x2(v[8 * i + 6], v[8 * i + 7]));
                    }
                }
            }
            tc_fence_before();
            mbar_arrive(&acc_empty[buf]);
        }
    }
    if (failed && lane == 0) atomicExch(p.status, 3);
    tc_fence_before();
    __syncthreads();
    if (warp == 4) tmem_free(tmem, kCols);
}

// ---- decode steps --------------------------------------------------------------------------------------------------------------
struct ChannelsParams {
    CUtensorMap x_map, w_map;
    MatmulParams p;
    int batch_m_tiles;           // row tiles per batch entry (blockIdx.z = batch * row tiles + row tile)
    int x_step, w_rows;
    int64_t y_step;
    const gptrs_row_tile* tiles; // grouped form: blockIdx.z counts the row tiles of the list
    const int* n_row_tiles;
};
constexpr int kChThreads = 320;  // warps 0-7 epilogue, 8 loader, 9 MMA + tensor memory

template <int BN, int STAGES, bool GROUPED = false>
__global__ void __launch_bounds__(kChThreads, BN <= 64 ? 2 : 1) dense_channels_kernel(const __grid_constant__ ChannelsParams cp) {
    constexpr int kStageBytes = kATile + BN * 128;
    constexpr uint32_t kCols = BN < 32 ? 32 : BN;
    constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kTileM >> 4) << 24);
    static_assert(STAGES * kStageBytes >= (BN + 7) * kRedStride * 4, "the receive slots alias the stages");
    extern __shared__ unsigned char smem_raw[];
    __shared__ __align__(8) uint64_t full[STAGES], empty[STAGES], done;
    __shared__ uint32_t tmem_holder;
    unsigned char* smem = smem_raw + ((1024 - (smem_u32(smem_raw) & 1023)) & 1023);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    MatmulParams p = cp.p;
    int b = blockIdx.z / cp.batch_m_tiles, m0 = (blockIdx.z % cp.batch_m_tiles) * BN;
    const int n0 = blockIdx.x * kTileM;
    if constexpr (GROUPED) {   // which weights to read is a result of the kernels in front
        pdl_wait();
        if ((int)blockIdx.z >= *cp.n_row_tiles) return;   // the whole cluster
        const gptrs_row_tile t = cp.tiles[blockIdx.z];
        b = t.group; m0 = t.row0;
        p.M = t.row0 + t.rows;
    }
    SplitReduce sr;
    sr.begin(p, false);
    const int k_tiles = (p.K + kBK - 1) / kBK;
    const int k0 = (int)((int64_t)k_tiles * blockIdx.y / p.n_split), k1 = (int)((int64_t)k_tiles * (blockIdx.y + 1) / p.n_split);
    const int n_k = k1 - k0;
    if (warp == 8) {
        if (lane == 0) {
            for (int s = 0; s < STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
            mbar_init(&done, 1);
            mbar_fence_init();
            fence_proxy_async();
            // weights are constants: the first stages of them travel while the kernel in front still runs
            for (int i = 0; i < STAGES && i < n_k; ++i) {
                const uint32_t bar = smem_u32(&full[i]);
                mbar_expect_tx_addr(bar, kStageBytes);
                tma_load_2d(smem + i * kStageBytes, &cp.w_map, (k0 + i) * kBK, b * cp.w_rows + n0, bar);
            }
        }
        __syncwarp();
    }
    if (warp == 9) tmem_alloc(&tmem_holder, kCols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_holder;
    pdl_launch_dependents();   // every CTA of this grid holds its tensor memory before a dependent grid may start
    if constexpr (!GROUPED) pdl_wait();
    bool failed = false;
    if (warp == 8) {
        for (int it = 0; it < n_k; ++it) {
            const int s = it % STAGES;
            if (it >= STAGES && !mbar_wait_relaxed(&empty[s], (uint32_t)(it / STAGES - 1) & 1u)) { failed = true; break; }
            if (lane == 0) {
                const uint32_t bar = smem_u32(&full[s]);
                if (it >= STAGES) {
                    mbar_expect_tx_addr(bar, kStageBytes);
                    tma_load_2d(smem + s * kStageBytes, &cp.w_map, (k0 + it) * kBK, b * cp.w_rows + n0, bar);
                }
                tma_load_2d(smem + s * kStageBytes + kATile, &cp.x_map, (GROUPED ? 0 : b * cp.x_step) + (k0 + it) * kBK, m0, bar);
            }
            __syncwarp();
        }
        // copies in flight write this CTA's stages (only after a timeout are there any left unread)
        if (!failed)
            for (int it = max(n_k - STAGES, 0); it < n_k; ++it) mbar_wait_relaxed(&full[it % STAGES], (uint32_t)(it / STAGES) & 1u);
    } else if (warp == 9) {
        for (int it = 0; it < n_k; ++it) {
            const int s = it % STAGES;
            if (!mbar_wait_relaxed(&full[s], (uint32_t)(it / STAGES) & 1u)) { failed = true; break; }
            tc_fence_after();
            if (lane == 0) {
                const uint64_t ad = make_smem_desc(smem_u32(smem + s * kStageBytes)), bd = make_smem_desc(smem_u32(smem + s * kStageBytes + kATile));
#pragma unroll
                for (int k4 = 0; k4 < 4; ++k4) umma_bf16(tmem, ad + 2 * k4, bd + 2 * k4, kIdesc, (it > 0 || k4 > 0) ? 1u : 0u);
                umma_commit(&empty[s]);
            }
            __syncwarp();
        }
        if (lane == 0 && !failed) umma_commit(&done);
        __syncwarp();
    }
    // every thread sees the MMAs of its own CTA complete before the cluster may write into the stage buffers
    if (!mbar_wait_relaxed(&done, 0)) failed = true;
    tc_fence_after();
    sr.barrier_all_done();
    float* slots = reinterpret_cast<float*>(smem);
    sr.ready(slots, BN);
    if (warp < 8) {
        const int quarter = warp & 3, col = quarter * 32 + lane;
        constexpr int kHalves = BN >= 64 ? 2 : 1;
        constexpr int kSpan = BN / kHalves;
        if ((warp >> 2) < kHalves) {
#pragma unroll 1
            for (int c0 = (warp >> 2) * kSpan; c0 < ((warp >> 2) + 1) * kSpan; c0 += 32) {
                float v[32];
                tmem_ld_32(tmem + ((uint32_t)(quarter * 32) << 16) + (uint32_t)c0, v);
                int owner = c0 % sr.S, local_row = c0 / sr.S;
#pragma unroll
                for (int i = 0; i < (BN < 32 ? BN : 32); ++i) {
                    sr.push(owner, local_row, col, v[i]);
                    if (++owner == sr.S) { owner = 0; ++local_row; }
                }
            }
        }
    }
    if (failed && lane == 0) atomicExch(p.status, 3);
    tc_fence_before();
    __syncthreads();
    if (warp == 9) tmem_free(tmem, kCols);
    if constexpr (!GROUPED) {
        if (p.out_f32) p.y = static_cast<float*>(p.y) + b * cp.y_step;
        else p.y = static_cast<__nv_bfloat16*>(p.y) + b * cp.y_step;
    }
    split_reduce_finish<BN, true>(p, sr, slots, tid, kChThreads, m0, n0);
}

int encode(CUtensorMap* map, const void* base, int64_t cols, int64_t rows, int64_t ld, int box_rows) {
    EncodeTiledFn enc = encode_fn();
    if (!enc) return fail(GPTRS_EXECUTION, "cuTensorMapEncodeTiled is not available");
    cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    cuuint32_t box[2] = {kBK, (cuuint32_t)box_rows};
    cuuint32_t estr[2] = {1, 1};
    CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                     CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(GPTRS_EXECUTION, "cuTensorMapEncodeTiled failed for a dense matmul (" + std::to_string((int)r) + ")");
    return GPTRS_OK;
}

struct Call {
    const void *x, *w;
    void* y;
    int M, N, K, batch;
    int64_t ldx, ldy, x_step, y_step;
    const gptrs_dense_epilogue* ep;
};

template <int BN, int STAGES>
int launch_rows(const Call& c, cudaStream_t st) {
    RowsParams p = {};
    int rc = encode(&p.x_map, c.x, c.ldx, c.M, c.ldx, kTileM);
    if (!rc) rc = encode(&p.w_map, c.w, c.K, (int64_t)c.batch * c.N, c.K, BN);
    if (rc) return rc;
    p.y = c.y; p.bias = c.ep->d_bias; p.status = c.ep->d_status;
    p.act = {c.ep->act, c.ep->act_pos, c.ep->act_neg, c.ep->softcap};
    p.gate = c.ep->swiglu;
    p.M = c.M; p.N = c.N; p.K = c.K; p.batch = c.batch; p.out_f32 = c.ep->out_dtype == GPTRS_F32;
    p.m_tiles = ceil_div(c.M, kTileM); p.n_tiles = ceil_div(c.N, BN);
    p.x_step = (int)c.x_step; p.w_rows = c.N; p.ldy = c.ldy; p.y_step = c.y_step;
    p.tiles = c.ep->d_tiles; p.n_row_tiles = c.ep->d_n_tiles;
    const int64_t tiles = (p.tiles ? c.ep->max_tiles : (int64_t)p.m_tiles * p.batch) * p.n_tiles;
    constexpr size_t smem = (size_t)STAGES * (kATile + BN * 128) + 1024;
    void (*kerns[8])(RowsParams) = {dense_rows_kernel<BN, STAGES, 0>, dense_rows_kernel<BN, STAGES, 1>, dense_rows_kernel<BN, STAGES, 4>,
                                    dense_rows_kernel<BN, STAGES, 2>, dense_rows_kernel<BN, STAGES, 3>, dense_rows_kernel<BN, STAGES, 0, true>,
                                    dense_rows_kernel<BN, STAGES, 4, true>, dense_rows_kernel<BN, STAGES, 3, true>};
    static PerDeviceOnce attr_once;
    if (attr_once.first_time())
        for (auto k : kerns) GPTRS_CUDA_OK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const auto kern = kerns[p.tiles ? (c.ep->swiglu ? 7 : c.ep->act == 2 ? 6 : 5) : c.ep->swiglu ? 4 : c.ep->softcap > 0.f ? 3 : c.ep->act];
    return launch_kernel(kern, dim3((unsigned)(tiles < sm_count() ? tiles : sm_count())), dim3(kRowsThreads), smem, st, 1, p);
}

template <int BN, int STAGES>
int launch_channels(const Call& c, cudaStream_t st) {
    ChannelsParams cp = {};
    int rc = encode(&cp.x_map, c.x, c.ldx, c.M, c.ldx, BN);
    if (!rc) rc = encode(&cp.w_map, c.w, c.K, (int64_t)c.batch * c.N, c.K, kTileM);
    if (rc) return rc;
    MatmulParams& p = cp.p;
    p.y = c.y; p.bias = c.ep->d_bias; p.status = c.ep->d_status;
    p.M = c.M; p.N = c.N; p.K = c.K; p.out_f32 = c.ep->out_dtype == GPTRS_F32;
    p.act = {c.ep->act, c.ep->act_pos, c.ep->act_neg, c.ep->softcap};
    p.ldy = c.ldy;
    p.best_val = c.ep->d_best_val; p.best_idx = c.ep->d_best_idx; p.skip_store = c.ep->skip_store;
    cp.batch_m_tiles = ceil_div(c.M, BN);
    cp.tiles = c.ep->d_tiles; cp.n_row_tiles = c.ep->d_n_tiles;
    p.swiglu = c.ep->swiglu;
    const int64_t z = cp.tiles ? c.ep->max_tiles : (int64_t)cp.batch_m_tiles * c.batch;
    GPTRS_REQUIRE(z <= 65535, "dense bf16 matmul: too many row tiles in one launch");
    cp.x_step = (int)c.x_step; cp.w_rows = c.N; cp.y_step = c.y_step;
    const int n_tiles = ceil_div(c.N, kTileM), k_tiles = ceil_div(c.K, kBK);
    const int64_t ctas = (int64_t)n_tiles * z;
    // fill the SMs (two CTAs each up to 64 rows) with at least two stages of K per CTA; clusters above 4 pack badly once
    // most of the slots are taken
    const int64_t slots = (int64_t)sm_count() * (BN <= 64 ? 2 : 1);
    int64_t split = slots / ctas;
    if (split > k_tiles / 2) split = k_tiles / 2;
    if (split > 8) split = 8;
    while (split > 3 && ctas * split * 100 > slots * 85) --split;
    p.n_split = (int)(split < 1 ? 1 : split);
    constexpr size_t smem = (size_t)STAGES * (kATile + BN * 128) + 1024;
    void (*kerns[2])(ChannelsParams) = {dense_channels_kernel<BN, STAGES>, dense_channels_kernel<BN, STAGES, true>};
    static PerDeviceOnce attr_once;
    if (attr_once.first_time())
        for (auto k : kerns) GPTRS_CUDA_OK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return launch_kernel(kerns[cp.tiles ? 1 : 0], dim3((unsigned)n_tiles, (unsigned)p.n_split, (unsigned)z), dim3(kChThreads), smem, st, p.n_split, cp);
}

}  // namespace
}  // namespace gptrs

using namespace gptrs;

extern "C" int gptrs_cuda_dense_bf16(const void* d_x, const void* d_w, void* d_y, int64_t m, int64_t n, int64_t k, const gptrs_dense_epilogue* ep,
                                     void* stream) {
    GPTRS_REQUIRE(d_x && d_w && d_y && ep && ep->d_status, "null pointer");
    GPTRS_REQUIRE(m >= 0 && n > 0 && k > 0 && m < (1ll << 30) && n < (1ll << 30) && k < (1ll << 30), "bad shape");
    Call c = {d_x, d_w, d_y, (int)m, (int)n, (int)k, ep->batch > 1 ? (int)ep->batch : 1, ep->ldx ? ep->ldx : k, ep->ldy ? ep->ldy : n,
              ep->x_step, ep->y_step, ep};
    if (ep->swiglu && !ep->ldy) c.ldy = n / 2;
    GPTRS_REQUIRE(((n | k | c.ldx | c.ldy | c.x_step | c.y_step) & 7) == 0, "dense bf16 matmul: sizes, strides and steps must be multiples of 8");
    GPTRS_REQUIRE(((reinterpret_cast<uintptr_t>(d_x) | reinterpret_cast<uintptr_t>(d_w) | reinterpret_cast<uintptr_t>(d_y)) & 15) == 0, "16-byte alignment");
    GPTRS_REQUIRE(c.ldx >= k && c.ldy >= (ep->swiglu ? n / 2 : n) && c.ldx < (1ll << 30), "row strides shorter than the rows");
    GPTRS_REQUIRE((int64_t)c.batch * n < (1ll << 31) && (c.batch == 1 || ep->d_tiles || (c.x_step > 0 && c.y_step > 0)), "batch");
    GPTRS_REQUIRE(ep->out_dtype == GPTRS_BF16 || ep->out_dtype == GPTRS_F32, "out_dtype must be bf16 or f32");
    GPTRS_REQUIRE(ep->act >= 0 && ep->act <= 2, "activation: 0 none, 1 xIELU, 2 squared relu");
    GPTRS_REQUIRE(!ep->d_best_val || (m <= 128 && c.batch == 1 && ep->out_dtype == GPTRS_F32 && ep->d_best_idx), "fused greedy head: up to 128 rows, f32");
    GPTRS_REQUIRE(!ep->swiglu || ((ep->swiglu == GPTRS_GATE_SILU || ep->swiglu == GPTRS_GATE_GELU_TANH) && ep->out_dtype == GPTRS_BF16 && n % 16 == 0 &&
                                  c.ldy == n / 2 && (c.batch == 1 || ep->d_tiles) && !ep->d_bias && !ep->act && ep->softcap == 0.f && !ep->d_best_val),
                  "gated output: compact bf16 rows, no other epilogue");
    if (m == 0) return GPTRS_OK;
    cudaStream_t st = as_stream(stream);
    if (ep->d_tiles) {
        GPTRS_REQUIRE(ep->d_n_tiles && ep->max_tiles > 0 && !ep->d_bias && ep->act != 1 && ep->softcap == 0.f && !ep->d_best_val, "grouped form: tile list, squared relu or no activation");
        if (ep->tile_rows == 16) return launch_channels<16, 5>(c, st);
        if (ep->tile_rows == 32) return launch_channels<32, 5>(c, st);
        if (ep->tile_rows == 64) return launch_channels<64, 4>(c, st);
        GPTRS_REQUIRE(ep->tile_rows == kTileM, "grouped form: tiles of 16, 32, 64 or 128 rows");
        if (n <= 64) return launch_rows<64, 8>(c, st);
        if (n > 128 && ep->max_tiles * ceil_div(n, 256) >= sm_count()) return launch_rows<256, 4>(c, st);
        return launch_rows<128, 6>(c, st);
    }
    if (m <= 16) return launch_channels<16, 5>(c, st);
    if (m <= 32) return launch_channels<32, 5>(c, st);
    if (m <= 64) return launch_channels<64, 4>(c, st);
    if (m <= 128) return launch_channels<128, 6>(c, st);
    if (n <= 64) return launch_rows<64, 8>(c, st);
    // a wide tile where it still gives every SM one; otherwise 128 columns
    if (n > 128 && (int64_t)ceil_div(m, kTileM) * ceil_div(n, 256) * c.batch >= sm_count()) return launch_rows<256, 4>(c, st);
    return launch_rows<128, 6>(c, st);
}
