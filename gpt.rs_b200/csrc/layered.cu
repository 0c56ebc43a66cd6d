// Models whose layers are configured one by one (engine kind "layered"): weight packing, cache and state set-up and the forward
// pass. A layer is a mixer (latent attention, latent_attention.cu; attention with grouped key / value heads, grouped_attention.cu; a
// gated delta rule, delta_rule.cu) and an optional feed-forward (dense xIELU, gated gelu or a polynomial of normed powers; a mixture of
// experts, moe_route.cu). The step between two sublayers is post_norm_conv.cu (output norm, residual sum, short convolution with its
// per-sequence state), norm_step.cu (norms on both sides of a sublayer), stream_step.cu (norms in front, several residual streams) or
// depth_step.cu (output norms in groups, an average over all layers' results), the matmuls are dense_bf16.cu or, in f32 mode,
// dense_f32.cu. Slots, pages, graphs, sampling and the generator are the engine's.
#include <cmath>
#include <cstdlib>
#include <cstring>

#include "engine.h"

namespace gptrs {
namespace {

int64_t pad8(int64_t v) { return (v + 7) / 8 * 8; }

// dst[b][..] = src[b][n][k] element by element, any strides (in elements), f32 or bf16 destination
struct PackParams {
    const float* src;
    void* dst;
    int64_t total, n, k;
    int64_t sb, sn, sk, db, dn, dk;
    int bf16;
};
__global__ void pack_kernel(const PackParams p) {
    for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < p.total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t k = i % p.k, n = (i / p.k) % p.n, b = i / (p.k * p.n);
        const float v = p.src[b * p.sb + n * p.sn + k * p.sk];
        const int64_t at = b * p.db + n * p.dn + k * p.dk;
        if (p.bf16) static_cast<__nv_bfloat16*>(p.dst)[at] = __float2bfloat16_rn(v);
        else static_cast<float*>(p.dst)[at] = v;
    }
}
int launch_pack(Model& m, const PackParams& pp) {
    const int64_t blocks = (pp.total + 255) / 256;
    pack_kernel<<<(unsigned)(blocks < 4096 ? blocks : 4096), 256, 0, m.stream>>>(pp);
    return cudaGetLastError() == cudaSuccess ? GPTRS_OK : fail(GPTRS_EXECUTION, "packing a weight failed");
}

// One block of a source leaf and where it goes in the packed weight: rows n (with a step between batches) and columns k.
struct Piece {
    int64_t batch, n, k;        // block: batch x n output channels x k inputs
    int64_t src, sb, sn, sk;    // first element and strides in the leaf
    int64_t row, row_b;         // first output channel in the packed weight, step between batches
    int64_t col, col_b;         // first input column, step between batches
    int64_t mat_b;              // step between batches in whole matrices (1: a batch entry is a matrix of its own)
    int64_t mat = 0;            // matrix of the first batch entry
    int64_t row_n = 1;          // step between packed rows
};
struct Leaf {
    std::string name;
    std::vector<int64_t> dims;
    std::vector<Piece> pieces;
    std::string bias;           // optional [dims[0]], placed like the pieces' rows
};
// a leaf [n][k] whose rows go to the rows from `row` on
Leaf rows_of(const std::string& name, int64_t n, int64_t k, int64_t row, const std::string& bias = "") {
    return {name, {n, k}, {{1, n, k, 0, 0, k, 1, row, 0, 0, 0, 0}}, bias};
}
// the same in `heads` groups of rows, `stride` rows apart
Leaf heads_of(const std::string& name, int64_t heads, int64_t n, int64_t k, int64_t row, int64_t stride, const std::string& bias = "") {
    return {name, {heads * n, k}, {{heads, n, k, 0, n * k, k, 1, row, stride, 0, 0, 0}}, bias};
}

// Packs the pieces of the leaves into a weight of `batch` matrices n x k: bf16 [n][k] with both sizes padded to 8 and zeros in
// between, or f32 [k][n]; biases into one vector of n. Memoised by the stable ids of the leaves like every derived layout. The
// names of the leaves are added to `used`.
int pack_weight(Model& m, const std::vector<Leaf>& leaves, int64_t batch, int64_t n, int64_t k, const std::string& tag, DenseWeight* w,
                std::vector<std::string>* used) {
    const bool bf16 = !m.f32();
    w->batch = batch; w->n = bf16 ? pad8(n) : n; w->k = bf16 ? pad8(k) : k;
    int rc = GPTRS_OK;
    std::vector<Tensor*> raw(leaves.size(), nullptr);
    auto drop = [&]() { for (Tensor* t : raw) tensor_release(t); };
    for (size_t i = 0; i < leaves.size(); ++i) {
        if ((rc = get_raw(m, leaves[i].name, leaves[i].dims, &raw[i]))) { drop(); return rc; }
        if (used) used->push_back(leaves[i].name);
    }
    for (size_t i = 0; i < leaves.size(); ++i) {
        if (leaves[i].bias.empty()) continue;
        if (!w->bias) {
            int64_t bd[1] = {w->n};
            if ((rc = tensor_alloc(GPTRS_F32, 1, bd, true, &w->bias))) { drop(); return rc; }
            if (cudaDeviceSynchronize() != cudaSuccess) { drop(); return fail(GPTRS_EXECUTION, "packing a bias failed"); }   // the zero fill is done
        }
        Tensor* b = nullptr;
        if ((rc = get_raw(m, leaves[i].bias, {leaves[i].dims[0]}, &b))) { drop(); return rc; }
        for (const Piece& p : leaves[i].pieces) {
            PackParams pp = {};
            pp.src = static_cast<const float*>(b->data); pp.dst = static_cast<float*>(w->bias->data) + p.row;
            pp.n = p.n; pp.k = 1; pp.total = p.batch * p.n;
            pp.sb = p.n; pp.sn = 1; pp.db = p.row_b; pp.dn = 1;
            if (!rc) rc = launch_pack(m, pp);
        }
        if (cudaStreamSynchronize(m.stream) != cudaSuccess && !rc) rc = fail(GPTRS_EXECUTION, "packing a bias failed");
        tensor_release(b);
        if (rc) { drop(); return rc; }
    }
    std::pair<uint64_t, uint64_t> key = m.ids[leaves[0].name];
    for (size_t i = 1; i < leaves.size(); ++i) {
        const auto id = m.ids[leaves[i].name];
        key.first = key.first * 3 ^ id.first * 31; key.second = key.second * 5 ^ id.second * 131;
    }
    const auto did = derived_id(key, (bf16 ? "dense_bf16:" : "dense_f32:") + tag + ":" + std::to_string(batch) + "x" + std::to_string(w->n) + "x" + std::to_string(w->k));
    const size_t need = (size_t)batch * w->n * w->k * (bf16 ? 2 : 4);
    if (Tensor* hit = param_lookup(did.first, did.second)) {
        if (hit->bytes == need) { w->w = hit; ++m.memo_hits; drop(); return GPTRS_OK; }
        tensor_release(hit);
    }
    int64_t wd[3] = {batch, bf16 ? w->n : w->k, bf16 ? w->k : w->n};
    if ((rc = tensor_alloc(bf16 ? GPTRS_BF16 : GPTRS_F32, 3, wd, true, &w->w))) { drop(); return rc; }
    if (cudaDeviceSynchronize() != cudaSuccess) { drop(); return fail(GPTRS_EXECUTION, "packing a weight failed"); }   // the zero fill is done
    for (size_t i = 0; i < leaves.size() && !rc; ++i)
        for (const Piece& p : leaves[i].pieces) {
            if (p.batch * p.n * p.k == 0) continue;
            PackParams pp = {};
            const int64_t dn = bf16 ? w->k : 1, dk = bf16 ? 1 : w->n;
            pp.src = static_cast<const float*>(raw[i]->data) + p.src;
            pp.dst = static_cast<unsigned char*>(w->w->data) + (p.mat * w->n * w->k + p.row * dn + p.col * dk) * (bf16 ? 2 : 4);
            pp.n = p.n; pp.k = p.k; pp.total = p.batch * p.n * p.k;
            pp.sb = p.sb; pp.sn = p.sn; pp.sk = p.sk;
            pp.db = p.row_b * dn + p.col_b * dk + p.mat_b * w->n * w->k; pp.dn = p.row_n * dn; pp.dk = dk;
            pp.bf16 = bf16;
            if ((rc = launch_pack(m, pp))) break;
        }
    if (cudaStreamSynchronize(m.stream) != cudaSuccess && !rc) rc = fail(GPTRS_EXECUTION, "packing a weight failed");
    drop();
    if (rc) return rc;
    param_store(did.first, did.second, w->w);
    ++m.quantised_now;
    return GPTRS_OK;
}
// a plain [out][in] leaf
int pack_plain(Model& m, const std::string& name, int64_t n, int64_t k, const std::string& bias, DenseWeight* w, std::vector<std::string>* used = nullptr) {
    return pack_weight(m, {rows_of(name, n, k, 0, bias)}, 1, n, k, "plain", w, used);
}

// rows of `ld` floats -> rows of `n` (a vocabulary that is no multiple of 8 is computed with padding columns)
struct CompactParams { const float* src; float* dst; int ld, n; };
__global__ void compact_rows_kernel(const CompactParams p) {
    pdl_launch_dependents();
    pdl_wait();
    for (int i = threadIdx.x; i < p.n; i += blockDim.x) p.dst[(size_t)blockIdx.x * p.n + i] = p.src[(size_t)blockIdx.x * p.ld + i];
}

struct DenseOpts {
    bool out_f32 = false;
    int act = 0;
    float pos = 0.f, neg = 0.f, softcap = 0.f;
    int64_t ldx = 0, ldy = 0, x_step = 0, y_step = 0;
    bool pick = false;
    // grouped form
    const gptrs_row_tile* tiles = nullptr;
    const int32_t* n_tiles = nullptr;
    int64_t max_tiles = 0, tile_rows = 0;
    int gate = 0;   // GPTRS_GATE_*
};
int dense(Model& m, const DenseWeight& w, const void* x, void* y, int64_t rows, const DenseOpts& o) {
    ++m.launches;
    gptrs_dense_epilogue ep = {};
    ep.out_dtype = (m.f32() || o.out_f32) ? GPTRS_F32 : GPTRS_BF16;
    ep.d_bias = w.bias ? static_cast<const float*>(w.bias->data) : nullptr;
    ep.act = o.act; ep.act_pos = o.pos; ep.act_neg = o.neg; ep.softcap = o.softcap;
    ep.ldx = o.ldx; ep.ldy = o.ldy; ep.batch = w.batch; ep.x_step = o.x_step; ep.y_step = o.y_step;
    if (o.pick) { ep.d_best_val = m.best_val.as<float>(); ep.d_best_idx = m.best_idx.as<int32_t>(); ep.skip_store = 1; }
    ep.d_status = m.d_status.as<int32_t>();
    ep.d_tiles = o.tiles; ep.d_n_tiles = o.n_tiles; ep.max_tiles = o.max_tiles; ep.tile_rows = o.tile_rows; ep.swiglu = o.gate;
    if (m.f32())
        return gptrs_cuda_dense_f32(static_cast<const float*>(x), static_cast<const float*>(w.w->data), static_cast<float*>(y), rows, w.n, w.k, &ep, m.stream);
    return gptrs_cuda_dense_bf16(x, w.w->data, y, rows, w.n, w.k, &ep, m.stream);
}

float softplus(float x) { return x > 20.f ? x : (float)std::log1p(std::exp((double)x)); }

// Rows of a tile of the experts' matmuls for a launch of `rows` rows: small tiles (weights on the M side of the MMA) while an
// expert has few rows on average, whole 128-row tiles beyond.
int expert_tile_rows(const Model& m, const gptrs_moe& a, int64_t rows) {
    if (m.f32()) return 8;
    const double mean = (double)rows * a.top / a.experts;
    return mean <= 8 ? 16 : mean <= 24 ? 32 : mean <= 48 ? 64 : 128;
}

// what the buffers of a forward pass must hold, over all layers (elements per row unless said otherwise)
struct Widths {
    int64_t qkv = 0, q = 0, q_latent = 0, qa = 0, lat = 0, attn = 0, up = 0, gate_up = 0, decay = 0, gate = 0;
    int64_t delta_scratch = 0, router = 0, sorted = 0, expert_y = 0, top = 0, work = 0, row_tiles = 0;
    size_t pool = 0, delta_state = 0, mix_conv = 0;
    int n_state = 0;
};

int build_latent(Model& m, LayeredLayer& L, const std::string& x, std::vector<std::string>* used) {
    const gptrs_latent_attention& a = L.att;
    LayerWeights& w = *L.w;
    const int64_t W = m.cfg.d_model, H = a.heads, dim = a.dim, rot = a.rot_dim, rank = a.kv_rank, vd = a.vdim;
    int rc;
    if ((rc = get_raw(m, x + "dkv.norm", {rank}, &w.latent_norm))) return rc;
    // queries (or the query latent) and the down-projection in one weight, laid out as the attention kernels expect a projection row
    // the rotated part, pairs next to one another whichever layout the design has
    auto rotated = [&](std::vector<Piece>* to, int64_t batch, int64_t k, int64_t src, int64_t sb, int64_t row, int64_t row_b) {
        const int64_t half = L.cfg.rope_halves ? a.rot_dims / 2 : 0, done = 2 * half;
        for (int64_t i = 0; i < 2 && half > 0; ++i) to->push_back({batch, half, k, src + i * half * k, sb, k, 1, row + i, row_b, 0, 0, 0, 0, 2});
        if (rot > done) to->push_back({batch, rot - done, k, src + done * k, sb, k, 1, row + done, row_b, 0, 0, 0});
    };
    auto queries = [&](const char* name, int64_t k) {
        Leaf l = {x + name, {H * (dim + rot), k}, {{H, dim, k, 0, (dim + rot) * k, k, 1, 0, a.q_head_stride, 0, 0, 0}}, ""};
        rotated(&l.pieces, H, k, dim * k, (dim + rot) * k, a.q_rot_offset, a.q_head_stride);
        return l;
    };
    Leaf down = {x + "dkv", {rank + rot, W}, {{1, rank, W, 0, 0, W, 1, a.dkv_offset, 0, 0, 0, 0}}, ""};
    rotated(&down.pieces, 1, W, rank * W, 0, a.rot_offset, 0);
    const std::string order = L.cfg.rope_halves ? "_halves" + std::to_string(a.rot_dims) : "";   // part of what the packed layout is memoised under
    if (L.cfg.sink && (rc = get_raw(m, x + "sink", {H}, &w.sink))) return rc;
    if ((rc = pack_weight(m, {a.q_rank > 0 ? rows_of(x + "dq", a.q_rank, W, 0) : queries("q", W), down}, 1, a.kv_row, W, "latent_qkv" + order, &w.qkv, used))) return rc;
    if (a.q_rank > 0 && ((rc = get_raw(m, x + "dq.norm", {a.q_rank}, &w.q_norm)) || (rc = pack_weight(m, {queries("uq", a.q_rank)}, 1, a.q_row, a.q_rank, "latent_uq" + order, &w.uq, used)))) return rc;
    // absorbed query: per head [rank] <- [dim], the stored key projection transposed
    if ((rc = pack_weight(m, {{x + "uk", {H * dim, rank}, {{H, rank, dim, 0, dim * rank, 1, rank, 0, 0, 0, 0, 1}}, ""}}, H, rank, dim, "latent_uk", &w.uk, used))) return rc;
    if ((rc = pack_weight(m, {{x + "uv", {H * vd, rank}, {{H, vd, rank, 0, vd * rank, rank, 1, 0, 0, 0, 0, 1}}, ""}}, H, vd, rank, "latent_uv", &w.uv, used))) return rc;
    return pack_weight(m, {{x + "o", {W, H * vd}, {{H, W, vd, 0, vd, H * vd, 1, 0, 0, 0, a.out_head_stride, 0}}, ""}}, 1, W, H * a.out_head_stride, "latent_o", &w.out, used);
}

// lambda of differential attention: exp(lq1 . lk1) - exp(lq2 . lk2) + diff
int read_lambda(Model& m, const std::string& x, int64_t dim, float diff, float* lambda) {
    std::vector<float> v[4];
    const char* names[4] = {"lq1", "lk1", "lq2", "lk2"};
    for (int i = 0; i < 4; ++i) {
        Tensor* t = nullptr;
        int rc = get_raw(m, x + names[i], {dim}, &t);
        if (rc) return rc;
        v[i].resize(dim);
        const cudaError_t e = cudaMemcpy(v[i].data(), t->data, (size_t)dim * 4, cudaMemcpyDeviceToHost);
        tensor_release(t);
        GPTRS_CUDA_OK(e);
    }
    double s1 = 0., s2 = 0.;
    for (int64_t i = 0; i < dim; ++i) { s1 += (double)v[0][i] * v[1][i]; s2 += (double)v[2][i] * v[3][i]; }
    *lambda = (float)(std::exp(s1) - std::exp(s2) + diff);
    return GPTRS_OK;
}

int read_floats(Model& m, const std::string& name, int64_t n, std::vector<float>* v) {
    Tensor* t = nullptr;
    const int rc = get_raw(m, name, {n}, &t);
    if (rc) return rc;
    v->resize(n);
    const cudaError_t e = cudaMemcpy(v->data(), t->data, (size_t)n * 4, cudaMemcpyDeviceToHost);
    tensor_release(t);
    GPTRS_CUDA_OK(e);
    return GPTRS_OK;
}
int write_floats(const std::vector<float>& v, Tensor** t) {
    int64_t d[1] = {(int64_t)v.size()};
    const int rc = tensor_alloc(GPTRS_F32, 1, d, false, t);
    if (rc) return rc;
    GPTRS_CUDA_OK(cudaMemcpy((*t)->data, v.data(), v.size() * 4, cudaMemcpyHostToDevice));
    return GPTRS_OK;
}

// Short convolutions and norms of queries and keys, slopes of a linear distance bias, and how far its heads can see at all: the norms bound a
// score by scale dim max |gain_q gain_k|, so a key at distance d weighs at most exp(2 bound - slope d) times as much as the position itself.
int build_grouped_prepare(Model& m, LayeredLayer& L, const std::string& x) {
    const gptrs_grouped_attention& a = L.gatt;
    LayerWeights& w = *L.w;
    int rc;
    if (a.taps > 0) {
        int64_t cd[2] = {a.taps, a.conv_channels};
        if ((rc = tensor_alloc(GPTRS_F32, 2, cd, true, &w.qk_conv))) return rc;
        if (cudaDeviceSynchronize() != cudaSuccess) return fail(GPTRS_EXECUTION, "packing a convolution failed");   // the zero fill is done
        for (int part = 0; part < 2; ++part) {
            const int heads = part ? a.kv_heads : a.heads;
            Tensor* t = nullptr;
            if ((rc = get_raw(m, x + (part ? "k.conv" : "q.conv"), {(int64_t)heads * a.dim, a.taps}, &t))) return rc;
            PackParams pp = {};
            pp.src = static_cast<const float*>(t->data); pp.dst = static_cast<float*>(w.qk_conv->data) + (part ? a.k_offset : 0);
            pp.n = a.dim; pp.k = a.taps; pp.total = (int64_t)heads * a.dim * a.taps;
            pp.sb = (int64_t)a.dim * a.taps; pp.sn = a.taps; pp.sk = 1;
            pp.db = a.q_head_stride; pp.dn = 1; pp.dk = a.conv_channels;
            rc = launch_pack(m, pp);
            if (cudaStreamSynchronize(m.stream) != cudaSuccess && !rc) rc = fail(GPTRS_EXECUTION, "packing a convolution failed");
            tensor_release(t);
            if (rc) return rc;
        }
    }
    std::vector<float> gq, gk;
    if (a.qk_norm) {
        if ((rc = read_floats(m, x + "q.norm", a.dim, &gq)) || (rc = read_floats(m, x + "k.norm", a.dim, &gk))) return rc;
        std::vector<float> both(gq);
        for (size_t i = 0; i < both.size(); ++i) both[i] *= gk[i];
        if ((rc = write_floats(a.tied ? both : gq, &w.q_gain)) || (!a.tied && (rc = write_floats(gk, &w.k_gain)))) return rc;
    }
    if (a.distance_bias != GPTRS_DISTANCE_LINEAR) return GPTRS_OK;
    std::vector<float> slope(a.heads);
    for (int h = 0; h < a.heads; ++h) slope[h] = (float)std::exp2(-8.0 * (h + 1) / a.heads);
    if ((rc = write_floats(slope, &w.r1)) || !a.qk_norm) return rc;
    double bound = 0.;
    for (int i = 0; i < a.dim; ++i) bound = std::max(bound, std::fabs((double)gq[i] * gk[i]));
    bound *= 1.02 * a.scale * a.dim;   // queries and keys that are rounded to bf16 may be a little longer
    std::vector<int32_t> reach(a.kv_heads);
    for (int g = 0; g < a.kv_heads; ++g) {
        const double least = slope[(g + 1) * (a.heads / a.kv_heads) - 1];   // slopes fall with the head
        reach[g] = (int32_t)std::min(std::ceil((2. * bound + 32.) / least), 1e9);
    }
    if ((rc = w.reach.alloc(reach.size() * 4))) return rc;
    GPTRS_CUDA_OK(cudaMemcpy(w.reach.p, reach.data(), reach.size() * 4, cudaMemcpyHostToDevice));
    return GPTRS_OK;
}

int build_grouped(Model& m, LayeredLayer& L, const std::string& x, std::vector<std::string>* used) {
    const gptrs_grouped_attention& a = L.gatt;
    LayerWeights& w = *L.w;
    const int64_t W = m.cfg.d_model, H = a.heads, G = a.kv_heads;
    auto bias = [&](const char* n) { return L.cfg.proj_bias ? x + n + ".b" : std::string(); };
    int rc;
    if (a.distance_bias == GPTRS_DISTANCE_LOG && ((rc = get_raw(m, x + "r1", {H}, &w.r1)) || (rc = get_raw(m, x + "r2", {H}, &w.r2)))) return rc;
    if ((rc = build_grouped_prepare(m, L, x))) return rc;
    const int64_t maps = a.maps > 1 ? a.maps : 1;
    if (maps > 1 && (rc = read_lambda(m, x, a.dim, L.cfg.diff, &w.lambda))) return rc;
    std::vector<Leaf> in = {heads_of(x + "q", H * maps, a.dim, W, 0, a.map_stride, bias("q"))};
    if (!a.shared_kv) {
        in.push_back(heads_of(x + "k", G * maps, a.dim, W, a.k_offset, a.map_stride, bias("k")));
        if (!a.tied) in.push_back(heads_of(x + "v", G, a.vdim, W, a.v_offset, a.v_head_stride, bias("v")));
    }
    if (a.gate) in.push_back(heads_of(x + "g", H, a.vdim, W, a.g_offset, a.g_head_stride));
    if ((rc = pack_weight(m, in, 1, a.q_row, W, "grouped_qkv", &w.qkv, used))) return rc;
    return pack_weight(m, {{x + "o", {W, H * a.vdim}, {{H, W, a.vdim, 0, a.vdim, H * a.vdim, 1, 0, 0, 0, a.out_head_stride, 0}}, ""}}, 1, W, H * a.out_head_stride, "heads_o", &w.out, used);
}

// bias of a weight whose rows are not placed by heads
int add_bias(Model& m, const std::string& name, int64_t n, DenseWeight* w) {
    Tensor* b = nullptr;
    int rc = get_raw(m, name, {n}, &b);
    if (rc) return rc;
    int64_t bd[1] = {w->n};
    if (!(rc = tensor_alloc(GPTRS_F32, 1, bd, true, &w->bias)) &&
        (cudaDeviceSynchronize() != cudaSuccess || cudaMemcpy(w->bias->data, b->data, (size_t)n * 4, cudaMemcpyDeviceToDevice) != cudaSuccess))
        rc = fail(GPTRS_EXECUTION, "bias copy failed");
    tensor_release(b);
    return rc;
}

int build_delta(Model& m, LayeredLayer& L, const std::string& x, std::vector<std::string>* used) {
    const gptrs_delta_rule& a = L.delta;
    LayerWeights& w = *L.w;
    const int64_t W = m.cfg.d_model, H = a.heads, kq = (int64_t)a.kv_heads * a.dim, hv = H * a.vdim, hd = H * a.dim;
    int rc;
    if ((rc = get_raw(m, x + "A_log", {H}, &w.a_log)) || (rc = get_raw(m, x + "dt_bias", {a.decay_rank > 0 ? hd : H}, &w.dt_bias)) || (rc = get_raw(m, x + "norm", {a.vdim}, &w.delta_norm))) return rc;
    if ((rc = pack_weight(m, {rows_of(x + "q", kq, W, a.q_offset), rows_of(x + "k", kq, W, a.k_offset), rows_of(x + "v", hv, W, a.v_offset), rows_of(x + "b", H, W, a.beta_offset),
                              a.decay_rank > 0 ? rows_of(x + "a1", a.decay_rank, W, a.a_offset) : rows_of(x + "a", H, W, a.a_offset),
                              a.gate_rank > 0 ? rows_of(x + "g1", a.gate_rank, W, a.g_offset) : rows_of(x + "g", hv, W, a.g_offset)}, 1, a.row, W, "delta_proj", &w.qkv, used))) return rc;
    if (a.decay_rank > 0 && (rc = pack_plain(m, x + "a2", hd, a.decay_rank, "", &w.decay, used))) return rc;
    if (a.gate_rank > 0 && (rc = pack_plain(m, x + "g2", hv, a.gate_rank, "", &w.gate, used))) return rc;
    if ((rc = pack_weight(m, {{x + "o", {W, hv}, {{H, W, a.vdim, 0, a.vdim, hv, 1, 0, 0, 0, a.out_head_stride, 0}}, ""}}, 1, W, H * a.out_head_stride, "heads_o", &w.out, used))) return rc;
    // the three convolutions behind one another
    int64_t cd[2] = {a.conv_channels, a.taps};
    if ((rc = tensor_alloc(GPTRS_F32, 2, cd, false, &w.delta_conv))) return rc;
    float* dst = static_cast<float*>(w.delta_conv->data);
    for (const auto& part : {std::make_pair("q.conv", kq), std::make_pair("k.conv", kq), std::make_pair("v.conv", hv)}) {
        Tensor* t = nullptr;
        if ((rc = get_raw(m, x + part.first, {part.second, a.taps}, &t))) return rc;
        const cudaError_t e = cudaMemcpy(dst, t->data, (size_t)part.second * a.taps * 4, cudaMemcpyDeviceToDevice);
        tensor_release(t);
        GPTRS_CUDA_OK(e);
        dst += part.second * a.taps;
    }
    return GPTRS_OK;
}

// gate and up of a gated feed-forward [F][W] as one matrix: 8 gates, then their 8 partners (matrix `mat` of a batch)
void add_gated(std::vector<Leaf>* leaves, const std::string& x, int64_t F, int64_t W, int64_t mat) {
    for (int part = 0; part < 2; ++part) {
        const int64_t full = F / 8, rest = F % 8;
        Leaf l = {x + (part ? "up" : "gate"), {F, W}, {{full, 8, W, 0, 8 * W, W, 1, part * 8, 16, 0, 0, 0, mat}}, ""};
        if (rest) l.pieces.push_back({1, rest, W, full * 8 * W, 0, W, 1, full * 16 + part * 8, 0, 0, 0, 0, mat});
        leaves->push_back(l);
    }
}

int build_experts(Model& m, LayeredLayer& L, const std::string& x, std::vector<std::string>* used) {
    LayerWeights& w = *L.w;
    const bool gated = L.cfg.expert_form == GPTRS_EXPERT_SWIGLU;
    const int64_t W = m.cfg.d_model, F = L.cfg.d_ff, Fp = pad8(F), E = L.moe.experts, S = L.cfg.shared_ff;
    std::vector<Leaf> up, down;
    for (int64_t e = 0; e < E; ++e) {
        const std::string n = x + "e" + std::to_string(e) + ".";
        if (gated) add_gated(&up, n, F, W, e);
        else up.push_back({n + "up", {F, W}, {{1, F, W, 0, 0, W, 1, 0, 0, 0, 0, 0, e}}, ""});
        down.push_back({n + "down", {W, F}, {{1, W, F, 0, 0, F, 1, 0, 0, 0, 0, 0, e}}, ""});
    }
    int rc;
    if ((rc = pack_weight(m, up, E, gated ? 2 * Fp : F, W, "experts_up", &w.up, used)) ||
        (rc = pack_weight(m, down, E, W, gated ? Fp : F, "experts_down", &w.down, used))) return rc;
    if (S > 0 && gated) {
        std::vector<Leaf> shared;
        add_gated(&shared, x + "shared.", S, W, 0);
        if ((rc = pack_weight(m, shared, 1, 2 * pad8(S), W, "gated_up", &w.shared_up, used)) ||
            (rc = pack_weight(m, {rows_of(x + "shared.down", W, S, 0)}, 1, W, pad8(S), "gated_down", &w.shared_down, used))) return rc;
    } else if (S > 0 && ((rc = pack_plain(m, x + "shared.up", S, W, "", &w.shared_up, used)) || (rc = pack_plain(m, x + "shared.down", W, S, "", &w.shared_down, used)))) {
        return rc;
    }
    if (L.cfg.correction && (rc = get_raw(m, x + "correction", {E}, &w.correction))) return rc;
    if (!L.cfg.shared_gate) return pack_plain(m, x + "router", E, W, "", &w.router, used);
    // the shared expert's gate is one more row of the router
    return pack_weight(m, {rows_of(x + "router", E, W, 0), rows_of(x + "shared.sg", 1, W, E)}, 1, E + 1, W, "router_gate", &w.router, used);
}

// what stands beside the norms of a sublayer (0: mixer, 1: feed-forward), depending on the block form
int build_block(Model& m, LayerWeights& w, const std::string& p, int sub) {
    const gptrs_layered_config& c = m.lay->cfg;
    const int64_t W = m.cfg.d_model;
    const std::string n = std::to_string(sub + 1);
    int rc;
    if ((rc = get_raw(m, p + "norm" + n, {W}, sub ? &w.norm2 : &w.norm1))) return rc;
    if (c.block == GPTRS_BLOCK_SANDWICH) return get_raw(m, p + "norm" + n + "b", {W}, sub ? &w.norm2b : &w.norm1b);
    if (c.block == GPTRS_BLOCK_DEPTH) return GPTRS_OK;
    if (c.block == GPTRS_BLOCK_OUTPUT_NORM) return get_raw(m, p + "canon" + n, {W, c.conv_taps}, sub ? &w.conv2 : &w.conv1);
    if (c.streams == 0) return GPTRS_OK;
    const std::string h = p + "hc" + n + ".";
    LayerWeights::Streams& s = w.streams[sub];
    if ((rc = get_raw(m, h + "in", {c.streams}, &s.in)) || (rc = get_raw(m, h + "out", {c.streams}, &s.out))) return rc;
    return get_raw(m, h + "mix", {c.streams, c.streams}, &s.mix);
}

int build_weights(Model& m, LayeredLayer& L, int l, bool drop_leaves) {
    const int64_t W = m.cfg.d_model;
    const std::string p = "l" + std::to_string(l) + ".", x = p + "mix.", f = p + "mlp.";
    L.w = std::make_shared<LayerWeights>();
    LayerWeights& w = *L.w;
    std::vector<std::string> used;
    int rc;
    if ((rc = build_block(m, w, p, 0))) return rc;
    if (m.lay->cfg.block == GPTRS_BLOCK_DEPTH && (rc = get_raw(m, p + "dwa", {l + 2}, &w.dwa))) return rc;
    if (L.cfg.mixer == GPTRS_MIXER_LATENT_ATTENTION) rc = build_latent(m, L, x, &used);
    else if (L.cfg.mixer == GPTRS_MIXER_GROUPED_ATTENTION) rc = build_grouped(m, L, x, &used);
    else rc = build_delta(m, L, x, &used);
    if (rc) return rc;
    if (L.cfg.mixer == GPTRS_MIXER_GROUPED_ATTENTION && L.cfg.proj_bias && (rc = add_bias(m, x + "o.b", W, &w.out))) return rc;
    if (L.cfg.mlp != GPTRS_MLP_NONE && (rc = build_block(m, w, p, 1))) return rc;
    if (L.cfg.mlp == GPTRS_MLP_DENSE_XIELU) {
        const int64_t F = L.cfg.d_ff;
        if ((rc = pack_plain(m, f + "up", F, W, f + "up.b", &w.up, &used)) || (rc = pack_plain(m, f + "down", W, F, f + "down.b", &w.down, &used))) return rc;
        Tensor* pq = nullptr;
        float v[2];
        if ((rc = get_raw(m, f + "act", {2}, &pq))) return rc;
        const cudaError_t e = cudaMemcpy(v, pq->data, 8, cudaMemcpyDeviceToHost);
        tensor_release(pq);
        GPTRS_CUDA_OK(e);
        w.act_pos = softplus(v[0]);
        w.act_neg = 0.5f + softplus(v[1]);
    } else if (L.cfg.mlp == GPTRS_MLP_DENSE_GELU) {
        const int64_t F = L.cfg.d_ff;
        std::vector<Leaf> up;
        add_gated(&up, f, F, W, 0);
        if ((rc = pack_weight(m, up, 1, 2 * pad8(F), W, "gated_up", &w.up, &used)) ||
            (rc = pack_weight(m, {rows_of(f + "down", W, F, 0)}, 1, W, pad8(F), "gated_down", &w.down, &used))) return rc;
    } else if (L.cfg.mlp == GPTRS_MLP_DENSE_POLY) {
        const int64_t F = L.cfg.d_ff;
        if ((rc = get_raw(m, f + "act", {4}, &w.act)) || (rc = pack_plain(m, f + "up", F, W, "", &w.up, &used)) || (rc = pack_plain(m, f + "down", W, F, "", &w.down, &used))) return rc;
    } else if (L.cfg.mlp == GPTRS_MLP_EXPERTS) {
        if ((rc = build_experts(m, L, f, &used))) return rc;
    }
    if (drop_leaves)
        for (const std::string& n : used) {
            auto it = m.raw.find(n);
            if (it != m.raw.end()) { tensor_release(it->second); m.raw.erase(it); }
        }
    return GPTRS_OK;
}

// Rotation tables, one pair per distinct rotation; angles in double, rounded once. With YaRN scaling (Peng et al., "YaRN: Efficient Context Window
// Extension of Large Language Models") dimensions that turn less than `slow` times over `original` positions are slowed down by `factor`,
// those that turn more than `fast` times stay, those in between are blended; cos and sin grow by 0.1 ln(factor) + 1.
int add_rope(Model& m, LayeredLayer& L) {
    Layered& y = *m.lay;
    const auto& c = m.cfg;
    const gptrs_latent_attention& a = L.att;
    for (size_t i = 0; i < y.ropes.size(); ++i)
        if (const Layered::Rope& o = *y.ropes[i]; o.base == L.cfg.rope_base && o.dims == a.rot_dims && o.factor == L.cfg.rope_factor && o.original == L.cfg.rope_original &&
                                                  o.fast == L.cfg.rope_fast && o.slow == L.cfg.rope_slow) L.rope = (int)i;
    if (L.rope >= 0) return GPTRS_OK;
    auto r = std::make_unique<Layered::Rope>();
    r->base = L.cfg.rope_base; r->dims = a.rot_dims;
    r->factor = L.cfg.rope_factor; r->original = L.cfg.rope_original; r->fast = L.cfg.rope_fast; r->slow = L.cfg.rope_slow;
    const int half = a.rot_dims / 2;
    const bool scaled = r->factor > 0. && half > 0;
    double lo = 0., hi = 0., mag = 1.;
    if (scaled) {
        constexpr double kTwoPi = 6.283185307179586;
        auto turning = [&](double turns) { return r->dims * std::log(r->original / (kTwoPi * turns)) / (2. * std::log(r->base)); };   // the dimension that turns so often
        lo = std::max(std::floor(turning(r->fast)), 0.);
        hi = std::min(std::ceil(turning(r->slow)), r->dims - 1.);
        mag = 0.1 * std::log(r->factor) + 1.;
    }
    std::vector<float> cs((size_t)c.context_length * half), sn(cs.size());
    for (int i = 0; i < half; ++i) {
        double f = std::pow(r->base, -2.0 * i / a.rot_dims);
        if (scaled) {
            const double slowed = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.), 1.);
            f = f / r->factor * slowed + f * (1. - slowed);
        }
        for (int q = 0; q < c.context_length; ++q) {
            cs[(size_t)q * half + i] = (float)(std::cos(q * f) * mag);
            sn[(size_t)q * half + i] = (float)(std::sin(q * f) * mag);
        }
    }
    int rc;
    if (half > 0) {
        if ((rc = r->cos_t.alloc(cs.size() * 4)) || (rc = r->sin_t.alloc(sn.size() * 4))) return rc;
        GPTRS_CUDA_OK(cudaMemcpy(r->cos_t.p, cs.data(), cs.size() * 4, cudaMemcpyHostToDevice));
        GPTRS_CUDA_OK(cudaMemcpy(r->sin_t.p, sn.data(), sn.size() * 4, cudaMemcpyHostToDevice));
    }
    L.rope = (int)y.ropes.size();
    y.ropes.push_back(std::move(r));
    return GPTRS_OK;
}

// query tiles of the tensor-core attention (GPTRS_LATENT_TC=0 / GPTRS_GROUPED_TC=0 keep the plain kernels)
int add_tiles(Model& m, LayeredLayer& L) {
    Layered& y = *m.lay;
    static const bool latent_on = [] { const char* e = getenv("GPTRS_LATENT_TC"); return !e || atoi(e) != 0; }();
    static const bool grouped_on = [] { const char* e = getenv("GPTRS_GROUPED_TC"); return !e || atoi(e) != 0; }();
    const int tokens = L.cfg.mixer == GPTRS_MIXER_LATENT_ATTENTION ? (latent_on ? gptrs_cuda_latent_tile_tokens(&L.att) : 0)
                                                                   : (grouped_on ? gptrs_cuda_grouped_tile_tokens(&L.gatt) : 0);
    L.tiles = -1;
    if (tokens <= 0) return GPTRS_OK;
    for (size_t i = 0; i < y.tile_sets.size(); ++i)
        if (y.tile_sets[i]->tokens == tokens) L.tiles = (int)i;
    if (L.tiles >= 0) return GPTRS_OK;
    auto t = std::make_unique<Layered::TileSet>();
    t->tokens = tokens;
    int rc;
    if ((rc = t->row.alloc((size_t)m.cfg.max_tokens * 4, true)) || (rc = t->rows.alloc((size_t)m.cfg.max_tokens * 4, true))) return rc;
    L.tiles = (int)y.tile_sets.size();
    y.tile_sets.push_back(std::move(t));
    return GPTRS_OK;
}

void count_widths(const Model& m, LayeredLayer& L, Widths* n) {
    const auto& c = m.cfg;
    const LayerWeights& w = *L.w;
    n->qkv = std::max(n->qkv, w.qkv.n);
    n->attn = std::max(n->attn, w.out.k);
    L.pool_off = n->pool;
    if (L.cfg.mixer == GPTRS_MIXER_LATENT_ATTENTION) {
        n->qa = std::max(n->qa, (int64_t)L.att.heads * L.att.qa_head_stride);
        n->lat = std::max(n->lat, (int64_t)L.att.heads * L.att.lat_head_stride);
        if (L.att.q_rank > 0) {
            n->q = std::max(n->q, (int64_t)L.att.q_row);
            n->q_latent = std::max(n->q_latent, (int64_t)L.att.q_latent_row);
        }
        n->pool += (size_t)c.kv_pages * L.att.page_bytes;
    } else if (L.cfg.mixer == GPTRS_MIXER_GROUPED_ATTENTION) {
        if (L.cfg.kv_from >= 0) L.pool_off = m.lay->layers[L.cfg.kv_from].pool_off;
        else n->pool += (size_t)c.kv_pages * L.gatt.page_bytes;
        if (L.prepared()) n->q = std::max(n->q, (int64_t)L.gatt.query_row);
        L.mix_conv_off = n->mix_conv;
        n->mix_conv += (size_t)c.max_seqs * L.gatt.conv_floats;
    } else {
        n->decay = std::max(n->decay, (int64_t)L.delta.decay_row);
        n->gate = std::max(n->gate, (int64_t)L.delta.gate_row);
        // a pass that is not one token per sequence: at most one run per slot
        n->delta_scratch = std::max(n->delta_scratch, gptrs_cuda_delta_scratch_floats(&L.delta, c.max_tokens, std::min(c.max_seqs, c.max_tokens - 1)));
        L.delta_state_off = n->delta_state;
        L.mix_conv_off = n->mix_conv;
        n->delta_state += (size_t)c.max_seqs * L.delta.state_floats;
        n->mix_conv += (size_t)c.max_seqs * L.delta.conv_floats;
    }
    n->pool = (n->pool + 255) / 256 * 256;
    n->delta_state = (n->delta_state + 63) / 64 * 64;
    n->mix_conv = (n->mix_conv + 63) / 64 * 64;
    if (m.lay->cfg.block == GPTRS_BLOCK_OUTPUT_NORM) {
        L.state1 = n->n_state++;
        if (L.cfg.mlp != GPTRS_MLP_NONE) L.state2 = n->n_state++;
    }
    if (L.cfg.mlp == GPTRS_MLP_DENSE_XIELU || L.cfg.mlp == GPTRS_MLP_DENSE_POLY) n->up = std::max(n->up, w.up.n);
    if (L.cfg.mlp == GPTRS_MLP_DENSE_GELU) {
        n->up = std::max(n->up, w.up.n / 2);
        n->gate_up = std::max(n->gate_up, w.up.n);
    }
    if (L.cfg.mlp == GPTRS_MLP_EXPERTS) {
        const int64_t T = c.max_tokens, top = L.moe.top;
        n->top = std::max(n->top, top);
        n->router = std::max(n->router, w.router.n);
        n->sorted = std::max(n->sorted, top * w.up.k);
        const bool gated = L.cfg.expert_form == GPTRS_EXPERT_SWIGLU;
        n->up = std::max({n->up, gated ? top * w.up.n / 2 : top * w.up.n, gated ? w.shared_up.n / 2 : w.shared_up.n});
        if (gated) n->gate_up = std::max({n->gate_up, top * w.up.n, w.shared_up.n});
        n->expert_y = std::max(n->expert_y, top * w.down.n);
        n->work = std::max(n->work, gptrs_cuda_moe_work_ints(&L.moe, T));
        gptrs_moe smallest = L.moe;   // most tiles: the smallest tile that a launch of this many rows, or of one, may get
        smallest.tile_rows = m.f32() ? 8 : 16;
        n->row_tiles = std::max(n->row_tiles, gptrs_cuda_moe_max_tiles(&smallest, T));
    }
}

bool same_shape(const gptrs_layer_config& a, const gptrs_layer_config& b) {
    auto key = [](const gptrs_layer_config& c) {
        return std::make_tuple(std::make_tuple(c.mixer, c.heads, c.dim, c.rot_dim, c.rot_dims, c.vdim, c.kv_rank, c.window, c.scale, c.rope_base, c.mlp, c.d_ff),
                               std::make_tuple(c.kv_heads, c.mask, c.mask_size, c.distance_bias, c.proj_bias, c.softcap, c.taps, c.decay_rank, c.gate_rank),
                               std::make_tuple(c.experts, c.top, c.groups, c.keep, c.expert_form, c.shared_ff, c.route, c.group_best, c.correction, c.weight_scale),
                               std::make_tuple(c.q_rank, c.maps, c.out_gate, c.kv_from, c.diff, c.sink, c.rope_halves, c.qk_norm, c.tied, c.gate_silu, c.shared_gate),
                               std::make_tuple(c.rope_factor, c.rope_original, c.rope_fast, c.rope_slow));
    };
    return key(a) == key(b);
}

}  // namespace

int layered_check_config(const gptrs_model_config& c) {
    GPTRS_REQUIRE(c.weight_mode == kModeF32 || c.weight_mode == kModeBf16, "the layered kind runs with f32 or bf16 weights");
    GPTRS_REQUIRE(c.n_layers > 0 && c.d_model > 0 && c.vocab > 0 && c.context_length > 0, "bad model dimensions");
    GPTRS_REQUIRE(c.max_seqs > 0 && c.max_tokens > 0 && c.kv_pages > 0 && c.max_pages_per_seq > 0, "max_seqs, max_tokens and the page counts must be positive");
    if (c.tp_size > 1) return fail(GPTRS_UNIMPLEMENTED, "tensor parallelism is implemented for the ministral kind");
    return GPTRS_OK;
}

int layered_set_layers(Model& m, const gptrs_layered_config& common, const gptrs_layer_config* layers) {
    const int n = m.cfg.n_layers;
    GPTRS_REQUIRE(common.block == GPTRS_BLOCK_OUTPUT_NORM || common.block == GPTRS_BLOCK_SANDWICH || common.block == GPTRS_BLOCK_PRE_NORM || common.block == GPTRS_BLOCK_DEPTH, "unknown block form");
    GPTRS_REQUIRE(common.block != GPTRS_BLOCK_DEPTH || (common.norm_groups >= 1 && m.cfg.d_model % common.norm_groups == 0), "norm groups: equal parts of the width");
    GPTRS_REQUIRE(common.streams >= 0 && (common.streams == 0 || common.block == GPTRS_BLOCK_PRE_NORM), "residual streams: for the block form with norms in front");
    if (common.streams > GPTRS_MAX_STREAMS) return fail(GPTRS_UNIMPLEMENTED, "more than 16 residual streams");
    GPTRS_REQUIRE(common.block != GPTRS_BLOCK_OUTPUT_NORM || (common.conv_taps >= 1 && common.conv_taps <= 16), "short convolutions of 1 to 16 taps");
    GPTRS_REQUIRE(common.learned_positions == 0 || (common.block == GPTRS_BLOCK_SANDWICH && common.learned_positions >= m.cfg.context_length),
                  "learned positions: for the block form with norms on both sides, one for every position of the context");
    m.lay->cfg = common;
    m.lay->layers.clear();
    m.lay->layers.resize(n);
    const int dtype = m.f32() ? GPTRS_F32 : GPTRS_BF16;
    for (int l = 0; l < n; ++l) {
        const gptrs_layer_config& c = layers[l];
        GPTRS_REQUIRE(c.mlp == GPTRS_MLP_NONE || c.d_ff > 0, "feed-forward size");
        GPTRS_REQUIRE(c.weights_of < n && (c.weights_of < 0 || layers[c.weights_of].weights_of < 0), "weights_of names a layer that has weights of its own");
        GPTRS_REQUIRE(common.block != GPTRS_BLOCK_DEPTH || c.weights_of < 0, "a layer whose output is averaged over depth has weights of its own");
        GPTRS_REQUIRE(!(c.rope_factor > 0.) || (c.rope_original > 0. && c.rope_fast > 0. && c.rope_slow > 0.), "rotation scaling: constants must be positive");
        LayeredLayer& L = m.lay->layers[l];
        L.cfg = c;
        int rc;
        if (c.mixer == GPTRS_MIXER_LATENT_ATTENTION) {
            L.att.dtype = dtype;
            L.att.heads = c.heads; L.att.dim = c.dim; L.att.rot_dim = c.rot_dim; L.att.vdim = c.vdim; L.att.kv_rank = c.kv_rank;
            L.att.window = c.window; L.att.rot_dims = c.rot_dims; L.att.scale = c.scale; L.att.q_rank = c.q_rank;
            rc = gptrs_cuda_latent_layout(&L.att);
        } else if (c.mixer == GPTRS_MIXER_GROUPED_ATTENTION) {
            L.gatt.dtype = dtype;
            L.gatt.heads = c.heads; L.gatt.kv_heads = c.kv_heads; L.gatt.dim = c.dim; L.gatt.vdim = c.vdim; L.gatt.mask = c.mask; L.gatt.mask_size = c.mask_size;
            L.gatt.scale = c.scale; L.gatt.softcap = c.softcap; L.gatt.distance_bias = c.distance_bias;
            L.gatt.maps = c.maps; L.gatt.gate = c.out_gate; L.gatt.shared_kv = c.kv_from >= 0;
            L.gatt.head_scale = 1.f - c.diff; L.gatt.head_eps = m.cfg.norm_eps;
            L.gatt.taps = c.taps; L.gatt.qk_norm = c.qk_norm; L.gatt.tied = c.tied;
            if (c.kv_from >= 0) {
                GPTRS_REQUIRE(c.kv_from < l && !c.proj_bias, "kv_from names an earlier layer (projections without biases)");
                const gptrs_layer_config& o = layers[c.kv_from];
                GPTRS_REQUIRE(o.mixer == c.mixer && o.kv_from < 0 && o.kv_heads == c.kv_heads && o.dim == c.dim && o.vdim == c.vdim && std::max(o.maps, 1) == std::max(c.maps, 1),
                              "kv_from names a layer with keys and values of its own and the same heads");
            }
            rc = gptrs_cuda_grouped_layout(&L.gatt);
        } else if (c.mixer == GPTRS_MIXER_CHANNEL_DELTA) {
            L.delta.dtype = dtype;
            L.delta.heads = c.heads; L.delta.kv_heads = c.kv_heads; L.delta.dim = c.dim; L.delta.vdim = c.vdim; L.delta.taps = c.taps;
            L.delta.decay_rank = c.decay_rank; L.delta.gate_rank = c.gate_rank; L.delta.eps = m.cfg.norm_eps; L.delta.gate_silu = c.gate_silu;
            rc = gptrs_cuda_delta_layout(&L.delta);
        } else {
            return fail(GPTRS_UNIMPLEMENTED, "unknown mixer");
        }
        if (rc) return rc;
        if (c.mlp == GPTRS_MLP_EXPERTS) {
            GPTRS_REQUIRE(common.block != GPTRS_BLOCK_OUTPUT_NORM, "experts: for the block forms without short convolutions between the sublayers");
            GPTRS_REQUIRE(c.shared_ff >= 0 && (c.shared_ff == 0 || common.block == GPTRS_BLOCK_PRE_NORM || common.block == GPTRS_BLOCK_DEPTH),
                          "shared expert: for the block forms with norms on one side only");
            GPTRS_REQUIRE(!c.shared_gate || (c.shared_ff > 0 && common.block == GPTRS_BLOCK_DEPTH), "gated shared expert: for the block form with an average over depth");
            GPTRS_REQUIRE(c.expert_form == GPTRS_EXPERT_SWIGLU || c.expert_form == GPTRS_EXPERT_RELU2, "unknown form of the experts");
            L.moe = {c.experts, c.top, c.groups, c.keep, 16, c.route, c.group_best, c.weight_scale};
            GPTRS_REQUIRE(c.experts > 0 && c.top > 0 && c.groups > 0 && c.keep > 0 && c.experts % c.groups == 0 && c.keep <= c.groups &&
                              c.top <= c.keep * (c.experts / c.groups), "experts: groups must be equal and hold enough experts");
            if (c.experts > 1024) return fail(GPTRS_UNIMPLEMENTED, "experts: more than 1024");
        } else if (c.mlp != GPTRS_MLP_NONE && c.mlp != GPTRS_MLP_DENSE_XIELU && c.mlp != GPTRS_MLP_DENSE_GELU && c.mlp != GPTRS_MLP_DENSE_POLY) {
            return fail(GPTRS_UNIMPLEMENTED, "unknown feed-forward kind");
        }
    }
    return GPTRS_OK;
}

int layered_finalize(Model& m, bool drop_leaves) {
    Layered& y = *m.lay;
    const auto& c = m.cfg;
    GPTRS_REQUIRE(!y.layers.empty(), "call gptrs_cuda_model_set_layers before finalize");
    const int64_t W = c.d_model, V = c.vocab, taps = y.cfg.conv_taps;
    const bool convs = y.cfg.block == GPTRS_BLOCK_OUTPUT_NORM;
    const int64_t streams = std::max(y.cfg.streams, 1);
    int rc;
    if ((rc = get_raw(m, "embed", {V, W}, &m.tok_emb)) || (rc = get_raw(m, "final.norm", {W}, &m.final_g))) return rc;
    if (convs && (rc = get_raw(m, "embed.norm", {W}, &y.embed_norm))) return rc;
    if (y.cfg.learned_positions > 0 && (rc = get_raw(m, "pos", {y.cfg.learned_positions, W}, &m.pos_emb))) return rc;
    if ((rc = pack_plain(m, "head", V, W, "", &y.head))) return rc;
    const size_t act = m.f32() ? 4 : 2;
    Widths n;
    for (int l = 0; l < c.n_layers; ++l)
        if (y.layers[l].cfg.weights_of < 0 && (rc = build_weights(m, y.layers[l], l, drop_leaves))) return rc;
    for (int l = 0; l < c.n_layers; ++l) {
        LayeredLayer& L = y.layers[l];
        if (L.cfg.weights_of >= 0) {
            GPTRS_REQUIRE(same_shape(L.cfg, y.layers[L.cfg.weights_of].cfg), "a layer that reuses another one's weights has an equal configuration");
            L.w = y.layers[L.cfg.weights_of].w;
        }
        L.gatt.lambda_ = L.w->lambda;
        count_widths(m, L, &n);
        if (L.cfg.mixer == GPTRS_MIXER_LATENT_ATTENTION && (rc = add_rope(m, L))) return rc;
        if (L.attends() && (rc = add_tiles(m, L))) return rc;
    }
    if (drop_leaves) {
        auto it = m.raw.find("head");
        if (it != m.raw.end()) { tensor_release(it->second); m.raw.erase(it); }
    }
    // activations (zeroed: padding columns that no kernel writes are multiplied by zero weights and must be finite)
    const size_t T = c.max_tokens, Wp = m.f32() ? W : pad8(W), Vp = y.head.n, rows = m.max_rows();
    if ((rc = m.hidden.alloc(T * streams * W * 4, true)) || (rc = y.x2.alloc(convs ? T * W * 4 : 0, true)) || (rc = y.h.alloc(T * Wp * act, true)) ||
        (rc = y.y.alloc(T * Wp * act, true)) || (rc = y.qkv.alloc(T * n.qkv * act, true)) || (rc = y.q.alloc(T * n.q * act, true)) ||
        (rc = y.q_latent.alloc(T * n.q_latent * act, true)) || (rc = y.qa.alloc(T * n.qa * act, true)) ||
        (rc = y.lat.alloc(T * n.lat * act, true)) || (rc = y.attn.alloc(T * n.attn * act, true)) || (rc = y.up.alloc(T * n.up * act, true)) ||
        (rc = m.xn_rows.alloc(rows * Wp * act, true)) || (rc = m.logits.alloc(rows * V * 4, true))) return rc;
    if ((rc = y.decay.alloc(T * n.decay * 4, true)) || (rc = y.gate.alloc(T * n.gate * act, true)) || (rc = y.delta_scratch.alloc(n.delta_scratch * 4, true)) ||
        (rc = y.delta_state.alloc(n.delta_state * 4, true)) || (rc = y.mix_conv.alloc(n.mix_conv * 4, true))) return rc;
    if (y.cfg.block == GPTRS_BLOCK_DEPTH && (rc = y.states.alloc((size_t)(c.n_layers + 1) * T * W * 4, true))) return rc;
    if ((rc = y.router.alloc(T * n.router * 4, true)) || (rc = y.sorted.alloc(T * n.sorted * act, true)) || (rc = y.gate_up.alloc(m.f32() ? T * n.gate_up * 4 : 0, true)) ||
        (rc = y.expert_y.alloc(T * n.expert_y * act, true)) || (rc = y.pair.alloc(T * n.top * 4, true)) || (rc = y.pair_weight.alloc(T * n.top * 4, true)) ||
        (rc = y.row_tiles.alloc(n.row_tiles * sizeof(gptrs_row_tile), true)) || (rc = y.n_row_tiles.alloc(4, true)) || (rc = y.moe_work.alloc(n.work * 4, true))) return rc;
    if ((int64_t)Vp != V && (rc = y.logits_pad.alloc(rows * Vp * 4, true))) return rc;
    if (!m.f32()) {
        const size_t tiles = (Vp + 127) / 128, r = std::min<size_t>(rows, 128);
        if ((rc = m.best_val.alloc(tiles * r * 4)) || (rc = m.best_idx.alloc(tiles * r * 4))) return rc;
        if (const char* e = getenv("GPTRS_FUSE_PICK")) m.fuse_pick = atoi(e) != 0;
    }
    y.state_stride = convs ? (size_t)c.max_seqs * 2 * (taps - 1) * W : 0;
    if ((rc = y.state.alloc(std::max<size_t>(1, (size_t)n.n_state * y.state_stride) * 4, true))) return rc;
    for (DevBuf* b : {&y.d_run_first, &y.d_run_last, &y.d_parity, &y.d_runs})
        if ((rc = b->alloc(T * 4, true))) return rc;
    GPTRS_CUDA_OK(cudaMallocHost(&y.h_tiles, T * 2 * 4));
    y.parity.assign(c.max_seqs, 0);
    if ((rc = alloc_step_buffers(m, 10))) return rc;
    if ((rc = m.kv_pool.alloc(n.pool, true))) return rc;
    if ((rc = alloc_page_tables(m))) return rc;
    // partial outputs of split keys: a launch splits only while its CTAs number at most the SMs
    size_t scratch = 0;
    for (const LayeredLayer& L : y.layers) {
        if (L.tiles < 0) continue;
        if (L.cfg.mixer == GPTRS_MIXER_LATENT_ATTENTION) scratch = std::max(scratch, gptrs_cuda_latent_scratch_bytes(&L.att, 1, sm_count() + 1));
        else {
            const int tile_rows = L.gatt.maps > 1 ? 64 : 128, per_split = L.gatt.kv_heads * ((L.gatt.heads / L.gatt.kv_heads + tile_rows - 1) / tile_rows);
            scratch = std::max(scratch, gptrs_cuda_grouped_scratch_bytes(&L.gatt, 1, 2 * sm_count() / per_split + 2));
        }
    }
    if ((rc = y.scratch.alloc(scratch))) return rc;
    GPTRS_CUDA_OK(cudaDeviceSynchronize());
    return GPTRS_OK;
}

namespace {

int copy_tiles(Model& m, Layered::TileSet& t) {
    GPTRS_CUDA_OK(cudaMemcpyAsync(t.row.p, m.lay->h_tiles, (size_t)t.n * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaMemcpyAsync(t.rows.p, m.lay->h_tiles + m.cfg.max_tokens, (size_t)t.n * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaStreamSynchronize(m.stream));   // the staging area is used again for the next list
    return GPTRS_OK;
}

}  // namespace

// Host rows -> runs (consecutive positions of one sequence), the halves of the convolution state they read, and query tiles.
// State and cache move forward only, so a run must start where its sequence stands.
int layered_stage_rows(Model& m, const int32_t* slots, const int32_t* positions, int n) {
    Layered& y = *m.lay;
    y.runs.clear();
    std::vector<char> seen(m.cfg.max_seqs, 0);
    for (int i = 0; i < n;) {
        int e = i + 1;
        while (e < n && slots[e] == slots[i] && positions[e] == positions[e - 1] + 1) ++e;
        GPTRS_REQUIRE(!seen[slots[i]], "the rows of a sequence must be consecutive positions in consecutive rows");
        GPTRS_REQUIRE(positions[i] == m.seq_len[slots[i]], "the rows of a sequence must continue at its length (reset_sequence starts a new one)");
        seen[slots[i]] = 1;
        y.runs.push_back(i);
        y.runs.push_back(e - i);
        i = e;
    }
    int32_t* st = m.h_stage;
    const int stride = m.stage_stride();
    const int n_runs = (int)y.runs.size() / 2;
    for (int r = 0; r < n_runs; ++r) {
        const int first = y.runs[2 * r], len = y.runs[2 * r + 1];
        for (int i = first; i < first + len; ++i) {
            st[6 * stride + i] = first;
            st[7 * stride + i] = first + len - 1;
            st[8 * stride + i] = y.parity[slots[i]];
        }
        st[9 * stride + r] = first;
    }
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_run_first.p, st + 6 * stride, (size_t)n * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_run_last.p, st + 7 * stride, (size_t)n * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_parity.p, st + 8 * stride, (size_t)n * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_runs.p, st + 9 * stride, (size_t)n_runs * 4, cudaMemcpyHostToDevice, m.stream));
    y.n_runs = n_runs;
    for (auto& t : y.tile_sets) {
        t->n = 0;
        for (size_t r = 0; r < y.runs.size(); r += 2)
            for (int o = 0; o < y.runs[r + 1]; o += t->tokens) {
                y.h_tiles[t->n] = y.runs[r] + o;
                y.h_tiles[m.cfg.max_tokens + t->n] = std::min(t->tokens, y.runs[r + 1] - o);
                ++t->n;
            }
        int rc = copy_tiles(m, *t);
        if (rc) return rc;
    }
    return GPTRS_OK;
}

// The generator's rows: slot b in row b, one token each.
int layered_stage_generator(Model& m, int batch) {
    Layered& y = *m.lay;
    int32_t* st = m.h_stage;
    const int stride = m.stage_stride();
    for (int b = 0; b < batch; ++b) { st[6 * stride + b] = b; st[8 * stride + b] = y.parity[b]; }
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_run_first.p, st + 6 * stride, (size_t)batch * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_run_last.p, st + 6 * stride, (size_t)batch * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_runs.p, st + 6 * stride, (size_t)batch * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_parity.p, st + 8 * stride, (size_t)batch * 4, cudaMemcpyHostToDevice, m.stream));
    y.n_runs = batch;
    for (int b = 0; b < batch; ++b) { y.h_tiles[b] = b; y.h_tiles[m.cfg.max_tokens + b] = 1; }
    for (auto& t : y.tile_sets) {
        t->n = batch;
        int rc = copy_tiles(m, *t);
        if (rc) return rc;
    }
    return GPTRS_OK;
}

// The first position whose cached keys some layer still reads from position `pos` on.
int layered_first_visible(const Model& m, int pos) {
    int first = pos;
    for (const LayeredLayer& L : m.lay->layers) {
        if (L.attends()) first = std::min(first, L.first_visible(pos));
    }
    return first;
}

// Beyond the widest mask a longer context changes nothing about the launches of a decode step.
int layered_graph_bucket(const Model& m, int bucket) {
    int widest = 1;
    for (const LayeredLayer& L : m.lay->layers) {
        if (L.attends()) widest = std::max(widest, L.span(bucket));
    }
    return (int)std::min<int64_t>(bucket, ((int64_t)widest + 511) / 512 * 512);
}

namespace {

// One forward pass: what its parts share.
struct Pass {
    Model& m;
    Layered& y;
    int T, max_ctx, act_dt;
    int64_t ldw;
    cudaStream_t st;
    static const float* fp(Tensor* t) { return t ? static_cast<const float*>(t->data) : nullptr; }

    unsigned char* pool(const LayeredLayer& L) const { return m.kv_pool.as<unsigned char>() + L.pool_off; }
    const int32_t* slot() const { return m.d_slot.as<int32_t>(); }
    const int32_t* pos() const { return m.d_pos.as<int32_t>(); }
    const int32_t* pages() const { return m.d_page_table.as<int32_t>(); }

    int latent(LayeredLayer& L) {
        const gptrs_latent_attention& a = L.att;
        const LayerWeights& w = *L.w;
        const Layered::Rope& rope = *y.ropes[L.rope];
        int rc;
        if ((rc = dense(m, w.qkv, y.h.p, y.qkv.p, T, {}))) return rc;
        const bool two_steps = a.q_rank > 0;
        const void* q = two_steps ? y.q.p : y.qkv.p;
        if (two_steps) {
            ++m.launches;
            if ((rc = gptrs_cuda_latent_append_keys(&a, y.qkv.p, pos(), slot(), pages(), m.cfg.max_pages_per_seq, fp(w.latent_norm), fp(w.q_norm), m.cfg.norm_eps,
                                                    rope.cos_t.as<float>(), rope.sin_t.as<float>(), y.q_latent.p, pool(L), T, st))) return rc;
            if ((rc = dense(m, w.uq, y.q_latent.p, y.q.p, T, {}))) return rc;
        }
        DenseOpts ok;
        ok.ldx = a.q_row; ok.x_step = a.q_head_stride; ok.ldy = (int64_t)a.heads * a.qa_head_stride; ok.y_step = a.qa_head_stride;
        if ((rc = dense(m, w.uk, q, y.qa.p, T, ok))) return rc;
        ++m.launches;
        if (two_steps) {
            if ((rc = gptrs_cuda_latent_rotate_queries(&a, q, pos(), rope.cos_t.as<float>(), rope.sin_t.as<float>(), y.qa.p, T, st))) return rc;
        } else if ((rc = gptrs_cuda_latent_append(&a, y.qkv.p, pos(), slot(), pages(), m.cfg.max_pages_per_seq, fp(w.latent_norm), m.cfg.norm_eps,
                                           rope.cos_t.as<float>(), rope.sin_t.as<float>(), y.qa.p, pool(L), T, st))) return rc;
        const Layered::TileSet* t = L.tiles >= 0 ? y.tile_sets[L.tiles].get() : nullptr;
        const int splits = t ? gptrs_cuda_latent_splits(&a, t->n, max_ctx) : 1;
        m.launches += splits > 1 ? 2 : 1;
        if ((rc = gptrs_cuda_latent_attention(&a, y.qa.p, pool(L), pages(), m.cfg.max_pages_per_seq, slot(), m.d_ctx.as<int32_t>(), fp(w.sink),
                                              t ? t->row.as<int32_t>() : nullptr, t ? t->rows.as<int32_t>() : nullptr, t ? t->n : 0, splits, y.lat.p, y.scratch.p,
                                              y.scratch.n, m.d_status.as<int32_t>(), T, st))) return rc;
        DenseOpts ov;
        ov.ldx = (int64_t)a.heads * a.lat_head_stride; ov.x_step = a.lat_head_stride; ov.ldy = w.out.k; ov.y_step = a.out_head_stride;
        if ((rc = dense(m, w.uv, y.lat.p, y.attn.p, T, ov))) return rc;
        return dense(m, w.out, y.attn.p, y.y.p, T, {});
    }

    int grouped(LayeredLayer& L) {
        const gptrs_grouped_attention& a = L.gatt;
        const LayerWeights& w = *L.w;
        int rc;
        if ((rc = dense(m, w.qkv, y.h.p, y.qkv.p, T, {}))) return rc;
        if (!a.shared_kv) ++m.launches;
        const void* q = y.qkv.p;
        if (L.prepared()) {
            gptrs_grouped_step s = {};
            s.d_qkv = y.qkv.p; s.d_conv = fp(w.qk_conv); s.d_q_gain = fp(w.q_gain); s.d_k_gain = fp(w.k_gain);
            s.d_conv_state = y.mix_conv.as<float>() + L.mix_conv_off;
            s.d_slot = slot(); s.d_pos = pos();
            s.d_run_first = y.d_run_first.as<int32_t>(); s.d_run_last = y.d_run_last.as<int32_t>(); s.d_parity = y.d_parity.as<int32_t>();
            s.d_page_table = pages(); s.max_pages = m.cfg.max_pages_per_seq; s.d_pool = pool(L); s.d_q = y.q.p; s.rows = T;
            if ((rc = gptrs_cuda_grouped_prepare(&a, &s, st))) return rc;
            q = y.q.p;
        } else if (!a.shared_kv && (rc = gptrs_cuda_grouped_append(&a, y.qkv.p, pos(), slot(), pages(), m.cfg.max_pages_per_seq, pool(L), T, st))) {
            return rc;
        }
        const Layered::TileSet* t = L.tiles >= 0 ? y.tile_sets[L.tiles].get() : nullptr;
        const int splits = t ? gptrs_cuda_grouped_splits(&a, T, t->n, max_ctx) : 1;
        m.launches += splits > 1 ? 2 : 1;
        if ((rc = gptrs_cuda_grouped_attention(&a, q, pool(L), pages(), m.cfg.max_pages_per_seq, slot(), m.d_ctx.as<int32_t>(), fp(w.r1), fp(w.r2), w.reach.as<int32_t>(),
                                               t ? t->row.as<int32_t>() : nullptr, t ? t->rows.as<int32_t>() : nullptr, t ? t->n : 0, splits, y.attn.p, y.scratch.p,
                                               y.scratch.n, m.d_status.as<int32_t>(), T, st))) return rc;
        return dense(m, w.out, y.attn.p, y.y.p, T, {});
    }

    int delta(LayeredLayer& L) {
        const gptrs_delta_rule& a = L.delta;
        const LayerWeights& w = *L.w;
        const size_t act = m.f32() ? 4 : 2;
        int rc;
        if ((rc = dense(m, w.qkv, y.h.p, y.qkv.p, T, {}))) return rc;
        auto column = [&](int off) { return y.qkv.as<unsigned char>() + off * act; };
        DenseOpts od;
        od.out_f32 = true; od.ldx = w.qkv.n; od.ldy = a.decay_row;
        if (a.decay_rank > 0 && (rc = dense(m, w.decay, column(a.a_offset), y.decay.p, T, od))) return rc;
        DenseOpts og;
        og.ldx = w.qkv.n; og.ldy = a.gate_row;
        if (a.gate_rank > 0 && (rc = dense(m, w.gate, column(a.g_offset), y.gate.p, T, og))) return rc;
        gptrs_delta_step s = {};
        s.d_proj = y.qkv.p; s.d_decay = y.decay.as<float>(); s.d_gate = y.gate.p;
        s.d_conv = fp(w.delta_conv); s.d_a_log = fp(w.a_log); s.d_dt_bias = fp(w.dt_bias); s.d_norm = fp(w.delta_norm);
        s.d_state = y.delta_state.as<float>() + L.delta_state_off;
        s.d_conv_state = y.mix_conv.as<float>() + L.mix_conv_off;
        s.d_slot = slot(); s.d_pos = pos();
        s.d_run_first = y.d_run_first.as<int32_t>(); s.d_run_last = y.d_run_last.as<int32_t>(); s.d_parity = y.d_parity.as<int32_t>();
        s.d_runs = y.d_runs.as<int32_t>(); s.n_runs = y.n_runs;
        s.d_out = y.attn.p; s.d_scratch = y.delta_scratch.as<float>(); s.rows = T; s.d_status = m.d_status.as<int32_t>();
        m.launches += y.n_runs == T ? 1 : 3;
        if ((rc = gptrs_cuda_delta_rule(&a, &s, st))) return rc;
        return dense(m, w.out, y.attn.p, y.y.p, T, {});
    }

    // leaves the experts' outputs in expert_y; the step behind sums them up
    int experts(LayeredLayer& L) {
        const LayerWeights& w = *L.w;
        gptrs_moe a = L.moe;
        a.tile_rows = expert_tile_rows(m, a, T);
        int rc;
        if (L.cfg.shared_ff > 0) {   // its output is a second one for the step behind
            DenseOpts os;
            os.act = 2;
            rc = L.cfg.expert_form == GPTRS_EXPERT_SWIGLU ? gated(w.shared_up, y.h.p, T, GPTRS_GATE_SILU, {}) : dense(m, w.shared_up, y.h.p, y.up.p, T, os);
            if (rc || (rc = dense(m, w.shared_down, y.up.p, y.y.p, T, {}))) return rc;
        }
        DenseOpts orr;
        orr.out_f32 = true;
        if ((rc = dense(m, w.router, y.h.p, y.router.p, T, orr))) return rc;
        m.launches += T > 128 ? 3 : 2;
        gptrs_row_tile* tiles = y.row_tiles.as<gptrs_row_tile>();
        int32_t* n_tiles = y.n_row_tiles.as<int32_t>();
        if ((rc = gptrs_cuda_moe_route(&a, y.router.as<float>(), w.router.n, fp(w.correction), y.h.p, act_dt, ldw, y.pair.as<int32_t>(), y.pair_weight.as<float>(), tiles, n_tiles,
                                       y.sorted.p, y.moe_work.as<int32_t>(), T, st))) return rc;
        DenseOpts o;
        o.tiles = tiles; o.n_tiles = n_tiles; o.tile_rows = a.tile_rows; o.max_tiles = gptrs_cuda_moe_max_tiles(&a, T);
        const int64_t pairs = (int64_t)T * a.top;
        if (L.cfg.expert_form == GPTRS_EXPERT_RELU2) {
            DenseOpts ou = o;
            ou.act = 2;
            rc = dense(m, w.up, y.sorted.p, y.up.p, pairs, ou);
        } else {
            rc = gated(w.up, y.sorted.p, pairs, GPTRS_GATE_SILU, o);
        }
        return rc ? rc : dense(m, w.down, y.up.p, y.expert_y.p, pairs, o);
    }

    // act(gate) up of a gated feed-forward -> y.up
    int gated(const DenseWeight& w, const void* x, int64_t rows, int gate, DenseOpts o) {
        if (!m.f32()) {
            o.gate = gate;
            return dense(m, w, x, y.up.p, rows, o);
        }
        const int rc = dense(m, w, x, y.gate_up.p, rows, o);
        ++m.launches;
        return rc ? rc : gptrs_cuda_gated_pairs_f32(y.gate_up.as<float>(), y.up.as<float>(), rows, w.n / 2, gate, st);
    }

    int mixer(LayeredLayer& L) {
        return L.cfg.mixer == GPTRS_MIXER_LATENT_ATTENTION ? latent(L) : L.cfg.mixer == GPTRS_MIXER_GROUPED_ATTENTION ? grouped(L) : delta(L);
    }
    int feed_forward(LayeredLayer& L) {
        if (L.cfg.mlp == GPTRS_MLP_EXPERTS) return experts(L);
        if (L.cfg.mlp == GPTRS_MLP_DENSE_GELU) {
            const int rg = gated(L.w->up, y.h.p, T, GPTRS_GATE_GELU_TANH, {});
            return rg ? rg : dense(m, L.w->down, y.up.p, y.y.p, T, {});
        }
        if (L.cfg.mlp == GPTRS_MLP_DENSE_POLY) {
            const LayerWeights& w = *L.w;
            int rp = dense(m, w.up, y.h.p, y.up.p, T, {});
            ++m.launches;
            if (!rp) rp = gptrs_cuda_poly_norm(y.up.p, fp(w.act), m.cfg.norm_eps, y.up.p, act_dt, T, L.cfg.d_ff, w.up.n, st);
            return rp ? rp : dense(m, w.down, y.up.p, y.y.p, T, {});
        }
        DenseOpts ou;
        ou.act = 1; ou.pos = L.w->act_pos; ou.neg = L.w->act_neg;
        int rc = dense(m, L.w->up, y.h.p, y.up.p, T, ou);
        return rc ? rc : dense(m, L.w->down, y.up.p, y.y.p, T, {});
    }
};

struct Capture {   // debug: the residual stream after every layer
    DevBuf buf;
    int begin(Model& m, int T) { return m.lay->h_residuals ? buf.alloc((size_t)m.cfg.n_layers * T * m.cfg.d_model * 4) : GPTRS_OK; }
    float* at(Model& m, int l, int T) { return buf.p ? buf.as<float>() + (size_t)l * T * m.cfg.d_model : nullptr; }
    int take(Model& m, int l, const float* x, int T) {
        const size_t n = (size_t)T * m.cfg.d_model;
        if (buf.p) GPTRS_CUDA_OK(cudaMemcpyAsync(buf.as<float>() + l * n, x, n * 4, cudaMemcpyDeviceToDevice, m.stream));
        return GPTRS_OK;
    }
    int end(Model& m) {
        if (!buf.p) return GPTRS_OK;
        GPTRS_CUDA_OK(cudaMemcpyAsync(m.lay->h_residuals, buf.p, buf.n, cudaMemcpyDeviceToHost, m.stream));
        GPTRS_CUDA_OK(cudaStreamSynchronize(m.stream));
        m.lay->h_residuals = nullptr;
        return GPTRS_OK;
    }
};

// norms on the outputs, sublayers that read the stream through short convolutions
int forward_output_norm(Pass& f, Capture& cap, int n_rows, bool rows_identity) {
    Model& m = f.m;
    Layered& y = f.y;
    const auto& c = m.cfg;
    const int W = c.d_model, T = f.T;
    float* x = m.hidden.as<float>();
    float* x_other = y.x2.as<float>();
    int rc;
    gptrs_conv_step base = {};
    base.y_dtype = f.act_dt; base.d_y = y.y.p; base.ldy = f.ldw;
    base.eps = c.norm_eps; base.taps = y.cfg.conv_taps;
    base.d_slot = f.slot(); base.d_pos = f.pos();
    base.d_run_first = y.d_run_first.as<int32_t>(); base.d_run_last = y.d_run_last.as<int32_t>(); base.d_parity = y.d_parity.as<int32_t>();
    base.d_h = y.h.p; base.h_dtype = f.act_dt; base.ldh = f.ldw;
    base.d_status = m.d_status.as<int32_t>();
    base.rows = T; base.dim = W;
    // closes a sublayer with its output norm (or opens the model with the normed embedding) and prepares the next one's input
    auto step = [&](Tensor* gamma, bool embed, Tensor* conv, int state) -> int {
        gptrs_conv_step s = base;
        if (embed) { s.d_embed = f.fp(m.tok_emb); s.d_tokens = m.d_tokens.as<int32_t>(); s.vocab = c.vocab; s.ldy = W; s.y_dtype = GPTRS_F32; }
        else s.d_x = x;
        s.d_x_out = x_other;
        s.d_gamma = f.fp(gamma);
        if (conv) { s.d_conv = f.fp(conv); s.d_state = y.state.as<float>() + (size_t)state * y.state_stride; }
        ++m.launches;
        int r = gptrs_cuda_post_norm_conv(&s, f.st);
        std::swap(x, x_other);
        return r;
    };
    if ((rc = step(y.embed_norm, true, y.layers[0].w->conv1, y.layers[0].state1))) return rc;
    for (int l = 0; l < c.n_layers; ++l) {
        LayeredLayer& L = y.layers[l];
        if ((rc = f.mixer(L))) return rc;
        const bool last = l + 1 == c.n_layers;
        Tensor* next = last ? nullptr : y.layers[l + 1].w->conv1;
        const int next_state = last ? 0 : y.layers[l + 1].state1;
        Tensor* gamma = L.w->norm1;
        if (L.cfg.mlp != GPTRS_MLP_NONE) {
            if ((rc = step(L.w->norm1, false, L.w->conv2, L.state2)) || (rc = f.feed_forward(L))) return rc;
            gamma = L.w->norm2;
        }
        if (!last) {
            if ((rc = step(gamma, false, next, next_state)) || (rc = cap.take(m, l, x, T))) return rc;
            continue;
        }
        ++m.launches;
        if ((rc = gptrs_cuda_post_norm_final(x, y.y.p, f.act_dt, f.ldw, f.fp(gamma), f.fp(m.final_g), c.norm_eps, rows_identity ? nullptr : m.d_rows.as<int32_t>(),
                                             m.xn_rows.p, f.act_dt, f.ldw, n_rows, W, f.st))) return rc;
        if (cap.buf.p && ((rc = step(gamma, false, nullptr, 0)) || (rc = cap.take(m, l, x, T)))) return rc;
    }
    return GPTRS_OK;
}

// norms on both sides of every sublayer
int forward_sandwich(Pass& f, Capture& cap, int n_rows, bool rows_identity) {
    Model& m = f.m;
    Layered& y = f.y;
    const auto& c = m.cfg;
    float* x = m.hidden.as<float>();
    gptrs_norm_step base = {};
    base.d_x = x; base.y_dtype = f.act_dt; base.eps = c.norm_eps;
    base.d_h = y.h.p; base.h_dtype = f.act_dt; base.ldh = f.ldw;
    base.d_status = m.d_status.as<int32_t>();
    base.rows = f.T; base.dim = c.d_model;
    auto launch = [&](const gptrs_norm_step& s) { ++m.launches; return gptrs_cuda_norm_step(&s, f.st); };
    // the output of the sublayer that has just run, normed by `gamma`
    auto closing = [&](const LayeredLayer& L, bool ff, Tensor* gamma) {
        gptrs_norm_step s = base;
        s.d_gamma_out = f.fp(gamma);
        if (ff && L.cfg.mlp == GPTRS_MLP_EXPERTS) {
            s.d_y = y.expert_y.p; s.ldy = L.w->down.n;
            s.d_pair = y.pair.as<int32_t>(); s.d_pair_weight = y.pair_weight.as<float>(); s.top = L.moe.top;
        } else {
            s.d_y = y.y.p; s.ldy = f.ldw;
        }
        return s;
    };
    gptrs_norm_step open = base;
    open.d_embed = f.fp(m.tok_emb); open.d_pos_embed = f.fp(m.pos_emb);
    open.d_tokens = m.d_tokens.as<int32_t>(); open.d_pos = f.pos();
    open.vocab = c.vocab; open.positions = y.cfg.learned_positions;
    open.d_gamma_in = f.fp(y.layers[0].w->norm1);
    int rc = launch(open);
    if (rc) return rc;
    for (int l = 0; l < c.n_layers; ++l) {
        LayeredLayer& L = y.layers[l];
        const bool last = l + 1 == c.n_layers, ff = L.cfg.mlp != GPTRS_MLP_NONE;
        if ((rc = f.mixer(L))) return rc;
        if (ff) {
            gptrs_norm_step s = closing(L, false, L.w->norm1b);
            s.d_gamma_in = f.fp(L.w->norm2);
            if ((rc = launch(s)) || (rc = f.feed_forward(L))) return rc;
        }
        gptrs_norm_step s = closing(L, ff, ff ? L.w->norm2b : L.w->norm1b);
        if (!last || cap.buf.p) {
            s.d_gamma_in = last ? nullptr : f.fp(y.layers[l + 1].w->norm1);
            if ((rc = launch(s)) || (rc = cap.take(m, l, x, f.T))) return rc;
        }
        if (last) {
            if (cap.buf.p) s.d_y = nullptr;   // the stream already holds it
            s.d_gamma_in = f.fp(m.final_g);
            s.d_rows = rows_identity ? nullptr : m.d_rows.as<int32_t>();
            s.d_h = m.xn_rows.p;
            s.rows = n_rows;
            if ((rc = launch(s))) return rc;
        }
    }
    return GPTRS_OK;
}

// norms in front of the sublayers, streams that are mixed behind them
int forward_pre_norm(Pass& f, Capture& cap, int n_rows, bool rows_identity) {
    Model& m = f.m;
    Layered& y = f.y;
    const auto& c = m.cfg;
    gptrs_stream_step base = {};
    base.d_x = m.hidden.as<float>(); base.streams = std::max(y.cfg.streams, 1);
    base.y_dtype = f.act_dt; base.eps = c.norm_eps;
    base.d_h = y.h.p; base.h_dtype = f.act_dt; base.ldh = f.ldw;
    base.d_status = m.d_status.as<int32_t>();
    base.rows = f.T; base.dim = c.d_model;
    auto launch = [&](const gptrs_stream_step& s) { ++m.launches; return gptrs_cuda_stream_step(&s, f.st); };
    // what a sublayer reads
    auto opens = [&](gptrs_stream_step& s, const LayeredLayer& L, int sub) {
        s.d_in = f.fp(L.w->streams[sub].in);
        s.d_gamma_in = f.fp(sub ? L.w->norm2 : L.w->norm1);
    };
    // the output of the sublayer that has just run
    auto closing = [&](const LayeredLayer& L, int sub) {
        gptrs_stream_step s = base;
        s.d_mix = f.fp(L.w->streams[sub].mix); s.d_out = f.fp(L.w->streams[sub].out);
        if (sub && L.cfg.mlp == GPTRS_MLP_EXPERTS) {
            s.d_y = y.expert_y.p; s.ldy = L.w->down.n;
            s.d_pair = y.pair.as<int32_t>(); s.d_pair_weight = y.pair_weight.as<float>(); s.top = L.moe.top;
            if (L.cfg.shared_ff > 0) { s.d_add = y.y.p; s.ld_add = f.ldw; }
        } else {
            s.d_y = y.y.p; s.ldy = f.ldw;
        }
        return s;
    };
    gptrs_stream_step open = base;
    open.d_embed = f.fp(m.tok_emb); open.embed_scale = y.cfg.embed_scale; open.d_tokens = m.d_tokens.as<int32_t>(); open.vocab = c.vocab;
    opens(open, y.layers[0], 0);
    int rc = launch(open);
    if (rc) return rc;
    for (int l = 0; l < c.n_layers; ++l) {
        LayeredLayer& L = y.layers[l];
        const bool last = l + 1 == c.n_layers, ff = L.cfg.mlp != GPTRS_MLP_NONE;
        if ((rc = f.mixer(L))) return rc;
        if (ff) {
            gptrs_stream_step s = closing(L, 0);
            opens(s, L, 1);
            if ((rc = launch(s)) || (rc = f.feed_forward(L))) return rc;
        }
        gptrs_stream_step s = closing(L, ff ? 1 : 0);
        if (!last || cap.buf.p) {
            if (!last) opens(s, y.layers[l + 1], 0);
            s.d_sum = cap.at(m, l, f.T);
            if ((rc = launch(s))) return rc;
        }
        if (last) {
            if (cap.buf.p) { s.d_y = s.d_add = nullptr; s.d_pair = nullptr; s.d_sum = nullptr; }   // the streams already hold it
            s.d_gamma_in = f.fp(m.final_g);
            s.d_rows = rows_identity ? nullptr : m.d_rows.as<int32_t>();
            s.d_h = m.xn_rows.p;
            s.rows = n_rows;
            if ((rc = launch(s))) return rc;
        }
    }
    return GPTRS_OK;
}

// norms on the outputs in groups, a weighted average of all results so far behind every layer
int forward_depth(Pass& f, Capture& cap, int n_rows, bool rows_identity) {
    Model& m = f.m;
    Layered& y = f.y;
    const auto& c = m.cfg;
    float *x = y.states.as<float>(), *running = m.hidden.as<float>();   // the first layer reads the embedding
    gptrs_depth_step base = {};
    base.y_dtype = f.act_dt; base.mult = y.cfg.residual_mult; base.groups = y.cfg.norm_groups; base.eps = c.norm_eps;
    base.d_states = y.states.as<float>(); base.state_stride = (int64_t)c.max_tokens * c.d_model;
    base.d_h = y.h.p; base.h_dtype = f.act_dt; base.ldh = f.ldw;
    base.d_status = m.d_status.as<int32_t>();
    base.rows = f.T; base.dim = c.d_model;
    auto launch = [&](const gptrs_depth_step& s) { ++m.launches; return gptrs_cuda_depth_step(&s, f.st); };
    // the output of the sublayer that has just run
    auto closing = [&](const LayeredLayer& L, int sub) {
        gptrs_depth_step s = base;
        s.d_x = x; s.d_x_out = running;
        s.d_gamma_out = f.fp(sub ? L.w->norm2 : L.w->norm1);
        if (sub && L.cfg.mlp == GPTRS_MLP_EXPERTS) {
            s.d_y = y.expert_y.p; s.ldy = L.w->down.n;
            s.d_pair = y.pair.as<int32_t>(); s.d_pair_weight = y.pair_weight.as<float>(); s.top = L.moe.top;
            if (L.cfg.shared_ff > 0) { s.d_add = y.y.p; s.ld_add = f.ldw; }
            if (L.cfg.shared_gate) { s.d_add_gate = y.router.as<float>() + L.moe.experts; s.ld_add_gate = L.w->router.n; }
        } else {
            s.d_y = y.y.p; s.ldy = f.ldw;
        }
        return s;
    };
    gptrs_depth_step open = base;
    open.d_embed = f.fp(m.tok_emb); open.d_tokens = m.d_tokens.as<int32_t>(); open.vocab = c.vocab;
    open.d_x_out = x;
    int rc = launch(open);
    if (rc) return rc;
    for (int l = 0; l < c.n_layers; ++l) {
        LayeredLayer& L = y.layers[l];
        const bool last = l + 1 == c.n_layers, ff = L.cfg.mlp != GPTRS_MLP_NONE;
        if ((rc = f.mixer(L))) return rc;
        if (ff) {
            if ((rc = launch(closing(L, 0)))) return rc;
            x = running;
            if ((rc = f.feed_forward(L))) return rc;
        }
        gptrs_depth_step s = closing(L, ff ? 1 : 0);
        s.d_weights = f.fp(L.w->dwa); s.n_states = l + 1;
        if (!last || cap.buf.p) {
            if (last) s.d_h = nullptr;
            if ((rc = launch(s)) || (rc = cap.take(m, l, running, f.T))) return rc;
            x = running;
        }
        if (last) {
            if (cap.buf.p) { s.d_x = running; s.d_y = s.d_add = nullptr; s.d_pair = nullptr; s.d_weights = nullptr; }   // the stream already holds it
            s.d_gamma_in = f.fp(m.final_g);
            s.d_rows = rows_identity ? nullptr : m.d_rows.as<int32_t>();
            if (rows_identity) s.d_x_out = nullptr;
            s.d_h = m.xn_rows.p;
            s.rows = n_rows;
            if ((rc = launch(s))) return rc;
        }
    }
    return GPTRS_OK;
}

}  // namespace

int layered_forward(Model& m, int T, int max_ctx, int n_rows, bool rows_identity, float temperature, bool skip_logits) {
    Layered& y = *m.lay;
    const auto& c = m.cfg;
    Pass f = {m, y, T, max_ctx, m.f32() ? GPTRS_F32 : GPTRS_BF16, m.f32() ? (int64_t)c.d_model : pad8(c.d_model), m.stream};
    cudaStream_t st = m.stream;
    Capture cap;
    int rc = cap.begin(m, T);
    if (!rc) {
        const auto forward = y.cfg.block == GPTRS_BLOCK_SANDWICH ? forward_sandwich : y.cfg.block == GPTRS_BLOCK_PRE_NORM ? forward_pre_norm
                           : y.cfg.block == GPTRS_BLOCK_DEPTH ? forward_depth : forward_output_norm;
        rc = forward(f, cap, n_rows, rows_identity);
    }
    if (!rc) rc = cap.end(m);
    if (rc) return rc;
    const bool padded = y.head.n != c.vocab;
    const bool pick = skip_logits && m.fuse_pick && temperature <= 0.f && !m.f32() && !padded && n_rows <= 128;
    DenseOpts oh;
    oh.out_f32 = true; oh.softcap = y.cfg.logit_softcap; oh.pick = pick;
    if ((rc = dense(m, y.head, m.xn_rows.p, padded ? y.logits_pad.p : m.logits.p, n_rows, oh))) return rc;
    if (padded) {
        CompactParams cp = {y.logits_pad.as<float>(), m.logits.as<float>(), (int)y.head.n, c.vocab};
        ++m.launches;
        if ((rc = launch_kernel(compact_rows_kernel, dim3(n_rows), dim3(256), 0, st, 1, cp))) return rc;
    }
    ++m.launches;
    if (pick) return gptrs_cuda_pick_best(m.best_val.as<float>(), m.best_idx.as<int32_t>(), (c.vocab + 127) / 128, n_rows, m.d_sampled.as<int32_t>(), st);
    return gptrs_cuda_sample_rows_top_k(m.logits.as<float>(), n_rows, c.vocab, temperature, m.top_k, m.sample_seed, m.d_sampled.as<int32_t>(), st);
}

}  // namespace gptrs
