// Models whose layers are configured one by one (engine kind "layered"): weight packing, cache and state set-up and the forward
// pass. A layer is a mixer (latent attention over the paged cache, latent_attention.cu) and an optional feed-forward; the step
// between two sublayers (output norm, residual sum, short convolution with its per-sequence state) is post_norm_conv.cu, the
// matmuls are dense_bf16.cu or, in f32 mode, dense_f32.cu. Slots, pages, graphs, sampling and the generator are the engine's.
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

// One block of a source leaf and where it goes in the packed weight: rows n (with a step between batches) and columns k.
struct Piece {
    int64_t batch, n, k;        // block: batch x n output channels x k inputs
    int64_t src, sb, sn, sk;    // first element and strides in the leaf
    int64_t row, row_b;         // first output channel in the packed weight, step between batches
    int64_t col, col_b;         // first input column, step between batches
    int64_t mat_b;              // step between batches in whole matrices (1: a batch entry is a matrix of its own)
};

// Packs the pieces of the leaves `names` (name i holds pieces[i]) into a weight of `batch` matrices n x k: bf16 [n][k] with
// both sizes padded to 8 and zeros in between, or f32 [k][n]. Memoised by the stable ids of the leaves like every derived layout.
int pack_weight(Model& m, const std::vector<std::string>& names, const std::vector<std::vector<int64_t>>& dims, const std::vector<std::vector<Piece>>& pieces,
                int64_t batch, int64_t n, int64_t k, const std::string& bias, const std::string& tag, DenseWeight* w) {
    const bool bf16 = !m.f32();
    w->batch = batch; w->n = bf16 ? pad8(n) : n; w->k = bf16 ? pad8(k) : k;
    int rc = GPTRS_OK;
    if (!bias.empty()) {
        Tensor* raw = nullptr;
        if ((rc = get_raw(m, bias, {n}, &raw))) return rc;
        int64_t bd[1] = {w->n};
        if (!(rc = tensor_alloc(GPTRS_F32, 1, bd, true, &w->bias)))
            if (cudaMemcpy(w->bias->data, raw->data, (size_t)n * 4, cudaMemcpyDeviceToDevice) != cudaSuccess) rc = fail(GPTRS_EXECUTION, "bias copy failed");
        tensor_release(raw);
        if (rc) return rc;
    }
    std::vector<Tensor*> leaves(names.size(), nullptr);
    auto drop = [&]() { for (Tensor* t : leaves) tensor_release(t); };
    for (size_t i = 0; i < names.size(); ++i)
        if ((rc = get_raw(m, names[i], dims[i], &leaves[i]))) { drop(); return rc; }
    std::pair<uint64_t, uint64_t> key = m.ids[names[0]];
    for (size_t i = 1; i < names.size(); ++i) { key.first ^= m.ids[names[i]].first * 31; key.second ^= m.ids[names[i]].second * 131; }
    const auto did = derived_id(key, (bf16 ? "dense_bf16:" : "dense_f32:") + tag + ":" + std::to_string(batch) + "x" + std::to_string(w->n) + "x" + std::to_string(w->k));
    const size_t need = (size_t)batch * w->n * w->k * (bf16 ? 2 : 4);
    if (Tensor* hit = param_lookup(did.first, did.second)) {
        if (hit->bytes == need) { w->w = hit; ++m.memo_hits; drop(); return GPTRS_OK; }
        tensor_release(hit);
    }
    int64_t wd[3] = {batch, bf16 ? w->n : w->k, bf16 ? w->k : w->n};
    if ((rc = tensor_alloc(bf16 ? GPTRS_BF16 : GPTRS_F32, 3, wd, true, &w->w))) { drop(); return rc; }
    if (cudaDeviceSynchronize() != cudaSuccess) { drop(); return fail(GPTRS_EXECUTION, "packing a weight failed"); }   // the zero fill is done
    for (size_t i = 0; i < names.size(); ++i)
        for (const Piece& p : pieces[i]) {
            PackParams pp = {};
            const int64_t dn = bf16 ? w->k : 1, dk = bf16 ? 1 : w->n;
            pp.src = static_cast<const float*>(leaves[i]->data) + p.src;
            pp.dst = static_cast<unsigned char*>(w->w->data) + (p.row * dn + p.col * dk) * (bf16 ? 2 : 4);
            pp.n = p.n; pp.k = p.k; pp.total = p.batch * p.n * p.k;
            pp.sb = p.sb; pp.sn = p.sn; pp.sk = p.sk;
            pp.db = p.row_b * dn + p.col_b * dk + p.mat_b * w->n * w->k; pp.dn = dn; pp.dk = dk;
            pp.bf16 = bf16;
            const int64_t blocks = (pp.total + 255) / 256;
            pack_kernel<<<(unsigned)(blocks < 4096 ? blocks : 4096), 256, 0, m.stream>>>(pp);
        }
    if (cudaGetLastError() != cudaSuccess || cudaStreamSynchronize(m.stream) != cudaSuccess) rc = fail(GPTRS_EXECUTION, "packing a weight failed");
    drop();
    if (rc) return rc;
    param_store(did.first, did.second, w->w);
    ++m.quantised_now;
    return GPTRS_OK;
}
// a plain [out][in] leaf
int pack_plain(Model& m, const std::string& name, int64_t n, int64_t k, const std::string& bias, DenseWeight* w) {
    return pack_weight(m, {name}, {{n, k}}, {{{1, n, k, 0, 0, k, 1, 0, 0, 0, 0, 0}}}, 1, n, k, bias, "plain", w);
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
};
int dense(Model& m, const DenseWeight& w, const void* x, void* y, int rows, const DenseOpts& o) {
    ++m.launches;
    gptrs_dense_epilogue ep = {};
    ep.out_dtype = (m.f32() || o.out_f32) ? GPTRS_F32 : GPTRS_BF16;
    ep.d_bias = w.bias ? static_cast<const float*>(w.bias->data) : nullptr;
    ep.act = o.act; ep.act_pos = o.pos; ep.act_neg = o.neg; ep.softcap = o.softcap;
    ep.ldx = o.ldx; ep.ldy = o.ldy; ep.batch = w.batch; ep.x_step = o.x_step; ep.y_step = o.y_step;
    if (o.pick) { ep.d_best_val = m.best_val.as<float>(); ep.d_best_idx = m.best_idx.as<int32_t>(); ep.skip_store = 1; }
    ep.d_status = m.d_status.as<int32_t>();
    if (m.f32())
        return gptrs_cuda_dense_f32(static_cast<const float*>(x), static_cast<const float*>(w.w->data), static_cast<float*>(y), rows, w.n, w.k, &ep, m.stream);
    return gptrs_cuda_dense_bf16(x, w.w->data, y, rows, w.n, w.k, &ep, m.stream);
}

float softplus(float x) { return x > 20.f ? x : (float)std::log1p(std::exp((double)x)); }

}  // namespace

int layered_check_config(const gptrs_model_config& c) {
    GPTRS_REQUIRE(c.weight_mode == kModeF32 || c.weight_mode == kModeBf16, "the layered kind runs with f32 or bf16 weights");
    GPTRS_REQUIRE(c.n_layers > 0 && c.d_model > 0 && c.vocab > 0 && c.context_length > 0, "bad model dimensions");
    GPTRS_REQUIRE(c.max_seqs > 0 && c.max_tokens > 0 && c.kv_pages > 0 && c.max_pages_per_seq > 0, "max_seqs, max_tokens and the page counts must be positive");
    if (c.tp_size > 1) return fail(GPTRS_UNIMPLEMENTED, "tensor parallelism is implemented for the ministral kind");
    return GPTRS_OK;
}

int layered_finalize(Model& m, bool drop_leaves) {
    Layered& y = *m.lay;
    const auto& c = m.cfg;
    GPTRS_REQUIRE(!y.layers.empty(), "call gptrs_cuda_model_set_layers before finalize");
    const int64_t W = c.d_model, V = c.vocab, taps = y.cfg.conv_taps;
    int rc;
    if ((rc = get_raw(m, "embed", {V, W}, &m.tok_emb)) || (rc = get_raw(m, "embed.norm", {W}, &y.embed_norm)) ||
        (rc = get_raw(m, "final.norm", {W}, &m.final_g))) return rc;
    if ((rc = pack_plain(m, "head", V, W, "", &y.head))) return rc;
    const size_t act = m.f32() ? 4 : 2;
    int64_t qkv_w = 0, qa_w = 0, lat_w = 0, attn_w = 0, up_w = 0;
    size_t pool = 0;
    int n_state = 0;
    for (int l = 0; l < c.n_layers; ++l) {
        LayeredLayer& L = y.layers[l];
        const gptrs_latent_attention& a = L.att;
        const std::string p = "l" + std::to_string(l) + ".", x = p + "mix.";
        const int64_t H = a.heads, dim = a.dim, rot = a.rot_dim, rank = a.kv_rank, vd = a.vdim;
        if ((rc = get_raw(m, p + "norm1", {W}, &L.norm1)) || (rc = get_raw(m, p + "canon1", {W, taps}, &L.conv1)) ||
            (rc = get_raw(m, x + "dkv.norm", {rank}, &L.latent_norm))) return rc;
        // queries and the down-projection in one weight, laid out as the attention kernels expect a projection row
        if ((rc = pack_weight(m, {x + "q", x + "dkv"}, {{H * (dim + rot), W}, {rank + rot, W}},
                              {{{H, dim, W, 0, (dim + rot) * W, W, 1, 0, a.q_head_stride, 0, 0, 0},
                                {H, rot, W, dim * W, (dim + rot) * W, W, 1, a.q_rot_offset, a.q_head_stride, 0, 0, 0}},
                               {{1, rank, W, 0, 0, W, 1, a.dkv_offset, 0, 0, 0, 0}, {1, rot, W, rank * W, 0, W, 1, a.rot_offset, 0, 0, 0, 0}}},
                              1, a.q_row, W, "", "latent_qkv", &L.qkv))) return rc;
        // absorbed query: per head [rank] <- [dim], the stored key projection transposed
        if ((rc = pack_weight(m, {x + "uk"}, {{H * dim, rank}}, {{{H, rank, dim, 0, dim * rank, 1, rank, 0, 0, 0, 0, 1}}}, H, rank, dim, "", "latent_uk", &L.uk))) return rc;
        if ((rc = pack_weight(m, {x + "uv"}, {{H * vd, rank}}, {{{H, vd, rank, 0, vd * rank, rank, 1, 0, 0, 0, 0, 1}}}, H, vd, rank, "", "latent_uv", &L.uv))) return rc;
        if ((rc = pack_weight(m, {x + "o"}, {{W, H * vd}}, {{{H, W, vd, 0, vd, H * vd, 1, 0, 0, 0, a.out_head_stride, 0}}}, 1, W, H * a.out_head_stride, "", "latent_o", &L.out))) return rc;
        L.state1 = n_state++;
        if (L.cfg.mlp == GPTRS_MLP_DENSE_XIELU) {
            const int64_t F = L.cfg.d_ff;
            if ((rc = get_raw(m, p + "norm2", {W}, &L.norm2)) || (rc = get_raw(m, p + "canon2", {W, taps}, &L.conv2))) return rc;
            if ((rc = pack_plain(m, p + "mlp.up", F, W, p + "mlp.up.b", &L.up)) || (rc = pack_plain(m, p + "mlp.down", W, F, p + "mlp.down.b", &L.down))) return rc;
            Tensor* pq = nullptr;
            float v[2];
            if ((rc = get_raw(m, p + "mlp.act", {2}, &pq))) return rc;
            const cudaError_t e = cudaMemcpy(v, pq->data, 8, cudaMemcpyDeviceToHost);
            tensor_release(pq);
            GPTRS_CUDA_OK(e);
            L.act_pos = softplus(v[0]);
            L.act_neg = 0.5f + softplus(v[1]);
            L.state2 = n_state++;
            up_w = std::max(up_w, L.up.n);
        }
        if (drop_leaves)
            for (const char* s : {"mix.q", "mix.dkv", "mix.uk", "mix.uv", "mix.o", "mlp.up", "mlp.down"}) {
                auto it = m.raw.find(p + s);
                if (it != m.raw.end()) { tensor_release(it->second); m.raw.erase(it); }
            }
        qkv_w = std::max(qkv_w, L.qkv.n);
        qa_w = std::max(qa_w, H * (int64_t)a.qa_head_stride);
        lat_w = std::max(lat_w, H * (int64_t)a.lat_head_stride);
        attn_w = std::max(attn_w, L.out.k);
        L.pool_off = pool;
        pool += (size_t)c.kv_pages * a.page_bytes;
        y.max_window = std::max(y.max_window, a.window);
        // rotation tables, one pair per distinct (base, dims); angles in double, rounded once
        L.rope = -1;
        for (size_t i = 0; i < y.ropes.size(); ++i)
            if (y.ropes[i]->base == L.cfg.rope_base && y.ropes[i]->dims == a.rot_dims) L.rope = (int)i;
        if (L.rope < 0) {
            auto r = std::make_unique<Layered::Rope>();
            r->base = L.cfg.rope_base; r->dims = a.rot_dims;
            const int half = a.rot_dims / 2;
            std::vector<float> cs((size_t)c.context_length * half), sn(cs.size());
            for (int i = 0; i < half; ++i) {
                const double f = std::pow(r->base, -2.0 * i / a.rot_dims);
                for (int q = 0; q < c.context_length; ++q) {
                    cs[(size_t)q * half + i] = (float)std::cos(q * f);
                    sn[(size_t)q * half + i] = (float)std::sin(q * f);
                }
            }
            if (half > 0) {
                if ((rc = r->cos_t.alloc(cs.size() * 4)) || (rc = r->sin_t.alloc(sn.size() * 4))) return rc;
                GPTRS_CUDA_OK(cudaMemcpy(r->cos_t.p, cs.data(), cs.size() * 4, cudaMemcpyHostToDevice));
                GPTRS_CUDA_OK(cudaMemcpy(r->sin_t.p, sn.data(), sn.size() * 4, cudaMemcpyHostToDevice));
            }
            L.rope = (int)y.ropes.size();
            y.ropes.push_back(std::move(r));
        }
        // GPTRS_LATENT_TC=0 keeps the plain attention kernel
        static const bool tc_on = [] { const char* e = getenv("GPTRS_LATENT_TC"); return !e || atoi(e) != 0; }();
        const int tokens = tc_on ? gptrs_cuda_latent_tile_tokens(&a) : 0;
        L.tiles = -1;
        if (tokens > 0) {
            for (size_t i = 0; i < y.tile_sets.size(); ++i)
                if (y.tile_sets[i]->tokens == tokens) L.tiles = (int)i;
            if (L.tiles < 0) {
                auto t = std::make_unique<Layered::TileSet>();
                t->tokens = tokens;
                if ((rc = t->row.alloc((size_t)c.max_tokens * 4, true)) || (rc = t->rows.alloc((size_t)c.max_tokens * 4, true))) return rc;
                L.tiles = (int)y.tile_sets.size();
                y.tile_sets.push_back(std::move(t));
            }
        }
    }
    if (drop_leaves) {
        auto it = m.raw.find("head");
        if (it != m.raw.end()) { tensor_release(it->second); m.raw.erase(it); }
    }
    // activations (zeroed: padding columns that no kernel writes are multiplied by zero weights and must be finite)
    const size_t T = c.max_tokens, Wp = m.f32() ? W : pad8(W), Vp = y.head.n, rows = m.max_rows();
    if ((rc = m.hidden.alloc(T * W * 4, true)) || (rc = y.x2.alloc(T * W * 4, true)) || (rc = y.h.alloc(T * Wp * act, true)) ||
        (rc = y.y.alloc(T * Wp * act, true)) || (rc = y.qkv.alloc(T * qkv_w * act, true)) || (rc = y.qa.alloc(T * qa_w * act, true)) ||
        (rc = y.lat.alloc(T * lat_w * act, true)) || (rc = y.attn.alloc(T * attn_w * act, true)) || (rc = y.up.alloc(T * up_w * act, true)) ||
        (rc = m.xn_rows.alloc(rows * Wp * act, true)) || (rc = m.logits.alloc(rows * V * 4, true))) return rc;
    if ((int64_t)Vp != V && (rc = y.logits_pad.alloc(rows * Vp * 4, true))) return rc;
    if (!m.f32()) {
        const size_t tiles = (Vp + 127) / 128, r = std::min<size_t>(rows, 128);
        if ((rc = m.best_val.alloc(tiles * r * 4)) || (rc = m.best_idx.alloc(tiles * r * 4))) return rc;
        if (const char* e = getenv("GPTRS_FUSE_PICK")) m.fuse_pick = atoi(e) != 0;
    }
    y.state_stride = (size_t)c.max_seqs * 2 * (taps - 1) * W;
    if ((rc = y.state.alloc(std::max<size_t>(1, (size_t)n_state * y.state_stride) * 4, true))) return rc;
    for (DevBuf* b : {&y.d_run_first, &y.d_run_last, &y.d_parity})
        if ((rc = b->alloc(T * 4, true))) return rc;
    GPTRS_CUDA_OK(cudaMallocHost(&y.h_tiles, T * 2 * 4));
    y.parity.assign(c.max_seqs, 0);
    if ((rc = alloc_step_buffers(m, 9))) return rc;
    if ((rc = m.kv_pool.alloc(pool, true))) return rc;
    if ((rc = alloc_page_tables(m))) return rc;
    // partial outputs of split keys: a launch splits only while its CTAs number at most the SMs
    size_t scratch = 0;
    for (const LayeredLayer& L : y.layers)
        if (L.tiles >= 0) scratch = std::max(scratch, gptrs_cuda_latent_scratch_bytes(&L.att, 1, sm_count() + 1));
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
// Convolution state and cache move forward only, so a run must start where its sequence stands.
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
    for (size_t r = 0; r < y.runs.size(); r += 2)
        for (int i = y.runs[r]; i < y.runs[r] + y.runs[r + 1]; ++i) {
            st[6 * stride + i] = y.runs[r];
            st[7 * stride + i] = y.runs[r] + y.runs[r + 1] - 1;
            st[8 * stride + i] = y.parity[slots[i]];
        }
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_run_first.p, st + 6 * stride, (size_t)n * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_run_last.p, st + 7 * stride, (size_t)n * 4, cudaMemcpyHostToDevice, m.stream));
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_parity.p, st + 8 * stride, (size_t)n * 4, cudaMemcpyHostToDevice, m.stream));
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
    GPTRS_CUDA_OK(cudaMemcpyAsync(y.d_parity.p, st + 8 * stride, (size_t)batch * 4, cudaMemcpyHostToDevice, m.stream));
    for (int b = 0; b < batch; ++b) { y.h_tiles[b] = b; y.h_tiles[m.cfg.max_tokens + b] = 1; }
    for (auto& t : y.tile_sets) {
        t->n = batch;
        int rc = copy_tiles(m, *t);
        if (rc) return rc;
    }
    return GPTRS_OK;
}

// Beyond the widest window a longer context changes nothing about the launches of a decode step.
int layered_graph_bucket(const Model& m, int bucket) { return std::min(bucket, (m.lay->max_window + 511) / 512 * 512); }

int layered_forward(Model& m, int T, int max_ctx, int n_rows, bool rows_identity, float temperature, bool skip_logits) {
    Layered& y = *m.lay;
    const auto& c = m.cfg;
    const int W = c.d_model, taps = y.cfg.conv_taps;
    const int act_dt = m.f32() ? GPTRS_F32 : GPTRS_BF16;
    const int64_t ldw = m.f32() ? W : pad8(W);
    cudaStream_t st = m.stream;
    float* x = m.hidden.as<float>();
    float* x_other = y.x2.as<float>();
    int rc;
    gptrs_conv_step base = {};
    base.y_dtype = act_dt; base.d_y = y.y.p; base.ldy = ldw;
    base.eps = c.norm_eps; base.taps = taps;
    base.d_slot = m.d_slot.as<int32_t>(); base.d_pos = m.d_pos.as<int32_t>();
    base.d_run_first = y.d_run_first.as<int32_t>(); base.d_run_last = y.d_run_last.as<int32_t>(); base.d_parity = y.d_parity.as<int32_t>();
    base.d_h = y.h.p; base.h_dtype = act_dt; base.ldh = ldw;
    base.d_status = m.d_status.as<int32_t>();
    base.rows = T; base.dim = W;
    auto fp = [](Tensor* t) { return static_cast<const float*>(t->data); };
    // closes a sublayer with its output norm (or opens the model with the normed embedding) and prepares the next one's input
    auto step = [&](Tensor* gamma, bool embed, Tensor* conv, int state) -> int {
        gptrs_conv_step s = base;
        if (embed) { s.d_embed = fp(m.tok_emb); s.d_tokens = m.d_tokens.as<int32_t>(); s.vocab = c.vocab; s.ldy = W; s.y_dtype = GPTRS_F32; }
        else s.d_x = x;
        s.d_x_out = x_other;
        s.d_gamma = fp(gamma);
        if (conv) { s.d_conv = fp(conv); s.d_state = y.state.as<float>() + (size_t)state * y.state_stride; }
        ++m.launches;
        int r = gptrs_cuda_post_norm_conv(&s, st);
        std::swap(x, x_other);
        return r;
    };
    DevBuf captured;
    if (y.h_residuals && (rc = captured.alloc((size_t)c.n_layers * T * W * 4))) return rc;
    auto capture = [&](int l) -> int {
        if (captured.p) GPTRS_CUDA_OK(cudaMemcpyAsync(captured.as<float>() + (size_t)l * T * W, x, (size_t)T * W * 4, cudaMemcpyDeviceToDevice, st));
        return GPTRS_OK;
    };

    if ((rc = step(y.embed_norm, true, y.layers[0].conv1, y.layers[0].state1))) return rc;
    for (int l = 0; l < c.n_layers; ++l) {
        LayeredLayer& L = y.layers[l];
        const gptrs_latent_attention& a = L.att;
        const Layered::Rope& rope = *y.ropes[L.rope];
        unsigned char* pool = m.kv_pool.as<unsigned char>() + L.pool_off;
        DenseOpts o;
        if ((rc = dense(m, L.qkv, y.h.p, y.qkv.p, T, o))) return rc;
        DenseOpts ok;
        ok.ldx = L.qkv.n; ok.x_step = a.q_head_stride; ok.ldy = (int64_t)a.heads * a.qa_head_stride; ok.y_step = a.qa_head_stride;
        if ((rc = dense(m, L.uk, y.qkv.p, y.qa.p, T, ok))) return rc;
        ++m.launches;
        if ((rc = gptrs_cuda_latent_append(&a, y.qkv.p, base.d_pos, base.d_slot, m.d_page_table.as<int32_t>(), c.max_pages_per_seq, fp(L.latent_norm), c.norm_eps,
                                           rope.cos_t.as<float>(), rope.sin_t.as<float>(), y.qa.p, pool, T, st))) return rc;
        const Layered::TileSet* t = L.tiles >= 0 ? y.tile_sets[L.tiles].get() : nullptr;
        const int splits = t ? gptrs_cuda_latent_splits(&a, t->n, max_ctx) : 1;
        m.launches += splits > 1 ? 2 : 1;
        if ((rc = gptrs_cuda_latent_attention(&a, y.qa.p, pool, m.d_page_table.as<int32_t>(), c.max_pages_per_seq, base.d_slot, m.d_ctx.as<int32_t>(),
                                              t ? t->row.as<int32_t>() : nullptr, t ? t->rows.as<int32_t>() : nullptr, t ? t->n : 0, splits, y.lat.p, y.scratch.p,
                                              y.scratch.n, base.d_status, T, st))) return rc;
        DenseOpts ov;
        ov.ldx = (int64_t)a.heads * a.lat_head_stride; ov.x_step = a.lat_head_stride; ov.ldy = L.out.k; ov.y_step = a.out_head_stride;
        if ((rc = dense(m, L.uv, y.lat.p, y.attn.p, T, ov))) return rc;
        if ((rc = dense(m, L.out, y.attn.p, y.y.p, T, o))) return rc;
        const bool last = l + 1 == c.n_layers;
        Tensor* next = last ? nullptr : y.layers[l + 1].conv1;
        const int next_state = last ? 0 : y.layers[l + 1].state1;
        Tensor* gamma = L.norm1;
        if (L.cfg.mlp == GPTRS_MLP_DENSE_XIELU) {
            if ((rc = step(L.norm1, false, L.conv2, L.state2))) return rc;
            DenseOpts ou;
            ou.act = 1; ou.pos = L.act_pos; ou.neg = L.act_neg;
            if ((rc = dense(m, L.up, y.h.p, y.up.p, T, ou))) return rc;
            if ((rc = dense(m, L.down, y.up.p, y.y.p, T, o))) return rc;
            gamma = L.norm2;
        }
        if (!last) {
            if ((rc = step(gamma, false, next, next_state)) || (rc = capture(l))) return rc;
            continue;
        }
        ++m.launches;
        if ((rc = gptrs_cuda_post_norm_final(x, y.y.p, act_dt, ldw, fp(gamma), fp(m.final_g), c.norm_eps, rows_identity ? nullptr : m.d_rows.as<int32_t>(),
                                             m.xn_rows.p, act_dt, ldw, n_rows, W, st))) return rc;
        if (captured.p && ((rc = step(gamma, false, nullptr, 0)) || (rc = capture(l)))) return rc;
    }
    if (captured.p) {
        GPTRS_CUDA_OK(cudaMemcpyAsync(y.h_residuals, captured.p, captured.n, cudaMemcpyDeviceToHost, st));
        GPTRS_CUDA_OK(cudaStreamSynchronize(st));
        y.h_residuals = nullptr;
    }
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
