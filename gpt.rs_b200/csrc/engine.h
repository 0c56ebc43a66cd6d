// Internal interface of the decode engine: the model object (weights, activations, KV storage, slots and pages) and the
// helpers shared by the translation units that implement its kinds (engine.cu: gpt and ministral; layered.cu: models whose
// layers are configured one by one).
#pragma once

#include <algorithm>
#include <map>
#include <memory>
#include <string>
#include <tuple>
#include <utility>
#include <vector>

#include "nccl_dl.h"
#include "peer_allreduce.h"
#include "gpt_decode_mega.h"
#include "tensor.h"

namespace gptrs {

enum { kKindGpt = 0, kKindMinistral = 1, kKindLayered = 2 };
enum { kModeF32 = 0, kModeW4 = 1, kModeW8 = 2, kModeBf16 = 3 };
constexpr int kPage = 16;

struct DevBuf {
    void* p = nullptr;
    size_t n = 0;
    int alloc(size_t bytes, bool zero = false) {
        release();
        if (bytes == 0) return GPTRS_OK;
        cudaError_t e = cudaMalloc(&p, bytes);
        if (e != cudaSuccess) return fail(GPTRS_EXECUTION, std::string("cudaMalloc(") + std::to_string(bytes) + "): " + cudaGetErrorString(e));
        n = bytes;
        if (zero) cudaMemset(p, 0, bytes);
        return GPTRS_OK;
    }
    void release() { if (p) cudaFree(p); p = nullptr; n = 0; }
    ~DevBuf() { release(); }
    template <typename T> T* as() const { return static_cast<T*>(p); }
};

struct Weight {        // one Linear
    Tensor* f32 = nullptr;     // [in][out] (f32 mode)
    Tensor* packed = nullptr;  // quantised + repacked (W4/W8 modes)
    Tensor* bias = nullptr;    // optional [out]
    int64_t in = 0, out = 0;
};

struct Layer {
    Tensor *ln1_g = nullptr, *ln1_b = nullptr, *ln2_g = nullptr, *ln2_b = nullptr;
    Weight qkv, attn_out, mlp_in, mlp_gate, mlp_up, mlp_gate_up, mlp_out;
};

struct GraphKey {
    int batch, chunk_pages, splits;
    bool operator<(const GraphKey& o) const {
        return std::tie(batch, chunk_pages, splits) < std::tie(o.batch, o.chunk_pages, o.splits);
    }
};


// ---- models whose layers are configured one by one (layered.cu) ----------------------------------------------------------
struct DenseWeight {   // [batch][n][k] bf16 with n and k padded to 8, or [batch][k][n] f32
    Tensor* w = nullptr;
    Tensor* bias = nullptr;
    int64_t n = 0, k = 0, batch = 1;
};
// What a layer multiplies with; layers that reuse another one's weights share the object.
struct LayerWeights {
    Tensor *norm1 = nullptr, *norm2 = nullptr, *norm1b = nullptr, *norm2b = nullptr, *conv1 = nullptr, *conv2 = nullptr, *latent_norm = nullptr;
    Tensor *r1 = nullptr, *r2 = nullptr;                                                              // distance penalty (linear: r1 alone, the slopes)
    DevBuf reach;                                                                                     // of the kv heads, where norms bound the scores
    Tensor *sink = nullptr, *dwa = nullptr, *act = nullptr;                                           // softmax sinks; average over depth; polynomial
    Tensor *qk_conv = nullptr, *q_gain = nullptr, *k_gain = nullptr;                                  // grouped attention: convolutions, norms per head
    Tensor *q_norm = nullptr, *correction = nullptr;                                                  // query latent; experts' choice
    struct Streams { Tensor *in = nullptr, *out = nullptr, *mix = nullptr; } streams[2];              // of the two sublayers
    Tensor *delta_conv = nullptr, *a_log = nullptr, *dt_bias = nullptr, *delta_norm = nullptr;        // delta rule
    DenseWeight qkv, uq, uk, uv, out, up, down, decay, gate, router, shared_up, shared_down;   // up: gates and ups of a gated layer or experts
    float act_pos = 0.f, act_neg = 0.f;
    float lambda = 0.f;   // differential attention
    ~LayerWeights() {
        for (Tensor* t : {norm1, norm2, norm1b, norm2b, conv1, conv2, latent_norm, r1, r2, q_norm, correction, delta_conv, a_log, dt_bias, delta_norm, sink, dwa, act, qk_conv, q_gain, k_gain}) tensor_release(t);
        for (Streams& s : streams) for (Tensor* t : {s.in, s.out, s.mix}) tensor_release(t);
        for (DenseWeight* w : {&qkv, &uq, &uk, &uv, &out, &up, &down, &decay, &gate, &router, &shared_up, &shared_down}) { tensor_release(w->w); tensor_release(w->bias); }
    }
};
struct LayeredLayer {
    gptrs_layer_config cfg = {};
    gptrs_latent_attention att = {};      // the mixer, whichever it is
    gptrs_grouped_attention gatt = {};
    gptrs_delta_rule delta = {};
    gptrs_moe moe = {};
    std::shared_ptr<LayerWeights> w;
    size_t pool_off = 0;   // byte offset of the layer's pages in Model::kv_pool
    int rope = -1;         // index into Layered::ropes
    int tiles = -1;        // index into Layered::tile_sets, -1 = plain attention kernel
    int state1 = 0, state2 = 0;                      // convolution states of the two sublayers
    size_t delta_state_off = 0, mix_conv_off = 0;    // floats: delta rule's state, inputs of the mixer's convolutions
    bool attends() const { return cfg.mixer != GPTRS_MIXER_CHANNEL_DELTA; }
    bool prepared() const { return cfg.mixer == GPTRS_MIXER_GROUPED_ATTENTION && (gatt.taps > 0 || gatt.qk_norm || gatt.tied); }   // queries in rows of their own
    // the first position that `pos` sees
    int first_visible(int pos) const {
        int f = 0;
        if (cfg.mixer == GPTRS_MIXER_LATENT_ATTENTION) f = att.window > 0 ? pos - att.window + 1 : 0;
        else if (gatt.mask == GPTRS_MASK_WINDOW) f = pos - gatt.mask_size + 1;
        else if (gatt.mask == GPTRS_MASK_CHUNK) f = pos / gatt.mask_size * gatt.mask_size;
        return f > 0 ? f : 0;
    }
    // most positions that one sees, of a sequence of `len`
    int span(int len) const {
        const int size = cfg.mixer == GPTRS_MIXER_LATENT_ATTENTION ? att.window : gatt.mask == GPTRS_MASK_CAUSAL ? 0 : gatt.mask_size;
        return size > 0 ? size : len;
    }
};
struct Layered {
    gptrs_layered_config cfg = {};
    std::vector<LayeredLayer> layers;
    Tensor* embed_norm = nullptr;
    DenseWeight head;
    struct Rope { double base, factor, original, fast, slow; int dims; DevBuf cos_t, sin_t; };
    std::vector<std::unique_ptr<Rope>> ropes;
    // query tiles of the tensor-core attention: one list per distinct tile size (layers may differ in their head counts)
    struct TileSet { int tokens = 1, n = 0; DevBuf row, rows; };
    std::vector<std::unique_ptr<TileSet>> tile_sets;
    int32_t* h_tiles = nullptr;   // pinned staging of one tile list (rows, then counts)
    DevBuf x2, h, qkv, q, q_latent, qa, lat, attn, up, y, logits_pad, state, scratch;
    DevBuf d_run_first, d_run_last, d_parity, d_runs;
    DevBuf decay, gate, delta_state, delta_scratch;   // delta rule
    DevBuf mix_conv;                                  // last inputs of the mixers' short convolutions
    DevBuf states;                                    // GPTRS_BLOCK_DEPTH: the embedding and every layer's result [layers + 1][max_tokens][d_model]
    // experts: logits, sorted rows and what comes of them, the place of every (row, choice) among them, row tiles
    DevBuf router, sorted, gate_up, expert_y, pair, pair_weight, row_tiles, n_row_tiles, moe_work;
    std::vector<int> parity;      // per slot: the half of the convolution state the next step reads
    int n_runs = 0;               // runs of the rows that are staged
    std::vector<int32_t> runs;    // host scratch: (first row, rows) of every run of the current call
    size_t state_stride = 0;      // floats of one sublayer's state
    float* h_residuals = nullptr; // debug: where the next forward pass leaves the residual stream after every layer
    ~Layered() {
        tensor_release(embed_norm);
        tensor_release(head.w);
        if (h_tiles) cudaFreeHost(h_tiles);
    }
};

struct Model {
    gptrs_model_config cfg;
    bool finalized = false;
    std::map<std::string, Tensor*> raw;  // name -> f32 leaf (retained)
    std::map<std::string, std::pair<uint64_t, uint64_t>> ids;
    Tensor *tok_emb = nullptr, *pos_emb = nullptr, *final_g = nullptr, *final_b = nullptr;
    Weight lm_head;
    std::vector<Layer> layers;
    int quantised_now = 0, memo_hits = 0;

    // activations
    DevBuf hidden, xn, qkv, q_rot, attn, mlp_h, mlp_g, mlp_u, logits, xn_rows;
    DevBuf d_tokens, d_slot, d_pos, d_ctx, d_rows, d_sampled, d_status, attn_scratch;
    DevBuf sumsq;  // [d_model / 128][max_tokens] row sums of squares of the folded RMSNorm
    DevBuf history;  // [max_seqs][context_length] token ids by position (the generator re-windows from it)
    bool fold_norm = true, fold_rope = true;
    DevBuf cos_tab, sin_tab;
    int n_rope_pos = 0;
    // KV
    DevBuf kv_pool;                 // bf16 modes: [layer][page][kv_head][K|V][16][128]
    size_t pool_layer_bytes = 0;
    DevBuf k_cache, v_cache;        // f32 mode: [layer][slot][kv_head][capacity][hd]
    size_t cache_layer_elems = 0;
    DevBuf d_page_table;
    int32_t* h_page_table = nullptr;  // pinned mirror [max_seqs][max_pages_per_seq]
    bool table_dirty = true;
    std::vector<int32_t> free_pages;
    std::vector<int> seq_pages, seq_len;
    std::vector<int> seq_first_page;  // first page a slot still holds (pages that every layer's window has passed go back)
    std::unique_ptr<Layered> lay;     // kind kKindLayered
    // staging (pinned)
    int32_t* h_stage = nullptr;  // 6 * max_tokens int32
    float* h_logits = nullptr;
    cudaStream_t stream = nullptr;
    // Optional (GPTRS_LANES=2): decode steps of >= 32 sequences run as two half-batches ("lanes") on two
    // streams, meant to overlap the HBM-bound attention of one half with the latency-bound projections of
    // the other. Off by default: on B200 the grids of both lanes fill every SM, the work distributor runs
    // them back to back, and the doubled weight traffic made a batch-64 step 15 % slower.
    cudaStream_t stream2 = nullptr;
    cudaEvent_t ev_fork = nullptr, ev_join = nullptr;
    std::vector<cudaEvent_t> ev_a, ev_b;  // per layer: attention of lane A / lane B finished
    int n_lanes = 1;
    bool lane_order = true;  // lanes take turns at the attention kernel
    int lane_priority = 0;   // launch priority of everything but attention in a two-lane step (0 = off)
    struct GraphEntry { cudaGraphExec_t exec; int64_t kernels; };
    std::map<GraphKey, GraphEntry> graphs;
    // tensor parallelism: cfg holds the LOCAL head / MLP sizes; the full sizes are kept here
    int tp = 1, tp_rank = 0, full_q = 0, full_kv = 0, full_mlp = 0, vocab_l = 0;
    NcclComm comm = nullptr;
    // one-shot all-reduce over peer memory (decode-sized messages); the regions of the peers are IPC mappings
    void* peer_region = nullptr;
    void* peer_maps[kMaxPeers] = {};
    PeerView peer = {};
    bool peer_on = false;
    bool fuse_peer_push = true;   // GPTRS_TP_FUSED_PUSH=0: a copy kernel pushes the tile instead of the matmul epilogue
    DevBuf partial, tp_vals, tp_idx, tp_gvals, tp_gidx;  // row-parallel partial sums; (max, argmax) exchange
    // greedy head of the quantised engine: per-tile (max, argmax) candidates from the lm_head epilogue
    DevBuf best_val, best_idx;
    bool fuse_pick = true;   // GPTRS_FUSE_PICK=0: logits + sampling kernel
    // f32 GPT kind, one sequence: the whole decode step as one cooperative kernel (gpt_decode_mega.cu)
    bool mega_on = false;
    DevBuf mega_wt, mega_scratch;   // transposed weights [out][in]; vectors + barrier word
    MegaParams mega = {};
    int gen_batch = 0;  // slots 0..gen_batch-1 are driven by generator_step
    int64_t launches = 0;
    uint32_t sample_seed = 0;
    int64_t top_k = 0;  // 0 = no top-k filter in temperature sampling

    int QKV() const { return (cfg.n_q_heads + 2 * cfg.n_kv_heads) * cfg.head_dim; }
    int QD() const { return cfg.n_q_heads * cfg.head_dim; }
    bool f32() const { return cfg.weight_mode == kModeF32; }
    bool layered() const { return cfg.kind == kKindLayered; }
    bool paged() const { return !f32() || layered(); }
    int max_rows() const { return cfg.max_logit_rows > 0 ? cfg.max_logit_rows : cfg.max_seqs; }
    int stage_stride() const { return std::max(cfg.max_tokens, max_rows()); }

    ~Model() {
        for (auto& g : graphs) cudaGraphExecDestroy(g.second.exec);
        for (auto& r : raw) tensor_release(r.second);
        auto relw = [](Weight& w) { tensor_release(w.f32); tensor_release(w.packed); tensor_release(w.bias); };
        for (auto& l : layers) {
            for (Tensor* t : {l.ln1_g, l.ln1_b, l.ln2_g, l.ln2_b}) tensor_release(t);
            for (Weight* w : {&l.qkv, &l.attn_out, &l.mlp_in, &l.mlp_gate, &l.mlp_up, &l.mlp_gate_up, &l.mlp_out}) relw(*w);
        }
        relw(lm_head);
        for (Tensor* t : {tok_emb, pos_emb, final_g, final_b}) tensor_release(t);
        if (h_page_table) cudaFreeHost(h_page_table);
        if (h_stage) cudaFreeHost(h_stage);
        if (h_logits) cudaFreeHost(h_logits);
        for (void* p : peer_maps) if (p) cudaIpcCloseMemHandle(p);
        if (peer_region) cudaFree(peer_region);
        if (comm) { std::string e; if (const NcclApi* api = nccl_api(&e)) api->CommDestroy(comm); }
        for (cudaEvent_t e : ev_a) cudaEventDestroy(e);
        for (cudaEvent_t e : ev_b) cudaEventDestroy(e);
        if (ev_fork) cudaEventDestroy(ev_fork);
        if (ev_join) cudaEventDestroy(ev_join);
        if (stream2) cudaStreamDestroy(stream2);
        if (stream) cudaStreamDestroy(stream);
    }
};

// engine.cu
std::pair<uint64_t, uint64_t> derived_id(std::pair<uint64_t, uint64_t> leaf, const std::string& tag);
int get_raw(Model& m, const std::string& name, std::vector<int64_t> want_dims, Tensor** out);
int alloc_step_buffers(Model& m, int stage_arrays);
int alloc_page_tables(Model& m);
// layered.cu
int layered_check_config(const gptrs_model_config& c);
int layered_finalize(Model& m, bool drop_leaves);
int layered_stage_rows(Model& m, const int32_t* slots, const int32_t* positions, int n);
int layered_stage_generator(Model& m, int batch);
int layered_set_layers(Model& m, const gptrs_layered_config& common, const gptrs_layer_config* layers);
int layered_first_visible(const Model& m, int pos);
int layered_graph_bucket(const Model& m, int bucket);
int layered_forward(Model& m, int rows, int max_ctx, int n_rows, bool rows_identity, float temperature, bool skip_logits);

}  // namespace gptrs
