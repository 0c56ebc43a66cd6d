"""Host-side mirror of gpt.rs' runtime surface for the decode path, over the C ABI.

  runtime::load_model / LoadedModel      crates/gpt-rs/src/runtime/loader.rs:243-309
  params::base_param_id / param_key      crates/gpt-rs/src/params.rs:29-48
  CausalLanguageModel                    crates/gpt-rs/src/inference/mod.rs:10-40
  Generator                              crates/gpt-rs/src/inference/generate.rs:59-203
  py bindings: logits / generate_tokens  crates/gpt-rs-py/src/runtime.rs:154-360

All arithmetic happens inside libgptrs_cuda.so; this file only marshals arguments.
"""
from __future__ import annotations

import ctypes
import os
from dataclasses import dataclass

import numpy as np

from . import check, lib

KIND_GPT, KIND_MINISTRAL, KIND_LAYERED = 0, 1, 2
MODE_F32, MODE_W4A16, MODE_W8A16, MODE_BF16 = 0, 1, 2, 3
MIXER_LATENT_ATTENTION, MIXER_GROUPED_ATTENTION, MIXER_CHANNEL_DELTA = 0, 1, 2
MLP_NONE, MLP_DENSE_XIELU, MLP_EXPERTS, MLP_DENSE_GELU, MLP_DENSE_POLY = 0, 1, 2, 3, 4
EXPERT_SWIGLU, EXPERT_RELU2 = 0, 1
ROUTE_SOFTMAX, ROUTE_SIGMOID = 0, 1
BLOCK_OUTPUT_NORM, BLOCK_SANDWICH, BLOCK_PRE_NORM, BLOCK_DEPTH = 0, 1, 2, 3
MASK_CAUSAL, MASK_WINDOW, MASK_CHUNK = 0, 1, 2
DISTANCE_NONE, DISTANCE_LOG, DISTANCE_LINEAR = 0, 1, 2


class _ModelConfig(ctypes.Structure):
    _fields_ = [
        ("kind", ctypes.c_int), ("weight_mode", ctypes.c_int),
        ("n_layers", ctypes.c_int), ("d_model", ctypes.c_int), ("n_q_heads", ctypes.c_int),
        ("n_kv_heads", ctypes.c_int), ("head_dim", ctypes.c_int), ("d_mlp", ctypes.c_int),
        ("vocab", ctypes.c_int), ("context_length", ctypes.c_int),
        ("norm_eps", ctypes.c_float), ("rope_theta", ctypes.c_float), ("rotary_dim", ctypes.c_int),
        ("max_seqs", ctypes.c_int), ("max_tokens", ctypes.c_int), ("max_logit_rows", ctypes.c_int),
        ("kv_pages", ctypes.c_int64), ("max_pages_per_seq", ctypes.c_int), ("use_pdl", ctypes.c_int),
        ("tp_size", ctypes.c_int), ("tp_rank", ctypes.c_int),
    ]


class _LayerConfig(ctypes.Structure):
    _fields_ = [
        ("mixer", ctypes.c_int), ("heads", ctypes.c_int), ("dim", ctypes.c_int), ("rot_dim", ctypes.c_int), ("rot_dims", ctypes.c_int),
        ("vdim", ctypes.c_int), ("kv_rank", ctypes.c_int), ("window", ctypes.c_int), ("scale", ctypes.c_float),
        ("rope_base", ctypes.c_double), ("mlp", ctypes.c_int), ("d_ff", ctypes.c_int),
        ("kv_heads", ctypes.c_int), ("mask", ctypes.c_int), ("mask_size", ctypes.c_int), ("distance_bias", ctypes.c_int), ("proj_bias", ctypes.c_int),
        ("softcap", ctypes.c_float), ("taps", ctypes.c_int), ("decay_rank", ctypes.c_int), ("gate_rank", ctypes.c_int),
        ("experts", ctypes.c_int), ("top", ctypes.c_int), ("groups", ctypes.c_int), ("keep", ctypes.c_int), ("weights_of", ctypes.c_int),
        ("q_rank", ctypes.c_int), ("maps", ctypes.c_int), ("out_gate", ctypes.c_int), ("kv_from", ctypes.c_int), ("diff", ctypes.c_float),
        ("expert_form", ctypes.c_int), ("shared_ff", ctypes.c_int), ("route", ctypes.c_int), ("group_best", ctypes.c_int), ("correction", ctypes.c_int),
        ("weight_scale", ctypes.c_float),
        ("sink", ctypes.c_int), ("rope_halves", ctypes.c_int), ("rope_factor", ctypes.c_double), ("rope_original", ctypes.c_double),
        ("rope_fast", ctypes.c_double), ("rope_slow", ctypes.c_double), ("qk_norm", ctypes.c_int), ("tied", ctypes.c_int), ("gate_silu", ctypes.c_int),
        ("shared_gate", ctypes.c_int),
    ]


class _LayeredConfig(ctypes.Structure):
    _fields_ = [("conv_taps", ctypes.c_int), ("logit_softcap", ctypes.c_float), ("block", ctypes.c_int), ("learned_positions", ctypes.c_int),
                ("streams", ctypes.c_int), ("embed_scale", ctypes.c_float), ("residual_mult", ctypes.c_float), ("norm_groups", ctypes.c_int)]


@dataclass
class LayerConfig:
    """One layer of a model of the layered kind: its mixer and its feed-forward. Latent attention (in a sliding window, or over
    everything) takes heads .. rot_dims, q_rank and sink .. rope_slow; attention with grouped key / value heads takes heads, dim, vdim, scale,
    kv_heads .. taps, maps .. diff, qk_norm and tied; the delta rule takes heads, dim, vdim, kv_heads, taps .. gate_rank and gate_silu.
    Experts have the size d_ff each."""
    heads: int
    dim: int            # query / key dimensions of a head (latent attention: those that are not rotated)
    rot_dim: int = 0    # and those that are (shared key part)
    vdim: int = 0
    kv_rank: int = 0
    window: int = 0     # 0 = none
    scale: float = 1.0
    rope_base: float = 10000.0
    rot_dims: int = 0   # rotated dimensions of the rot_dim part (0 = all)
    mixer: int = MIXER_LATENT_ATTENTION
    mlp: int = MLP_DENSE_XIELU
    d_ff: int = 0
    kv_heads: int = 0
    mask: int = MASK_CAUSAL
    mask_size: int = 0
    distance_bias: int = DISTANCE_NONE   # a penalty per head: r1 ln(1 + r2 distance), or 2^(-8 (h + 1) / heads) distance
    proj_bias: int = 0       # biases on the four projections
    softcap: float = 0.0     # of the scores
    taps: int = 0            # of the short convolutions (grouped attention: 0 = none)
    decay_rank: int = 0      # 0: one decay per head
    gate_rank: int = 0       # 0: a gate projected at once
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep: int = 1
    weights_of: int = -1     # layer whose weights this one uses
    q_rank: int = 0          # queries through a latent of this size
    maps: int = 1            # 2: differential attention
    out_gate: int = 0        # the heads' outputs are gated
    kv_from: int = -1        # earlier layer whose keys and values this one reads
    diff: float = 0.0        # constant of differential attention
    expert_form: int = EXPERT_SWIGLU
    shared_ff: int = 0       # size of a shared expert
    route: int = ROUTE_SOFTMAX
    group_best: int = 1      # experts that make a group's score
    correction: int = 0      # a vector added to the scores that choose
    weight_scale: float = 0.0   # > 0: the experts' weights are in proportion and sum to this
    sink: int = 0            # exp(sink) per head in the denominator of the softmax
    rope_halves: int = 0     # rotated pairs are (i, i + rot_dims / 2) instead of (2i, 2i + 1)
    rope_factor: float = 0.0    # YaRN scaling of the rotation (0 = none)
    rope_original: float = 0.0
    rope_fast: float = 0.0
    rope_slow: float = 0.0
    qk_norm: int = 0         # norms per head on queries and keys
    tied: int = 0            # values are the keys in front of their norm
    gate_silu: int = 0       # the delta rule's gate: silu instead of sigmoid
    shared_gate: int = 0     # the shared expert's output times sigmoid(shared.sg h)

    def _struct(self):
        values = {f: getattr(self, f) for f, _ in _LayerConfig._fields_}
        values["rot_dims"] = self.rot_dims or self.rot_dim
        return _LayerConfig(**values)

    def shapes(self, p: str, d: int, block: int, conv_taps: int, streams: int = 0) -> dict[str, tuple[int, ...]]:
        """Names and shapes of the layer's parameters (prefix `p`, width `d`)."""
        if self.weights_of >= 0:
            return {}

        def beside(n):   # a sublayer's norms and what the block form has beside them
            out = {f"{p}.norm{n}": (d,)}
            if block == BLOCK_SANDWICH:
                out[f"{p}.norm{n}b"] = (d,)
            elif block == BLOCK_OUTPUT_NORM:
                out[f"{p}.canon{n}"] = (d, conv_taps)
            elif block == BLOCK_PRE_NORM and streams:
                out.update({f"{p}.hc{n}.in": (streams,), f"{p}.hc{n}.out": (streams,), f"{p}.hc{n}.mix": (streams, streams)})
            return out

        out: dict[str, tuple[int, ...]] = beside(1)
        x, qk, v = f"{p}.mix", self.heads * self.dim, self.heads * self.vdim
        if self.mixer == MIXER_LATENT_ATTENTION:
            rows = self.heads * (self.dim + self.rot_dim)
            out.update({f"{x}.dq": (self.q_rank, d), f"{x}.dq.norm": (self.q_rank,), f"{x}.uq": (rows, self.q_rank)} if self.q_rank else {f"{x}.q": (rows, d)})
            out.update({f"{x}.dkv": (self.kv_rank + self.rot_dim, d), f"{x}.dkv.norm": (self.kv_rank,),
                        f"{x}.uk": (qk, self.kv_rank), f"{x}.uv": (v, self.kv_rank), f"{x}.o": (d, v)})
            if self.sink:
                out[f"{x}.sink"] = (self.heads,)
        elif self.mixer == MIXER_GROUPED_ATTENTION:
            rows = {"q": qk * self.maps}
            if self.kv_from < 0:
                rows["k"] = self.kv_heads * self.dim * self.maps
                if not self.tied:
                    rows["v"] = self.kv_heads * self.vdim
            out.update({f"{x}.{n}": (r, d) for n, r in rows.items()})
            for n in "qk":
                if self.taps:
                    out[f"{x}.{n}.conv"] = (rows[n], self.taps)
                if self.qk_norm:
                    out[f"{x}.{n}.norm"] = (self.dim,)
            out[f"{x}.o"] = (d, v)
            if self.proj_bias:
                out.update({f"{x}.{n}.b": (r,) for n, r in {**rows, "o": d}.items()})
            if self.distance_bias == DISTANCE_LOG:
                out.update({f"{x}.r1": (self.heads,), f"{x}.r2": (self.heads,)})
            if self.out_gate:
                out[f"{x}.g"] = (v, d)
            if self.maps == 2:
                out.update({f"{x}.{n}": (self.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
        else:
            kq = self.kv_heads * self.dim
            for n, r in (("q", kq), ("k", kq), ("v", v)):
                out.update({f"{x}.{n}": (r, d), f"{x}.{n}.conv": (r, self.taps)})
            out.update({f"{x}.b": (self.heads, d), f"{x}.A_log": (self.heads,), f"{x}.norm": (self.vdim,), f"{x}.o": (d, v)})
            out.update({f"{x}.a1": (self.decay_rank, d), f"{x}.a2": (qk, self.decay_rank), f"{x}.dt_bias": (qk,)} if self.decay_rank else
                       {f"{x}.a": (self.heads, d), f"{x}.dt_bias": (self.heads,)})
            out.update({f"{x}.g1": (self.gate_rank, d), f"{x}.g2": (v, self.gate_rank)} if self.gate_rank else {f"{x}.g": (v, d)})
        if self.mlp == MLP_NONE:
            return out
        f = f"{p}.mlp"
        out.update(beside(2))
        if self.mlp == MLP_DENSE_XIELU:
            out.update({f"{f}.up": (self.d_ff, d), f"{f}.up.b": (self.d_ff,), f"{f}.down": (d, self.d_ff), f"{f}.down.b": (d,), f"{f}.act": (2,)})
        elif self.mlp == MLP_DENSE_GELU:
            out.update({f"{f}.gate": (self.d_ff, d), f"{f}.up": (self.d_ff, d), f"{f}.down": (d, self.d_ff)})
        elif self.mlp == MLP_DENSE_POLY:
            out.update({f"{f}.up": (self.d_ff, d), f"{f}.down": (d, self.d_ff), f"{f}.act": (4,)})
        else:
            for e in range(self.experts):
                if self.expert_form == EXPERT_SWIGLU:
                    out[f"{f}.e{e}.gate"] = (self.d_ff, d)
                out.update({f"{f}.e{e}.up": (self.d_ff, d), f"{f}.e{e}.down": (d, self.d_ff)})
            out[f"{f}.router"] = (self.experts, d)
            if self.correction:
                out[f"{f}.correction"] = (self.experts,)
            if self.shared_ff and self.expert_form == EXPERT_SWIGLU:
                out[f"{f}.shared.gate"] = (self.shared_ff, d)
            if self.shared_gate:
                out[f"{f}.shared.sg"] = (1, d)
            if self.shared_ff:
                out.update({f"{f}.shared.up": (self.shared_ff, d), f"{f}.shared.down": (d, self.shared_ff)})
        return out


@dataclass
class ModelConfig:
    kind: int
    n_layers: int
    d_model: int
    n_q_heads: int
    n_kv_heads: int
    head_dim: int
    d_mlp: int
    vocab: int
    context_length: int
    norm_eps: float = 1e-5
    rope_theta: float = 1e6
    rotary_dim: int = 0
    weight_mode: int = MODE_F32
    max_seqs: int = 1
    max_tokens: int = 64
    max_logit_rows: int = 0
    kv_pages: int = 0
    max_pages_per_seq: int = 0
    use_pdl: int = 0
    tp_size: int = 1
    tp_rank: int = 0
    layers: list | None = None     # layered kind: one LayerConfig per layer (the head and MLP sizes above are unused)
    conv_taps: int = 1
    logit_softcap: float = 0.0
    block: int = BLOCK_OUTPUT_NORM
    learned_positions: int = 0     # position vectors added to the embedding
    streams: int = 0               # copies of the residual that are mixed at every sublayer (BLOCK_PRE_NORM)
    embed_scale: float = 1.0       # of the embedding (BLOCK_PRE_NORM)
    residual_mult: float = 1.0     # of the sublayers' normed outputs (BLOCK_DEPTH)
    norm_groups: int = 1           # equal parts of a row, each with a norm of its own (BLOCK_DEPTH)

    @staticmethod
    def layered(layers, d_model: int, vocab: int, context_length: int, norm_eps: float, conv_taps: int = 1, logit_softcap: float = 0.0, **kw):
        return ModelConfig(KIND_LAYERED, len(layers), d_model, 0, 0, 0, 0, vocab, context_length, norm_eps, layers=list(layers),
                           conv_taps=conv_taps, logit_softcap=logit_softcap, **kw)

    @staticmethod
    def gpt2_small(**kw):
        """GPT-2 small as run by the reference (crates/gpt-rs/src/model/gpt.rs; eps gpt.rs:170)."""
        return ModelConfig(KIND_GPT, 12, 768, 12, 12, 64, 3072, 50257, 1024, 1e-5, **kw)

    @staticmethod
    def ministral_3b(**kw):
        """Ministral-3B-shaped GQA decoder (26 layers, hidden 3072, 32 q / 8 kv heads of 128,
        SwiGLU 9216, RMSNorm eps 1e-5, RoPE theta 1e6, vocab 131072)."""
        kw.setdefault("rotary_dim", 128)
        kw.setdefault("context_length", 8192)
        ctx = kw.pop("context_length")
        return ModelConfig(KIND_MINISTRAL, 26, 3072, 32, 8, 128, 9216, 131072, ctx, 1e-5, 1e6, **kw)

    def param_shapes(self) -> dict[str, tuple[int, ...]]:
        """Parameter names and shapes in the reference's layout (model/gpt.rs:222-291,
        model/ministral.rs:376-421); Linear weights are [in, out]."""
        if self.kind == KIND_LAYERED:
            return self._layered_shapes()
        d, qd = self.d_model, self.n_q_heads * self.head_dim
        qkv = (self.n_q_heads + 2 * self.n_kv_heads) * self.head_dim
        out: dict[str, tuple[int, ...]] = {"tok_embeddings.weight": (self.vocab, d)}
        if self.kind == KIND_GPT:
            out["pos_embeddings"] = (self.context_length, d)
        for l in range(self.n_layers):
            p = f"blocks.{l}"
            out[f"{p}.attention.w_qkv"] = (d, qkv)
            out[f"{p}.attention.w_out"] = (qd, d)
            if self.kind == KIND_GPT:
                out[f"{p}.attention.b_qkv"] = (qkv,)
                out[f"{p}.attention.b_out"] = (d,)
                out[f"{p}.feed_forward.w_in"] = (d, self.d_mlp)
                out[f"{p}.feed_forward.b_in"] = (self.d_mlp,)
                out[f"{p}.feed_forward.w_out"] = (self.d_mlp, d)
                out[f"{p}.feed_forward.b_out"] = (d,)
                for n in ("ln_1", "ln_2"):
                    out[f"{p}.{n}.gamma"] = (d,)
                    out[f"{p}.{n}.beta"] = (d,)
            else:
                out[f"{p}.feed_forward.w_gate"] = (d, self.d_mlp)
                out[f"{p}.feed_forward.w_up"] = (d, self.d_mlp)
                out[f"{p}.feed_forward.w_down"] = (self.d_mlp, d)
                out[f"{p}.norm_1.gamma"] = (d,)
                out[f"{p}.norm_2.gamma"] = (d,)
        if self.kind == KIND_GPT:
            out["final_ln.gamma"] = (d,)
            out["final_ln.beta"] = (d,)
        else:
            out["final_norm.gamma"] = (d,)
        out["lm_head"] = (d, self.vocab)
        return out

    def _layered_shapes(self) -> dict[str, tuple[int, ...]]:
        """Names and shapes of the layered kind; Linear weights are [out, in]."""
        d = self.d_model
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab, d)}
        if self.block == BLOCK_OUTPUT_NORM:
            out["embed.norm"] = (d,)
        if self.learned_positions:
            out["pos"] = (self.learned_positions, d)
        for l, c in enumerate(self.layers):
            out.update(c.shapes(f"l{l}", d, self.block, self.conv_taps, self.streams))
            if self.block == BLOCK_DEPTH:
                out[f"l{l}.dwa"] = (l + 2,)
        out["final.norm"] = (d,)
        out["head"] = (self.vocab, d)
        return out


def base_param_id(name: str) -> int:
    """first 16 bytes of blake3(name), little endian (crates/gpt-rs/src/params.rs:29-36)."""
    import blake3
    return int.from_bytes(blake3.blake3(name.encode("ascii")).digest()[:16], "little")


def param_key(namespace: int, base_id: int) -> int:
    """crates/gpt-rs/src/params.rs:38-48."""
    import blake3
    h = blake3.blake3()
    h.update(b"gpt-rs:param-key:v1")
    h.update(int(namespace).to_bytes(16, "little"))
    h.update(int(base_id).to_bytes(16, "little"))
    return int.from_bytes(h.digest()[:16], "little")


class LoadedModel:
    """A model resident on the current CUDA device."""

    def __init__(self, config: ModelConfig, namespace: int = 0):
        self.config = config
        self.namespace = namespace
        c = _ModelConfig(**{f: getattr(config, f) for f, _ in _ModelConfig._fields_})
        self._h = ctypes.c_void_p()
        check(lib().gptrs_cuda_model_create(ctypes.byref(c), ctypes.byref(self._h)))
        if config.kind == KIND_LAYERED:
            rows = (_LayerConfig * len(config.layers))(*[l._struct() for l in config.layers])
            common = _LayeredConfig(config.conv_taps, config.logit_softcap, config.block, config.learned_positions, config.streams, config.embed_scale,
                                    config.residual_mult, config.norm_groups)
            check(lib().gptrs_cuda_model_set_layers(self._h, ctypes.byref(common), rows, len(config.layers)))
        self._finalized = False

    def close(self):
        if getattr(self, "_h", None) and self._h.value:
            lib().gptrs_cuda_model_destroy(self._h)
            self._h = ctypes.c_void_p()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    # ---- parameters ---------------------------------------------------------------------------
    def load_param(self, name: str, value, stable_id: int | None = None):
        """value: numpy f32 array (host) or torch CUDA f32 tensor."""
        if stable_id is None:
            stable_id = param_key(self.namespace, base_param_id(name))
        lo, hi = stable_id & (2 ** 64 - 1), stable_id >> 64
        if isinstance(value, np.ndarray):
            arr = np.ascontiguousarray(value, dtype=np.float32)
            dims = (ctypes.c_int64 * arr.ndim)(*arr.shape)
            check(lib().gptrs_cuda_model_load_param(self._h, name.encode(), lo, hi, arr.ctypes.data, 0, arr.ndim, dims))
        else:
            import torch
            assert value.is_cuda and value.dtype == torch.float32 and value.is_contiguous()
            dims = (ctypes.c_int64 * value.dim())(*value.shape)
            torch.cuda.current_stream().synchronize()
            check(lib().gptrs_cuda_model_load_param(self._h, name.encode(), lo, hi, value.data_ptr(), 1, value.dim(), dims))

    def set_rope_tables(self, cos: np.ndarray, sin: np.ndarray):
        cos = np.ascontiguousarray(cos, dtype=np.float32)
        sin = np.ascontiguousarray(sin, dtype=np.float32)
        check(lib().gptrs_cuda_model_set_rope_tables(self._h, cos.ctypes.data, sin.ctypes.data, cos.shape[0]))

    def init_tensor_parallel(self, unique_id: bytes):
        """Joins the NCCL communicator of the tensor-parallel group (call on every rank before finalize)."""
        assert len(unique_id) == 128
        buf = (ctypes.c_uint8 * 128).from_buffer_copy(unique_id)
        check(lib().gptrs_cuda_model_init_tensor_parallel(self._h, buf))

    def tp_allreduce_kind(self) -> str:
        """The collective behind the row-parallel projections of decode-sized steps (after finalize)."""
        return {0: "none", 1: "nccl", 2: "peer-store one-shot"}[int(lib().gptrs_cuda_model_tp_allreduce_kind(self._h))]

    def finalize(self, drop_f32_leaves: bool = True):
        check(lib().gptrs_cuda_model_finalize(self._h, int(drop_f32_leaves)))
        self._finalized = True

    def stats(self) -> dict:
        v = [ctypes.c_int64() for _ in range(4)]
        check(lib().gptrs_cuda_model_stats(self._h, *[ctypes.byref(x) for x in v]))
        return dict(zip(("quantised_now", "memo_hits", "free_pages", "kernel_launches"), (x.value for x in v)))

    # ---- forward --------------------------------------------------------------------------------
    def reset_sequence(self, slot: int = 0):
        check(lib().gptrs_cuda_model_reset_sequence(self._h, slot))

    def set_top_k(self, top_k: int | None):
        """Sampler::with_top_k for temperature draws (None or 0 = keep every logit)."""
        check(lib().gptrs_cuda_model_set_top_k(self._h, int(top_k or 0)))

    def sequence_length(self, slot: int = 0) -> int:
        n = ctypes.c_int()
        check(lib().gptrs_cuda_model_sequence_length(self._h, slot, ctypes.byref(n)))
        return n.value

    def forward_with_decode_cache(self, tokens, slots, positions, logit_rows=(), want_logits=True,
                                  temperature: float = 0.0, seed: int = 0):
        """Returns (logits [rows][vocab] or None, sampled ids [rows])."""
        tok = np.ascontiguousarray(tokens, dtype=np.int32)
        sl = np.ascontiguousarray(slots, dtype=np.int32)
        pos = np.ascontiguousarray(positions, dtype=np.int32)
        rows = np.ascontiguousarray(logit_rows, dtype=np.int32)
        n, r = len(tok), len(rows)
        vocab_local = self.config.vocab // max(self.config.tp_size, 1)
        logits = np.empty((r, vocab_local), dtype=np.float32) if (want_logits and r) else None
        sampled = np.empty(r, dtype=np.int32)
        check(lib().gptrs_cuda_model_forward_with_decode_cache(
            self._h, tok.ctypes.data, sl.ctypes.data, pos.ctypes.data, n, rows.ctypes.data if r else None, r,
            logits.ctypes.data if logits is not None else None, sampled.ctypes.data if r else None,
            float(temperature), int(seed)))
        return logits, sampled

    def layer_residuals(self, tokens, slots, positions) -> np.ndarray:
        """Debug, layered kind: one forward pass that returns the residual stream after every layer [layer][row][d_model]."""
        out = np.empty((self.config.n_layers, len(tokens), self.config.d_model), dtype=np.float32)
        check(lib().gptrs_cuda_debug_layer_residuals(self._h, out.ctypes.data))
        try:
            self.forward_with_decode_cache(tokens, slots, positions)
        finally:
            check(lib().gptrs_cuda_debug_layer_residuals(self._h, None))
        return out

    def prefill(self, slot: int, tokens, chunk: int | None = None, want_logits: bool = False):
        """Appends a prompt to `slot` in chunks of at most `chunk` tokens; returns the logits
        (optional) and greedy id of the LAST prompt row (the generator's first sampled token)."""
        chunk = chunk or self.config.max_tokens
        start = self.sequence_length(slot)
        tokens = list(tokens)
        logits, sampled = None, None
        for o in range(0, len(tokens), chunk):
            part = tokens[o:o + chunk]
            last = o + len(part) == len(tokens)
            lg, sm = self.forward_with_decode_cache(
                part, [slot] * len(part), list(range(start + o, start + o + len(part))),
                [len(part) - 1] if last else [], want_logits=want_logits and last)
            if last:
                logits, sampled = lg, sm
        return (logits[0] if logits is not None else None), int(sampled[0])

    def prefill_many(self, slots, prompts, chunk: int | None = None):
        """Appends one prompt to each of `slots` with the rows of all prompts packed into forward passes of up to
        `chunk` rows, so a pass may hold the tail of one sequence and the head of the next: the matmuls then see
        full row tiles whatever the prompt lengths are. Where the grouped attention kernel would run, a pass is cut early
        if the next sequence would start off the row alignment that lets the rows of a group share one K/V stream.
        Returns the greedy id that follows each prompt, in the order given."""
        cfg = self.config
        chunk = min(chunk or cfg.max_tokens, cfg.max_tokens)
        group = max(cfg.n_q_heads // max(cfg.n_kv_heads, 1), 1)
        align = max(16 // group, 1)
        # passes the engine gives to the tensor-core prefill attention (the rule of gptrs_cuda_model_forward: paged bf16
        # cache, heads of 128, at least two 256-row tiles) need no alignment: a tile may hold two sequences
        if cfg.kind == KIND_LAYERED:   # query tiles are cut at sequence boundaries
            align = 1
        elif (cfg.weight_mode != MODE_F32 and cfg.head_dim == 128 and group in (1, 2, 4, 8) and chunk >= 2 * (256 // group)
                and os.environ.get("GPTRS_PREFILL_TC", "1") != "0"):
            align = 1
        max_rows = cfg.max_logit_rows if cfg.max_logit_rows > 0 else cfg.max_seqs
        first = [None] * len(prompts)
        tok, sl, pos, rows, owners = [], [], [], [], []

        def flush():
            if not tok:
                return
            _, sampled = self.forward_with_decode_cache(tok, sl, pos, rows, want_logits=False)
            for r, o in enumerate(owners):
                first[o] = int(sampled[r])
            tok.clear(), sl.clear(), pos.clear(), rows.clear(), owners.clear()

        for i, (slot, prompt) in enumerate(zip(slots, prompts)):
            prompt = np.asarray(prompt, dtype=np.int32)
            start = self.sequence_length(slot)
            done = 0
            while done < len(prompt):
                n = min(len(prompt) - done, chunk - len(tok))
                tok.extend(prompt[done:done + n].tolist())
                sl.extend([slot] * n)
                pos.extend(range(start + done, start + done + n))
                done += n
                if done == len(prompt):
                    rows.append(len(tok) - 1)
                    owners.append(i)
                if len(tok) == chunk or (done == len(prompt) and (len(tok) % align != 0 or len(rows) == max_rows)):
                    flush()
        flush()
        return first

    def logits(self, tokens) -> np.ndarray:
        """LoadedModel.logits of the py bindings: logits of every row of one fresh sequence."""
        self.reset_sequence(0)
        n = len(tokens)
        lg, _ = self.forward_with_decode_cache(tokens, [0] * n, list(range(n)), list(range(n)))
        return lg


def nccl_unique_id() -> bytes:
    """128-byte NCCL id created on the calling rank (distribute it to the group yourself)."""
    buf = (ctypes.c_uint8 * 128)()
    check(lib().gptrs_cuda_nccl_unique_id(buf))
    return bytes(buf)


class Generator:
    """Greedy batched generator over slots 0..batch-1 (Generator::step, generate.rs:123-169)."""

    def __init__(self, model: LoadedModel, first_tokens, use_graph: bool = True):
        self.model = model
        self.batch = len(first_tokens)
        self.use_graph = use_graph
        ft = np.ascontiguousarray(first_tokens, dtype=np.int32)
        check(lib().gptrs_cuda_generator_begin(model._h, self.batch, ft.ctypes.data))
        self._out = np.empty(self.batch, dtype=np.int32)

    def step(self, tokens_in=None, read_back: bool = True):
        """One decode step; returns the sampled ids (host) when read_back, else None."""
        tin = None
        if tokens_in is not None:
            tin = np.ascontiguousarray(tokens_in, dtype=np.int32)
        check(lib().gptrs_cuda_generator_step(self.model._h, tin.ctypes.data if tin is not None else None,
                                              self._out.ctypes.data if read_back else None, int(self.use_graph)))
        return self._out.copy() if read_back else None

    def sync(self):
        check(lib().gptrs_cuda_generator_sync(self.model._h))


def generate_tokens(model: LoadedModel, prompt, max_new_tokens: int, use_graph: bool = True):
    """py-binding style helper for one sequence in slot 0: prefill, then greedy decode."""
    model.reset_sequence(0)
    _, first = model.prefill(0, prompt)
    out = [first]
    if max_new_tokens > 1:
        gen = Generator(model, [first], use_graph=use_graph)
        for _ in range(max_new_tokens - 1):
            out.append(int(gen.step()[0]))
    return out
