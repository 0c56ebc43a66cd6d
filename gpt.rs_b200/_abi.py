"""Declares the ctypes signatures of libgptrs_cuda.so from include/gptrs_cuda.h.

The header is the single source of truth: every `gptrs_cuda_*` prototype in it is parsed and
bound, so a symbol declared there but not exported by the library fails at load time.
"""
from __future__ import annotations

import ctypes
import re
from pathlib import Path

HEADER = Path(__file__).resolve().parent.parent / "include" / "gptrs_cuda.h"

_SCALARS = {
    "int": ctypes.c_int,
    "unsigned": ctypes.c_uint,
    "int32_t": ctypes.c_int32,
    "uint32_t": ctypes.c_uint32,
    "int64_t": ctypes.c_int64,
    "uint64_t": ctypes.c_uint64,
    "size_t": ctypes.c_size_t,
    "float": ctypes.c_float,
    "double": ctypes.c_double,
}


class MatmulEpilogue(ctypes.Structure):
    """gptrs_matmul_epilogue."""
    _fields_ = [
        ("out_dtype", ctypes.c_int),
        ("d_bias", ctypes.c_void_p),
        ("d_residual", ctypes.c_void_p),
        ("swiglu", ctypes.c_int),
        ("d_norm_gamma", ctypes.c_void_p),
        ("d_norm_x", ctypes.c_void_p),
        ("d_sumsq_out", ctypes.c_void_p),
        ("d_sumsq_in", ctypes.c_void_p),
        ("sumsq_tiles", ctypes.c_int),
        ("norm_dim", ctypes.c_int),
        ("norm_eps", ctypes.c_float),
        ("d_rope_positions", ctypes.c_void_p),
        ("d_rope_slot", ctypes.c_void_p),
        ("d_rope_page_table", ctypes.c_void_p),
        ("rope_max_pages", ctypes.c_int64),
        ("d_rope_cos", ctypes.c_void_p),
        ("d_rope_sin", ctypes.c_void_p),
        ("d_rope_q_out", ctypes.c_void_p),
        ("d_rope_kv_pool", ctypes.c_void_p),
        ("rope_q_heads", ctypes.c_int),
        ("rope_kv_heads", ctypes.c_int),
        ("d_status", ctypes.c_void_p),
        ("peer_push", ctypes.c_void_p),
        ("d_best_val", ctypes.c_void_p),
        ("d_best_idx", ctypes.c_void_p),
        ("skip_store", ctypes.c_int),
    ]


class DenseEpilogue(ctypes.Structure):
    """gptrs_dense_epilogue."""
    _fields_ = [
        ("out_dtype", ctypes.c_int), ("d_bias", ctypes.c_void_p), ("act", ctypes.c_int), ("act_pos", ctypes.c_float), ("act_neg", ctypes.c_float),
        ("softcap", ctypes.c_float), ("ldx", ctypes.c_int64), ("ldy", ctypes.c_int64), ("batch", ctypes.c_int64), ("x_step", ctypes.c_int64),
        ("y_step", ctypes.c_int64), ("d_best_val", ctypes.c_void_p), ("d_best_idx", ctypes.c_void_p), ("skip_store", ctypes.c_int),
        ("d_status", ctypes.c_void_p), ("d_tiles", ctypes.c_void_p), ("d_n_tiles", ctypes.c_void_p), ("max_tiles", ctypes.c_int64),
        ("tile_rows", ctypes.c_int64), ("swiglu", ctypes.c_int),
    ]


class NormStep(ctypes.Structure):
    """gptrs_norm_step."""
    _fields_ = [
        ("d_x", ctypes.c_void_p), ("d_y", ctypes.c_void_p), ("y_dtype", ctypes.c_int), ("ldy", ctypes.c_int64), ("d_pair", ctypes.c_void_p),
        ("d_pair_weight", ctypes.c_void_p), ("top", ctypes.c_int64), ("d_embed", ctypes.c_void_p), ("d_pos_embed", ctypes.c_void_p),
        ("d_tokens", ctypes.c_void_p), ("d_pos", ctypes.c_void_p), ("vocab", ctypes.c_int64), ("positions", ctypes.c_int64), ("d_gamma_out", ctypes.c_void_p),
        ("d_gamma_in", ctypes.c_void_p), ("eps", ctypes.c_float), ("d_rows", ctypes.c_void_p), ("d_h", ctypes.c_void_p), ("h_dtype", ctypes.c_int),
        ("ldh", ctypes.c_int64), ("d_status", ctypes.c_void_p), ("rows", ctypes.c_int64), ("dim", ctypes.c_int64),
    ]


class StreamStep(ctypes.Structure):
    """gptrs_stream_step."""
    _fields_ = [
        ("d_x", ctypes.c_void_p), ("streams", ctypes.c_int), ("d_y", ctypes.c_void_p), ("y_dtype", ctypes.c_int), ("ldy", ctypes.c_int64),
        ("d_pair", ctypes.c_void_p), ("d_pair_weight", ctypes.c_void_p), ("top", ctypes.c_int64), ("d_add", ctypes.c_void_p), ("ld_add", ctypes.c_int64),
        ("d_embed", ctypes.c_void_p), ("embed_scale", ctypes.c_float), ("d_tokens", ctypes.c_void_p), ("vocab", ctypes.c_int64), ("d_mix", ctypes.c_void_p),
        ("d_out", ctypes.c_void_p), ("d_in", ctypes.c_void_p), ("d_gamma_in", ctypes.c_void_p), ("eps", ctypes.c_float), ("d_rows", ctypes.c_void_p),
        ("d_h", ctypes.c_void_p), ("h_dtype", ctypes.c_int), ("ldh", ctypes.c_int64), ("d_sum", ctypes.c_void_p), ("d_status", ctypes.c_void_p),
        ("rows", ctypes.c_int64), ("dim", ctypes.c_int64),
    ]


class DepthStep(ctypes.Structure):
    """gptrs_depth_step."""
    _fields_ = [
        ("d_x", ctypes.c_void_p), ("d_x_out", ctypes.c_void_p), ("d_y", ctypes.c_void_p), ("y_dtype", ctypes.c_int), ("ldy", ctypes.c_int64),
        ("d_pair", ctypes.c_void_p), ("d_pair_weight", ctypes.c_void_p), ("top", ctypes.c_int64), ("d_add", ctypes.c_void_p), ("ld_add", ctypes.c_int64),
        ("d_add_gate", ctypes.c_void_p), ("ld_add_gate", ctypes.c_int64), ("d_embed", ctypes.c_void_p), ("d_tokens", ctypes.c_void_p), ("vocab", ctypes.c_int64),
        ("d_gamma_out", ctypes.c_void_p), ("mult", ctypes.c_float), ("groups", ctypes.c_int), ("eps", ctypes.c_float), ("d_states", ctypes.c_void_p),
        ("state_stride", ctypes.c_int64), ("n_states", ctypes.c_int64), ("d_weights", ctypes.c_void_p), ("d_gamma_in", ctypes.c_void_p),
        ("d_rows", ctypes.c_void_p), ("d_h", ctypes.c_void_p), ("h_dtype", ctypes.c_int), ("ldh", ctypes.c_int64), ("d_status", ctypes.c_void_p),
        ("rows", ctypes.c_int64), ("dim", ctypes.c_int64),
    ]


class GroupedStep(ctypes.Structure):
    """gptrs_grouped_step."""
    _fields_ = [(n, ctypes.c_void_p) for n in ("d_qkv", "d_conv", "d_q_gain", "d_k_gain", "d_conv_state", "d_slot", "d_pos", "d_run_first", "d_run_last", "d_parity",
                                               "d_page_table")] + \
        [("max_pages", ctypes.c_int64), ("d_pool", ctypes.c_void_p), ("d_q", ctypes.c_void_p), ("rows", ctypes.c_int64)]


class GroupedAttention(ctypes.Structure):
    """gptrs_grouped_attention."""
    _fields_ = [(n, ctypes.c_int) for n in ("dtype", "heads", "kv_heads", "dim", "vdim", "mask", "mask_size")] + \
        [("scale", ctypes.c_float), ("softcap", ctypes.c_float), ("distance_bias", ctypes.c_int)] + \
        [(n, ctypes.c_int) for n in ("maps", "gate", "shared_kv")] + [(n, ctypes.c_float) for n in ("lambda_", "head_scale", "head_eps")] + \
        [(n, ctypes.c_int) for n in ("taps", "qk_norm", "tied")] + \
        [(n, ctypes.c_int) for n in ("q_head_stride", "k_offset", "k_head_stride", "v_offset", "v_head_stride", "q_row", "map_stride", "g_offset",
                                     "g_head_stride", "out_head_stride", "query_row", "conv_channels")] + \
        [("conv_floats", ctypes.c_int64), ("page_bytes", ctypes.c_int64)]


class DeltaRule(ctypes.Structure):
    """gptrs_delta_rule."""
    _fields_ = [(n, ctypes.c_int) for n in ("dtype", "heads", "kv_heads", "dim", "vdim", "taps", "decay_rank", "gate_rank")] + [("eps", ctypes.c_float), ("gate_silu", ctypes.c_int)] + \
        [(n, ctypes.c_int) for n in ("q_offset", "k_offset", "v_offset", "beta_offset", "a_offset", "g_offset", "row", "decay_row", "gate_row",
                                     "out_head_stride", "conv_channels")] + \
        [(n, ctypes.c_int64) for n in ("state_floats", "conv_floats")]


class DeltaStep(ctypes.Structure):
    """gptrs_delta_step."""
    _fields_ = [(n, ctypes.c_void_p) for n in ("d_proj", "d_decay", "d_gate", "d_conv", "d_a_log", "d_dt_bias", "d_norm", "d_state", "d_conv_state", "d_slot",
                                               "d_pos", "d_run_first", "d_run_last", "d_parity", "d_runs")] + \
        [("n_runs", ctypes.c_int64), ("d_out", ctypes.c_void_p), ("d_scratch", ctypes.c_void_p), ("rows", ctypes.c_int64), ("d_status", ctypes.c_void_p)]


class Moe(ctypes.Structure):
    """gptrs_moe."""
    _fields_ = [(n, ctypes.c_int) for n in ("experts", "top", "groups", "keep", "tile_rows", "scores", "group_best")] + [("weight_scale", ctypes.c_float)]


class ConvStep(ctypes.Structure):
    """gptrs_conv_step."""
    _fields_ = [
        ("d_x", ctypes.c_void_p), ("d_x_out", ctypes.c_void_p), ("d_y", ctypes.c_void_p), ("y_dtype", ctypes.c_int), ("ldy", ctypes.c_int64),
        ("d_embed", ctypes.c_void_p), ("d_tokens", ctypes.c_void_p), ("vocab", ctypes.c_int64), ("d_gamma", ctypes.c_void_p),
        ("eps", ctypes.c_float), ("d_conv", ctypes.c_void_p), ("taps", ctypes.c_int64), ("d_state", ctypes.c_void_p), ("d_slot", ctypes.c_void_p),
        ("d_pos", ctypes.c_void_p), ("d_run_first", ctypes.c_void_p), ("d_run_last", ctypes.c_void_p), ("d_parity", ctypes.c_void_p),
        ("d_h", ctypes.c_void_p), ("h_dtype", ctypes.c_int), ("ldh", ctypes.c_int64), ("d_status", ctypes.c_void_p), ("rows", ctypes.c_int64),
        ("dim", ctypes.c_int64),
    ]


class LatentAttention(ctypes.Structure):
    """gptrs_latent_attention."""
    _fields_ = [(n, ctypes.c_int) for n in ("dtype", "heads", "dim", "rot_dim", "vdim", "kv_rank", "window", "rot_dims")] + [("scale", ctypes.c_float)] + \
        [(n, ctypes.c_int) for n in ("q_rank", "q_head_stride", "q_rot_offset", "dkv_offset", "rot_offset", "q_row", "kv_row", "q_latent_row", "qa_head_stride", "qa_rot_offset",
                                     "lat_head_stride", "out_head_stride")] + [("page_bytes", ctypes.c_int64)]


def prototypes(header_text: str | None = None) -> dict[str, tuple[str, list[str]]]:
    """Returns {name: (return type, [parameter declarations])} for every exported function."""
    text = header_text if header_text is not None else HEADER.read_text()
    text = re.sub(r"/\*.*?\*/", " ", text, flags=re.S)
    text = re.sub(r"//[^\n]*", " ", text)
    text = re.sub(r"typedef\s+(struct|enum)\s*\w*\s*\{.*?\}\s*\w+\s*;", " ", text, flags=re.S)
    out = {}
    for m in re.finditer(r"([\w\s\*]+?)\b(gptrs_cuda_\w+)\s*\(([^)]*)\)\s*;", text):
        ret, name, params = m.group(1).strip(), m.group(2), m.group(3).strip()
        plist = [] if params in ("", "void") else [p.strip() for p in params.split(",")]
        out[name] = (ret, plist)
    return out


def _ctype_of(decl: str):
    if "*" in decl:
        if re.match(r"(const\s+)?char\s*\*", decl) and decl.count("*") == 1:
            return ctypes.c_char_p
        return ctypes.c_void_p
    base = decl.replace("const", " ").split()
    # last token is the parameter name when there are two or more tokens
    ty = base[0] if len(base) >= 1 else "int"
    if ty in _SCALARS:
        return _SCALARS[ty]
    return ctypes.c_int  # enums


def load(path: str) -> ctypes.CDLL:
    lib = ctypes.CDLL(path, mode=ctypes.RTLD_GLOBAL)
    missing = []
    for name, (ret, params) in prototypes().items():
        try:
            fn = getattr(lib, name)
        except AttributeError:
            missing.append(name)
            continue
        fn.argtypes = [_ctype_of(p) for p in params]
        if "*" in ret:
            fn.restype = ctypes.c_char_p if "char" in ret else ctypes.c_void_p
        else:
            fn.restype = _SCALARS.get(ret.replace("const", "").split()[0], ctypes.c_int)
    if missing:
        raise RuntimeError(f"libgptrs_cuda.so does not export: {', '.join(missing)}")
    return lib
