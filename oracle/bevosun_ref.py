"""TEST INFRASTRUCTURE ONLY — plain numpy restatement of the Bevosun decoder, one function per mechanism, written from the
design's equations and slow on purpose: every position is computed from the whole sequence, there is no cache, no state and
no batch. Arithmetic is float64 on the stored (bfloat16-valued) weights.

The decoder: a normed embedding, then per layer up to two sublayers that read the residual stream through a short causal
convolution and add an RMS-normed output back to it,

    x <- x + rms(mixer(conv(x))),    x <- x + rms(ff(conv(x))),

with latent attention in a sliding window as the mixer and an xIELU feed-forward, then a final norm and soft-capped logits.
Nothing under gpt.rs_b200/ may import this module.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np

D = np.float64


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def short_conv(x, w):
    """x [T][C], w [C][taps]: the taps last inputs of every channel, the newest under the last tap, zeros before position 0."""
    taps = w.shape[1]
    out = np.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return out


def conv_input(x, w):
    """What a sublayer reads: its input plus the convolution of it."""
    return x + short_conv(x, w)


def rotate_interleaved(x, positions, base, dims):
    """x [T][...][n]: the pairs (2i, 2i + 1) of the first `dims` dimensions turn by position * base^(-2i / dims)."""
    out = x.copy()
    for i in range(dims // 2):
        ang = np.asarray(positions, D) * D(base) ** (-2.0 * i / dims)
        ang = ang.reshape((-1,) + (1,) * (x.ndim - 2))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(ang) - v * np.sin(ang)
        out[..., 2 * i + 1] = v * np.cos(ang) + u * np.sin(ang)
    return out


def window_softmax_attention(q, k, v, scale, window):
    """q [T][H][a], k [T][H][a], v [T][H][b]: position i sees positions i - window + 1 .. i."""
    t_n, heads, _ = q.shape
    out = np.zeros((t_n, heads, v.shape[2]), D)
    for i in range(t_n):
        lo = max(0, i - window + 1)
        s = np.einsum("ha,jha->hj", q[i], k[lo:i + 1]) * scale
        p = np.exp(s - s.max(axis=1, keepdims=True))
        p /= p.sum(axis=1, keepdims=True)
        out[i] = np.einsum("hj,jhb->hb", p, v[lo:i + 1])
    return out


def latent_attention(h, w, c, eps):
    """h [T][width]; w: the mixer's tensors by short name; c: the mixer's configuration."""
    t_n = h.shape[0]
    heads, dim, rot, vdim, rank = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    pos = np.arange(t_n)
    q = (h @ w["q"].T).reshape(t_n, heads, dim + rot)
    dkv = h @ w["dkv"].T
    lat = rms_norm(dkv[:, :rank], w["dkv.norm"], eps)
    k_rot = rotate_interleaved(dkv[:, rank:], pos, c["rot"]["base"], c["rot"]["dims"])
    q_rot = rotate_interleaved(q[:, :, dim:], pos, c["rot"]["base"], c["rot"]["dims"])
    k = (lat @ w["uk"].T).reshape(t_n, heads, dim)
    v = (lat @ w["uv"].T).reshape(t_n, heads, vdim)
    k_full = np.concatenate([k, np.broadcast_to(k_rot[:, None, :], (t_n, heads, rot))], axis=2)
    q_full = np.concatenate([q[:, :, :dim], q_rot], axis=2)
    o = window_softmax_attention(q_full, k_full, v, c["scale"], c["mask"]["size"])
    return o.reshape(t_n, heads * vdim) @ w["o"].T


def softplus(x):
    return np.log1p(np.exp(x))


def xielu(z, p, q):
    pos = softplus(p) * z * z + z / 2
    zn = np.minimum(z, 0.0)
    neg = (0.5 + softplus(q)) * (np.expm1(zn) - zn) + zn / 2
    return np.where(z > 0, pos, neg)


def feed_forward(h, w):
    up = h @ w["up"].T + w["up.b"]
    return xielu(up, w["act"][0], w["act"][1]) @ w["down"].T + w["down.b"]


def soft_cap(logits, cap):
    return cap * np.tanh(logits / cap)


def forward(cfg, tensors, tokens, streams=False):
    """Logits [T][vocab] of a whole sequence from position 0; with `streams` also the residual after every layer."""
    w = {n: np.asarray(t, D) for n, t in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = rms_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = {n[len(p) + 4:]: t for n, t in w.items() if n.startswith(p + "mix.")}
        x = x + rms_norm(latent_attention(conv_input(x, w[p + "canon1"]), mix, layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp"):
            mlp = {n[len(p) + 4:]: t for n, t in w.items() if n.startswith(p + "mlp.")}
            x = x + rms_norm(feed_forward(conv_input(x, w[p + "canon2"]), mlp), w[p + "norm2"], eps)
        after.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    if cfg.get("logit_softcap"):
        logits = soft_cap(logits, cfg["logit_softcap"])
    return (logits, np.stack(after)) if streams else logits


# ---- small models for the tests ---------------------------------------------------------------------------------------
def to_bf16(x):
    b = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((b + 0x7FFF + ((b >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def layer_config(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=24, window=20, base=10000.0, scale=None, ff=48):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot_dim}, "scale": float(scale if scale is not None else (dim + rot_dim) ** -0.5)},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model_config(layers, width=40, vocab=72, taps=3, eps=1e-5, softcap=20.0):
    return {"architecture": "Bevosun", "vocab": vocab, "width": width, "layers": layers, "canon": {"taps": taps}, "norm": {"eps": eps},
            "logit_softcap": softcap}


def tensor_shapes(cfg):
    n, v = cfg["width"], cfg["vocab"]
    out = {"embed": (v, n), "embed.norm": (n,)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        out.update({p + "norm1": (n,), p + "canon1": (n, cfg["canon"]["taps"]),
                    p + "mix.q": (m["heads"] * (m["dim"] + m["rot_dim"]), n), p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], n),
                    p + "mix.dkv.norm": (m["kv_rank"],), p + "mix.uk": (m["heads"] * m["dim"], m["kv_rank"]),
                    p + "mix.uv": (m["heads"] * m["vdim"], m["kv_rank"]), p + "mix.o": (n, m["heads"] * m["vdim"])})
        if layer["mlp"]:
            f = layer["mlp"]["ff"]
            out.update({p + "norm2": (n,), p + "canon2": (n, cfg["canon"]["taps"]), p + "mlp.up": (f, n), p + "mlp.up.b": (f,),
                        p + "mlp.down": (n, f), p + "mlp.down.b": (n,), p + "mlp.act": (2,)})
    out.update({"final.norm": (n,), "head": (v, n)})
    return out


def random_tensors(cfg, seed=0, gain=1.0):
    """bfloat16-valued weights; norm gains around 1, projections of unit output scale times `gain`."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        if "norm" in name:
            w = 1.0 + 0.2 * rng.standard_normal(shape)
        elif "canon" in name:
            w = 0.4 * rng.standard_normal(shape)
        elif name.endswith(".b") or name.endswith(".act"):
            w = 0.3 * rng.standard_normal(shape)
        elif name == "embed":
            w = rng.standard_normal(shape)
        else:
            w = gain * rng.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = to_bf16(w.astype(np.float32))
    return out


def write_model(folder, cfg, tensors):
    """config.json and model.safetensors (bfloat16) as a user would have them."""
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    head, blobs, at = {}, [], 0
    for name, w in tensors.items():
        blob = (np.ascontiguousarray(w, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(w.shape), "data_offsets": [at, at + len(blob)]}
        blobs.append(blob)
        at += len(blob)
    text = json.dumps(head).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(text)) + text + b"".join(blobs))
    return folder
