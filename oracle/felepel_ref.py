"""TEST INFRASTRUCTURE ONLY — plain numpy restatement of the Felepel decoder, one function per mechanism, written from the
design's equations and slow on purpose: every position is computed from the whole sequence, there is no cache, no state that
outlives a call and no batch. Arithmetic is float64 on the stored (bfloat16-valued) weights.

The decoder: embedding plus a learned position vector, then per layer up to two sublayers with a norm on either side,

    x <- x + rms(mixer(rms(x))),    x <- x + rms(experts(rms(x))),

where the mixer is either grouped-query attention inside fixed chunks (soft-capped scores, a logarithmic distance penalty) or a
gated delta rule with a decay per key channel, and the feed-forward is a mixture of experts chosen from the best groups. Layers
may reuse an earlier layer's weights. Nothing under gpt.rs_b200/ may import this module.
"""
from __future__ import annotations

import copy
import json
import struct
from pathlib import Path

import numpy as np

D = np.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def embed(tokens, table, positions):
    """Row t: table[token t] + positions[t]."""
    return table[tokens] + positions[np.arange(len(tokens))]


# ---- attention -----------------------------------------------------------------------------------------------------------
def soft_cap(s, cap):
    return cap * np.tanh(s / cap)


def distance_penalty(r1, r2, distance):
    """r1 ln(1 + r2 distance), taken off a score."""
    return r1 * np.log(1.0 + r2 * distance)


def chunk_visible(i, j, size):
    """Position i sees j: not later, and in the same run of `size` positions counted from the start of the sequence."""
    return j <= i and i // size == j // size


def chunked_attention(q, k, v, r1, r2, scale, cap, size):
    """q [T][H][a], k [T][G][a], v [T][G][b], r1 and r2 [H] -> [T][H][b]."""
    t_n, heads, _ = q.shape
    group = heads // k.shape[1]
    out = np.zeros((t_n, heads, v.shape[2]), D)
    for i in range(t_n):
        js = [j for j in range(i // size * size, i + 1) if chunk_visible(i, j, size)]
        lo, hi = js[0], js[-1] + 1
        dist = i - np.arange(lo, hi)
        for h in range(heads):
            s = k[lo:hi, h // group] @ q[i, h] * scale
            s = soft_cap(s, cap) - distance_penalty(r1[h], r2[h], dist)
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:hi, h // group]
    return out


def attention(h, w, c):
    """h [T][width]; w: the mixer's tensors by short name; c: the mixer's configuration."""
    t_n, heads, kv = h.shape[0], c["heads"], c["kv_heads"]
    q = (h @ w["q"].T + w["q.b"]).reshape(t_n, heads, c["dim"])
    k = (h @ w["k"].T + w["k.b"]).reshape(t_n, kv, c["dim"])
    v = (h @ w["v"].T + w["v.b"]).reshape(t_n, kv, c["vdim"])
    o = chunked_attention(q, k, v, w["r1"], w["r2"], c["scale"], c["softcap"], c["mask"]["size"])
    return o.reshape(t_n, heads * c["vdim"]) @ w["o"].T + w["o.b"]


# ---- delta rule ----------------------------------------------------------------------------------------------------------
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


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def channel_decay(a, a_log, dt_bias):
    """a, dt_bias [..][H][dim], a_log [H]: exp(-exp(a_log_h) softplus(a + dt_bias))."""
    return np.exp(-np.exp(a_log)[:, None] * softplus(a + dt_bias))


def delta_rule(q, k, v, decay, beta):
    """q, k, decay [T][H][dim], v [T][H][vdim], beta [T][H]; the state S [H][dim][vdim] starts at zero. Per token the rows of S
    decay, S takes up beta (v - S^T k) under k, and q reads S."""
    t_n, heads, dim = k.shape
    s = np.zeros((heads, dim, v.shape[2]), D)
    out = np.zeros_like(v)
    for t in range(t_n):
        s = decay[t][:, :, None] * s
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", s, k[t]))
        s = s + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", s, q[t])
    return out


def channel_delta(h, w, c, eps):
    t_n, heads, kv, dim, vdim = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(short_conv(h @ w[n].T, w[n + ".conv"])) for n in "qkv")
    of = np.arange(heads) // (heads // kv)          # the q/k head of every head
    q = (unit(q.reshape(t_n, kv, dim)) * dim ** -0.5)[:, of]
    k = unit(k.reshape(t_n, kv, dim))[:, of]
    beta = sigmoid(h @ w["b"].T)
    a = ((h @ w["a1"].T) @ w["a2"].T).reshape(t_n, heads, dim)
    decay = channel_decay(a, w["A_log"], w["dt_bias"].reshape(heads, dim))
    o = delta_rule(q, k, v.reshape(t_n, heads, vdim), decay, beta)
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T).reshape(t_n, heads, vdim)
    return (rms(o, eps) * w["norm"] * gate).reshape(t_n, heads * vdim) @ w["o"].T


# ---- experts -------------------------------------------------------------------------------------------------------------
def route(z, top, count, keep):
    """Logits z [E] of one token -> (chosen experts, their weights). The experts form `count` groups of neighbours; only those of
    the `keep` groups with the largest best score take part, the `top` best of them are chosen."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    groups = s.reshape(count, -1)
    best = np.argsort(-groups.max(axis=1), kind="stable")[:keep]
    allowed = np.full(groups.shape, -1.0)
    allowed[best] = groups[best]
    chosen = np.argsort(-allowed.ravel(), kind="stable")[:top]
    return chosen, s[chosen]


def expert(h, w, e):
    return (silu(h @ w[f"e{e}.gate"].T) * (h @ w[f"e{e}.up"].T)) @ w[f"e{e}.down"].T


def mixture(h, w, c):
    r = c["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(*route(h[t] @ w["router"].T, r["top"], g["count"], g["keep"])):
            out[t] += s * expert(h[t], w, e)
    return out


# ---- the model -----------------------------------------------------------------------------------------------------------
def forward(cfg, tensors, tokens, streams=False):
    """Logits [T][vocab] of a whole sequence from position 0; with `streams` also the residual after every layer."""
    w = {n: np.asarray(t, D) for n, t in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = embed(np.asarray(tokens), w["embed"], w["pos"])
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        part = lambda s: {n[len(p + s) + 1:]: t for n, t in w.items() if n.startswith(p + s + ".")}  # noqa: E731
        h = rms(x, eps) * w[p + "norm1"]
        m = attention(h, part("mix"), layer["mixer"]) if layer["type"] == "attention" else channel_delta(h, part("mix"), layer["mixer"], eps)
        x = x + rms(m, eps) * w[p + "norm1b"]
        if layer.get("mlp"):
            y = mixture(rms(x, eps) * w[p + "norm2"], part("mlp"), layer["mlp"])
            x = x + rms(y, eps) * w[p + "norm2b"]
        after.append(x)
    logits = (rms(x, eps) * w["final.norm"]) @ w["head"].T
    return (logits, np.stack(after)) if streams else logits


# ---- small models for the tests ---------------------------------------------------------------------------------------
def to_bf16(x):
    b = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((b + 0x7FFF + ((b >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def moe(experts=6, top=2, count=2, keep=1, ff=40):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "groups": {"count": count, "keep": keep}, "top": top}}


def attention_layer(heads=4, kv_heads=2, dim=16, vdim=24, chunk=20, softcap=12.0, scale=None, mlp=moe()):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "softcap": softcap,
                      "scale": float(scale if scale is not None else dim ** -0.5)}}


def delta_layer(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, mlp=moe()):
    return {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def again(layers, j):
    """The entry of a layer that reuses layer j's weights."""
    return {**copy.deepcopy(layers[j]), "weights_of": j}


def model_config(layers, width=40, vocab=72, eps=1e-5, positions=1024):
    return {"architecture": "Felepel", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "max_positions": positions}


def tensor_shapes(cfg, decay_rank=10, gate_rank=6):
    n, v = cfg["width"], cfg["vocab"]
    out = {"embed": (v, n), "pos": (cfg["max_positions"], n)}
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        m, p = layer["mixer"], f"l{i}."
        x = p + "mix."
        qh, kh, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (n,), p + "norm1b": (n,)})
        if layer["type"] == "attention":
            for name, rows in (("q", qh * dim), ("k", kh * dim), ("v", kh * vdim)):
                out.update({x + name: (rows, n), x + name + ".b": (rows,)})
            out.update({x + "r1": (qh,), x + "r2": (qh,), x + "o": (n, qh * vdim), x + "o.b": (n,)})
        else:
            for name, rows in (("q", kh * dim), ("k", kh * dim), ("v", qh * vdim)):
                out.update({x + name: (rows, n), x + name + ".conv": (rows, m["conv"])})
            out.update({x + "b": (qh, n), x + "A_log": (qh,), x + "norm": (vdim,), x + "a1": (decay_rank, n), x + "a2": (qh * dim, decay_rank),
                        x + "dt_bias": (qh * dim,), x + "g1": (gate_rank, n), x + "g2": (qh * vdim, gate_rank), x + "o": (n, qh * vdim)})
        if layer["mlp"]:
            f = layer["mlp"]["expert"]["ff"]
            out.update({p + "norm2": (n,), p + "norm2b": (n,)})
            for e in range(layer["mlp"]["router"]["experts"]):
                out.update({f"{p}mlp.e{e}.gate": (f, n), f"{p}mlp.e{e}.up": (f, n), f"{p}mlp.e{e}.down": (n, f)})
            out[p + "mlp.router"] = (layer["mlp"]["router"]["experts"], n)
    out.update({"final.norm": (n,), "head": (v, n)})
    return out


def random_tensors(cfg, seed=0, **ranks):
    """bfloat16-valued weights; norm gains around 1, projections of unit output scale, decays spread between quick and slow."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, **ranks).items():
        last = name.rsplit(".", 1)[-1]
        if "norm" in last:
            w = 1.0 + 0.2 * rng.standard_normal(shape)
        elif last == "conv":
            w = 0.5 * rng.standard_normal(shape)
            w[:, -1] += 0.7
        elif last == "r1":
            w = rng.uniform(0.2, 1.0, shape)
        elif last == "r2":
            w = rng.uniform(0.05, 1.5, shape)
        elif last == "A_log":
            w = np.log(rng.uniform(0.3, 3.0, shape))
        elif last == "dt_bias":
            w = rng.uniform(-6.0, 0.0, shape)
        elif last == "b" and len(shape) == 1:
            w = 0.3 * rng.standard_normal(shape)
        elif last == "router":
            w = 2.0 * rng.standard_normal(shape) / np.sqrt(shape[-1])
        elif name in ("embed", "pos"):
            w = rng.standard_normal(shape)
        else:
            w = rng.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = to_bf16(w.astype(np.float32))
    return out


CODE = 8   # width reserved by `steady_routing`


def steady_routing(cfg, tensors, seed=0, margin=0.12):
    """Weights whose routers read the last CODE channels of the stream only, where every token keeps a code of its own that no layer
    adds to, drawn so that no choice of experts or groups is close: rounding then never changes an expert."""
    rng = np.random.default_rng(seed)
    t = {n: w.copy() for n, w in tensors.items()}
    routers = []
    t["pos"][:, -CODE:] = 0
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        t[f"l{i}.norm1b"][-CODE:] = 0
        if not layer["mlp"]:
            continue
        t[f"l{i}.norm2b"][-CODE:] = 0
        t[f"l{i}.norm2"][-CODE:] = 1
        w = t[f"l{i}.mlp.router"]
        w[:, :-CODE] = 0
        w[:, -CODE:] = to_bf16(rng.standard_normal((w.shape[0], CODE)).astype(np.float32))
        r = layer["mlp"]["router"]
        routers.append((w[:, -CODE:].astype(D), r["top"], r["groups"]["count"], r["groups"]["keep"]))

    def decided(z, top, count, keep):
        best = np.sort(z.reshape(count, -1).max(axis=1))[::-1]
        if keep < count and best[keep - 1] - best[keep] < margin * np.abs(z).max():
            return False
        chosen, _ = route(z, top, count, keep)
        allowed = np.isin(np.arange(len(z)) // (len(z) // count), np.argsort(-z.reshape(count, -1).max(axis=1), kind="stable")[:keep])
        rest = np.setdiff1d(np.nonzero(allowed)[0], chosen)
        return len(rest) == 0 or z[chosen].min() - z[rest].max() >= margin * np.abs(z).max()

    for v in range(cfg["vocab"]):
        for _ in range(20000):
            code = to_bf16((1.5 * rng.standard_normal(CODE)).astype(np.float32))
            if all(decided(w @ code, *r) for w, *r in routers):
                break
        else:
            raise ValueError("no code with this margin")
        t["embed"][v, -CODE:] = code
    return t


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
