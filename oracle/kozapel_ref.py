"""TEST INFRASTRUCTURE ONLY — plain numpy restatement of the Kozapel decoder, one function per mechanism, written from the
design's equations and slow on purpose: every position is computed from the whole sequence, there is no cache and no batch.
Arithmetic is float64 on the stored (bfloat16-valued) weights.

The decoder keeps `streams` copies of the residual. A sublayer reads a weighted sum of them through a norm; its output is added
to all of them while they are mixed with one another,

    u = sum_s in_s x_s,    y = f(rms(u)),    x_t <- sum_s mix_st x_s + out_t y.

Mixers are latent attention (queries through a latent too, no window) and differential attention with grouped heads in a sliding
window, whose keys and values may be an earlier layer's; feed-forwards are gated tanh-gelu or a mixture of squared-relu experts
with a shared one. Nothing under gpt.rs_b200/ may import this module.
"""
from __future__ import annotations

import numpy as np

from .felepel_ref import rms, sigmoid, to_bf16, write_model  # noqa: F401  (the same norm and the same file format)

D = np.float64


def embed(tokens, table, scale):
    return table[tokens] * scale


# ---- residual streams ------------------------------------------------------------------------------------------------------
def stream_input(x, w_in):
    """x [s][T][width] -> what a sublayer's norm reads [T][width]."""
    return np.einsum("s,stw->tw", w_in, x)


def stream_update(x, y, mix, w_out):
    """mix [from][to]; every new stream is made from all the old ones."""
    return np.einsum("st,snw->tnw", mix, x) + w_out[:, None, None] * y


# ---- attention -------------------------------------------------------------------------------------------------------------
def rotate(x, pos, base):
    """x [T][..][dims]: the pair (2i, 2i + 1) turns by pos base^(-2i / dims)."""
    dims = x.shape[-1]
    a = pos.reshape(-1, *[1] * (x.ndim - 1)) * base ** (-np.arange(0, dims, 2) / dims)
    out = np.empty_like(x)
    u, v = x[..., 0::2], x[..., 1::2]
    out[..., 0::2], out[..., 1::2] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


def softmax_attention(q, k, v, scale, window=None):
    """q [T][H][a], k [T][G][a], v [T][G][b] -> [T][H][b]; position i sees i - window + 1 .. i (no window: 0 .. i)."""
    t_n, heads, _ = q.shape
    group = heads // k.shape[1]
    out = np.zeros((t_n, heads, v.shape[2]), D)
    for i in range(t_n):
        lo = 0 if window is None else max(0, i - window + 1)
        for h in range(heads):
            s = k[lo:i + 1, h // group] @ q[i, h] * scale
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, h // group]
    return out


def latent_attention(h, w, c, eps):
    """Keys and values expanded per head from the latent."""
    t_n, heads, dim, rd, rank = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["kv_rank"]
    pos = np.arange(t_n)
    cq = rms(h @ w["dq"].T, eps) * w["dq.norm"]
    q = (cq @ w["uq"].T).reshape(t_n, heads, dim + rd)
    both = h @ w["dkv"].T
    lat = rms(both[:, :rank], eps) * w["dkv.norm"]
    base = c["rot"]["base"]
    kr = rotate(both[:, rank:], pos, base)
    q = np.concatenate([q[..., :dim], rotate(q[..., dim:], pos, base)], -1)
    k = np.concatenate([(lat @ w["uk"].T).reshape(t_n, heads, dim), np.repeat(kr[:, None], heads, 1)], -1)
    v = (lat @ w["uv"].T).reshape(t_n, heads, c["vdim"])
    return softmax_attention(q, k, v, c["scale"]).reshape(t_n, -1) @ w["o"].T


def diff_lambda(w, diff):
    return np.exp(np.sum(w["lq1"] * w["lk1"])) - np.exp(np.sum(w["lq2"] * w["lk2"])) + diff


def diff_combine(a1, a2, lam, diff, eps):
    """Two maps' outputs [T][H][vdim] -> one, of unit root mean square per head, times 1 - diff."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def keys_values(h, w, c):
    t_n, kv = h.shape[0], c["kv_heads"]
    return (h @ w["k"].T).reshape(t_n, kv, 2, c["dim"]), (h @ w["v"].T).reshape(t_n, kv, c["vdim"])


def diff_attention(h, w, c, kv, eps):
    """kv: this layer's keys and values, or those of the layer it takes them from."""
    t_n, heads = h.shape[0], c["heads"]
    q = (h @ w["q"].T).reshape(t_n, heads, 2, c["dim"])
    k, v = kv
    window = (c.get("mask") or {}).get("size")
    a1, a2 = (softmax_attention(q[:, :, m], k[:, :, m], v, c["scale"], window) for m in (0, 1))
    o = diff_combine(a1, a2, diff_lambda(w, c["diff"]), c["diff"], eps)
    return (o.reshape(t_n, -1) * sigmoid(h @ w["g"].T)) @ w["o"].T


# ---- feed-forward ----------------------------------------------------------------------------------------------------------
def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def dense(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def relu2(z):
    return np.maximum(z, 0.0) ** 2


def expert(h, w, name):
    return relu2(h @ w[name + ".up"].T) @ w[name + ".down"].T


def route(z, correction, top, count, keep, scale):
    """Logits z [E] of one token -> (chosen experts, their weights). Choices go by sigmoid + correction, a group's score is the
    sum of its two largest; weights are the chosen sigmoids in proportion."""
    s = sigmoid(z)
    choice = s + correction
    groups = choice.reshape(count, -1)
    score = np.sort(groups, axis=1)[:, -2:].sum(axis=1)
    best = np.argsort(-score, kind="stable")[:keep]
    allowed = np.full(groups.shape, -np.inf)
    allowed[best] = groups[best]
    chosen = np.argsort(-allowed.ravel(), kind="stable")[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20) * scale


def mixture(h, w, c):
    r = c["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    out = expert(h, w, "shared") if c.get("shared") else np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(*route(h[t] @ w["router"].T, w["correction"], r["top"], g["count"], g["keep"], r["scale"])):
            out[t] += s * expert(h[t], w, f"e{e}")
    return out


# ---- the model -------------------------------------------------------------------------------------------------------------
def forward(cfg, tensors, tokens, streams=False):
    """Logits [T][vocab] of a whole sequence from position 0; with `streams` also the sum of the streams after every layer."""
    w = {n: np.asarray(t, D) for n, t in tensors.items()}
    eps = cfg["norm"]["eps"]
    x0 = embed(np.asarray(tokens), w["embed"], cfg["embedding"]["scale"])
    x = np.repeat(x0[None], cfg["streams"], axis=0)
    after, kv = [], {}

    def sublayer(x, p, q, f):
        hc = {n: w[f"{p}hc{q}.{n}"] for n in ("in", "mix", "out")}
        u = stream_input(x, hc["in"])
        y = f(rms(u, eps) * w[f"{p}norm{q}"])
        return stream_update(x, y, hc["mix"], hc["out"])

    for i, layer in enumerate(cfg["layers"]):
        p, c = f"l{i}.", layer["mixer"]
        part = lambda s: {n[len(p + s) + 1:]: t for n, t in w.items() if n.startswith(p + s + ".")}  # noqa: E731, B023
        mix, mlp = part("mix"), part("mlp")

        def mixer(h):
            if layer["type"] == "latent_attention":
                return latent_attention(h, mix, c, eps)
            if "kv_from" not in c:
                kv[i] = keys_values(h, mix, c)
            return diff_attention(h, mix, c, kv[c.get("kv_from", i)], eps)

        x = sublayer(x, p, 1, mixer)
        if layer.get("mlp"):
            x = sublayer(x, p, 2, (lambda h: dense(h, mlp)) if layer["mlp"]["kind"] == "dense" else (lambda h: mixture(h, mlp, layer["mlp"])))
        after.append(x.sum(axis=0))
    logits = (rms(x.sum(axis=0), eps) * w["final.norm"]) @ w["head"].T
    return (logits, np.stack(after)) if streams else logits
