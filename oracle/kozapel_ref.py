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


# ---- small models for the tests ---------------------------------------------------------------------------------------------
def dense_mlp(ff=48):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, count=3, keep=2, ff=24, scale=1.7, shared=40):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None,
            "router": {"experts": experts, "groups": {"count": count, "keep": keep}, "scale": scale, "top": top}}


def latent_layer(heads=4, dim=16, rot_dim=8, vdim=12, kv_rank=24, q_rank=20, base=300.0, scale=None, mlp=dense_mlp()):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "rot": {"base": base, "dims": rot_dim}, "scale": float(scale if scale is not None else (dim + rot_dim) ** -0.5)}}


def diff_layer(heads=4, kv_heads=2, dim=16, vdim=24, window=20, diff=0.4, scale=None, kv_from=None, mlp=dense_mlp()):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "diff": diff,
         "scale": float(scale if scale is not None else dim ** -0.5)}
    return {"type": "attention", "mlp": mlp, "mixer": m if kv_from is None else {**m, "kv_from": kv_from}}


def model_config(layers, width=40, vocab=72, eps=1e-5, streams=2, embed_scale=3.0):
    return {"architecture": "Kozapel", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "streams": streams,
            "embedding": {"scale": embed_scale}}


def tensor_shapes(cfg):
    n, v, s = cfg["width"], cfg["vocab"], cfg["streams"]
    out = {"embed": (v, n)}
    for i, layer in enumerate(cfg["layers"]):
        m, p, mlp = layer["mixer"], f"l{i}.", layer["mlp"]
        x, f = p + "mix.", p + "mlp."
        for q in (1, 2) if mlp else (1,):
            out.update({f"{p}norm{q}": (n,), f"{p}hc{q}.in": (s,), f"{p}hc{q}.out": (s,), f"{p}hc{q}.mix": (s, s)})
        heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "latent_attention":
            rank, rd, qr = m["kv_rank"], m["rot_dim"], m["q_rank"]
            out.update({x + "dq": (qr, n), x + "dq.norm": (qr,), x + "uq": (heads * (dim + rd), qr), x + "dkv": (rank + rd, n), x + "dkv.norm": (rank,),
                        x + "uk": (heads * dim, rank), x + "uv": (heads * vdim, rank)})
        else:
            out.update({x + "q": (heads * 2 * dim, n), x + "g": (heads * vdim, n), **{x + a: (dim,) for a in ("lq1", "lk1", "lq2", "lk2")}})
            if "kv_from" not in m:
                out.update({x + "k": (m["kv_heads"] * 2 * dim, n), x + "v": (m["kv_heads"] * vdim, n)})
        out[x + "o"] = (n, heads * vdim)
        if mlp and mlp["kind"] == "dense":
            out.update({f + "gate": (mlp["ff"], n), f + "up": (mlp["ff"], n), f + "down": (n, mlp["ff"])})
        elif mlp:
            names = [f"e{e}." for e in range(mlp["router"]["experts"])]
            for name, ff in [(a, mlp["expert"]["ff"]) for a in names] + ([("shared.", mlp["shared"]["ff"])] if mlp["shared"] else []):
                out.update({f + name + "up": (ff, n), f + name + "down": (n, ff)})
            out.update({f + "router": (mlp["router"]["experts"], n), f + "correction": (mlp["router"]["experts"],)})
    out.update({"final.norm": (n,), "head": (v, n)})
    return out


def random_tensors(cfg, seed=0, sharp=1.0):
    """bfloat16-valued weights; norm gains around 1, projections of unit output scale (queries times `sharp`), streams that differ, choices
    that the correction changes (some of them negative)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if "norm" in last:
            w = 1.0 + 0.2 * rng.standard_normal(shape)
        elif ".hc" in name:
            w = 0.25 * rng.standard_normal(shape)
            w += np.eye(*shape) if last == "mix" else 1.0 / shape[0] if last == "in" else 0.8
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            w = 0.6 * rng.standard_normal(shape) / shape[0] ** 0.25
        elif last == "correction":
            w = rng.uniform(-0.9, 0.3, shape)
        elif last == "router":
            w = 2.0 * rng.standard_normal(shape) / np.sqrt(shape[-1])
        elif name == "embed":
            w = 0.4 * rng.standard_normal(shape)
        else:
            w = rng.standard_normal(shape) / np.sqrt(shape[-1]) * (sharp if last in ("q", "uq") else 1.0)
        out[name] = to_bf16(w.astype(np.float32))
    return out


CODE = 8   # width reserved by `steady_routing`


def steady_routing(cfg, tensors, seed=0, margin=0.02):
    """Weights whose routers read the last CODE channels of the streams only, which no sublayer adds to, so that there every token keeps a
    code of its own times a number that depends on the layer. Codes are drawn so that no choice of experts or groups is close, whatever
    the norm makes of their size within a wide range: rounding then never changes an expert."""
    rng = np.random.default_rng(seed)
    t = {n: w.copy() for n, w in tensors.items()}
    coef, routers = np.ones(cfg["streams"]), []
    for i, layer in enumerate(cfg["layers"]):
        t[f"l{i}.mix.o"][-CODE:] = 0
        for n in t:
            if n.startswith(f"l{i}.mlp.") and n.endswith("down"):
                t[n][-CODE:] = 0
        for q in (1, 2) if layer["mlp"] else (1,):
            if q == 2 and layer["mlp"]["kind"] == "moe":
                # inputs scaled so that the code arrives with the size of the embedding, whatever the mixing has made of it
                w_in = t[f"l{i}.hc2.in"]
                t[f"l{i}.hc2.in"] = to_bf16(w_in / np.float32(w_in @ coef)) if abs(w_in @ coef) > 0.2 else to_bf16(np.float32(coef / (coef @ coef)))
                t[f"l{i}.norm2"][-CODE:] = 1
                w = t[f"l{i}.mlp.router"]
                w[:, :-CODE] = 0
                w[:, -CODE:] = to_bf16((1.5 * rng.standard_normal((w.shape[0], CODE))).astype(np.float32))
                routers.append((w[:, -CODE:].astype(D), t[f"l{i}.mlp.correction"].astype(D), layer["mlp"]["router"]))
            coef = t[f"l{i}.hc{q}.mix"].astype(D).T @ coef

    def picks(codes, w, corr, r):
        """Chosen experts [N][E] (bool) and whether nothing was close."""
        g = r["groups"]
        choice = sigmoid(codes @ w.T) + corr
        groups = choice.reshape(len(codes), g["count"], -1)
        score = np.sort(groups, axis=2)[:, :, -2:].sum(axis=2)
        order = np.sort(score, axis=1)[:, ::-1]
        ok = order[:, g["keep"] - 1] - order[:, g["keep"]] > margin if g["keep"] < g["count"] else np.full(len(codes), True)
        allowed = np.where((score >= order[:, [g["keep"] - 1]])[:, :, None], groups, -np.inf).reshape(len(codes), -1)
        best = np.sort(allowed, axis=1)[:, ::-1]
        if r["top"] < allowed.shape[1]:
            ok &= best[:, r["top"] - 1] - best[:, r["top"]] > margin
        return allowed >= best[:, [r["top"] - 1]], ok

    drawn = rng.standard_normal((60000, CODE))
    drawn *= 0.8 * CODE ** 0.5 / np.linalg.norm(drawn, axis=1, keepdims=True)
    drawn = to_bf16(drawn.astype(np.float32))
    good = np.full(len(drawn), True)
    for w, corr, r in routers:
        first = None
        for size in (0.35, 0.5, 0.7, 1.0, 1.4, 2.0):
            chosen, ok = picks(drawn * size, w, corr, r)
            first = chosen if first is None else first
            good &= ok & (chosen == first).all(axis=1)
    codes = drawn[good]
    if len(codes) < cfg["vocab"]:
        raise ValueError(f"only {len(codes)} codes with this margin")
    t["embed"][:, -CODE:] = to_bf16(codes[:cfg["vocab"]] * np.float32(1.5 / cfg["embedding"]["scale"]))
    return t
