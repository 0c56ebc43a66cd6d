"""TEST INFRASTRUCTURE ONLY — plain numpy restatement of the Domorax decoder, one function per mechanism, written from the
design's equations and slow on purpose: every position is computed from the whole sequence, there is no cache, no state that
outlives a call and no batch. Arithmetic is float64 on the stored (bfloat16-valued) weights.

The decoder keeps every layer's result. A layer reads the running stream x and adds the normed outputs of its sublayers, each
norm taken over equal groups of channels; what goes on is a weighted sum of the embedding and of all results so far,

    x <- x + m groupnorm(mixer(x)),    x <- x + m groupnorm(ff(x)),    X_(i+1) = x,    x <- sum_j a_ij X_j.

Mixers are latent attention in a window (queries through a latent too, a sink per head, rotation with stretched wavelengths),
attention whose values are its keys before their norm (short convolutions on both, norms per head, a linear distance bias) and a
gated delta rule with one decay per head; feed-forwards are dense with a polynomial activation of normed powers, or a mixture of
gated experts with a gated shared one. Nothing under gpt.rs_b200/ may import this module.
"""
from __future__ import annotations

import numpy as np

from .felepel_ref import delta_rule, rms, short_conv, sigmoid, silu, softplus, to_bf16, unit, write_model  # noqa: F401

D = np.float64


# ---- the stream ------------------------------------------------------------------------------------------------------------
def group_rms(x, groups, eps):
    """Every one of `groups` equal consecutive parts of the last axis divided by its own root mean square."""
    return rms(x.reshape(*x.shape[:-1], groups, -1), eps).reshape(x.shape)


def depth_average(states, a):
    """states: the embedding and the results of the layers so far; a: a weight for each."""
    return sum(w * s for w, s in zip(a, states, strict=True))


# ---- latent attention --------------------------------------------------------------------------------------------------------
def yarn(dims, base, scaling=None):
    """Frequencies [dims / 2] and the factor on cos and sin."""
    i = np.arange(dims // 2)
    f = base ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0
    s = scaling["factor"]
    dim_of = lambda turns: dims * np.log(scaling["original"] / (2 * np.pi * turns)) / (2 * np.log(base))  # noqa: E731
    lo, hi = max(np.floor(dim_of(scaling["fast"])), 0), min(np.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0, 1)
    return f / s * ramp + f * (1 - ramp), 0.1 * np.log(s) + 1


def rotate_halves(x, pos, dims, freq, mag):
    """x [T][..][n]: dimensions i and i + dims / 2 turn together, those from `dims` on stay."""
    a = pos.reshape(-1, *[1] * (x.ndim - 1)) * freq
    cos, sin = np.cos(a) * mag, np.sin(a) * mag
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return np.concatenate([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def softmax_sink(s, sink=None):
    """Weights of the scores s; the exponential of `sink` counts in the denominator and has no weight of its own."""
    top = s.max() if sink is None else max(s.max(), sink)
    p = np.exp(s - top)
    return p / (p.sum() + (0.0 if sink is None else np.exp(sink - top)))


def latent_attention(h, w, c, eps):
    """Keys and values expanded per head from the latent; position i sees i - window + 1 .. i."""
    t_n, heads, dim, rd, rank = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["kv_rank"]
    pos = np.arange(t_n)
    cq = rms(h @ w["dq"].T, eps) * w["dq.norm"]
    q = (cq @ w["uq"].T).reshape(t_n, heads, dim + rd)
    both = h @ w["dkv"].T
    lat = rms(both[:, :rank], eps) * w["dkv.norm"]
    r = c["rot"]
    turn = (pos, r["dims"], *yarn(r["dims"], r["base"], r.get("scaling")))
    kr, qr = rotate_halves(both[:, rank:], *turn), rotate_halves(q[..., dim:], *turn)
    k = (lat @ w["uk"].T).reshape(t_n, heads, dim)
    v = (lat @ w["uv"].T).reshape(t_n, heads, c["vdim"])
    window = (c.get("mask") or {}).get("size")
    out = np.zeros((t_n, heads, c["vdim"]), D)
    for i in range(t_n):
        lo = 0 if window is None else max(0, i - window + 1)
        for n in range(heads):
            s = (k[lo:i + 1, n] @ q[i, n, :dim] + kr[lo:i + 1] @ qr[i, n]) * c["scale"]
            out[i, n] = softmax_sink(s, w["sink"][n]) @ v[lo:i + 1, n]
    return out.reshape(t_n, -1) @ w["o"].T


# ---- attention whose values are keys ---------------------------------------------------------------------------------------
def slope(head, heads):
    return 2.0 ** (-8.0 * (head + 1) / heads)


def biased_attention(q, k, v, scale):
    """q [T][H][a], k [T][G][a], v [T][G][b] -> [T][H][b]: all of 0 .. i, less the head's slope per position of distance."""
    t_n, heads, _ = q.shape
    group = heads // k.shape[1]
    out = np.zeros((t_n, heads, v.shape[2]), D)
    for i in range(t_n):
        away = i - np.arange(i + 1)
        for n in range(heads):
            s = k[:i + 1, n // group] @ q[i, n] * scale - slope(n, heads) * away
            out[i, n] = softmax_sink(s) @ v[:i + 1, n // group]
    return out


def attention(h, w, c, eps):
    t_n, heads, kv, dim = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q = short_conv(h @ w["q"].T, w["q.conv"]).reshape(t_n, heads, dim)
    k = short_conv(h @ w["k"].T, w["k.conv"]).reshape(t_n, kv, dim)
    o = biased_attention(rms(q, eps) * w["q.norm"], rms(k, eps) * w["k.norm"], k, c["scale"])
    return o.reshape(t_n, -1) @ w["o"].T


# ---- delta rule ----------------------------------------------------------------------------------------------------------------
def head_decay(a, a_log, dt_bias):
    """One per head: exp(-exp(A_log) softplus(a + dt_bias))."""
    return np.exp(-np.exp(a_log) * softplus(a + dt_bias))


def gated_delta(h, w, c, eps):
    t_n, heads, kv, dim, vdim = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(short_conv(h @ w[n].T, w[n + ".conv"])) for n in "qkv")
    of = np.arange(heads) // (heads // kv)          # the q/k head of every head
    q = (unit(q.reshape(t_n, kv, dim)) * dim ** -0.5)[:, of]
    k = unit(k.reshape(t_n, kv, dim))[:, of]
    decay = head_decay(h @ w["a"].T, w["A_log"], w["dt_bias"])
    o = delta_rule(q, k, v.reshape(t_n, heads, vdim), np.repeat(decay[:, :, None], dim, 2), sigmoid(h @ w["b"].T))
    gate = silu(h @ w["g"].T).reshape(t_n, heads, vdim)
    return (rms(o, eps) * w["norm"] * gate).reshape(t_n, -1) @ w["o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------------------------
def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense(h, w, eps):
    return poly_norm(h @ w["up"].T, w["act"], eps) @ w["down"].T


def expert(h, w, name):
    return (silu(h @ w[name + ".gate"].T) * (h @ w[name + ".up"].T)) @ w[name + ".down"].T


def route(z, top):
    """Logits z [E] of one token -> (chosen experts, the softmax over their logits)."""
    chosen = np.argsort(-z, kind="stable")[:top]
    return chosen, softmax_sink(z[chosen])


def mixture(h, w, c):
    out = np.zeros_like(h)
    if c.get("shared"):
        out += expert(h, w, "shared") * sigmoid(h @ w["shared.sg"].T)
    for t in range(h.shape[0]):
        for e, s in zip(*route(h[t] @ w["router"].T, c["router"]["top"])):
            out[t] += s * expert(h[t], w, f"e{e}")
    return out


# ---- the model -----------------------------------------------------------------------------------------------------------------
def forward(cfg, tensors, tokens, streams=False):
    """Logits [T][vocab] of a whole sequence from position 0; with `streams` also what goes on after every layer."""
    w = {n: np.asarray(t, D) for n, t in tensors.items()}
    eps, groups, m = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["residual_mult"]
    x = w["embed"][np.asarray(tokens)]
    states, after = [x], []
    mixers = {"latent_attention": latent_attention, "attention": attention, "delta": gated_delta}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        part = lambda s: {n[len(p + s) + 1:]: t for n, t in w.items() if n.startswith(p + s + ".")}  # noqa: E731, B023
        x = x + m * group_rms(mixers[layer["type"]](x, part("mix"), layer["mixer"], eps), groups, eps) * w[p + "norm1"]
        if layer.get("mlp"):
            y = dense(x, part("mlp"), eps) if layer["mlp"]["kind"] == "dense" else mixture(x, part("mlp"), layer["mlp"])
            x = x + m * group_rms(y, groups, eps) * w[p + "norm2"]
        states.append(x)
        x = depth_average(states, w[p + "dwa"])
        after.append(x)
    logits = (group_rms(x, groups, eps) * w["final.norm"]) @ w["head"].T
    return (logits, np.stack(after)) if streams else logits


# ---- small models for the tests -----------------------------------------------------------------------------------------------
def dense_mlp(ff=48):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, shared=40):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, **({"shared": {"ff": shared}} if shared else {})}


def latent_layer(heads=4, dim=16, rot_dim=8, vdim=12, kv_rank=24, q_rank=20, window=20, base=300.0, scaling=(4.0, 64, 8.0, 1.0), scale=None, mlp=dense_mlp()):
    """scaling: (factor, original, fast, slow) or None."""
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "rot": rot,
         "scale": float(scale if scale is not None else (dim + rot_dim) ** -0.5)}
    return {"type": "latent_attention", "mlp": mlp, "mixer": {**m, "mask": {"size": window}} if window else m}


def attention_layer(heads=4, kv_heads=2, dim=16, conv=3, scale=None, mlp=dense_mlp()):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv,
                                                      "scale": float(scale if scale is not None else dim ** -0.5)}}


def delta_layer(heads=4, kv_heads=2, dim=16, vdim=24, conv=4, mlp=dense_mlp()):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def model_config(layers, width=40, vocab=72, eps=1e-5, groups=2, mult=0.6):
    return {"architecture": "Domorax", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps, "groups": groups}, "residual_mult": mult}


def tensor_shapes(cfg):
    n, v = cfg["width"], cfg["vocab"]
    out = {"embed": (v, n)}
    for i, layer in enumerate(cfg["layers"]):
        m, p, mlp = layer["mixer"], f"l{i}.", layer["mlp"]
        x, f = p + "mix.", p + "mlp."
        heads, dim, vdim, kv = m["heads"], m["dim"], m["vdim"], m.get("kv_heads")
        out.update({p + "norm1": (n,), p + "dwa": (i + 2,), x + "o": (n, heads * vdim)})
        if layer["type"] == "latent_attention":
            rank, rd, qr = m["kv_rank"], m["rot_dim"], m["q_rank"]
            out.update({x + "dq": (qr, n), x + "dq.norm": (qr,), x + "uq": (heads * (dim + rd), qr), x + "dkv": (rank + rd, n), x + "dkv.norm": (rank,),
                        x + "uk": (heads * dim, rank), x + "uv": (heads * vdim, rank), x + "sink": (heads,)})
        elif layer["type"] == "attention":
            for name, rows in (("q", heads * dim), ("k", kv * dim)):
                out.update({x + name: (rows, n), x + name + ".conv": (rows, m["conv"]), x + name + ".norm": (dim,)})
        else:
            for name, rows in (("q", kv * dim), ("k", kv * dim), ("v", heads * vdim)):
                out.update({x + name: (rows, n), x + name + ".conv": (rows, m["conv"])})
            out.update({x + "b": (heads, n), x + "a": (heads, n), x + "A_log": (heads,), x + "dt_bias": (heads,), x + "g": (heads * vdim, n), x + "norm": (vdim,)})
        if not mlp:
            continue
        out[p + "norm2"] = (n,)
        if mlp["kind"] == "dense":
            out.update({f + "up": (mlp["ff"], n), f + "down": (n, mlp["ff"]), f + "act": (4,)})
            continue
        names = [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if mlp.get("shared"):
            names.append(("shared.", mlp["shared"]["ff"]))
            out[f + "shared.sg"] = (1, n)
        for name, ff in names:
            out.update({f + name + "gate": (ff, n), f + name + "up": (ff, n), f + name + "down": (n, ff)})
        out[f + "router"] = (mlp["router"]["experts"], n)
    out.update({"final.norm": (n,), "head": (v, n)})
    return out


def random_tensors(cfg, seed=0, sharp=1.0):
    """bfloat16-valued weights; norm gains around 1, projections of unit output scale (what makes scores larger times `sharp`), sinks that take a
    share of the softmax, decays between quick and slow, averages over depth that lean on the newest result."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if "norm" in last:
            w = (1.0 + 0.2 * rng.standard_normal(shape)) * (sharp if name.endswith("q.norm") and not name.endswith("dq.norm") else 1.0)
        elif last == "conv":
            w = 0.5 * rng.standard_normal(shape)
            w[:, -1] += 0.7
        elif last == "sink":
            w = rng.uniform(0.5, 3.0, shape)
        elif last == "dwa":
            w = 0.25 * rng.standard_normal(shape)
            w[-1] += 0.8
        elif last == "act":
            w = rng.uniform(0.3, 1.0, shape) * np.array([1, 1, -1, 1])
        elif last == "A_log":
            w = np.log(rng.uniform(0.3, 3.0, shape))
        elif last == "dt_bias":
            w = rng.uniform(-6.0, 0.0, shape)
        elif last == "router":
            w = 2.0 * rng.standard_normal(shape) / np.sqrt(shape[-1])
        elif name == "embed":
            w = rng.standard_normal(shape)
        else:
            w = rng.standard_normal(shape) / np.sqrt(shape[-1]) * (sharp if last == "uq" else 1.0)
        out[name] = to_bf16(w.astype(np.float32))
    return out


CODE = 8   # width reserved by `steady_routing`


def steady_routing(cfg, tensors, seed=0, margin=0.12):
    """Weights whose routers read the last CODE channels of the stream only, which no sublayer adds to: there every token keeps a code of its
    own times a number that depends on the layer. Codes are drawn so that no choice is close: rounding then never changes an expert."""
    rng = np.random.default_rng(seed)
    t = {n: w.copy() for n, w in tensors.items()}
    routers, states, now = [], [1.0], 1.0   # what the averages over depth have made of a code of 1
    for i, layer in enumerate(cfg["layers"]):
        t[f"l{i}.norm1"][-CODE:] = 0
        if layer["mlp"]:
            t[f"l{i}.norm2"][-CODE:] = 0
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            w = t[f"l{i}.mlp.router"]
            w[:, :-CODE] = 0
            w[:, -CODE:] = to_bf16(rng.standard_normal((w.shape[0], CODE)).astype(np.float32))
            routers.append((w[:, -CODE:].astype(D) * now, layer["mlp"]["router"]["top"]))
        states.append(now)
        now = float(np.dot(t[f"l{i}.dwa"].astype(D), states))
        if abs(now) < 0.3:   # codes would fade: lean on the newest result
            t[f"l{i}.dwa"] = to_bf16(np.eye(i + 2)[-1].astype(np.float32))
            now = states[-1]

    def decided(z, top):
        order = np.sort(z)[::-1]
        return top == len(z) or order[top - 1] - order[top] >= margin * np.abs(z).max()

    for v in range(cfg["vocab"]):
        for _ in range(20000):
            code = to_bf16((1.5 * rng.standard_normal(CODE)).astype(np.float32))
            if all(decided(w @ code, top) for w, top in routers):
                break
        else:
            raise ValueError("no code with this margin")
        t["embed"][v, -CODE:] = code
    return t
