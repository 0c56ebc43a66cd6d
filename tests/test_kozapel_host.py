"""Kozapel without a GPU: configuration and weight readers, layouts, and the oracle's own properties (the mistakes that the GPU tests
must be able to see are planted here, in the oracle)."""
import copy
import ctypes

import numpy as np
import pytest

import gptrs_b200
from gptrs_b200 import BackendError, _abi
from gptrs_b200 import checkpoint as ck
from gptrs_b200 import model as gm
from oracle import kozapel_ref as kr

A, L, M = kr.diff_layer, kr.latent_layer, kr.moe
MIXED = kr.model_config([A(heads=6, kv_heads=2, dim=24, vdim=16, window=14, diff=0.3, scale=0.2, mlp=M(experts=12, top=3, count=4, keep=2, ff=20, scale=2.5, shared=36)),
                         L(heads=3, dim=10, rot_dim=6, vdim=14, kv_rank=22, q_rank=9, base=77.0, scale=0.4, mlp=None),
                         A(heads=12, kv_heads=2, dim=24, vdim=16, window=31, diff=0.7, kv_from=0), L(mlp=M(shared=0))], streams=4, embed_scale=5.5, eps=1e-4)


def _config(cfg, **kw):
    return ck.engine_config({"kind": "kozapel", "config": cfg}, gm.MODE_BF16, None, **kw)[0]


def test_folder_reader_round_trip(tmp_path):
    t = kr.random_tensors(MIXED, 3)
    kr.write_model(tmp_path, MIXED, t)
    r = ck.open_model(tmp_path)
    assert r.kind == "kozapel" and r.kind in ck.LAYERED_KINDS and r.model_config["config"] == MIXED
    assert ck.shapes_of(r) == {n: w.shape for n, w in t.items()}
    assert all(np.array_equal(r.get(n), w) for n, w in t.items())


def test_config_gives_every_size_and_constant():
    c = _config(MIXED, context_length=99, max_seqs=2)
    assert c.kind == gm.KIND_LAYERED and c.block == gm.BLOCK_PRE_NORM
    assert (c.d_model, c.vocab, c.n_layers, c.context_length, c.streams, c.embed_scale, c.norm_eps, c.learned_positions) == (40, 72, 4, 99, 4, 5.5, 1e-4, 0)
    l0, l1, l2, l3 = c.layers
    assert (l0.mixer, l0.heads, l0.kv_heads, l0.dim, l0.vdim, l0.scale, l0.maps, l0.out_gate, l0.diff) == (gm.MIXER_GROUPED_ATTENTION, 6, 2, 24, 16, 0.2, 2, 1, 0.3)
    assert (l0.mask, l0.mask_size, l0.kv_from, l0.softcap, l0.distance_bias, l0.proj_bias) == (gm.MASK_WINDOW, 14, -1, 0.0, 0, 0)
    assert (l0.mlp, l0.expert_form, l0.d_ff, l0.experts, l0.top, l0.groups, l0.keep, l0.shared_ff) == (gm.MLP_EXPERTS, gm.EXPERT_RELU2, 20, 12, 3, 4, 2, 36)
    assert (l0.route, l0.group_best, l0.correction, l0.weight_scale) == (gm.ROUTE_SIGMOID, 2, 1, 2.5)
    assert (l1.mixer, l1.heads, l1.dim, l1.rot_dim, l1.rot_dims, l1.vdim, l1.kv_rank, l1.q_rank, l1.rope_base, l1.scale, l1.window, l1.mlp) == \
        (gm.MIXER_LATENT_ATTENTION, 3, 10, 6, 6, 14, 22, 9, 77.0, 0.4, 0, gm.MLP_NONE)
    assert (l2.kv_from, l2.mask_size, l2.diff, l2.heads, l2.mlp, l2.d_ff) == (0, 31, 0.7, 12, gm.MLP_DENSE_GELU, 48)
    assert l3.shared_ff == 0
    assert c.param_shapes() == kr.tensor_shapes(MIXED)


def test_optional_parts():
    cfg = copy.deepcopy(MIXED)
    del cfg["layers"][0]["mlp"]["router"]["groups"], cfg["layers"][0]["mlp"]["shared"], cfg["layers"][0]["mixer"]["mask"], cfg["streams"]
    cfg["layers"][1]["mixer"]["mask"] = {"size": 40}
    c = _config(cfg)
    l0, l1 = c.layers[:2]
    assert (l0.groups, l0.keep, l0.shared_ff, l0.mask, l1.window, c.streams) == (1, 1, 0, gm.MASK_CAUSAL, 40, 0)
    assert not any(".hc" in n for n in c.param_shapes())


@pytest.mark.parametrize("change", ["type", "kind"])
def test_unknown_parts_are_refused(change):
    cfg = copy.deepcopy(MIXED)
    if change == "type":
        cfg["layers"][2]["type"] = "other_mixer"
    else:
        cfg["layers"][2]["mlp"]["kind"] = "other"
    with pytest.raises(BackendError):
        _config(cfg)


@pytest.mark.parametrize("dtype,want", [
    (0, dict(map_stride=13, q_head_stride=26, k_offset=104, k_head_stride=26, v_offset=156, v_head_stride=70, g_offset=296, g_head_stride=70, q_row=576, out_head_stride=70,
             page_bytes=2 * 16 * 96 * 4)),
    (2, dict(map_stride=16, q_head_stride=32, k_offset=128, k_head_stride=32, v_offset=192, v_head_stride=72, g_offset=336, g_head_stride=72, q_row=624, out_head_stride=72,
             page_bytes=2 * 16 * 256 * 2))])
def test_differential_layout(dtype, want):
    def layout(**kw):
        a = _abi.GroupedAttention(dtype=dtype, heads=4, kv_heads=2, dim=13, vdim=70, mask=gm.MASK_WINDOW, mask_size=33, scale=0.25, maps=2, gate=1)
        for k, v in kw.items():
            setattr(a, k, v)
        return gptrs_b200.lib().gptrs_cuda_grouped_layout(ctypes.byref(a)), a
    rc, a = layout()
    assert rc == 0 and {k: getattr(a, k) for k in want} == want
    _, b = layout(shared_kv=1)   # queries and gates only; the pages are the other layer's
    assert b.g_offset == b.k_offset == want["k_offset"] and b.q_row == b.g_offset + 4 * want["g_head_stride"] and b.page_bytes == a.page_bytes
    _, b = layout(gate=0)
    assert b.q_row == want["g_offset"]
    assert layout(maps=3)[0] != 0 and layout(maps=1)[1].q_head_stride == want["map_stride"]


@pytest.mark.parametrize("dtype,want", [(0, dict(q_row=60, q_latent_row=5, dkv_offset=5, rot_offset=26, kv_row=32)),
                                        (2, dict(q_row=72, q_latent_row=8, dkv_offset=8, rot_offset=32, kv_row=40))])
def test_latent_layout_with_query_latent(dtype, want):
    a = _abi.LatentAttention(dtype, 3, 14, 6, 11, 21, 0, 6, 0.25, 5)
    assert gptrs_b200.lib().gptrs_cuda_latent_layout(ctypes.byref(a)) == 0
    assert {k: getattr(a, k) for k in want} == want


# ---- the oracle --------------------------------------------------------------------------------------------------------
SHOW = kr.model_config([A(window=20, mlp=M()), L(mlp=None), A(window=13, kv_from=0, diff=0.6), L(mlp=M(experts=8, top=3, count=2, keep=1))], streams=3)


def test_sharp_weights_show_every_planted_mistake():
    """With the query projections scaled up a few keys dominate most rows, so an edge that is one token off, a lost stream or a constant
    that is wrong moves the logits far beyond the tolerances of the GPU tests."""
    t = kr.random_tensors(SHOW, 5, sharp=3.0)
    tok = np.random.default_rng(1).integers(0, SHOW["vocab"], 90)
    good = kr.forward(SHOW, t, tok)

    def moved(change_cfg=None, change_t=None, **patched):
        c, w = copy.deepcopy(SHOW), dict(t)
        if change_cfg:
            change_cfg(c)
        if change_t:
            change_t(w)
        old = {n: getattr(kr, n) for n in patched}
        try:
            for n, f in patched.items():
                setattr(kr, n, f)
            got = kr.forward(c, w, tok)
        finally:
            for n, f in old.items():
                setattr(kr, n, f)
        return float(np.sqrt(np.mean((got - good) ** 2)) / np.sqrt(np.mean(good ** 2)))

    mixer = lambda i: (lambda c: c["layers"][i]["mixer"])  # noqa: E731
    assert moved(lambda c: mixer(0)(c)["mask"].update(size=21)) > 0.01
    assert moved(lambda c: mixer(2)(c)["mask"].update(size=12)) > 0.01
    assert moved(lambda c: mixer(2)(c).update(diff=0.4)) > 0.01
    assert moved(lambda c: mixer(1)(c)["rot"].update(base=400.0)) > 0.01
    assert moved(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3)) > 0.01
    assert moved(lambda c: c["layers"][3]["mlp"]["router"].update(scale=1.8)) > 0.005
    assert moved(lambda c: c["embedding"].update(scale=1.0)) > 0.01
    for name in ("l0.mix.g", "l1.mix.dq.norm", "l3.mix.dkv.norm", "l0.mlp.correction", "l0.mlp.shared.down", "l2.mix.lq1", "l2.mix.lq2"):
        assert moved(None, lambda w: w.update({name: 0 * w[name]})) > 0.01, name
    for n in ("l0.hc1", "l0.hc2", "l3.hc2"):
        assert moved(None, lambda w: w.update({n + ".mix": np.ascontiguousarray(w[n + ".mix"].T)})) > 0.01, n
        if n != "l0.hc1":   # where all streams are still equal
            assert moved(None, lambda w: w.update({n + ".in": w[n + ".in"][::-1]})) > 0.01, n
    route = kr.route
    assert moved(route=route_by_best) > 0.01
    assert moved(route=lambda z, c, *a: (lambda ch, w: (ch, w * 0 + a[-1] / len(ch)))(*route(z, c, *a))) > 0.01
    assert moved(diff_combine=lambda a1, a2, lam, diff, eps: kr.rms(a1 - lam * a2, eps)) > 0.01   # the factor 1 - diff is lost
    # a stream that is updated before the next one has read it
    def one_after_another(x, y, mix, w_out):
        x = x.copy()
        for s in range(len(x)):
            x[s] = np.einsum("s,snw->nw", mix[:, s], x) + w_out[s] * y
        return x
    assert moved(stream_update=one_after_another) > 0.01


def route_by_best(z, correction, top, count, keep, scale):
    """A group counts as much as its best expert alone."""
    s = kr.sigmoid(z)
    groups = (s + correction).reshape(count, -1)
    allowed = np.full(groups.shape, -np.inf)
    best = np.argsort(-groups.max(axis=1), kind="stable")[:keep]
    allowed[best] = groups[best]
    chosen = np.argsort(-allowed.ravel(), kind="stable")[:top]
    return chosen, s[chosen] / s[chosen].sum() * scale


def test_oracle_is_causal_and_windowed():
    cfg = kr.model_config([A(window=8, mlp=None)])
    t = kr.random_tensors(cfg, 2)
    tok = np.random.default_rng(2).integers(0, cfg["vocab"], 30)
    full = kr.forward(cfg, t, tok)
    assert np.allclose(kr.forward(cfg, t, tok[:17]), full[:17], atol=1e-12)
    other = tok.copy()
    other[10] = (other[10] + 1) % cfg["vocab"]   # one layer: the eight positions from there on, nothing else
    d = np.abs(kr.forward(cfg, t, other) - full).max(axis=1)
    assert np.all(d[:10] == 0) and np.all(d[10:18] > 1e-9) and np.all(d[18:] == 0)


def test_route_on_paper():
    """Groups by the sum of their two best, choices by score + correction (a group that is out stays out even where its scores are above
    negative ones), weights by the score alone."""
    z = np.array([2.0, -2.0, 0.5, 0.4, 1.0, -5.0])
    s = kr.sigmoid(z)
    chosen, w = kr.route(z, np.zeros(6), 2, 3, 1, 3.0)
    assert chosen.tolist() == [2, 3] and np.allclose(w, 3.0 * s[[2, 3]] / s[[2, 3]].sum())
    chosen, w = kr.route(z, np.array([0, 0, -0.5, -0.5, 0, 0]), 2, 3, 1, 3.0)
    assert chosen.tolist() == [0, 1]
    chosen, w = kr.route(z, np.full(6, -2.0), 3, 3, 2, 1.0)   # every choice score is negative
    assert chosen.tolist() == [0, 2, 3] and np.allclose(w.sum(), 1.0)


def test_steady_routing_survives_rounding(monkeypatch):
    t = kr.steady_routing(SHOW, kr.random_tensors(SHOW, 4), 4)
    tok = np.random.default_rng(3).integers(0, SHOW["vocab"], 60)
    route, picks = kr.route, []
    for noise in (0.0, 0.02):
        rng = np.random.default_rng(0)
        picks.append([])

        def noisy(z, *a):
            chosen = route(z + noise * rng.standard_normal(z.shape), *a)
            picks[-1].append(tuple(sorted(chosen[0])))
            return chosen
        monkeypatch.setattr(kr, "route", noisy)
        kr.forward(SHOW, t, tok)
    assert picks[0] == picks[1] and len(set(picks[0])) > 3
