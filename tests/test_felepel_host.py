"""Felepel without a GPU: configuration and weight readers, layouts, and the oracle's own properties (the mistakes that the GPU tests
must be able to see are planted here, in the oracle)."""
import copy
import ctypes

import numpy as np
import pytest

import gptrs_b200
from gptrs_b200 import BackendError, _abi
from gptrs_b200 import checkpoint as ck
from gptrs_b200 import model as gm
from oracle import felepel_ref as fr

A, DL = fr.attention_layer, fr.delta_layer
LAYERS = [DL(heads=6, kv_heads=3, dim=8, vdim=12, conv=5, mlp=None), A(heads=6, kv_heads=2, dim=24, vdim=16, chunk=14, softcap=7.5, scale=0.3),
          A(heads=3, kv_heads=3, mlp=fr.moe(experts=12, top=3, count=4, keep=2, ff=20))]
MIXED = fr.model_config(LAYERS + [fr.again(LAYERS, 1), fr.again(LAYERS, 0)], positions=200)


def _config(cfg, **kw):
    shapes = fr.tensor_shapes(MIXED)
    return ck.engine_config({"kind": "felepel", "config": cfg}, gm.MODE_BF16, shapes, **kw)[0]


def test_folder_reader_round_trip(tmp_path):
    t = fr.random_tensors(MIXED, 3)
    fr.write_model(tmp_path, MIXED, t)
    r = ck.open_model(tmp_path)
    assert r.kind == "felepel" and r.kind in ck.LAYERED_KINDS and r.model_config["config"] == MIXED
    assert ck.shapes_of(r) == {n: w.shape for n, w in t.items()}
    assert all(np.array_equal(r.get(n), w) for n, w in t.items())


def test_config_gives_every_size_and_constant():
    c = _config(MIXED, context_length=99, max_seqs=2)
    assert c.kind == gm.KIND_LAYERED and c.block == gm.BLOCK_SANDWICH
    assert (c.d_model, c.vocab, c.n_layers, c.context_length, c.learned_positions, c.norm_eps) == (40, 72, 5, 99, 200, 1e-5)
    l0, l1, l2, l3, l4 = c.layers
    assert (l0.mixer, l0.heads, l0.kv_heads, l0.dim, l0.vdim, l0.taps, l0.decay_rank, l0.gate_rank, l0.mlp) == (gm.MIXER_CHANNEL_DELTA, 6, 3, 8, 12, 5, 10, 6, gm.MLP_NONE)
    assert (l1.mixer, l1.heads, l1.kv_heads, l1.dim, l1.vdim, l1.scale, l1.softcap) == (gm.MIXER_GROUPED_ATTENTION, 6, 2, 24, 16, 0.3, 7.5)
    assert (l1.mask, l1.mask_size, l1.distance_bias, l1.proj_bias) == (gm.MASK_CHUNK, 14, 1, 1)
    assert (l1.mlp, l1.d_ff, l1.experts, l1.top, l1.groups, l1.keep) == (gm.MLP_EXPERTS, 40, 6, 2, 2, 1)
    assert (l2.experts, l2.top, l2.groups, l2.keep, l2.d_ff) == (12, 3, 4, 2, 20)
    assert [l.weights_of for l in c.layers] == [-1, -1, -1, 1, 0] and (l4.decay_rank, l3.mask_size) == (10, 14)
    assert c.param_shapes() == fr.tensor_shapes(MIXED)


def test_context_is_bounded_by_the_position_table():
    assert _config(MIXED).context_length == 200
    assert _config(MIXED, context_length=10 ** 6).context_length == 200


def test_ranks_come_from_the_tensors_or_the_config():
    shapes = fr.tensor_shapes(MIXED, decay_rank=17, gate_rank=33)
    c = ck.felepel_config(MIXED, shapes)
    assert (c.layers[0].decay_rank, c.layers[0].gate_rank, c.layers[4].decay_rank) == (17, 33, 17)
    with pytest.raises(BackendError, match="rank"):
        ck.felepel_config(MIXED)
    named = copy.deepcopy(MIXED)
    for i in (0, 4):
        named["layers"][i]["mixer"].update(decay_rank=5, gate_rank=7)
    c = ck.felepel_config(named)
    assert (c.layers[0].decay_rank, c.layers[4].gate_rank) == (5, 7)


def test_router_without_groups():
    cfg = copy.deepcopy(MIXED)
    del cfg["layers"][2]["mlp"]["router"]["groups"]
    c = _config(cfg)
    assert (c.layers[2].groups, c.layers[2].keep) == (1, 1)


@pytest.mark.parametrize("change", ["type", "kind", "reuse"])
def test_unknown_parts_are_refused(change):
    cfg = copy.deepcopy(MIXED)
    if change == "type":
        cfg["layers"][2]["type"] = "other_mixer"
    elif change == "kind":
        cfg["layers"][2]["mlp"]["kind"] = "dense"
    else:
        cfg["layers"][3]["mixer"]["heads"] = 4
    with pytest.raises(BackendError):
        _config(cfg)


@pytest.mark.parametrize("dtype,want", [
    (0, dict(q_head_stride=14, k_offset=84, k_head_stride=14, v_offset=112, v_head_stride=70, q_row=252, out_head_stride=70, page_bytes=2 * 16 * 84 * 4)),
    (2, dict(q_head_stride=16, k_offset=96, k_head_stride=16, v_offset=128, v_head_stride=72, q_row=272, out_head_stride=72, page_bytes=2 * 16 * 192 * 2))])
def test_grouped_layout(dtype, want):
    def layout(**kw):
        v = dict(dtype=dtype, heads=6, kv_heads=2, dim=14, vdim=70, mask=gm.MASK_CHUNK, mask_size=33, scale=0.25, softcap=9.0, distance_bias=1)
        a = _abi.GroupedAttention(*{**v, **kw}.values())
        return gptrs_b200.lib().gptrs_cuda_grouped_layout(ctypes.byref(a)), a
    rc, a = layout()
    assert rc == 0 and {k: getattr(a, k) for k in want} == want
    for bad in (dict(mask_size=0), dict(mask=5), dict(heads=5), dict(scale=0.0), dict(softcap=-1.0), dict(vdim=2000), dict(dim=0)):
        assert layout(**bad)[0] != 0, bad
    assert layout(mask=gm.MASK_CAUSAL, mask_size=0)[0] == 0


@pytest.mark.parametrize("dtype,want", [
    (0, dict(q_offset=0, k_offset=21, v_offset=42, beta_offset=96, a_offset=102, g_offset=105, row=114, decay_row=42, gate_row=54, out_head_stride=9, conv_channels=96)),
    (2, dict(q_offset=0, k_offset=24, v_offset=48, beta_offset=104, a_offset=112, g_offset=120, row=136, decay_row=48, gate_row=56, out_head_stride=16, conv_channels=96))])
def test_delta_layout(dtype, want):
    def layout(**kw):
        v = dict(dtype=dtype, heads=6, kv_heads=3, dim=7, vdim=9, taps=4, decay_rank=3, gate_rank=9, eps=1e-5)
        a = _abi.DeltaRule(*{**v, **kw}.values())
        return gptrs_b200.lib().gptrs_cuda_delta_layout(ctypes.byref(a)), a
    rc, a = layout()
    assert rc == 0 and {k: getattr(a, k) for k in want} == want
    assert (a.state_floats, a.conv_floats) == (6 * 7 * 9, 2 * 3 * 96)
    for bad in (dict(kv_heads=4), dict(taps=0), dict(dim=1000), dict(decay_rank=-1), dict(vdim=0)):
        assert layout(**bad)[0] != 0, bad


# ---- the oracle --------------------------------------------------------------------------------------------------------
SHOW = fr.model_config([A(chunk=20, softcap=3.0), DL(), A(chunk=13, softcap=3.0, mlp=None), DL(mlp=None)], positions=120)


def _sharp(cfg, seed, factor=3.0):
    t = fr.random_tensors(cfg, seed)
    return {n: fr.to_bf16(w * factor) if n.endswith("mix.q") else w for n, w in t.items()}


def test_sharp_weights_show_every_planted_mistake(monkeypatch):
    """With the query projections scaled up a few keys dominate most rows, so an edge that is one token off, a lost state or a
    constant that is wrong moves the logits far beyond the tolerances of the GPU tests."""
    t = _sharp(SHOW, 5)
    tok = np.random.default_rng(1).integers(0, SHOW["vocab"], 90)
    good = fr.forward(SHOW, t, tok)

    def moved(change_cfg=None, change_t=None):
        c, w = copy.deepcopy(SHOW), dict(t)
        if change_cfg:
            change_cfg(c)
        if change_t:
            change_t(w)
        return float(np.sqrt(np.mean((fr.forward(c, w, tok) - good) ** 2)) / np.sqrt(np.mean(good ** 2)))

    mixer = lambda i: (lambda c: c["layers"][i]["mixer"])  # noqa: E731
    assert moved(lambda c: mixer(0)(c)["mask"].update(size=21)) > 0.03
    assert moved(lambda c: mixer(2)(c)["mask"].update(size=12)) > 0.03
    assert moved(lambda c: mixer(0)(c).update(softcap=6.0)) > 0.03
    assert moved(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=2)) > 0.03
    assert moved(lambda c: c["layers"][1]["mlp"]["router"].update(top=1)) > 0.03
    for name, rows in (("l0.mix.r1", None), ("l0.mix.r2", None), ("l0.mix.k.b", None), ("l0.mix.o.b", None), ("pos", None), ("l1.mix.dt_bias", None),
                       ("l1.mix.A_log", None), ("l1.mix.b", None), ("l3.mix.a2", None), ("l3.mix.g2", None)):
        assert moved(None, lambda w: w.update({name: 0 * w[name]})) > 0.01, name
    assert moved(None, lambda w: w.update({"l1.mix.q.conv": np.concatenate([0 * w["l1.mix.q.conv"][:, :1], w["l1.mix.q.conv"][:, 1:]], 1)})) > 0.01
    # a recurrence that forgets its state after 40 tokens, and a read-out in front of the write
    rule = fr.delta_rule

    def forgets(q, k, v, d, b):
        return np.concatenate([rule(q[s], k[s], v[s], d[s], b[s]) for s in (slice(0, 40), slice(40, None))])
    monkeypatch.setattr(fr, "delta_rule", forgets)
    assert moved() > 0.02


def test_oracle_is_causal_and_chunked():
    cfg = fr.model_config([A(chunk=8, mlp=None)])
    t = fr.random_tensors(cfg, 2)
    tok = np.random.default_rng(2).integers(0, cfg["vocab"], 30)
    full = fr.forward(cfg, t, tok)
    assert np.allclose(fr.forward(cfg, t, tok[:17]), full[:17], atol=1e-12)
    other = tok.copy()
    other[10] = (other[10] + 1) % cfg["vocab"]   # one layer: its own chunk from there on, nothing else
    d = np.abs(fr.forward(cfg, t, other) - full).max(axis=1)
    assert np.all(d[:10] == 0) and np.all(d[10:16] > 1e-9) and np.all(d[16:] == 0)


def test_oracle_state_reaches_far():
    cfg = fr.model_config([DL(mlp=None)])
    t = fr.random_tensors(cfg, 2)
    tok = np.random.default_rng(2).integers(0, cfg["vocab"], 80)
    other = tok.copy()
    other[3] = (other[3] + 1) % cfg["vocab"]
    d = np.abs(fr.forward(cfg, t, other) - fr.forward(cfg, t, tok)).max(axis=1)
    assert np.all(d[:3] == 0) and d[79] > 1e-4


def test_route_keeps_the_best_groups():
    z = np.array([5.0, 0.0, 4.9, 4.8, 1.0, 4.0])
    for count, keep, top, want in ((3, 1, 2, [0, 1]), (3, 2, 2, [0, 2]), (3, 2, 3, [0, 2, 3]), (1, 1, 3, [0, 2, 3]), (6, 3, 3, [0, 2, 3])):
        chosen, s = fr.route(z, top, count, keep)
        assert chosen.tolist() == want
        assert np.allclose(s, (np.exp(z) / np.exp(z).sum())[want])   # scores over all experts, not renormalized
