"""Domorax without a GPU: configuration and weight readers, layouts, and the oracle's own properties (the mistakes that the GPU tests
must be able to see are planted here, in the oracle)."""
import copy
import ctypes

import numpy as np
import pytest

import gptrs_b200
from gptrs_b200 import BackendError, _abi
from gptrs_b200 import checkpoint as ck
from gptrs_b200 import model as gm
from oracle import domorax_ref as dr

L, A, DL, M, F = dr.latent_layer, dr.attention_layer, dr.delta_layer, dr.moe, dr.dense_mlp
MIXED = dr.model_config([A(heads=6, kv_heads=3, dim=10, conv=5, scale=0.2, mlp=M(experts=12, top=3, ff=20, shared=36)),
                         L(heads=3, dim=10, rot_dim=6, vdim=14, kv_rank=22, q_rank=9, window=31, base=77.0, scaling=(3.5, 48, 6.0, 0.5), scale=0.4, mlp=None),
                         DL(heads=6, kv_heads=2, dim=12, vdim=7, conv=2, mlp=F(52)), L(scaling=None, window=None, mlp=M(shared=0))], width=45, groups=3, mult=0.7, eps=1e-4)


def _config(cfg, **kw):
    return ck.engine_config({"kind": "domorax", "config": cfg}, gm.MODE_BF16, None, **kw)[0]


def test_folder_reader_round_trip(tmp_path):
    t = dr.random_tensors(MIXED, 3)
    dr.write_model(tmp_path, MIXED, t)
    r = ck.open_model(tmp_path)
    assert r.kind == "domorax" and r.kind in ck.LAYERED_KINDS and r.model_config["config"] == MIXED
    assert ck.shapes_of(r) == {n: w.shape for n, w in t.items()}
    assert all(np.array_equal(r.get(n), w) for n, w in t.items())


def test_config_gives_every_size_and_constant():
    c = _config(MIXED, context_length=99, max_seqs=2)
    assert c.kind == gm.KIND_LAYERED and c.block == gm.BLOCK_DEPTH
    assert (c.d_model, c.vocab, c.n_layers, c.context_length, c.norm_eps, c.norm_groups, c.residual_mult, c.learned_positions, c.streams) == (45, 72, 4, 99, 1e-4, 3, 0.7, 0, 0)
    l0, l1, l2, l3 = c.layers
    assert (l0.mixer, l0.heads, l0.kv_heads, l0.dim, l0.vdim, l0.scale, l0.taps, l0.qk_norm, l0.tied) == (gm.MIXER_GROUPED_ATTENTION, 6, 3, 10, 10, 0.2, 5, 1, 1)
    assert (l0.mask, l0.distance_bias, l0.softcap, l0.proj_bias, l0.kv_from, l0.maps, l0.out_gate) == (gm.MASK_CAUSAL, gm.DISTANCE_LINEAR, 0.0, 0, -1, 1, 0)
    assert (l0.mlp, l0.expert_form, l0.d_ff, l0.experts, l0.top, l0.groups, l0.shared_ff, l0.shared_gate) == (gm.MLP_EXPERTS, gm.EXPERT_SWIGLU, 20, 12, 3, 1, 36, 1)
    assert (l0.route, l0.correction, l0.weight_scale) == (gm.ROUTE_SOFTMAX, 0, 1.0)
    assert (l1.mixer, l1.heads, l1.dim, l1.rot_dim, l1.rot_dims, l1.vdim, l1.kv_rank, l1.q_rank, l1.rope_base, l1.scale, l1.window, l1.sink, l1.rope_halves, l1.mlp) == \
        (gm.MIXER_LATENT_ATTENTION, 3, 10, 6, 6, 14, 22, 9, 77.0, 0.4, 31, 1, 1, gm.MLP_NONE)
    assert (l1.rope_factor, l1.rope_original, l1.rope_fast, l1.rope_slow) == (3.5, 48.0, 6.0, 0.5)
    assert (l2.mixer, l2.heads, l2.kv_heads, l2.dim, l2.vdim, l2.taps, l2.decay_rank, l2.gate_rank, l2.gate_silu) == (gm.MIXER_CHANNEL_DELTA, 6, 2, 12, 7, 2, 0, 0, 1)
    assert (l2.mlp, l2.d_ff) == (gm.MLP_DENSE_POLY, 52)
    assert (l3.rope_factor, l3.window, l3.shared_ff, l3.shared_gate) == (0.0, 0, 0, 0)
    assert c.param_shapes() == dr.tensor_shapes(MIXED)


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
    (0, dict(q_head_stride=13, k_offset=52, v_offset=78, g_offset=78, q_row=78, query_row=52, out_head_stride=13, conv_channels=78, conv_floats=2 * 3 * 78,
             page_bytes=2 * 16 * 13 * 4 + 2 * 16 * 4)),
    (2, dict(q_head_stride=16, k_offset=64, v_offset=96, g_offset=96, q_row=96, query_row=64, out_head_stride=16, conv_channels=96, conv_floats=2 * 3 * 96,
             page_bytes=2 * 16 * 64 * 2 + 2 * 16 * 4))])
def test_layout_of_values_that_are_keys(dtype, want):
    """The cache holds one vector and one number per key, the projection rows no values; without tied values the page is that of [value | key]."""
    def layout(**kw):
        a = _abi.GroupedAttention(dtype=dtype, heads=4, kv_heads=2, dim=13, vdim=13, scale=0.25, distance_bias=gm.DISTANCE_LINEAR, taps=4, qk_norm=1, tied=1)
        for k, v in kw.items():
            setattr(a, k, v)
        return gptrs_b200.lib().gptrs_cuda_grouped_layout(ctypes.byref(a)), a
    rc, a = layout()
    assert rc == 0 and {k: getattr(a, k) for k in want} == want
    rc, b = layout(tied=0, vdim=70)
    assert rc == 0 and b.page_bytes == 2 * 16 * ((13 + 70) * 4 if dtype == 0 else 192 * 2) and b.q_row == want["v_offset"] + 2 * b.v_head_stride and b.query_row == want["query_row"]
    rc, b = layout(tied=0, qk_norm=0, taps=0)   # nothing to prepare: attention reads the projection rows
    assert rc == 0 and b.query_row == b.q_row and b.conv_floats == 0
    for bad in (dict(vdim=12), dict(maps=2), dict(gate=1), dict(shared_kv=1), dict(distance_bias=gm.DISTANCE_LOG), dict(distance_bias=3), dict(taps=-1)):
        assert layout(**bad)[0] != 0, bad


@pytest.mark.parametrize("dtype,want", [(0, dict(a_offset=102, g_offset=108, row=162, decay_row=0, gate_row=162)), (2, dict(a_offset=112, g_offset=120, row=176, decay_row=0, gate_row=176))])
def test_delta_layout_with_one_decay_per_head(dtype, want):
    a = _abi.DeltaRule(dtype, 6, 3, 7, 9, 4, 0, 0, 1e-5, 1)
    assert gptrs_b200.lib().gptrs_cuda_delta_layout(ctypes.byref(a)) == 0
    assert {k: getattr(a, k) for k in want} == want


# ---- the oracle --------------------------------------------------------------------------------------------------------
SHOW = dr.model_config([L(mlp=F()), A(mlp=M()), DL(mlp=None), L(window=13, mlp=M(experts=8, top=3, shared=0)), A(heads=3, kv_heads=1, conv=2)], width=42, groups=3)


def test_sharp_weights_show_every_planted_mistake():
    """With larger scores a few keys dominate most rows, so an edge that is one token off, a lost state or a constant that is wrong moves
    the logits far beyond the tolerances of the GPU tests."""
    t = dr.random_tensors(SHOW, 5, sharp=3.0)
    tok = np.random.default_rng(1).integers(0, SHOW["vocab"], 90)
    good = dr.forward(SHOW, t, tok)

    def moved(change_cfg=None, change_t=None, **patched):
        c, w = copy.deepcopy(SHOW), dict(t)
        if change_cfg:
            change_cfg(c)
        if change_t:
            change_t(w)
        old = {n: getattr(dr, n) for n in patched}
        try:
            for n, f in patched.items():
                setattr(dr, n, f)
            got = dr.forward(c, w, tok)
        finally:
            for n, f in old.items():
                setattr(dr, n, f)
        return float(np.sqrt(np.mean((got - good) ** 2)) / np.sqrt(np.mean(good ** 2)))

    mixer = lambda i: (lambda c: c["layers"][i]["mixer"])  # noqa: E731
    assert moved(lambda c: mixer(0)(c)["mask"].update(size=21)) > 0.01
    assert moved(lambda c: mixer(3)(c)["mask"].update(size=12)) > 0.01
    assert moved(lambda c: mixer(0)(c)["rot"].update(base=400.0)) > 0.005
    for key in ("factor", "original"):
        assert moved(lambda c: mixer(0)(c)["rot"]["scaling"].update({key: 2 * mixer(0)(c)["rot"]["scaling"][key]})) > 0.003, key
    assert moved(lambda c: c.update(residual_mult=0.63)) > 0.005
    assert moved(lambda c: c["norm"].update(groups=1)) > 0.005
    for name in ("l0.mix.dq.norm", "l3.mix.dkv.norm", "l1.mix.k.norm", "l2.mix.g", "l2.mix.norm", "l1.mlp.shared.down", "l0.dwa", "l4.dwa"):
        assert moved(None, lambda w: w.update({name: 0 * w[name]})) > 0.01, name
    for name in ("l0.mix.sink", "l3.mix.sink"):   # no sink
        assert moved(None, lambda w: w.update({name: w[name] - 100})) > 0.01, name
    for name in ("l0.mlp.act", "l0.dwa", "l3.dwa", "l2.mix.A_log", "l2.mix.dt_bias"):
        assert moved(None, lambda w: w.update({name: w[name][::-1]})) > 0.01, name
    for name in ("l1.mix.q.conv", "l4.mix.k.conv", "l2.mix.v.conv"):   # the oldest input lost
        assert moved(None, lambda w: w.update({name: np.concatenate([0 * w[name][:, :1], w[name][:, 1:]], 1)})) > 0.005, name

    def interleaved(x, pos, dims, freq, mag):
        a = pos.reshape(-1, *[1] * (x.ndim - 1)) * freq
        out = x.copy()
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = (u * np.cos(a) - v * np.sin(a)) * mag, (v * np.cos(a) + u * np.sin(a)) * mag
        return out
    assert moved(rotate_halves=interleaved) > 0.005
    rotate = dr.rotate_halves
    assert moved(rotate_halves=lambda x, pos, dims, freq, mag: rotate(x, pos, dims, freq, 1.0)) > 0.003
    slope = dr.slope
    assert moved(slope=lambda n, heads: slope(n - 1, heads)) > 0.005
    assert moved(slope=lambda n, heads: 0.0) > 0.005
    biased = dr.biased_attention   # values behind the norm, or of the next kv head
    assert moved(biased_attention=lambda q, k, v, s: biased(q, k, dr.rms(v, 1e-5), s)) > 0.005
    assert moved(biased_attention=lambda q, k, v, s: biased(q, k, v[:, ::-1], s)) > 0.005
    conv = dr.short_conv
    assert moved(short_conv=lambda x, w: conv(x, w[:, ::-1])) > 0.01
    delta = dr.delta_rule

    def reads_first(q, k, v, decay, beta):   # the read-out before the token's own write
        own = beta[..., None] * np.einsum("thd,thd->th", k, q)[..., None]
        return delta(q, k, v, decay, beta) - own * v
    assert moved(delta_rule=reads_first) > 0.005
    assert moved(route=lambda z, top: (np.argsort(-z)[:top], dr.softmax_sink(z)[np.argsort(-z)[:top]])) > 0.005   # softmax over all
    assert moved(poly_norm=lambda z, act, eps: act[0] * dr.rms(z, eps) + act[1] * dr.rms(z, eps) ** 2 + act[2] * dr.rms(z, eps) ** 3 + act[3]) > 0.005
    assert moved(depth_average=lambda states, a: a[-1] * states[-1] + sum(w * s for w, s in zip(a[:-1], states[1:]))) > 0.01   # one result off


def test_oracle_is_causal_and_windowed():
    cfg = dr.model_config([L(window=8, mlp=None)])
    t = dr.random_tensors(cfg, 2)
    tok = np.random.default_rng(2).integers(0, cfg["vocab"], 30)
    full = dr.forward(cfg, t, tok)
    assert np.allclose(dr.forward(cfg, t, tok[:17]), full[:17], atol=1e-12)
    other = tok.copy()
    other[10] = (other[10] + 1) % cfg["vocab"]   # one layer: the eight positions from there on, nothing else
    d = np.abs(dr.forward(cfg, t, other) - full).max(axis=1)
    assert np.all(d[:10] == 0) and np.all(d[10:18] > 1e-9) and np.all(d[18:] == 0)


def test_mechanisms_on_paper():
    assert np.allclose(dr.group_rms(np.array([3.0, 4.0, 1.0, 1.0]), 2, 0.0), [3 / 12.5 ** 0.5, 4 / 12.5 ** 0.5, 1, 1])
    assert np.allclose(dr.softmax_sink(np.log([1.0, 3.0]), np.log(4.0)), [1 / 8, 3 / 8])
    assert np.allclose([dr.slope(h, 4) for h in range(4)], [1 / 4, 1 / 16, 1 / 64, 1 / 256])
    z = np.array([1.0, -2.0])
    n = lambda v: v / np.sqrt(np.mean(v * v))  # noqa: E731
    assert np.allclose(dr.poly_norm(z, np.array([1.0, 2.0, 3.0, 4.0]), 0.0), n(z) + 2 * n(z * z) + 3 * n(z ** 3) + 4)
    chosen, w = dr.route(np.array([0.0, 2.0, 1.0]), 2)
    assert chosen.tolist() == [1, 2] and np.allclose(w, [1 / (1 + np.exp(-1)), 1 / (1 + np.exp(1))])
    f, mag = dr.yarn(8, 10000.0, {"factor": 4.0, "original": 1000, "fast": 32.0, "slow": 1.0})
    plain, one = dr.yarn(8, 10000.0)
    assert one == 1.0 and abs(mag - (0.1 * np.log(4.0) + 1)) < 1e-12
    # 1000 / (2 pi 32) turns: dimension 8 ln(4.97) / (2 ln 1e4) = 0.70 -> 0; 1000 / (2 pi): 2.20 -> 3: a ramp of thirds
    assert np.allclose(f, plain * [1, 1 - 0.75 / 3, 1 - 0.75 * 2 / 3, 0.25])


def test_steady_routing_survives_rounding(monkeypatch):
    t = dr.steady_routing(SHOW, dr.random_tensors(SHOW, 4), 4)
    tok = np.random.default_rng(3).integers(0, SHOW["vocab"], 60)
    route, picks = dr.route, []
    for noise in (0.0, 0.02):
        rng = np.random.default_rng(0)
        picks.append([])

        def noisy(z, top):
            chosen = route(z + noise * rng.standard_normal(z.shape), top)
            picks[-1].append(tuple(sorted(chosen[0])))
            return chosen
        monkeypatch.setattr(dr, "route", noisy)
        dr.forward(SHOW, t, tok)
    assert picks[0] == picks[1] and len(set(picks[0])) > 3
