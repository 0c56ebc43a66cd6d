"""Bevosun without a GPU: configuration and weight readers, the replay's slot and batch logic, and the oracle's own properties
(the mistakes that the GPU tests must be able to see are planted here, in the oracle)."""
import copy
import ctypes
import json

import numpy as np
import pytest

import gptrs_b200
from gptrs_b200 import BackendError, _abi
from gptrs_b200 import checkpoint as ck
from gptrs_b200 import model as gm
from gptrs_b200 import trace
from oracle import bevosun_ref as br

MIXED = br.model_config([br.layer_config(), br.layer_config(heads=3, dim=24, rot_dim=12, vdim=20, kv_rank=40, window=9, ff=None),
                         br.layer_config(heads=1, window=33, base=500.0, ff=64)])


def test_folder_reader_round_trip(tmp_path):
    t = br.random_tensors(MIXED, 3)
    br.write_model(tmp_path, MIXED, t)
    r = ck.open_model(tmp_path)
    assert r.kind == "bevosun" and r.model_config["config"] == MIXED
    assert {e.name: e.dims for e in r.entries} == {n: w.shape for n, w in t.items()}
    for n, w in t.items():
        assert np.array_equal(r.get(n), w)
    with pytest.raises(BackendError):
        r.get("l9.mix.q")


def test_config_gives_every_size_and_constant():
    c, scaling = ck.engine_config({"kind": "bevosun", "config": MIXED}, gm.MODE_BF16, context_length=99, max_seqs=2)
    assert scaling is None and c.kind == gm.KIND_LAYERED and (c.d_model, c.vocab, c.n_layers, c.context_length) == (40, 72, 3, 99)
    assert (c.norm_eps, c.conv_taps, c.logit_softcap) == (1e-5, 3, 20.0)
    l0, l1, l2 = c.layers
    assert (l1.heads, l1.dim, l1.rot_dim, l1.vdim, l1.kv_rank, l1.window) == (3, 24, 12, 20, 40, 9)
    assert l1.mlp == gm.MLP_NONE and (l0.d_ff, l2.d_ff) == (48, 64) and l2.rope_base == 500.0
    assert l1.scale == pytest.approx(36 ** -0.5)
    assert c.param_shapes() == br.tensor_shapes(MIXED)


@pytest.mark.parametrize("change", [("architecture", "Other"), ("type", "other_mixer"), ("kind", "other")])
def test_unknown_parts_are_refused(tmp_path, change):
    cfg = copy.deepcopy(MIXED)
    if change[0] == "architecture":
        cfg["architecture"] = change[1]
    elif change[0] == "type":
        cfg["layers"][1]["type"] = change[1]
    else:
        cfg["layers"][0]["mlp"]["kind"] = change[1]
    br.write_model(tmp_path, cfg, br.random_tensors(MIXED))
    with pytest.raises(BackendError):
        ck.engine_config(ck.open_model(tmp_path).model_config)


def test_truncated_safetensors_are_refused(tmp_path):
    br.write_model(tmp_path, MIXED, br.random_tensors(MIXED))
    f = tmp_path / "model.safetensors"
    whole = f.read_bytes()
    f.write_bytes(whole[:-10])
    r = ck.open_model(tmp_path)
    with pytest.raises(BackendError):
        r.get("head")
    f.write_bytes(whole[:20])
    with pytest.raises(BackendError):
        ck.open_model(tmp_path)


@pytest.mark.parametrize("dtype,want", [
    (0, dict(q_head_stride=20, q_rot_offset=14, dkv_offset=60, rot_offset=81, q_row=87, qa_head_stride=27, qa_rot_offset=21, lat_head_stride=21,
             out_head_stride=11, page_bytes=16 * 27 * 4)),
    (2, dict(q_head_stride=24, q_rot_offset=16, dkv_offset=72, rot_offset=96, q_row=104, qa_head_stride=128, qa_rot_offset=64, lat_head_stride=24,
             out_head_stride=16, page_bytes=16 * 128 * 2))])
def test_latent_layout(dtype, want):
    a = _abi.LatentAttention(dtype, 3, 14, 6, 11, 21, 8, 6, 0.25)
    assert gptrs_b200.lib().gptrs_cuda_latent_layout(ctypes.byref(a)) == 0
    assert {k: getattr(a, k) for k in want} == want
    for bad in (dict(window=-1), dict(rot_dims=5), dict(rot_dims=8), dict(scale=0.0), dict(heads=0), dict(kv_rank=2000)):
        b = _abi.LatentAttention(dtype, 3, 14, 6, 11, 21, 8, 6, 0.25)
        for k, v in bad.items():
            setattr(b, k, v)
        assert gptrs_b200.lib().gptrs_cuda_latent_layout(ctypes.byref(b)) != 0


# ---- replay ------------------------------------------------------------------------------------------------------------
class _Engine:
    """Stands in for LoadedModel: logits of a row name its token, slot and position."""

    def __init__(self, max_tokens=64, max_logit_rows=64):
        self.config = gm.ModelConfig.layered([], 8, 3, 512, 1e-5, 3, max_seqs=4, max_tokens=max_tokens, max_logit_rows=max_logit_rows)
        self.len, self.calls, self.resets = {}, [], []

    def forward_with_decode_cache(self, tok, sl, pos, rows, **kw):
        assert 0 < len(tok) <= self.config.max_tokens and len(rows) <= self.config.max_logit_rows
        for s, p in zip(sl, pos):
            assert p == self.len.get(s, 0)
            self.len[s] = p + 1
        self.calls.append(list(sl))
        lg = np.array([[tok[r], sl[r], pos[r]] for r in rows], np.float32).reshape(-1, 3)
        return (lg if len(rows) else None), None

    def reset_sequence(self, slot):
        self.len[slot] = 0
        self.resets.append(slot)


@pytest.mark.parametrize("max_tokens,max_rows", [(64, 64), (4, 64), (64, 2), (5, 1)])
def test_replay_batches_and_reuses_slots(max_tokens, max_rows):
    eng = _Engine(max_tokens, max_rows)
    r = trace.Replay(eng)
    out = r.step([{"id": "a", "tokens": [1, 2, 3, 4, 5], "want": [4, 0, 2]}, {"id": "b", "tokens": [7], "want": []}, {"id": "c", "tokens": [8, 9], "want": [1]}])
    assert [list(v) for v in out] == [[5, 0, 4], [1, 0, 0], [3, 0, 2], [9, 2, 1]]
    if max_tokens >= 8 and max_rows >= 4:
        assert len(eng.calls) == 1   # one batch
    r.end("b")
    out = r.step([{"id": "d", "tokens": [4, 4], "want": [0]}, {"id": "a", "tokens": [6], "want": [0]}])   # b's slot, from position 0; c sits out
    assert [list(v) for v in out] == [[4, 1, 0], [6, 0, 5]]
    assert r.step([{"id": "c", "tokens": [3], "want": []}]).shape == (0, 3)
    assert eng.resets == [1] and eng.len == {0: 6, 1: 2, 2: 3}


def test_trace_run_loop(tmp_path, monkeypatch):
    import io
    monkeypatch.setattr(trace, "load", lambda *a: _Engine())
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": [5, 6], "want": [1]}], "end": []},
             {"step": 3, "entries": [{"id": "x", "tokens": [7], "want": []}], "end": ["x"]}]
    out = io.StringIO()
    assert trace.run("m", "float32", tmp_path, 64, io.StringIO("\n".join(map(json.dumps, lines)) + "\n\n"), out) == 0
    assert out.getvalue() == "done 0\ndone 3\n"
    assert [p.name for p in tmp_path.iterdir()] == ["0.f32"]
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [6, 0, 1]


def test_prefill_many_packs_layered_prompts_across_boundaries():
    class Rec(gm.LoadedModel):
        def __init__(self, config):
            self.config, self._h, self.passes, self.len = config, None, [], {}

        def __del__(self):
            pass

        def sequence_length(self, slot=0):
            return self.len.get(slot, 0)

        def forward_with_decode_cache(self, tok, sl, pos, rows=(), **kw):
            self.passes.append(len(tok))
            for s in sl:
                self.len[s] = self.len.get(s, 0) + 1
            return None, np.array([tok[r] for r in rows], np.int32)

    m = Rec(gm.ModelConfig.layered([], 8, 3, 512, 1e-5, 3, max_seqs=4, max_tokens=16, max_logit_rows=4))
    assert m.prefill_many([0, 1, 2], [list(range(11)), list(range(9)), list(range(7))]) == [10, 8, 6]
    assert m.passes == [16, 11]


# ---- the oracle --------------------------------------------------------------------------------------------------------
def test_sharp_weights_show_a_wrong_window_state_or_rotation():
    """With the query projection scaled up a single key dominates most rows, so an edge that is one token off, a lost
    convolution input or a missing rotation moves the logits far beyond the tolerances of the GPU tests."""
    cfg = br.model_config([br.layer_config(window=20), br.layer_config(window=13)], softcap=4.0)
    t = br.random_tensors(cfg, 5)
    for n in t:
        if n.endswith("mix.q"):
            t[n] = br.to_bf16(t[n] * 4)
    tok = np.random.default_rng(1).integers(0, cfg["vocab"], 90)
    good = br.forward(cfg, t, tok)

    def moved(change_cfg=None, change_t=None):
        c, w = copy.deepcopy(cfg), dict(t)
        if change_cfg:
            change_cfg(c)
        if change_t:
            change_t(w)
        return float(np.sqrt(np.mean((br.forward(c, w, tok) - good) ** 2)) / np.sqrt(np.mean(good ** 2)))

    assert moved(lambda c: c["layers"][0]["mixer"]["mask"].update(size=21)) > 0.03
    assert moved(lambda c: c["layers"][1]["mixer"]["mask"].update(size=12)) > 0.03
    assert moved(lambda c: c["layers"][0]["mixer"]["rot"].update(base=1e30)) > 0.03
    assert moved(None, lambda w: w.update({"l1.canon2": np.concatenate([0 * w["l1.canon2"][:, :1], w["l1.canon2"][:, 1:]], 1)})) > 0.03
    assert moved(lambda c: c.update(logit_softcap=8.0)) > 0.03
    assert moved(None, lambda w: w.update({"l0.mlp.act": w["l0.mlp.act"][::-1]})) > 0.003


def test_oracle_is_causal_and_windowed():
    cfg = br.model_config([br.layer_config(window=5)], taps=2)
    t = br.random_tensors(cfg, 2)
    tok = np.random.default_rng(2).integers(0, cfg["vocab"], 30)
    full = br.forward(cfg, t, tok)
    assert np.allclose(br.forward(cfg, t, tok[:17]), full[:17], atol=1e-12)
    other = tok.copy()
    other[3] = (other[3] + 1) % cfg["vocab"]   # one layer: it reaches the window behind it and one more input of either convolution
    d = np.abs(br.forward(cfg, t, other) - full).max(axis=1)
    assert np.all(d[:3] == 0) and d[3] > 1e-6 and np.all(d[3 + 5 + 2:] == 0)
    assert d[3 + 5 + 1] > 0
