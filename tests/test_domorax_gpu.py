"""Domorax through the engine against the plain oracle: whole prompts, token-by-token decoding, portions of any size, mixed batches,
pages and slots that are used again, window edges and far keys, long decoding, many layers to average over, generation through the
framework's own entry points. f32 is held to 1e-4 of the logit range on sharp weights (scaled queries), where a single wrong key moves the
logits far beyond that; bf16 to the rounding of bf16 activations, on less sharp ones with routers that leave no close call: two keys, or two
experts, that are nearly equal change places under bf16 rounding."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

from gptrs_b200 import BackendError
from gptrs_b200 import checkpoint as ck
from gptrs_b200 import model as gm
from gptrs_b200 import parallel
from oracle import domorax_ref as dr

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
MODES = [gm.MODE_F32, gm.MODE_BF16]

L, A, DL, M, F = dr.latent_layer, dr.attention_layer, dr.delta_layer, dr.moe, dr.dense_mlp

CONFIGS = {
    "small": dr.model_config([L(), A(mlp=M()), DL(mlp=M(experts=8, top=3, shared=0)), L(heads=2, window=33, mlp=None), A(heads=3, kv_heads=1, conv=2, mlp=None)]),
    # sizes that are multiples of nothing, windows of one and of a prime, convolutions of one and of many taps, a vocabulary that needs
    # padding, groups of 13 channels, one expert of one, all experts at once
    "odd": dr.model_config([A(heads=3, kv_heads=1, dim=5, conv=1, mlp=M(5, 5, 11, shared=3)), L(heads=3, dim=7, rot_dim=2, vdim=9, kv_rank=11, q_rank=3, window=1, mlp=F(19)),
                            DL(heads=3, kv_heads=3, dim=7, vdim=5, conv=2, mlp=M(1, 1, 13, shared=0)), DL(heads=4, kv_heads=2, dim=5, vdim=13, conv=1, mlp=None),
                            A(heads=6, kv_heads=6, dim=7, conv=7, mlp=F(21)), L(heads=5, dim=3, rot_dim=6, vdim=21, window=47, scaling=None)], width=39, vocab=61, groups=3),
    # wider than one block of anything: heads over 64 and over 128, more than 64 heads on a kv head, windows around 64 and 128, many experts,
    # a latent of three blocks; groups of 128 channels
    "wide": dr.model_config([L(heads=20, dim=24, rot_dim=72, vdim=40, kv_rank=136, q_rank=72, window=65, scaling=(8.0, 100, 16.0, 0.5)), A(heads=8, kv_heads=2, dim=72, conv=4, mlp=M(40, 4, 136, shared=72)),
                             A(heads=70, kv_heads=1, dim=8, mlp=None), DL(heads=4, kv_heads=2, dim=72, vdim=136, mlp=M(4, 4, 24)), A(heads=4, kv_heads=2, dim=136, conv=3, mlp=F(136)),
                             L(heads=70, window=130, mlp=None)], width=256, vocab=136),
    # heads and latents too wide for the tensor-core kernels beside layers that take them; one group
    "tall": dr.model_config([A(heads=2, kv_heads=1, dim=264, mlp=M(4, 2, 24)), L(heads=2, kv_rank=264, q_rank=40, window=24), DL(heads=2, kv_heads=1, dim=264, vdim=24, mlp=None), A()], width=64, groups=1),
    # windows only: pages go back; more results to average than are read at once
    "windows": dr.model_config([L(window=20), L(window=33, mlp=None), L(window=7, heads=2), DL(mlp=None), L(window=16, mlp=None), L(window=17), DL(mlp=None)], width=48, groups=4, mult=0.3, eps=1e-3),
}


def _tensors(name, mode, seed=11):
    if mode == gm.MODE_BF16:
        return dr.steady_routing(CONFIGS[name], dr.random_tensors(CONFIGS[name], seed), seed)
    return dr.random_tensors(CONFIGS[name], seed, sharp=3.0)


_CACHE = {}


def _oracle(name, n, mode=gm.MODE_F32, seed=0):
    """(config, tensors, tokens, logits) of one long sequence, computed once."""
    key = (name, n, mode, seed)
    if key not in _CACHE:
        t = _tensors(name, mode)
        tok = np.random.default_rng(seed).integers(0, CONFIGS[name]["vocab"], n)
        _CACHE[key] = (CONFIGS[name], t, tok, dr.forward(CONFIGS[name], t, tok))
    return _CACHE[key]


def _load(cfg, tensors, mode, pages=64, **kw):
    kw = {**dict(max_seqs=4, max_tokens=512, max_logit_rows=512, kv_pages=pages, max_pages_per_seq=pages, context_length=1024), **kw}
    c = ck.domorax_config(cfg, weight_mode=mode, **kw)
    m = gm.LoadedModel(c, namespace=ck.next_namespace())
    for name in c.param_shapes():
        m.load_param(name, tensors[name])
    m.finalize()
    return m


def _close(got, want, mode, what=""):
    scale = np.sqrt(np.mean(want ** 2))
    if mode == gm.MODE_F32:
        assert np.abs(got - want).max() < 1e-4 * max(1.0, np.abs(want).max()), what
    else:   # root mean square over the vocabulary, every position by itself
        err = np.sqrt(np.mean((got - want) ** 2, axis=-1)) / scale
        assert err.max() < 0.08 and np.mean(err) < 0.02, (what, err.max(), err.mean(), int(err.argmax()))


def _same(got, want, mode, what=""):
    """The same positions computed along two ways."""
    if mode == gm.MODE_F32:
        assert np.abs(got - want).max() < 1e-4 * max(1.0, np.abs(want).max()), what
    else:
        err = np.sqrt(np.mean((got - want) ** 2, axis=-1)) / np.sqrt(np.mean(want ** 2))
        assert err.max() < 0.06 and np.mean(err) < 0.015, (what, err.max(), err.mean())


def _feed(m, slot, tok, cuts):
    """A sequence in portions of the given sizes (cycled); logits of every position."""
    out, at, i = [], m.sequence_length(slot), 0
    while at < len(tok):
        n = min(cuts[i % len(cuts)], len(tok) - at)
        lg, _ = m.forward_with_decode_cache(tok[at:at + n], [slot] * n, list(range(at, at + n)), list(range(n)))
        out.append(lg)
        at += n
        i += 1
    return np.concatenate(out)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", CONFIGS)
def test_residual_after_every_layer(cuda, name, mode):
    cfg, t, tok, _ = _oracle(name, 300, mode)
    _, sums = dr.forward(cfg, t, tok[:50], True)
    m = _load(cfg, t, mode)
    got = m.layer_residuals(tok[:50], [0] * 50, list(range(50)))
    for l in range(len(sums)):
        d, scale = got[l] - sums[l], np.sqrt(np.mean(sums[l] ** 2))
        assert (np.abs(d).max() < 5e-5 * max(1.0, np.abs(sums[l]).max()) if mode == gm.MODE_F32 else np.sqrt(np.mean(d ** 2)) < 0.02 * scale), l
    lg, _ = m.forward_with_decode_cache(tok[50:51], [0], [50], [0])   # the pass that was looked into left its cache behind
    _close(lg, dr.forward(cfg, t, tok[:51])[-1:], mode)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_portions_and_decoding(cuda, name, mode):
    cfg, t, tok, want = _oracle(name, 300, mode)
    m = _load(cfg, t, mode)
    whole = None
    for cuts in ([300], [1], [2], [3, 1, 16, 2], [15, 17, 64, 1, 1], [129, 1, 1, 1, 100]):
        m.reset_sequence(0)
        got = _feed(m, 0, tok, cuts)
        _close(got, want, mode, cuts)
        whole = got if whole is None else whole
        _same(got, whole, mode, cuts)
    assert m.stats()["free_pages"] >= 64 - 300 // 16 - 1
    m.reset_sequence(0)
    assert m.stats()["free_pages"] == 64


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", ["small", "odd"])
def test_mixed_batches_equal_each_request_alone(cuda, name, mode):
    """Four live requests of ten, portions beside single tokens, some left out for a while; a pool that only holds what is live, so
    pages and slots come around again and again."""
    rng = np.random.default_rng(5)
    cfg, t, _, _ = _oracle(name, 300, mode)
    reqs = [rng.integers(0, cfg["vocab"], n) for n in (70, 3, 41, 120, 16, 1, 65, 33, 90, 7)]
    want = [dr.forward(cfg, t, r) for r in reqs]
    m = _load(cfg, t, mode, pages=24, max_tokens=256)
    live, free, todo, done = {}, [0, 1, 2, 3], list(range(len(reqs))), 0
    got = [[] for _ in reqs]
    while done < len(reqs):
        while free and todo:
            live[todo.pop(0)] = free.pop(rng.integers(len(free)))
        tok, sl, pos, owner = [], [], [], []
        for r, s in rng.permutation(list(live.items())):
            if rng.random() < 0.25 and len(live) > 1:
                continue
            at = sum(len(g) for g in got[r])
            n = min(len(reqs[r]) - at, 1 if rng.random() < 0.4 else int(rng.integers(2, 40)))
            tok.extend(reqs[r][at:at + n]), sl.extend([s] * n), pos.extend(range(at, at + n)), owner.extend([r] * n)
        if not tok:
            continue
        lg, _ = m.forward_with_decode_cache(tok, sl, pos, list(range(len(tok))))
        for r in dict.fromkeys(owner):
            got[r].append(lg[[i for i, o in enumerate(owner) if o == r]])
            if sum(len(g) for g in got[r]) == len(reqs[r]):
                m.reset_sequence(live[r])
                free.append(live.pop(r))
                done += 1
    for r in range(len(reqs)):
        _close(np.concatenate(got[r]), want[r], mode, r)
    assert m.stats()["free_pages"] == 24


@pytest.mark.parametrize("mode", MODES)
def test_pages_behind_the_windows_are_given_back(cuda, mode):
    """The widest window is 33 positions: a sequence of 300 tokens lives in four pages. With a layer that sees everything no page is given
    back."""
    cfg, t, tok, want = _oracle("windows", 300, mode)
    m = _load(cfg, t, mode, pages=4, max_pages_per_seq=64)
    _close(_feed(m, 0, tok, [7, 1, 1, 12, 2]), want, mode)
    m.reset_sequence(0)
    assert m.stats()["free_pages"] == 4
    with pytest.raises(BackendError, match="page pool"):
        m.forward_with_decode_cache(tok[:80], [1] * 80, list(range(80)))
    cfg, t, tok, want = _oracle("small", 300, mode)
    m = _load(cfg, t, mode, pages=19, max_pages_per_seq=64)
    _close(_feed(m, 0, tok, [100, 1, 12, 2]), want, mode)
    assert m.stats()["free_pages"] == 0


@pytest.mark.parametrize("mode", MODES)
def test_without_optional_parts(cuda, mode):
    """No window, no scaling of the rotation, no feed-forwards: a delta rule alone, and latent attention over everything."""
    for layers in ([DL(mlp=None)], [L(window=None, scaling=None, mlp=None)], [A(mlp=None)]):
        cfg = dr.model_config(layers, groups=1, mult=1.0)
        t = dr.random_tensors(cfg, 9, sharp=3.0 if mode == gm.MODE_F32 else 1.0)
        tok = np.arange(90) % cfg["vocab"]
        _close(_feed(_load(cfg, t, mode), 0, tok, [25, 1, 3, 2]), dr.forward(cfg, t, tok), mode)


def test_a_copied_token_far_back_is_found(cuda):
    """Queries that carry their token's code and keys, by their convolution, that of the token before: the last position attends to what came
    behind its own token hundreds of positions before, past every block border, in a prompt, in portions and when it is decoded alone."""
    cfg = dr.model_config([A(heads=8, kv_heads=2, dim=32, conv=2, scale=0.5, mlp=None)], width=64, vocab=300, groups=1, mult=1.0)
    rng = np.random.default_rng(4)
    t = {n: w.copy() for n, w in dr.random_tensors(cfg, 4).items()}
    code = dr.to_bf16((rng.standard_normal((32, 64)) / 8).astype(np.float32))   # keys and queries of all heads are the same projection
    t["l0.mix.k"], t["l0.mix.q"] = np.concatenate([code] * 2), np.concatenate([code] * 8)
    for n in ("q", "k"):
        t[f"l0.mix.{n}.conv"] = np.tile(np.array([0, 1] if n == "q" else [1, 0], np.float32), (t[f"l0.mix.{n}"].shape[0], 1))
        t[f"l0.mix.{n}.norm"] = np.full(32, 2.0, np.float32)
    tok = rng.permutation(np.arange(1, 300))[:280]
    for far in (0, 15, 16, 47, 63, 64, 200):
        ids = tok.copy()
        ids[-1] = tok[far]
        want, other = dr.forward(cfg, t, ids)[-1], dr.forward(cfg, t, np.concatenate([ids[:far], [0], ids[far + 1:]]))[-1]
        assert np.sqrt(np.mean((want - other) ** 2)) > 0.2 * np.sqrt(np.mean(want ** 2)), far   # the far token matters
        for mode in MODES:
            for cuts in ([280], [279, 1], [100, 2, 61, 1, 116]):
                m = _load(cfg, t, mode)
                _close(_feed(m, 0, ids, cuts)[-1:], want[None], mode, (far, cuts))


def _greedy(cfg, t, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(dr.forward(cfg, t, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("name", ["small", "odd"])
def test_greedy_generation_f32(cuda, name):
    """prefill + Generator, with and without a graph, with programmatic launches, and for a batch of unequal prompts."""
    cfg, t, tok, _ = _oracle(name, 300)
    prompts = [tok[:37].tolist(), tok[40:41].tolist(), tok[50:64].tolist()]
    want = [_greedy(cfg, t, p, 24) for p in prompts]
    m = _load(cfg, t, gm.MODE_F32, use_pdl=1)
    for use_graph in (False, True):
        assert gm.generate_tokens(m, prompts[0], 24, use_graph=use_graph) == want[0]
        out = parallel.run_requests(m, dict(enumerate(prompts)), 23, max_batch=3, prefill_chunk=16)
        assert [out[i] for i in range(3)] == want
    out = parallel.run_requests(m, dict(enumerate(prompts)), 23, max_batch=2)   # waves: slots are used again
    assert [out[i] for i in range(3)] == want


@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation_bf16(cuda, name):
    """Generated ids equal the argmax of the logits that the same tokens give as a prompt, wherever that is decided."""
    cfg, t, tok, _ = _oracle(name, 300, gm.MODE_BF16)
    m = _load(cfg, t, gm.MODE_BF16, use_pdl=1, max_seqs=20, pages=20 * 8)
    rng = np.random.default_rng(8)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in rng.integers(1, 60, 20)]
    first = m.prefill_many(list(range(20)), prompts)
    gens = {}
    for use_graph in (True, False):
        if not use_graph:
            for s in range(20):
                m.reset_sequence(s)
            m.prefill_many(list(range(20)), prompts, chunk=33)
        gen = gm.Generator(m, first, use_graph=use_graph)
        gens[use_graph] = np.stack([gen.step() for _ in range(20)])
    ids = gens[True]
    checked = 0
    for s in range(20):
        seq = prompts[s] + [first[s]] + ids[:, s].tolist()
        want = dr.forward(cfg, t, seq[:-1])[len(prompts[s]) - 1:]
        top = np.sort(want, axis=1)
        sure = top[:, -1] - top[:, -2] > 0.4 * np.sqrt(np.mean(want ** 2))
        checked += int(sure.sum())
        assert np.array_equal(np.asarray(seq[len(prompts[s]):])[sure], want.argmax(axis=1)[sure]), s
    assert checked > 80


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", ["small", "windows"])
def test_long_decoding_through_the_generator(cuda, name, mode):
    """600 steps under graphs: the context grows through several of them (or pages are given back and taken again); then the logits of the
    next token."""
    cfg, t, tok, _ = _oracle(name, 300, mode)
    m = _load(cfg, t, mode, pages=12 if name == "windows" else 80, max_pages_per_seq=64, max_seqs=2)
    first = m.prefill_many([0, 1], [tok[:20], tok[20:23]])
    gen = gm.Generator(m, first)
    ids = np.stack([gen.step() for _ in range(600)])
    for s, p in ((0, tok[:20]), (1, tok[20:23])):
        seq = p.tolist() + [first[s]] + ids[:, s].tolist()
        lg, _ = m.forward_with_decode_cache([seq[-1]], [s], [len(seq) - 1], [0])
        _close(lg, dr.forward(cfg, t, seq)[-1:], mode, s)


def test_context_window_slides_like_the_other_kinds(cuda):
    cfg, t, tok, _ = _oracle("small", 300)
    m = _load(cfg, t, gm.MODE_F32, context_length=48)
    got = gm.generate_tokens(m, tok[:40].tolist(), 12)
    seq, start = tok[:40].tolist(), 0
    for i in range(12):
        if len(seq) - start > 48:
            start = len(seq) - 48
        seq.append(int(dr.forward(cfg, t, seq[start:])[-1].argmax()))
    assert got == seq[40:]


@pytest.mark.parametrize("mode", MODES)
def test_temperature_sampling_draws_from_the_logits(cuda, mode):
    cfg, t, tok, want = _oracle("small", 300, mode)
    m = _load(cfg, t, mode, max_seqs=1)
    m.set_top_k(3)
    ids = set()
    for seed in range(200):
        m.reset_sequence(0)
        _, s = m.forward_with_decode_cache(tok[:9], [0] * 9, list(range(9)), [8], want_logits=False, temperature=3.0, seed=seed)
        ids.add(int(s[0]))
    assert ids <= set(np.argsort(want[8])[-5:].tolist()) and len(ids) >= 2


def test_many_rows_take_the_large_tiles(cuda):
    """Prompts long enough for whole 128-row tiles of all matmuls and for several CTAs of routing; far keys hundreds of positions back."""
    cfg = dr.model_config([L(window=100, mlp=M(4, 2, 40)), A(heads=8, dim=24, mlp=F(72)), DL(mlp=M(3, 2, 24, shared=0)), L(window=300, mlp=None)])
    t = dr.steady_routing(cfg, dr.random_tensors(cfg, 6))
    tok = np.random.default_rng(2).integers(0, cfg["vocab"], 640)
    want = dr.forward(cfg, t, tok)
    for mode in MODES:
        m = _load(cfg, t, mode, max_tokens=1300, max_logit_rows=700, pages=128)
        for s in (0, 1):
            n = len(tok)
            lg, _ = m.forward_with_decode_cache(tok, [s] * n, list(range(n)), list(range(n)))
            _close(lg, want, mode, s)
        m.reset_sequence(0), m.reset_sequence(1)
        first = m.prefill_many([0, 1], [tok, tok[:639]])   # both in one pass
        sure = np.sort(want[-1])[-1] - np.sort(want[-1])[-2] > 0.4 * np.sqrt(np.mean(want ** 2))
        assert not sure or first[0] == int(want[-1].argmax())


def test_command_line_and_trace_replay(cuda, tmp_path):
    cfg, t, tok, want = _oracle("small", 300, gm.MODE_BF16)
    dr.write_model(tmp_path / "m", cfg, t)
    prompt = tok[:12].tolist()
    cli = [sys.executable, str(ROOT / "gpt.rs_b200" / "cli.py")]
    r = subprocess.run(cli + ["generate", "--checkpoint", str(tmp_path / "m"), "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "8"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(x) for x in r.stdout.split(",")] == _greedy(cfg, t, prompt, 8)
    r = subprocess.run(cli + ["export-random", "--out", str(tmp_path / "r.gptrschk"), "--kind", "domorax", "--config", json.dumps(cfg)], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    r = subprocess.run(cli + ["generate", "--checkpoint", str(tmp_path / "r.gptrschk"), "--prompt-ids", "1,2", "--max-tokens", "3", "--weight-mode", "bf16"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and len(r.stdout.split(",")) == 3, r.stderr[-2000:]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tok[:30].tolist(), "want": [29, 3]}, {"id": "b", "tokens": tok[:2].tolist(), "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tok[2:3].tolist(), "want": [0]}, {"id": "a", "tokens": tok[30:47].tolist(), "want": [16]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "c", "tokens": tok[:64].tolist(), "want": [63]}], "end": ["c", "b"]}]
    rows = [[29, 3], [2, 46], [63]]
    for dtype, mode in (("float32", gm.MODE_F32), ("bfloat16", gm.MODE_BF16)):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                           input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
        for i, w in enumerate(rows):
            _close(np.fromfile(out / f"{i}.f32", "<f4").reshape(len(w), -1), want[w], mode, i)
