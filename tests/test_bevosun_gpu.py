"""Bevosun through the engine against the plain oracle: whole prompts, token-by-token decoding, portions of any size, mixed
batches, pages and slots that are used again, far keys and window edges, long decoding, generation through the framework's own
entry points. f32 is held to 1e-4 of the logit range on sharp weights (scaled query projections), where a single wrong key
moves the logits far beyond that; bf16 to the rounding of bf16 activations, on less sharp ones: two keys that are nearly equal
in a sharp softmax change places under bf16 rounding."""
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
from oracle import bevosun_ref as br

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
MODES = [gm.MODE_F32, gm.MODE_BF16]

L = br.layer_config
CONFIGS = {
    "small": br.model_config([L(), L(heads=3, dim=24, rot_dim=12, vdim=20, kv_rank=40, window=9, ff=None), L(heads=1, window=33, base=500.0, ff=64)]),
    # sizes that are multiples of nothing, one tap, one-token window, a vocabulary that needs padding
    "odd": br.model_config([L(heads=5, dim=7, rot_dim=6, vdim=9, kv_rank=13, window=1, ff=21), L(heads=2, dim=3, rot_dim=2, vdim=5, kv_rank=7, window=50, ff=11)],
                           width=37, vocab=61, taps=1, softcap=5.0),
    # wider than one block of anything: rank and rotated part over 64 columns, more than 128 heads, windows around 64 and 128
    "wide": br.model_config([L(heads=9, dim=32, rot_dim=72, vdim=24, kv_rank=136, window=65, ff=200), L(heads=131, dim=8, rot_dim=8, vdim=8, kv_rank=16, window=130, ff=72)],
                            width=104, vocab=136, taps=5),
    # a latent too large for the tensor-core kernel beside a layer that takes it, no soft cap
    "rank": br.model_config([L(heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=272, window=24, ff=None), L(heads=2, window=24, ff=None)], width=64, taps=2, softcap=0.0),
}


def _sharp(cfg, seed, factor=3.0):
    t = br.random_tensors(cfg, seed)
    return {n: br.to_bf16(w * factor) if n.endswith("mix.q") else w for n, w in t.items()}


_CACHE = {}


def _oracle(name, n, mode=gm.MODE_F32, seed=0):
    """(config, tensors, tokens, logits) of one long sequence, computed once."""
    key = (name, n, mode, seed)
    if key not in _CACHE:
        cfg = CONFIGS[name]
        t = _sharp(cfg, 11, 3.0 if mode == gm.MODE_F32 else 1.0)
        tok = np.random.default_rng(seed).integers(0, cfg["vocab"], n)
        _CACHE[key] = (cfg, t, tok, br.forward(cfg, t, tok))
    return _CACHE[key]


def _load(cfg, tensors, mode, pages=64, **kw):
    kw = {**dict(max_seqs=4, max_tokens=512, max_logit_rows=512, kv_pages=pages, max_pages_per_seq=pages, context_length=1024), **kw}
    c = ck.bevosun_config(cfg, weight_mode=mode, **kw)
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
        assert err.max() < 0.08 and np.mean(err) < 0.025, (what, err.max(), err.mean(), int(err.argmax()))


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
    _, streams = br.forward(cfg, t, tok[:50], True)
    got = _load(cfg, t, mode).layer_residuals(tok[:50], [0] * 50, list(range(50)))
    for l in range(len(streams)):
        d = got[l] - streams[l]
        assert (np.abs(d).max() < 1e-4 if mode == gm.MODE_F32 else np.sqrt(np.mean(d ** 2)) < 0.05), l


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", CONFIGS)
def test_prompt_portions_and_decoding(cuda, name, mode):
    cfg, t, tok, want = _oracle(name, 300, mode)
    m = _load(cfg, t, mode)
    for cuts in ([300], [1], [2], [3, 1, 16, 2], [15, 17, 64, 1, 1], [129, 1, 1, 1, 100]):
        m.reset_sequence(0)
        _close(_feed(m, 0, tok, cuts), want, mode, cuts)
    assert m.stats()["free_pages"] >= 64 - 300 // 16 - 1
    m.reset_sequence(0)
    assert m.stats()["free_pages"] == 64


@pytest.mark.parametrize("mode", MODES)
def test_mixed_batches_equal_each_request_alone(cuda, mode):
    """Four live requests of ten, portions beside single tokens, some left out for a while; a pool that only holds what is
    live, so pages and slots come around again and again."""
    rng = np.random.default_rng(5)
    cfg, t, _, _ = _oracle("small", 300, mode)
    reqs = [rng.integers(0, cfg["vocab"], n) for n in (70, 3, 41, 120, 16, 1, 65, 33, 90, 7)]
    want = [br.forward(cfg, t, r) for r in reqs]
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
    """Windows of 20, 9 and 33 positions: a sequence of 300 tokens lives in four pages, however long it gets."""
    cfg, t, tok, want = _oracle("small", 300, mode)
    m = _load(cfg, t, mode, pages=4, max_pages_per_seq=64)
    _close(_feed(m, 0, tok, [7, 1, 1, 12, 2]), want, mode)
    assert m.stats()["free_pages"] <= 2
    m.reset_sequence(0)
    assert m.stats()["free_pages"] == 4
    with pytest.raises(BackendError, match="page pool"):
        m.forward_with_decode_cache(tok[:80], [1] * 80, list(range(80)))


def test_rows_must_continue_their_sequence(cuda):
    cfg, t, tok, want = _oracle("small", 300)
    m = _load(cfg, t, gm.MODE_F32)
    m.forward_with_decode_cache(tok[:5], [2] * 5, list(range(5)))
    for sl, pos in (([2], [4]), ([2], [6]), ([1], [1]), ([2, 1, 2], [5, 0, 6])):
        with pytest.raises(BackendError, match="rows of a sequence"):
            m.forward_with_decode_cache(tok[:len(sl)], sl, pos)
    lg, _ = m.forward_with_decode_cache(tok[5:6], [2], [5], [0])   # the refused calls changed nothing
    _close(lg, want[5:6], gm.MODE_F32)


def _greedy(cfg, t, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(br.forward(cfg, t, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("name", ["small", "odd", "wide"])
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


@pytest.mark.parametrize("name", ["small", "odd", "wide", "rank"])
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
        gens[use_graph] = np.stack([gen.step() for _ in range(30)])
    ids = gens[True]
    checked = 0
    for s in range(20):
        seq = prompts[s] + [first[s]] + ids[:, s].tolist()
        want = br.forward(cfg, t, seq[:-1])[len(prompts[s]) - 1:]
        top = np.sort(want, axis=1)
        sure = top[:, -1] - top[:, -2] > 0.4 * np.sqrt(np.mean(want ** 2))
        checked += int(sure.sum())
        assert np.array_equal(np.asarray(seq[len(prompts[s]):])[sure], want.argmax(axis=1)[sure]), s
    assert checked > 100


@pytest.mark.parametrize("mode", MODES)
def test_long_decoding_through_the_generator(cuda, mode):
    """600 steps under a graph: many windows, pages given back and taken again; then the logits of the next token."""
    cfg, t, tok, _ = _oracle("small", 300, mode)
    m = _load(cfg, t, mode, pages=12, max_pages_per_seq=64, max_seqs=2)
    first = m.prefill_many([0, 1], [tok[:20], tok[20:23]])
    gen = gm.Generator(m, first)
    ids = np.stack([gen.step() for _ in range(600)])
    for s, p in ((0, tok[:20]), (1, tok[20:23])):
        seq = p.tolist() + [first[s]] + ids[:, s].tolist()
        lg, _ = m.forward_with_decode_cache([seq[-1]], [s], [len(seq) - 1], [0])
        want = br.forward(cfg, t, seq)[-1:]
        _close(lg, want, mode, s)


def test_context_window_slides_like_the_other_kinds(cuda):
    cfg, t, tok, _ = _oracle("small", 300)
    m = _load(cfg, t, gm.MODE_F32, context_length=48)
    got = gm.generate_tokens(m, tok[:40].tolist(), 12)
    seq, start = tok[:40].tolist(), 0
    for i in range(12):
        if len(seq) - start > 48:
            start = len(seq) - 48
        seq.append(int(br.forward(cfg, t, seq[start:])[-1].argmax()))
    assert got == seq[40:]


@pytest.mark.parametrize("mode", MODES)
def test_temperature_sampling_draws_from_the_capped_logits(cuda, mode):
    cfg, t, tok, want = _oracle("small", 300, mode)
    m = _load(cfg, t, mode, max_seqs=1)
    m.set_top_k(3)
    ids = set()
    for seed in range(200):
        m.reset_sequence(0)
        _, s = m.forward_with_decode_cache(tok[:9], [0] * 9, list(range(9)), [8], want_logits=False, temperature=3.0, seed=seed)
        ids.add(int(s[0]))
    assert ids <= set(np.argsort(want[8])[-4:].tolist()) and len(ids) >= 2


def test_command_line_and_trace_replay(cuda, tmp_path):
    cfg, t, tok, want = _oracle("small", 300, gm.MODE_BF16)
    br.write_model(tmp_path / "m", cfg, t)
    prompt = tok[:12].tolist()
    r = subprocess.run([sys.executable, str(ROOT / "gpt.rs_b200" / "cli.py"), "generate", "--checkpoint", str(tmp_path / "m"), "--prompt-ids",
                        ",".join(map(str, prompt)), "--max-tokens", "8"], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(x) for x in r.stdout.split(",")] == _greedy(cfg, t, prompt, 8)
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
