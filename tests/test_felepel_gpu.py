"""Felepel through the engine against the plain oracle: whole prompts, token-by-token decoding, portions of any size, mixed batches,
pages and slots that are used again, chunk edges and far keys, long decoding, reused weights, generation through the framework's own
entry points. f32 is held to 1e-4 of the logit range on sharp weights (scaled query projections), where a single wrong key moves the
logits far beyond that; bf16 to the rounding of bf16 activations, on less sharp ones with routers that leave no close call: two keys,
or two experts, that are nearly equal change places under bf16 rounding."""
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
from oracle import felepel_ref as fr

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
MODES = [gm.MODE_F32, gm.MODE_BF16]

A, DL, M = fr.attention_layer, fr.delta_layer, fr.moe


def _with_reuse(layers, *of, **kw):
    return fr.model_config(layers + [fr.again(layers, j) for j in of], **kw)


CONFIGS = {
    "small": _with_reuse([A(), DL(), A(heads=3, kv_heads=3, chunk=33, mlp=None), DL(heads=2, kv_heads=2, dim=32, vdim=16, conv=4)], 1, 0),
    # sizes that are multiples of nothing, chunks of one and of a prime, one tap, a vocabulary that needs padding, no groups to choose from
    "odd": _with_reuse([DL(heads=3, kv_heads=1, dim=5, vdim=7, conv=1, mlp=M(5, 3, 1, 1, 11)), A(heads=6, kv_heads=2, dim=7, vdim=9, chunk=1, mlp=M(9, 1, 3, 2, 13)),
                        A(heads=5, kv_heads=1, dim=3, vdim=21, chunk=47, softcap=4.0, mlp=None)], 2, width=37, vocab=61),
    # wider than one block of anything: head sizes over 64 and 128, more than 128 heads on a kv head, chunks around 64 and 128, many experts
    "wide": _with_reuse([A(heads=8, kv_heads=2, dim=136, vdim=72, chunk=65, mlp=M(40, 4, 5, 2, 136)), DL(heads=4, kv_heads=2, dim=72, vdim=136, conv=5),
                         A(heads=132, kv_heads=1, dim=8, vdim=16, chunk=130)], 0, width=104, vocab=136),
    # values too wide for the tensor-core kernel beside a layer that takes it; all experts chosen; the delta rule alone
    "tall": fr.model_config([A(heads=2, kv_heads=1, dim=16, vdim=264, chunk=24, mlp=M(4, 4, 2, 2, 24)), A(heads=2, kv_heads=2, chunk=24)], width=64),
    "delta": _with_reuse([DL(dim=24, vdim=8, mlp=None), DL(heads=2, kv_heads=1, dim=130, vdim=20)], 0, 1, width=48),
}
RANKS = {"odd": dict(decay_rank=3, gate_rank=17), "wide": dict(decay_rank=72, gate_rank=40)}


def _tensors(name, mode, seed=11):
    t = fr.random_tensors(CONFIGS[name], seed, **RANKS.get(name, {}))
    if mode == gm.MODE_BF16:
        return fr.steady_routing(CONFIGS[name], t, seed)
    return {n: fr.to_bf16(w * 3.0) if n.endswith("mix.q") else w for n, w in t.items()}


_CACHE = {}


def _oracle(name, n, mode=gm.MODE_F32, seed=0):
    """(config, tensors, tokens, logits) of one long sequence, computed once."""
    key = (name, n, mode, seed)
    if key not in _CACHE:
        t = _tensors(name, mode)
        tok = np.random.default_rng(seed).integers(0, CONFIGS[name]["vocab"], n)
        _CACHE[key] = (CONFIGS[name], t, tok, fr.forward(CONFIGS[name], t, tok))
    return _CACHE[key]


def _load(cfg, tensors, mode, pages=64, **kw):
    kw = {**dict(max_seqs=4, max_tokens=512, max_logit_rows=512, kv_pages=pages, max_pages_per_seq=pages, context_length=1024), **kw}
    c = ck.felepel_config(cfg, {n: w.shape for n, w in tensors.items()}, weight_mode=mode, **kw)
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
    _, streams = fr.forward(cfg, t, tok[:50], True)
    m = _load(cfg, t, mode)
    got = m.layer_residuals(tok[:50], [0] * 50, list(range(50)))
    for l in range(len(streams)):
        d = got[l] - streams[l]
        assert (np.abs(d).max() < 1e-4 if mode == gm.MODE_F32 else np.sqrt(np.mean(d ** 2)) < 0.04), l
    lg, _ = m.forward_with_decode_cache(tok[50:51], [0], [50], [0])   # the pass that was looked into left its cache and states behind
    _close(lg, fr.forward(cfg, t, tok[:51])[-1:], mode)


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
    want = [fr.forward(cfg, t, r) for r in reqs]
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
def test_pages_behind_the_chunks_are_given_back(cuda, mode):
    """Chunks of 20 and 33 positions: a sequence of 300 tokens lives in four pages, however long it gets; a model without attention
    holds one."""
    cfg, t, tok, want = _oracle("small", 300, mode)
    m = _load(cfg, t, mode, pages=4, max_pages_per_seq=64)
    _close(_feed(m, 0, tok, [7, 1, 1, 12, 2]), want, mode)
    m.reset_sequence(0)
    assert m.stats()["free_pages"] == 4
    with pytest.raises(BackendError, match="page pool"):
        m.forward_with_decode_cache(tok[:80], [1] * 80, list(range(80)))
    cfg, t, tok, want = _oracle("delta", 300, mode)
    m = _load(cfg, t, mode, pages=2, max_pages_per_seq=64)
    _close(_feed(m, 0, tok, [7, 1, 1, 12, 2]), want, mode)
    assert m.stats()["free_pages"] >= 0


def test_rows_must_continue_their_sequence(cuda):
    cfg, t, tok, want = _oracle("small", 300)
    m = _load(cfg, t, gm.MODE_F32)
    m.forward_with_decode_cache(tok[:5], [2] * 5, list(range(5)))
    for sl, pos in (([2], [4]), ([2], [6]), ([1], [1]), ([2, 1, 2], [5, 0, 6])):
        with pytest.raises(BackendError, match="rows of a sequence"):
            m.forward_with_decode_cache(tok[:len(sl)], sl, pos)
    lg, _ = m.forward_with_decode_cache(tok[5:6], [2], [5], [0])   # the refused calls changed nothing
    _close(lg, want[5:6], gm.MODE_F32)


def test_positions_beyond_the_table_are_refused(cuda):
    cfg = fr.model_config([A()], positions=40)
    t = fr.random_tensors(cfg, 1)
    m = _load(cfg, t, gm.MODE_F32)
    assert m.config.context_length == 40
    tok = np.arange(40) % cfg["vocab"]
    _close(m.logits(tok), fr.forward(cfg, t, tok), gm.MODE_F32)
    with pytest.raises(BackendError, match="context_length"):
        m.forward_with_decode_cache([1], [0], [40])


def test_reused_weights_are_stored_once(cuda):
    cfg, t, tok, _ = _oracle("small", 300)
    m = _load(cfg, t, gm.MODE_BF16)
    alone = _load(fr.model_config(cfg["layers"][:4]), {n: w for n, w in t.items()}, gm.MODE_BF16)
    assert m.stats()["quantised_now"] == alone.stats()["quantised_now"]


def _greedy(cfg, t, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(fr.forward(cfg, t, ids)[-1].argmax()))
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
        want = fr.forward(cfg, t, seq[:-1])[len(prompts[s]) - 1:]
        top = np.sort(want, axis=1)
        sure = top[:, -1] - top[:, -2] > 0.4 * np.sqrt(np.mean(want ** 2))
        checked += int(sure.sum())
        assert np.array_equal(np.asarray(seq[len(prompts[s]):])[sure], want.argmax(axis=1)[sure]), s
    assert checked > 100


@pytest.mark.parametrize("mode", MODES)
def test_long_decoding_through_the_generator(cuda, mode):
    """600 steps under a graph: many chunks, pages given back and taken again, a state that lives on; then the logits of the next token."""
    cfg, t, tok, _ = _oracle("small", 300, mode)
    m = _load(cfg, t, mode, pages=12, max_pages_per_seq=64, max_seqs=2)
    first = m.prefill_many([0, 1], [tok[:20], tok[20:23]])
    gen = gm.Generator(m, first)
    ids = np.stack([gen.step() for _ in range(600)])
    for s, p in ((0, tok[:20]), (1, tok[20:23])):
        seq = p.tolist() + [first[s]] + ids[:, s].tolist()
        lg, _ = m.forward_with_decode_cache([seq[-1]], [s], [len(seq) - 1], [0])
        _close(lg, fr.forward(cfg, t, seq)[-1:], mode, s)


def test_context_window_slides_like_the_other_kinds(cuda):
    cfg, t, tok, _ = _oracle("small", 300)
    m = _load(cfg, t, gm.MODE_F32, context_length=48)
    got = gm.generate_tokens(m, tok[:40].tolist(), 12)
    seq, start = tok[:40].tolist(), 0
    for i in range(12):
        if len(seq) - start > 48:
            start = len(seq) - 48
        seq.append(int(fr.forward(cfg, t, seq[start:])[-1].argmax()))
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
    """Prompts long enough for whole 128-row tiles of the experts' matmuls and for several CTAs of routing."""
    cfg = fr.model_config([DL(mlp=M(4, 2, 2, 1, 40)), A(chunk=100, mlp=M(3, 2, 1, 1, 24))], positions=700)
    t = fr.steady_routing(cfg, fr.random_tensors(cfg, 6))
    tok = np.random.default_rng(2).integers(0, cfg["vocab"], 640)
    want = fr.forward(cfg, t, tok)
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
    fr.write_model(tmp_path / "m", cfg, t)
    prompt = tok[:12].tolist()
    cli = [sys.executable, str(ROOT / "gpt.rs_b200" / "cli.py")]
    r = subprocess.run(cli + ["generate", "--checkpoint", str(tmp_path / "m"), "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "8"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(x) for x in r.stdout.split(",")] == _greedy(cfg, t, prompt, 8)
    r = subprocess.run(cli + ["generate", "--checkpoint", str(tmp_path / "m"), "--prompt-ids", "1,2", "--max-tokens", "2000"], capture_output=True, text=True, timeout=300)
    assert r.returncode != 0 and "context_length" in r.stderr
    small = fr.model_config([A(), DL()])
    small["layers"][1]["mixer"].update(decay_rank=6, gate_rank=9)
    r = subprocess.run(cli + ["export-random", "--out", str(tmp_path / "r.gptrschk"), "--kind", "felepel", "--config", json.dumps(small)], capture_output=True, text=True, timeout=300)
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
