"""Trace replay: given token ids go through a model step by step, through the same forward pass, page pool and state slots that
generation uses, and the logits of the wanted places are written out. Nothing is sampled.

Steps come as one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
All entries of a step form one batch (prompt portions beside single decoded tokens). A request takes a slot with its first
entry and gives it and its pages back after the step that lists it in "end". A step with wanted places leaves <step>.f32 in
the output folder; after every step "done <step>" is printed.
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np

from . import checkpoint as ck
from . import model as gm

SLOTS = 4
PAGE = 16


class Replay:
    """Requests by name on the slots of one engine."""

    def __init__(self, model: gm.LoadedModel):
        self.model = model
        self.free = list(range(model.config.max_seqs - 1, -1, -1))
        self.slot: dict[str, int] = {}
        self.length: dict[str, int] = {}

    def step(self, entries) -> np.ndarray:
        """Runs one batch; returns the wanted logits in the order of the entries and of their "want" lists."""
        cfg = self.model.config
        tok, sl, pos, order = [], [], [], []   # order: (row of the batch) of every wanted place
        for e in entries:
            name = e["id"]
            if name not in self.slot:
                self.slot[name] = self.free.pop()
                self.length[name] = 0
            start, first = self.length[name], len(tok)
            tok.extend(e["tokens"])
            sl.extend([self.slot[name]] * len(e["tokens"]))
            pos.extend(range(start, start + len(e["tokens"])))
            self.length[name] = start + len(e["tokens"])
            order.extend(first + w for w in e.get("want", []))
        wanted = sorted(set(order))
        rows = {}
        limit = cfg.max_logit_rows or cfg.max_seqs
        at = k = 0
        while at < len(tok):   # one forward pass unless the step exceeds what the engine was sized for
            end = min(len(tok), at + cfg.max_tokens)
            take = [w for w in wanted[k:k + limit] if w < end]
            if len(take) == limit and k + limit < len(wanted):
                end = min(end, wanted[k + limit])
            lg, _ = self.model.forward_with_decode_cache(tok[at:end], sl[at:end], pos[at:end], [w - at for w in take])
            for i, w in enumerate(take):
                rows[w] = lg[i]
            k += len(take)
            at = end
        return np.stack([rows[w] for w in order]) if order else np.empty((0, cfg.vocab), np.float32)

    def end(self, name: str):
        slot = self.slot.pop(name)
        del self.length[name]
        self.model.reset_sequence(slot)
        self.free.append(slot)


def load(model_dir, dtype: str, max_tokens: int) -> gm.LoadedModel:
    mode = gm.MODE_BF16 if dtype == "bfloat16" else gm.MODE_F32
    pool = (max_tokens + 63) // 64 * 64
    reader = ck.open_model(model_dir)
    kw = dict(context_length=pool) if reader.kind in ck.LAYERED_KINDS else {}   # the other kinds name theirs
    vocab = ck.engine_config(reader.model_config, mode, ck.shapes_of(reader), **kw)[0].vocab
    logit_rows = max(1, min(pool, 2 ** 26 // vocab))
    return ck.load_model(model_dir, weight_mode=mode, max_seqs=SLOTS, max_tokens=min(pool, 8192), max_logit_rows=logit_rows, kv_pages=pool // PAGE,
                         max_pages_per_seq=pool // PAGE, **kw)


def run(model_dir, dtype: str, out_dir, max_tokens: int, lines, answer) -> int:
    replay = Replay(load(model_dir, dtype, max_tokens))
    for line in lines:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"])
        if len(logits):
            logits.astype("<f4").tofile(Path(out_dir) / f"{s['step']}.f32")
        for name in s.get("end", []):
            replay.end(name)
        answer.write(f"done {s['step']}\n")
        answer.flush()
    return 0
