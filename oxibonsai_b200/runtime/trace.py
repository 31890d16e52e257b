"""Replays a trace of given tokens through an engine, step by step, and writes logits.

A step is one JSON object: ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}``.
Its entries are one batch (:meth:`LayeredEngine.feed`): portions of prompts beside single tokens, from the cache and state that
earlier steps left.  Nothing is sampled.  A request gets a slot, and pages as it grows, from its first entry to the step that
names it in ``end``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Iterable, TextIO

import numpy as np


@dataclass
class _Live:
    slot: int
    length: int = 0


class TraceSession:
    """Requests of a trace by their ids, over the slots of one engine."""

    def __init__(self, engine):
        self.engine = engine
        self.live: dict[str, _Live] = {}
        self._free = list(range(engine.max_batch))

    def step(self, entries: list[dict], end: Iterable[str] = ()) -> np.ndarray:
        """Runs one step; returns the wanted logits, f32 [wanted, vocab]."""
        eng, batch, want = self.engine, [], []
        for e in entries:
            toks = e["tokens"]
            if not toks:
                continue
            r = self.live.get(e["id"])
            if r is None:
                if not self._free:
                    raise RuntimeError(f"request {e['id']!r}: all {eng.max_batch} slots are in use")
                r = self.live[e["id"]] = _Live(self._free.pop(0))
            eng.reserve(r.slot, r.length + len(toks))
            batch.append((r.slot, toks, r.length))
            want.append(e.get("want", []))
            r.length += len(toks)
        out = eng.feed(batch, want).cpu().numpy() if batch else np.zeros((0, eng.config.vocab), dtype=np.float32)
        for i in end:
            r = self.live.pop(i)
            eng.close_sequence(r.slot)
            self._free.insert(0, r.slot)
        return out


def replay(engine, steps: Iterable[str], out_dir: str, answer: TextIO) -> int:
    """Replays the steps (JSON lines), writes ``out_dir/<step>.f32`` for steps in which something is wanted and prints
    ``done <step>`` after every step.  Returns the number of steps."""
    session, n = TraceSession(engine), 0
    for line in steps:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = session.step(s["entries"], s.get("end", ()))
        if len(logits):
            logits.astype("<f4").tofile(os.path.join(out_dir, f"{s['step']}.f32"))
        print(f"done {s['step']}", file=answer, flush=True)
        n += 1
    return n
