"""Replays a trace of token ids through a model, step by step, and writes the logits it asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

One step per input line:  {"step": 4, "entries": [{"id": "q7", "tokens": [11, 8], "want": [1]}], "end": ["q7"]}
An entry feeds a request's next tokens and names (`want`) which of them need logits; these go to DIR/<step>.f32 (float32,
[wanted, vocab], entries in order).  `end` releases requests.  `done <step>` on standard output answers each line.  All
entries of a step are one right-padded batch for Model.forward_rows, on top of what the cache and states already hold.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List

import numpy as np

DTYPES = {"bfloat16": "BF16", "float32": "F32"}


class Replay:
    """The live requests of a trace on one model.  The model is created when the first step shows how large a batch is,
    and again, between batches, when a later one needs more room."""

    def __init__(self, folder: str, dtype: int, max_tokens: int):
        from .device import Cuda
        self.folder, self.dtype, self.max_tokens = folder, dtype, max(1, max_tokens)
        self.device = Cuda(0)
        self.model = None
        self.live: List[str] = []           # request of each sequence of the batch
        self.held: Dict[str, int] = {}      # tokens fed so far

    def _make_room(self, batch: int, seq: int) -> None:
        m = self.model
        # a right-padded call needs capacity for the padding too
        need_seq = max([self.max_tokens, seq] + [n + seq for n in self.held.values()])
        if m is not None and batch <= m.max_batch and batch * seq <= m.max_tokens and need_seq <= m.max_seq:
            return
        if self.live:
            raise RuntimeError("a larger batch cannot start while requests of an earlier one are live")
        from .models import Model
        if m is not None:
            batch, need_seq = max(batch, m.max_batch), max(need_seq, m.max_seq)
            seq = max(seq, -(-m.max_tokens // batch))
            m.close()
        self.model = Model.from_pretrained(self.folder, self.dtype, self.device, batch, need_seq, batch * seq)

    def step(self, entries: List[dict], end: List[str]) -> np.ndarray:
        """Feeds one step's tokens; the wanted logits, float32 [wanted, vocab], in the entries' order."""
        tokens = {e["id"]: e["tokens"] for e in entries}
        if len(tokens) != len(entries):
            raise ValueError("a request is listed twice in one step")
        fresh = [e["id"] for e in entries if e["id"] not in self.held]
        vocab_rows = None
        if entries:
            batch = self.live + fresh
            seq = max(1, max(len(t) for t in tokens.values()))
            self._make_room(len(batch), seq)
            self.live = batch
            self.held.update({i: 0 for i in fresh})
            ids = np.zeros((len(batch), seq), dtype=np.int64)
            lens = np.zeros(len(batch), dtype=np.int32)
            for b, i in enumerate(batch):
                t = tokens.get(i, [])
                ids[b, :len(t)] = t
                lens[b] = len(t)
                self.held[i] += len(t)
            at = {i: b for b, i in enumerate(batch)}
            rows = [at[e["id"]] * seq + w for e in entries for w in e["want"]]
            full = bool((lens == seq).all())
            vocab_rows = self.model.forward_rows(ids, None if full else lens, rows)
        if end:
            gone = set(end)
            keep = [b for b, i in enumerate(self.live) if i not in gone]
            if self.model is not None and len(keep) < len(self.live):
                self.model.keep_sequences(keep)
            self.live = [self.live[b] for b in keep]
            for i in gone:
                self.held.pop(i, None)
        return np.zeros((0, 0), np.float32) if vocab_rows is None else vocab_rows.float().cpu().numpy()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="checkpoint folder: config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    from . import _lib, build
    if not build.LIB.exists():
        build.build()
    replay = Replay(a.model, getattr(_lib, DTYPES[a.dtype]), a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"], s.get("end", []))
        if logits.shape[0]:
            np.ascontiguousarray(logits, dtype="<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0
