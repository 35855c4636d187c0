"""Trace runner: given token ids are fed through a model step by step, logits at chosen places come out.  Nothing is sampled.

    bin/trace_run --model PATH --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input has one JSON object a line,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}

A step runs all its entries as one batch on the serving backend (``CudaBackend.forward_at``): portions of prompts beside single
decoded tokens, from the pages and state slots that earlier steps left.  ``want`` are the places among an entry's tokens whose
logits are written to ``DIR/<step>.f32`` (little-endian fp32 [wanted, vocab], in order); the sequences in ``end`` are closed after the
step.  After every step a line ``done <step>`` is printed.

``--max-tokens``: the most tokens that live sequences hold together, each rounded up to whole pages; the page pool is made for
that many, and the model's state slots for four sequences.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4


class TraceRunner:
    """The protocol over a backend with ``begin`` / ``forward_at`` / ``end``."""

    def __init__(self, backend, out_dir: str):
        self.backend, self.out = backend, out_dir
        self.live: dict[str, int] = {}
        self._next = 1

    def step(self, msg: dict) -> int:
        n = msg["step"]
        seqs, feeds, wants = [], [], []
        for e in msg["entries"]:
            if e["id"] not in self.live:
                self.backend.begin(self._next, None)
                self.live[e["id"]] = self._next
                self._next += 1
            seqs.append(self.live[e["id"]])
            feeds.append([int(t) for t in e["tokens"]])
            wants.append([int(w) for w in e.get("want", [])])
        if len(set(seqs)) != len(seqs) or any(not t for t in feeds):
            raise ValueError(f"step {n}: every entry needs tokens and a sequence of its own")
        if any(not 0 <= w < len(t) for t, want in zip(feeds, wants) for w in want):
            raise ValueError(f"step {n}: a wanted place is outside its entry's tokens")
        if any(not 0 <= t < self.backend.cfg.vocab for toks in feeds for t in toks):
            raise ValueError(f"step {n}: a token is outside the vocabulary")
        if seqs:
            logits = self.backend.forward_at(seqs, feeds, wants)
            if any(wants):
                tmp = os.path.join(self.out, f".{n}.part")
                with open(tmp, "wb") as f:
                    f.write(logits.numpy().astype("<f4").tobytes())
                os.replace(tmp, os.path.join(self.out, f"{n}.f32"))
        for name in msg.get("end", []):
            seq = self.live.pop(name, None)
            if seq is not None:
                self.backend.end(seq)
        return n


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="checkpoint folder (config.json, model.safetensors) or GGUF file")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live sequences hold at most")
    return ap.parse_args(argv)


def main(argv=None) -> int:
    a = parse_args(argv)
    from .. import _native
    from ..models.config import HYBRID_ARCHS
    from ..models.registry import peek_architecture
    if peek_architecture(a.model) in HYBRID_ARCHS:
        _native.use_subset("hybrid")                 # build no more than these families need
    from ..models.paged import PAGE
    from .backend import CudaBackend
    pages = max(1, (a.max_tokens + PAGE - 1) // PAGE)
    backend = CudaBackend.open(a.model, max_num_seqs=MAX_LIVE, max_ctx=pages * PAGE, max_tokens=pages * PAGE, dtype=a.dtype, n_pages=pages,
                               state_slots=MAX_LIVE)
    runner = TraceRunner(backend, a.out)
    for line in sys.stdin:
        if line.strip():
            n = runner.step(json.loads(line))
            backend.engine.check_status()
            print(f"done {n}", flush=True)
    return 0
