"""Replay a trace of token ids through the engine, step by step, and write the logits of chosen places.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

A step is one JSON line: {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}], "end": ["b"]}.  All entries of a step
are one batch of `engine.step` - prompt portions beside single decoded tokens, each from the cache and state that earlier steps left.
A request gets its sequence slot at its first entry and gives pages and slot back when it is named in `end`.  `want` names places
among the entry's tokens; their logits go to OUT/<step>.f32 (little-endian fp32, [wanted, vocab]).  "done <step>" is printed after
every step.  The page pool holds N tokens (every live request rounded up to whole pages) and there are four sequence slots.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE, SLOTS = 64, 4


class TraceRunner:
    def __init__(self, engine):
        self.eng = engine
        self.sids: dict[str, int] = {}

    def step(self, entries: list[dict], end: list[str]):
        """Run one step; returns the wanted logits [n, vocab] or None when nothing is wanted."""
        for e in entries:
            if e["id"] not in self.sids:
                self.sids[e["id"]] = self.eng.alloc_seq()
        lg = None
        if entries:
            lg = self.eng.step([(self.sids[e["id"]], e["tokens"]) for e in entries], [e.get("want", []) for e in entries])
        for i in end:
            if i in self.sids:
                self.eng.free_seq(self.sids.pop(i))
        return lg if lg is not None and lg.shape[0] else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids through the engine and write logits")
    ap.add_argument("--model", required=True, help="model folder (config.json, model.safetensors)")
    ap.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"), help="storage type of weights, activations and cache")
    ap.add_argument("--out", required=True, help="folder of the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at any time, each rounded up to whole pages")
    ap.add_argument("--batch-tokens", type=int, default=2048, help="rows of one forward; a larger step runs as several")
    a = ap.parse_args(argv)
    import torch

    from ..models.modeldir import make_engine
    from ..models.weights import load_weights
    if not torch.cuda.is_available():
        print("trace_run: no CUDA device", file=sys.stderr)
        return 2
    pages = max(1, (a.max_tokens + PAGE - 1) // PAGE)
    w = load_weights(a.model, "cuda:0", dtype=a.dtype)
    eng = make_engine(w, n_ctx=pages * PAGE, max_seqs=SLOTS, page_size=PAGE, n_pages=pages, max_batch_tokens=min(a.batch_tokens, pages * PAGE))
    run = TraceRunner(eng)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        lg = run.step(s.get("entries", []), s.get("end", []))
        if lg is not None:
            path = os.path.join(a.out, f"{s['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(lg.cpu().numpy().astype("<f4", copy=False).tobytes())
            os.replace(path + ".part", path)
        print(f"done {s['step']}", flush=True)
    return 0
