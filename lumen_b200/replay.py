"""Trace replay: given token ids go through a model step by step and the logits at the places asked for are written out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

A step is one JSON line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  An entry's tokens continue the
sequence `id` from the cache its earlier steps left; `want` are places among these tokens.  The logits land in
OUT/<step>.f32 (little-endian f32, [wanted, vocab]); "done <step>" is printed after every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from pathlib import Path

import numpy as np


class TraceReplay:
    """Keeps the caches of live sequences; those of finished ones are reset and used again."""

    def __init__(self, model):
        self.model = model
        self.live: dict = {}
        self.free: list = []

    def _caches(self, rid):
        if rid not in self.live:
            self.live[rid] = self.free.pop() if self.free else self.model.init_kv_caches(1)
        return self.live[rid]

    def entry(self, rid, tokens, want) -> np.ndarray:
        """Logits [len(want), vocab] at the wanted places of this portion."""
        ids = np.asarray(tokens, dtype=np.float32)[None]
        n = ids.shape[1]
        last_only = all(w == n - 1 for w in want)  # also when nothing is wanted
        logits = self.model.forward(ids, self._caches(rid), last_only=last_only)
        rows = logits if last_only else logits[0]
        return np.ascontiguousarray(rows[[0 if last_only else w for w in want]], dtype="<f4")

    def end(self, rid) -> None:
        caches = self.live.pop(rid, None)
        if caches is not None:
            self.model.reset_kv_caches(caches)
            self.free.append(caches)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], required=True)
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live sequences hold at any time")
    args = ap.parse_args(argv)
    f32 = args.dtype == "float32"
    if f32:  # true 32-bit products in every model: none on the (bf16) tensor cores.  Read by the library at its first product.
        os.environ["LUMEN_NO_TC"] = os.environ["LUMEN_NO_TC_ATTN"] = "1"
    from .registry import load_model
    from .tensor import no_grad
    model = load_model(args.model, max(args.max_tokens, 1), "f32" if f32 else "bf16")
    replay = TraceReplay(model)
    with no_grad():
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            rows = [replay.entry(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"] if e["tokens"]]
            if any(len(r) for r in rows):
                (Path(args.out) / f"{step['step']}.f32").write_bytes(b"".join(r.tobytes() for r in rows))
            for rid in step.get("end", []):
                replay.end(rid)
            print(f"done {step['step']}", flush=True)
    return 0
