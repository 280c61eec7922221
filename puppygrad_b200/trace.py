"""Replays a trace of token ids through a model, step by step, and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every line of the input is one step, a JSON object {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: each
entry appends its tokens to the sequence `id` (a new name starts a new sequence), `want` lists the places among these
tokens whose logits are written, in order, to DIR/<n>.f32 ([wanted, vocab] little-endian FP32); `end` lists the sequences
that give back what they hold. After a step the line `done <n>` is printed. Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional, Sequence, TextIO

import numpy as np

from .decoder import CudaConfig, DecoderModel
from .errors import Gpt2Error
from .registry import load_model

MODES = {"bfloat16": "bf16", "float32": "fp32"}


class TraceReplay:
    """Sequences by name over one cache: a name holds a slot from its first entry until it ends."""

    def __init__(self, model: DecoderModel, max_batch: int = 1):
        self.model = model
        self.cache = model.new_kv_cache(max_batch)
        self.free: List[int] = list(range(max_batch - 1, -1, -1))
        self.slot_of: Dict[str, int] = {}

    def _slot(self, name: str) -> int:
        if name not in self.slot_of:
            if not self.free:
                raise Gpt2Error("InvalidInput", f"more than {self.cache.max_batch} sequences are live")
            self.slot_of[name] = self.free.pop()
        return self.slot_of[name]

    def step(self, entries: Sequence[dict], end: Sequence[str]) -> np.ndarray:
        slots, portions, want, base = [], [], [], 0
        for e in entries:
            if e["tokens"]:
                slots.append(self._slot(e["id"]))
                portions.append(e["tokens"])
                want += [base + int(w) for w in e.get("want", [])]
                base += len(e["tokens"])
        logits = self.model.extend(slots, portions, self.cache, want) if portions else np.empty((0, self.model.config.vocab_size), np.float32)
        for name in end:
            slot = self.slot_of.pop(name, None)
            if slot is not None:
                self.cache.clear_slot(slot)
                self.free.append(slot)
        return logits


def main(argv: Optional[Sequence[str]] = None, stdin: TextIO = sys.stdin, stdout: TextIO = sys.stdout) -> int:
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=sorted(MODES))
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens that live sequences hold at any time")
    ap.add_argument("--max-sequences", type=int, default=1, help="the most sequences that are live at any time")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    model = load_model(a.model, CudaConfig(device=a.device, math_mode=MODES[a.dtype], max_context=max(a.max_tokens, 1)))
    replay = TraceReplay(model, a.max_sequences)
    for line in stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"], step.get("end", []))
        if len(logits):
            logits.astype("<f4", copy=False).tofile(os.path.join(a.out, f"{step['step']}.f32"))
        stdout.write(f"done {step['step']}\n")
        stdout.flush()
    return 0


if __name__ == "__main__":
    sys.exit(main())
