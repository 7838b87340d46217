"""Replays a trace of token ids through a model, step by step, and writes logits (bin/trace_run).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input holds one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every step is one batched pass of the model's own step function over its slot cache: `entries` bring the next tokens of their
requests and the places whose logits are wanted, `end` lists the requests that are finished after the step and give back their
slots.  The wanted logits go to OUT/<step>.f32 (little-endian f32, [wanted, vocab]); after every step a line "done <step>" is
printed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


class Replay:
    """Requests by name over the slots of one cache; the cache grows (while nothing lives in it) with the batches it meets."""

    def __init__(self, model, max_tokens: int):
        self.model, self.max_tokens = model, max_tokens
        self.slot_of: dict[str, int] = {}
        self.slots = 0

    def _room(self, needed: int) -> None:
        if needed <= self.slots:
            return
        if self.slot_of:
            raise ValueError(f"{needed} live requests do not fit the {self.slots} slots of the running batch")
        self.model.new_cache(needed, self.max_tokens)
        self.slots = needed

    def step(self, entries: list[dict], end: list[str]) -> np.ndarray:
        fresh = [e["id"] for e in entries if e["id"] not in self.slot_of]
        self._room(len(self.slot_of) + len(fresh))
        free = sorted(set(range(self.slots)) - set(self.slot_of.values()))
        for name, slot in zip(fresh, free):
            self.slot_of[name] = slot
        logits = self.model.run([(self.slot_of[e["id"]], e["tokens"], e.get("want", [])) for e in entries])
        for name in end:
            self.model.cache.release(self.slot_of.pop(name))
        return logits


def main(argv: list[str] | None = None) -> int:
    parser = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    parser.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    parser.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    parser.add_argument("--out", required=True, help="folder for the logits")
    parser.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = parser.parse_args(argv)

    import ctorch_b200 as B
    replay = Replay(B.LanguageModel.load(args.model, dtype=args.dtype), max(1, args.max_tokens))
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"], step.get("end", []))
        if logits.shape[0]:
            logits.astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
