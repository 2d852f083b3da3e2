"""Replays a trace: given token ids go through a model portion by portion, and the logits of chosen places are written.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Every line of standard input is a step in JSON,

    {"step": 7, "entries": [{"id": "x", "tokens": [11, 4], "want": [1]}], "end": ["x"]}

entries: the next tokens of each request and the places among them whose logits are wanted; end: requests that are over
after the step. For a step that wants something DIR/<step>.f32 receives the logits, little-endian FP32 [wanted, vocab]
in the order of entries and want; after every step `done <step>` is printed. Nothing is sampled. Every request is a
session of the model (its caches and recurrent state); a finished one is reset and serves the next request.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Dict, List

import numpy as np

from . import checkpoint, runtime


class Replay:
    def __init__(self, model: runtime.Model, capacity: int):
        self.model, self.capacity = model, capacity
        self.live: Dict[str, runtime.Session] = {}
        self.idle: List[runtime.Session] = []

    def _session(self, request: str) -> runtime.Session:
        if request not in self.live:
            self.live[request] = self.idle.pop() if self.idle else self.model.new_session(self.capacity, graph=True)
        return self.live[request]

    def step(self, entries, end) -> np.ndarray:
        """Runs the entries in order; returns the wanted logits, [wanted, vocab]."""
        rows = [np.empty((0, self.model.shape.vocab_size), dtype=np.float32)]
        for entry in entries:
            want = [int(w) for w in entry.get("want", [])]
            order = sorted(set(want))
            logits = self._session(entry["id"]).extend(entry["tokens"], order)
            rows.append(logits[[order.index(w) for w in want]])
        for request in end:
            session = self.live.pop(request, None)
            if session is not None:
                session.reset()
                self.idle.append(session)
        return np.concatenate(rows)


def main(argv=None) -> int:
    parser = argparse.ArgumentParser(description="Replay a trace of token portions and write the wanted logits.")
    parser.add_argument("--model", required=True, help="checkpoint folder (config.json, safetensors)")
    parser.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    parser.add_argument("--out", required=True, help="folder for <step>.f32")
    parser.add_argument("--max-tokens", type=int, required=True, help="capacity of a request, in tokens")
    args = parser.parse_args(argv)
    config, weights = checkpoint.load_directory(args.model)
    try:
        model_type = checkpoint.model_type_of(config, args.dtype)
    except NotImplementedError as error:
        print(error, file=sys.stderr)
        return 3
    shape, tensors = checkpoint.admit(config, weights, model_type)
    capacity = min(max(args.max_tokens, 1), shape.max_position_embeddings)
    replay = Replay(runtime.Model(shape, tensors), capacity)
    out = Path(args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"], step.get("end", []))
        if len(logits):
            logits.astype("<f4").tofile(out / f"{step['step']}.f32")
        print("done", step["step"], flush=True)
    return 0
