"""Replays a trace of given token ids through the serving engine, step by step, and writes the logits that it asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line: {"step": n, "entries": [{"id": ..., "tokens": [...],
"want": [...]}], "end": [...]}.  The engine runs every entry's tokens from the pages and the state that earlier steps
left; a step in which places are wanted leaves their logits in DIR/<step>.f32 (little-endian 32-bit floats,
[wanted, vocab], in the order of the entries and of `want`), and 'done <step>' is printed after every step.  The ids in
`end` give back what they hold.
"""
from __future__ import annotations

import argparse
import itertools
import json
import os
import sys

import numpy as np

MAX_SEQUENCES = 64
MAX_STEP_TOKENS = 4096


def build_engine(model_dir: str, dtype: str, max_tokens: int, device):
    from . import registry, serving
    from .stack import PAGE_SIZE, round_up
    capacity = round_up(max(max_tokens, PAGE_SIZE), PAGE_SIZE)
    # every live sequence may leave part of its last page unused
    model = registry.load_model(model_dir, device, capacity // PAGE_SIZE + MAX_SEQUENCES, MAX_SEQUENCES, dtype)
    engine = serving.ServingEngine(model, device, max_slots=MAX_SEQUENCES, max_sequence_tokens=capacity,
                                   max_prefill_tokens=min(capacity, MAX_STEP_TOKENS), radix_pages=1,
                                   checkpoint_capacity=1, use_fp8=False)
    return model, engine


def replay(engine, vocab: int, lines, out_dir: str, answer=sys.stdout) -> None:
    numbers = {}                       # name of a live request -> the engine's request id, never used twice
    fresh = itertools.count()
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries, order = [], []
        for entry in step["entries"]:
            if entry["id"] not in numbers:
                numbers[entry["id"]] = next(fresh)
            number = numbers[entry["id"]]
            wanted = sorted(set(entry["want"]))
            order.append([wanted.index(place) for place in entry["want"]])
            entries.append((number, entry["tokens"], wanted))
        logits = engine.forced_step(entries, vocab) if entries else np.empty((0, vocab), np.float32)
        rows, base = [], 0
        for (_, _, wanted), places in zip(entries, order):
            rows += [base + place for place in places]
            base += len(wanted)
        if rows:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            np.ascontiguousarray(logits[rows], dtype="<f4").tofile(path)
        for name in step.get("end", []):
            if name in numbers:
                engine.end_forced(numbers.pop(name))
        print(f"done {step['step']}", file=answer, flush=True)


def main(arguments=None) -> int:
    parser = argparse.ArgumentParser(prog="trace_run", description="Replay given tokens and write logits.")
    parser.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    parser.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    parser.add_argument("--out", required=True, help="folder for <step>.f32")
    parser.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    options = parser.parse_args(arguments)

    import torch

    from . import registry
    device = torch.device("cuda:0")
    with torch.cuda.stream(torch.cuda.Stream(device)):      # decode steps are captured: a stream of their own
        try:
            model, engine = build_engine(options.model, options.dtype, options.max_tokens, device)
        except registry.UnsupportedType as error:
            print(error, file=sys.stderr)
            return 3
        replay(engine, model.vocab, sys.stdin, options.out)
        engine.close()
    return 0
