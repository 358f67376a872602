"""Command line of the framework.

    bin/lfm25 models                                            known model families
    bin/lfm25 info --model DIR                                  what a model folder holds
    bin/lfm25 generate --model DIR --tokens 5,17,3 [--tokens ...] --max-new-tokens 16
    bin/lfm25 trace ...                                         the same as bin/trace_run

Prompts and continuations are token ids: no tokenizer is part of this repository.
"""
from __future__ import annotations

import argparse
import json


def _generate(options) -> int:
    import torch

    from . import registry, serving
    from .stack import PAGE_SIZE, round_up
    prompts = [[int(token) for token in text.split(",")] for text in options.tokens]
    longest = round_up(max(len(prompt) for prompt in prompts) + options.max_new_tokens, PAGE_SIZE)
    slots = min(len(prompts), 64)
    device = torch.device("cuda:0")
    with torch.cuda.stream(torch.cuda.Stream(device)):
        model = registry.load_model(options.model, device, (slots + 1) * longest // PAGE_SIZE + 64, slots, options.dtype)
        for prompt in prompts:
            if any(token < 0 or token >= model.vocab for token in prompt):
                raise SystemExit(f"token ids must lie in 0..{model.vocab - 1}")
        engine = serving.ServingEngine(model, device, max_slots=slots, max_sequence_tokens=longest,
                                       max_prefill_tokens=512, radix_pages=64, checkpoint_capacity=4,
                                       use_fp8=options.fp8)
        engine.calibrate()
        for tokens in serving.generate(engine, prompts, options.max_new_tokens):
            print(",".join(str(token) for token in tokens))
        engine.close()
    return 0


def _info(options) -> int:
    from . import registry
    config = registry.read_config(options.model)
    family = registry.family_of(config)
    print(json.dumps({"architecture": family.architecture, "dtypes": family.dtypes, "config": config}, indent=1))
    return 0


def main(arguments=None) -> int:
    parser = argparse.ArgumentParser(prog="lfm25", description=__doc__, formatter_class=argparse.RawTextHelpFormatter)
    commands = parser.add_subparsers(dest="command", required=True)
    commands.add_parser("models", help="known model families")
    info = commands.add_parser("info", help="what a model folder holds")
    info.add_argument("--model", required=True)
    generate = commands.add_parser("generate", help="greedy continuations through the serving engine")
    generate.add_argument("--model", required=True)
    generate.add_argument("--tokens", action="append", required=True, help="a prompt as comma-separated token ids")
    generate.add_argument("--max-new-tokens", type=int, default=16)
    generate.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    generate.add_argument("--fp8", action="store_true", help="families with an FP8 policy: use it for decode")
    commands.add_parser("trace", help="replay given tokens", add_help=False)
    options, rest = parser.parse_known_args(arguments)
    if options.command == "trace":
        from . import trace_runner
        return trace_runner.main(rest)
    if rest:
        parser.error(f"unknown arguments: {' '.join(rest)}")
    if options.command == "models":
        from . import registry
        for name, family in sorted(registry.FAMILIES.items()):
            print(f"{name}\t{', '.join(family.dtypes)}")
        return 0
    return {"info": _info, "generate": _generate}[options.command](options)
