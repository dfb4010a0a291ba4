"""Command line: ``python -m singe_b200 generate --model DIR --prompt 1,2,3 --max-new-tokens 16``.

Prompts and results are token ids (the package holds no tokenizer).  Several ``--prompt`` run as one batch, joining rows
as they come free.
"""
from __future__ import annotations

import argparse


def _tokens(text: str) -> list:
    return [int(part) for part in text.replace(",", " ").split()]


def generate(arguments) -> None:
    from . import build
    from .decoder import CachedDecoder
    from .generation import GenerationOptions, RunningBatch
    from .models import load_decoder

    build.build()
    prompts = [_tokens(text) for text in arguments.prompt]
    capacity = arguments.capacity or max(len(prompt) for prompt in prompts) + arguments.max_new_tokens
    rows = min(arguments.sequences or len(prompts), len(prompts))
    model = load_decoder(arguments.model, rows, capacity, arguments.dtype)
    if arguments.graph:
        model.capture()
    batch = RunningBatch.create(CachedDecoder(model), GenerationOptions(arguments.max_new_tokens, arguments.stop))
    results, waiting = {}, list(prompts)
    while waiting or not batch.is_empty():
        while waiting:
            joined = batch.join(waiting[0])
            if joined is None:
                break
            results[joined] = []
            waiting.pop(0)
        for generated in batch.advance():
            results[generated.sequence].append(generated.token)
    for sequence in sorted(results):
        print(",".join(str(token) for token in results[sequence]))


def main(argv=None) -> None:
    parser = argparse.ArgumentParser(prog="singe_b200", description=__doc__.split("\n")[0])
    commands = parser.add_subparsers(dest="command", required=True)
    command = commands.add_parser("generate", help="greedy generation after token-id prompts")
    command.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    command.add_argument("--prompt", action="append", required=True, help="token ids, separated by commas or spaces")
    command.add_argument("--max-new-tokens", type=int, default=16)
    command.add_argument("--stop", type=_tokens, default=[], help="token ids that end a sequence")
    command.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    command.add_argument("--sequences", type=int, default=0, help="rows of the batch (default: one per prompt)")
    command.add_argument("--capacity", type=int, default=0, help="most tokens of a sequence (default: what the run needs)")
    command.add_argument("--no-graph", dest="graph", action="store_false", help="do not capture the decode step")
    generate(parser.parse_args(argv))


if __name__ == "__main__":
    main()
