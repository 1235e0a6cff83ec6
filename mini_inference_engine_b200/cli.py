"""Command line: ``python -m mini_inference_engine_b200 <command>``.

    models                                          registered model designs
    generate --model DIR --prompt 1,2,3 ...         greedy continuation of token-id prompts, continuously batched
    trace --model DIR --dtype T --out DIR ...       replay given tokens step by step and write logits

There is no tokenizer here: prompts and results are token ids.
"""

from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

EXIT_UNSUPPORTED_DTYPE = 3


def _parser() -> argparse.ArgumentParser:
    parser = argparse.ArgumentParser(prog="mini_inference_engine_b200", description=__doc__.split("\n\n")[0])
    commands = parser.add_subparsers(dest="command", required=True)

    commands.add_parser("models", help="list the registered model designs")

    generate = commands.add_parser("generate", help="greedy generation through the continuous batcher")
    generate.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    generate.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    generate.add_argument("--prompt", action="append", default=[], help="comma-separated token ids; may be repeated")
    generate.add_argument("--prompts-file", help="a JSON list of token ids per line")
    generate.add_argument("--max-new-tokens", type=int, default=16)
    generate.add_argument("--max-batch", type=int, default=8)
    generate.add_argument("--max-prefill-tokens", type=int, default=512)
    generate.add_argument("--mixed", action="store_true", help="prompt chunks ride along with decode rows")
    generate.add_argument("--prefix-cache", action="store_true", help="requests share the pages of equal prefixes")
    generate.add_argument("--random-weights", type=int, metavar="SEED",
                          help="seeded random weights of the folder's configuration instead of its checkpoint")

    trace = commands.add_parser("trace", help="replay steps read from standard input and write their logits")
    trace.add_argument("--model", required=True)
    trace.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    trace.add_argument("--out", required=True, help="folder for <step>.f32 files")
    trace.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time")
    return parser


def run_generate(args: argparse.Namespace) -> int:
    from .engine.model_runner.continuous import ContinuousBatcher
    from .engine.registry import DTYPES, load_runner

    prompts = [[int(t) for t in text.split(",")] for text in args.prompt]
    if args.prompts_file:
        prompts += [json.loads(line) for line in Path(args.prompts_file).read_text().splitlines() if line.strip()]
    if not prompts:
        print("no prompts given", file=sys.stderr)
        return 2
    longest = max(len(p) for p in prompts) + args.max_new_tokens
    page = 16
    pages = args.max_batch * (-(-longest // page) + 1)
    runner = load_runner(args.model, dtype=DTYPES[args.dtype], random_seed=args.random_weights, num_pages=pages,
                         max_batch=args.max_batch, max_context=max(longest, 1024),
                         state_slots=args.max_batch * (2 if args.prefix_cache else 1))
    batcher = ContinuousBatcher(runner, max_prefill_tokens=args.max_prefill_tokens, mixed=args.mixed,
                                prefix_cache=args.prefix_cache)
    for index, prompt in enumerate(prompts):
        batcher.submit(index, prompt, args.max_new_tokens)
    results = batcher.run()
    for index in range(len(prompts)):
        print(json.dumps({"id": index, "tokens": results[index]}), flush=True)
    runner.release_graphs()
    return 0


def run_trace(args: argparse.Namespace) -> int:
    """Steps come as JSON lines ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``; a step in
    which something is wanted writes ``<out>/<n>.f32`` (little-endian fp32 ``[wanted, vocab]``), and every step
    prints ``done <n>``."""

    from .engine.model_runner.replay import TraceEntry, TraceSession
    from .engine.registry import DTYPES, load_runner

    page = 16
    pages = -(-max(args.max_tokens, 1) // page) + 256  # every live request may leave one page partly filled
    runner = load_runner(args.model, dtype=DTYPES[args.dtype], num_pages=pages, max_batch=8,
                         max_context=args.max_tokens + page, state_slots=256)
    session = TraceSession(runner)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = session.step([TraceEntry(e["id"], [int(t) for t in e["tokens"]], [int(w) for w in e.get("want", [])])
                               for e in step.get("entries", [])])
        session.end(step.get("end", []))
        if logits is not None:
            (Path(args.out) / f"{step['step']}.f32").write_bytes(logits.numpy().astype("<f4").tobytes())
        print(f"done {step['step']}", flush=True)
    return 0


def main(argv: list[str] | None = None) -> int:
    args = _parser().parse_args(argv)
    from . import build

    if args.command == "models":
        from .engine.registry import DESIGNS

        for name, design in DESIGNS.items():
            print(name, " ".join(str(d).removeprefix("torch.") for d in design.dtypes))
        return 0
    build.build_library()  # compiles what is missing or stale, otherwise returns at once
    from .engine.registry import UnsupportedDtype

    try:
        return run_generate(args) if args.command == "generate" else run_trace(args)
    except UnsupportedDtype as error:
        print(error, file=sys.stderr)
        return EXIT_UNSUPPORTED_DTYPE


if __name__ == "__main__":
    sys.exit(main())
