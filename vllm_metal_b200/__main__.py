"""Command line: ``python -m vllm_metal_b200 generate|trace|build``."""

from __future__ import annotations

import argparse
import json
import sys


def _generate(argv: list[str]) -> int:
    ap = argparse.ArgumentParser(prog="vllm_metal_b200 generate",
                                 description="Greedy continuations of token-id prompts, continuously batched.")
    ap.add_argument("--model", required=True, help="folder with config.json (and *.safetensors)")
    ap.add_argument("--prompts", default="-", help="JSON lines, one list of token ids each; '-' = standard input")
    ap.add_argument("--max-new-tokens", type=int, default=16)
    ap.add_argument("--stop-token", type=int, default=None)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-tokens", type=int, default=65536, help="tokens the cache pool holds")
    ap.add_argument("--max-num-seqs", type=int, default=64)
    ap.add_argument("--max-batched-tokens", type=int, default=2048)
    args = ap.parse_args(argv)

    from .lm.registry import family_of, read_config
    from .metal.build import ensure

    ensure(family_of(read_config(args.model)).component)

    from .v1.engine import Engine

    with (sys.stdin if args.prompts == "-" else open(args.prompts, encoding="utf-8")) as f:
        prompts = [json.loads(line) for line in f if line.strip()]
    engine = Engine.from_folder(args.model, dtype=args.dtype, max_tokens=args.max_tokens, max_num_seqs=args.max_num_seqs,
                                max_batched_tokens=args.max_batched_tokens)
    for out in engine.generate(prompts, args.max_new_tokens, args.stop_token):
        print(json.dumps(out), flush=True)
    return 0


def main(argv: list[str] | None = None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    command = argv.pop(0) if argv else "--help"
    if command == "generate":
        return _generate(argv)
    if command == "trace":
        from .v1.trace import main as trace

        return trace(argv)
    if command == "build":
        from .metal.build import build

        print(build(force="--force" in argv))
        return 0
    print("usage: python -m vllm_metal_b200 generate|trace|build [options]", file=sys.stderr)
    return 0 if command in ("-h", "--help") else 2


if __name__ == "__main__":
    sys.exit(main())
