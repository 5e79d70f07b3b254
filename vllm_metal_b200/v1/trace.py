"""Trace replay: JSON steps on standard input, logits to files.

Each input line is ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``: all entries run as one batch
through ``Engine.advance`` (the engine's own pages, state slots, runner and kernels), the logits at the wanted places go
to ``OUT/<n>.f32`` (little-endian fp32 ``[wanted, vocab]``), the requests of ``end`` give back what they hold, and
``done <n>`` is printed.  Nothing is sampled."""

from __future__ import annotations

import argparse
import json
import os
import sys

EXIT_UNSUPPORTED_DTYPE = 3
LIVE_REQUESTS = 4
TOKEN_UNIT = 64  # --max-tokens counts every request's tokens rounded up to this


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay given tokens through a model, step by step.")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", required=True, type=int,
                    help=f"most tokens live requests hold at a time, each rounded up to a multiple of {TOKEN_UNIT}")
    ap.add_argument("--max-requests", type=int, default=LIVE_REQUESTS, help="state slots (live requests)")
    args = ap.parse_args(argv)

    from ..lm.registry import family_of, read_config

    family = family_of(read_config(args.model))
    from .engine import DTYPES

    if DTYPES[args.dtype] not in family.dtypes:
        print(f"model family '{family.name}' does not run in {args.dtype}", file=sys.stderr)
        return EXIT_UNSUPPORTED_DTYPE
    from ..metal.build import ensure

    ensure(family.component)

    import torch

    from .engine import Engine, StepEntry

    torch.cuda.set_device(0)
    engine = Engine.from_folder(args.model, dtype=args.dtype, max_tokens=args.max_tokens,
                                max_num_seqs=args.max_requests)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = engine.advance([StepEntry(str(e["id"]), e["tokens"], e.get("want", ())) for e in step["entries"]])
        if logits.shape[0]:
            data = logits.float().cpu().contiguous().numpy().astype("<f4", copy=False)
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data.tobytes())
        for req_id in step.get("end", ()):
            engine.finish(str(req_id))
        print(f"done {step['step']}", flush=True)
    return 0
