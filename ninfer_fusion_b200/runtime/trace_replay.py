"""Token-trace replay: feeds given token ids through a model step by step and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps are read from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step are one batch of the engine's ragged step (`GpuProgram.step`): portions of prompts beside single
tokens, on lanes that are opened at a request's first entry and given back by "end".  A step with wanted places writes
`<step>.f32` to --out (little-endian fp32, [wanted, vocab], order of the entries and their places); after every step
"done <step>" is printed.  --max-tokens sizes the page pool: the most tokens that live requests hold at any time.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Iterable, TextIO

import torch

MAX_LIVE = 4
PAGE = 64


def open_program(model_dir: str, dtype: torch.dtype, max_tokens: int, device="cuda:0"):
    """The engine's program for a model folder, with a pool of `max_tokens` cache positions and slots for four lanes."""
    from ..models.architectures import load_folder
    from .gpu_program import GpuProgram
    max_tokens = max(PAGE, (max_tokens + PAGE - 1) // PAGE * PAGE)
    cfg, weights = load_folder(model_dir, device, dtype)
    return GpuProgram(cfg, weights, device, max_lanes=MAX_LIVE, max_context=max_tokens, kv_pages=max_tokens // PAGE,
                      page_size=PAGE, prefill_chunk=max_tokens, checkpoint_slots=0, use_graph=False)


def replay(program, lines: Iterable[str], out_dir: str, log: TextIO) -> None:
    lanes: Dict[str, object] = {}
    for line in lines:
        if not line.strip():
            continue
        rec = json.loads(line)
        entries = []
        for e in rec["entries"]:
            lane = lanes.get(e["id"])
            if lane is None:
                lane = lanes[e["id"]] = program.open_empty()
            if e["tokens"]:
                entries.append((lane, [int(t) for t in e["tokens"]], [int(w) for w in e.get("want", ())]))
        if entries:
            logits = program.step(entries)
            if logits.shape[0]:
                path = os.path.join(out_dir, f"{rec['step']}.f32")
                with open(path, "wb") as f:
                    f.write(logits.contiguous().numpy().astype("<f4", copy=False).tobytes())
        for name in rec.get("end", ()):
            lane = lanes.pop(name, None)
            if lane is not None:
                program.close(lane)
        print(f"done {rec['step']}", file=log, flush=True)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace through a model folder and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"],
                    help="float32: activations, cache and matrix products in true 32-bit")
    ap.add_argument("--out", required=True, help="folder the <step>.f32 files are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    if args.max_tokens < 1:
        raise SystemExit("--max-tokens must be positive")
    os.makedirs(args.out, exist_ok=True)
    program = open_program(args.model, torch.float32 if args.dtype == "float32" else torch.bfloat16, args.max_tokens)
    replay(program, sys.stdin, args.out, sys.stdout)
    return 0


if __name__ == "__main__":
    sys.exit(main())
