"""Replays a trace of token ids through a model, step by step, and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps are read from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step run as one batch on the serving backend (`GpuBackend`: its runner, paged pool and kernels); an id is
admitted at its first entry and gives its pages back when it is listed in "end". A step that wants logits writes
OUT/<step>.f32 (little-endian fp32 [wanted, vocab], entry by entry), and every step prints "done <step>". The pool holds
--max-tokens tokens and at most four requests are live. Exit codes: 0 at the end of the input, 3 when the model's decoder
does not run in the requested type."""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4


def replay(backend, lines, out_dir: str, report) -> None:
    """Feeds `lines` to any decode backend; `report(step)` is called after each step."""
    live: dict[str, object] = {}
    try:
        for line in lines:
            if not line.strip():
                continue
            step = json.loads(line)
            entries = [e for e in step["entries"] if e["tokens"]]
            for e in entries:
                if not all(isinstance(t, int) and 0 <= t < backend.vocab_size for t in e["tokens"]):
                    raise ValueError(f"step {step['step']}: token id outside the vocabulary")
                if not all(0 <= w < len(e["tokens"]) for w in e.get("want", [])):
                    raise ValueError(f"step {step['step']}: `want` outside the entry's tokens")
                if e["id"] not in live:
                    if len(live) >= MAX_LIVE:
                        raise ValueError(f"step {step['step']}: more than {MAX_LIVE} live requests")
                    live[e["id"]] = backend.new_sequence()
                if backend.length(live[e["id"]]) + len(e["tokens"]) > backend.max_context:
                    raise ValueError(f"step {step['step']}: request {e['id']!r} exceeds --max-tokens")
            if entries:
                logits = backend.forward_at([live[e["id"]] for e in entries], [list(e["tokens"]) for e in entries],
                                            [list(e.get("want", [])) for e in entries])
                if logits is not None:
                    path = os.path.join(out_dir, f"{step['step']}.f32")
                    logits.float().cpu().contiguous().numpy().astype("<f4").tofile(path)
            for rid in step.get("end", []):
                if rid in live:
                    backend.release(live.pop(rid))
            report(step["step"])
    finally:
        for s in live.values():
            backend.release(s)


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    args = ap.parse_args(argv)

    from .. import _native

    _native.prefer_text_kernels()
    import torch

    from ..contracts.errors import Unsupported
    from ..io.safetensors_io import load_dir
    from ..models.config import ModelConfig
    from ..ops import check_status
    from .loading import gpu_backend

    dtype = getattr(torch, args.dtype)
    cfg = ModelConfig.from_dir(args.model)
    try:
        backend = gpu_backend(cfg, load_dir(args.model), dtype=dtype, max_batch=MAX_LIVE, max_context=args.max_tokens,
                              kv_tokens=args.max_tokens)
    except Unsupported as e:
        print(f"trace_run: {e}", file=sys.stderr)
        return 3 if args.dtype == "float32" else 2
    os.makedirs(args.out, exist_ok=True)

    def report(step: int) -> None:
        check_status()              # a device-side wait that ran out is an error, not a wrong answer
        print(f"done {step}", flush=True)
    replay(backend, sys.stdin, args.out, report)
    return 0
