"""Trace replay: given token ids through a served model step by step, logits out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come as JSON lines on standard input::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step run as one batch of the paged engine (``LLMEngine.forced_step``): its
scheduler admits new ids and takes pages and state slots, its runner executes the batch with the
kernels and graphs that generation uses; nothing is sampled.  The logits at the wanted places go
to ``OUT/<step>.f32`` (little-endian FP32, [wanted, vocab]); ``done <step>`` is printed after
every step.  ``--max-tokens`` sizes the cache pool: the tokens live requests hold at a time, each
request rounded up to whole pages; four requests are live at most.  Exit code 3: no GPU path of
this model runs in the requested type.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 16
LIVE_REQUESTS = 4


def _open(args):
    """(engine, its vocabulary size) for the model directory, chosen by its configuration."""
    from ..checkpoint.safetensors_io import resolve_family
    from ..models.registry import PAGED_DECODERS
    family = resolve_family(args.model)
    if family not in PAGED_DECODERS:
        raise SystemExit(f"{args.model}: {family} is not a decoder of the paged engine")
    entry = PAGED_DECODERS[family]
    import torch
    dtype = getattr(torch, args.dtype)
    if dtype not in entry.gpu_dtypes:
        print(f"{family} does not run in {args.dtype}", file=sys.stderr)
        raise SystemExit(3)
    from .. import build
    from ..ops import native
    build.build(group=entry.build_group)       # compiles what changed since the last build
    native.use_group(entry.build_group)
    if not torch.cuda.is_available():
        raise RuntimeError("no CUDA device")
    from ..checkpoint.quantized import open_checkpoint
    from ..engine.engine import LLMEngine
    ld = open_checkpoint(args.model, dtype)
    cfg = entry.config(ld.config)
    model = entry.model(cfg, torch.device("cuda", 0), dtype, None).load_state(ld)
    tokens = (args.max_tokens + PAGE - 1) // PAGE * PAGE
    engine = LLMEngine(model, num_pages=tokens // PAGE + 1, page_size=PAGE,     # page 0: padding
                       max_num_seqs=LIVE_REQUESTS, max_model_len=tokens, enable_prefix_cache=False)
    return engine


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for the logits of every step")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens that live requests hold at a time (sizes the cache pool)")
    args = ap.parse_args(argv)
    engine = _open(args)
    os.makedirs(args.out, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want") or []) for e in step["entries"]]
        logits = engine.forced_step(entries, step.get("end") or [])
        if logits is not None:
            logits.numpy().astype("<f4", copy=False).tofile(
                os.path.join(args.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
