"""Trace runner: feeds given token ids through a model step by step and writes logits (``bin/trace_run``).

Steps come on standard input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

A step's entries are one batch; ``want`` are the places among an entry's tokens whose logits are written to
``OUT/<step>.f32`` (little-endian fp32 ``[wanted, vocab]``); ``end`` lists requests that give back what they hold.
After every step the line ``done <step>`` is printed. The engine is the one that generates: its scheduler's place is
taken by :class:`~tokenweave_b200.engine.replay.StepReplayer`.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64
MAX_LIVE = 4


def parse_args(argv=None) -> argparse.Namespace:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay given steps through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help=f"most tokens live requests hold at any time (each rounded up to {PAGE}): sizes the cache pool")
    ap.add_argument("--max-requests", type=int, default=MAX_LIVE, help="most requests live at any time")
    ap.add_argument("--device", default="cuda", help="cuda, or cpu to replay on the plain PyTorch path")
    return ap.parse_args(argv)


def main(argv=None) -> int:
    args = parse_args(argv)
    if args.device == "cuda":
        from .. import build
        build.build()
    from ..config import EngineArgs
    from ..engine.core import EngineCore
    from ..engine.replay import StepReplayer
    blocks = (args.max_tokens + PAGE - 1) // PAGE
    tokens = blocks * PAGE
    config = EngineArgs(model=args.model, dtype=args.dtype, device=args.device, skip_tokenizer_init=True,
                        block_size=PAGE, num_gpu_blocks_override=blocks + 1, max_num_seqs=args.max_requests,
                        max_model_len=tokens, max_num_batched_tokens=tokens).create_engine_config()
    core = EngineCore(config)
    replayer = StepReplayer(core)
    os.makedirs(args.out, exist_ok=True)
    try:
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            logits = replayer.step([(e["id"], e["tokens"], e.get("want", ())) for e in step["entries"]],
                                   step.get("end", ()))
            if logits is not None:
                path = os.path.join(args.out, f"{step['step']}.f32")
                logits.numpy().astype("<f4").tofile(path)
            print(f"done {step['step']}", flush=True)
    finally:
        core.shutdown()
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
