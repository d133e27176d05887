"""Trace replay: given token ids through the serving engine, step by step, logits out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every input line is one engine step, ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}],
"end": ["b"]}``: the next tokens of some sequences (portions of prompts beside single tokens, one batch), the places
among them whose logits are wanted, and the sequences whose cache is given back afterwards.  A step with wanted places
writes ``DIR/<step>.f32`` (little-endian fp32 [wanted, vocab], entries in order); ``done <step>`` is printed after every
step.  The model is loaded like any other (``ModelLoader``), and the steps run on the engine of
``engine.factory.build_engine`` through ``LLMEngine.score_step``: the block pool, batch packing, step function and
kernels of the generation path.  Needs a CUDA device.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import List, Optional

LIVE_SEQUENCES = 4
BLOCK = 16
CHUNK = 64          # a live sequence's tokens count in multiples of this against --max-tokens


def build_parser() -> argparse.ArgumentParser:
    p = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model and write logits")
    p.add_argument("--model", required=True, help="model directory (config.json and weights)")
    p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"],
                   help="bfloat16: as the model is served; float32: weights, cache and arithmetic in 32 bits")
    p.add_argument("--out", required=True, help="directory for <step>.f32")
    p.add_argument("--max-tokens", type=int, required=True, help="most tokens that live sequences hold at any time")
    return p


def replay(engine, lines, out_dir: str, write=print) -> None:
    for line in lines:
        if not line.strip():
            continue
        d = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want") or []) for e in d.get("entries", [])]
        logits = engine.score_step(entries, d.get("end") or [])
        check = getattr(engine.runner, "raise_on_device_error", None)
        if check is not None:
            check()
        if logits is not None and logits.shape[0]:
            path = os.path.join(out_dir, f"{d['step']}.f32")
            logits.float().cpu().contiguous().numpy().astype("<f4", copy=False).tofile(path)
        write(f"done {d['step']}", flush=True)


def main(argv: Optional[List[str]] = None) -> int:
    a = build_parser().parse_args(argv)
    import torch

    from ..weights import ModelLoader
    from .factory import build_engine

    tokens = -(-max(a.max_tokens, 1) // CHUNK) * CHUNK
    os.makedirs(a.out, exist_ok=True)
    model = ModelLoader().load_model(a.model, device="cpu")
    engine = build_engine(model, device="cuda", dtype=getattr(torch, a.dtype), max_num_seqs=LIVE_SEQUENCES,
                          max_num_batched_tokens=tokens, max_model_len=tokens, block_size=BLOCK, num_blocks=tokens // BLOCK,
                          enable_prefix_caching=False, use_cuda_graphs=False)
    replay(engine, sys.stdin, a.out)
    return 0
