"""Replays a recorded schedule of token ids through the continuous-batching engine and writes the logits it asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Each input line is one engine step:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

All entries of a line run as one batch (`Engine.run_given`): prompt portions beside single tokens, each request continuing from its
cache blocks and recurrent state.  The logits at the wanted places go to OUT/<step>.f32 ([wanted, vocab], little-endian fp32, in the
order of the entries); the requests under "end" give their blocks and state slot back after the step; "done <step>" is printed."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

BLOCK = 16            # tokens per cache block
STATE_SLOTS = 4       # most live requests


def open_engine(model_dir: str, dtype: str, max_tokens: int):
    import onnxruntime_genai_b200 as og
    blocks = -(-max_tokens // BLOCK)
    cfg = og.Config(model_dir)
    cfg.set_provider_option("cuda", "compute_dtype", dtype)
    cfg.overlay(json.dumps({"model": {"context_length": max(cfg.context_length, max_tokens + 1)}, "search": {"max_length": max(cfg.context_length, max_tokens + 1)},
                            "engine": {"dynamic_batching": {"block_size": BLOCK, "num_blocks": blocks, "max_batch_size": STATE_SLOTS,
                                                            "max_scheduled_tokens": max(max_tokens, STATE_SLOTS)}}}))
    model = og.Model(cfg)
    return model, og.Engine(model)


def replay(model, engine, lines, out_dir: str, say) -> None:
    import onnxruntime_genai_b200 as og
    live = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = og.Request(og.GeneratorParams(model))
            entries.append((live[e["id"]], e["tokens"], e.get("want", [])))
        logits = engine.run_given(entries) if entries else []
        if any(want for _, _, want in entries):
            rows = np.concatenate([t.float().cpu().numpy() for t in logits], axis=0)
            rows.astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for rid in step.get("end", []):
            if rid in live:
                engine.remove_request(live.pop(rid))
        say(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay given token ids through the engine and write logits")
    ap.add_argument("--model", required=True, help="model directory")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory of the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold together (sizes the cache pool)")
    a = ap.parse_args(argv)
    model, engine = open_engine(a.model, a.dtype, a.max_tokens)
    from . import ops
    replay(model, engine, sys.stdin, a.out, lambda t: print(t, flush=True))
    ops.check_kernel_status()
    return 0
