"""Replays a trace of given token ids through a model, step by step, and writes logits (``bin/trace_run``).

Steps come on standard input, one JSON object a line: {"step": 0, "entries": [{"id": "a", "tokens": [..], "want": [..]}],
"end": [..]}.  A step with wanted places writes DIR/<step>.f32 (little-endian fp32, [wanted, vocab]); every step prints
"done <step>".  ``end`` names the sequences to release after the step.
"""

import argparse
import json
import os
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=32768, help="tokens that live sequences hold at most")
    a = ap.parse_args(argv)

    import torch
    from .checkpoint import read_config
    from .engine import Engine
    from .registry import build_kernels, load_model
    build_kernels(read_config(a.model))
    model = load_model(a.model, getattr(torch, a.dtype))
    engine = Engine(model, max_tokens=max(a.max_tokens, 1), max_seqs=64)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = engine.feed([(e["id"], e["tokens"], e["want"]) for e in step["entries"]])
        if logits is not None:
            logits.float().cpu().numpy().astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        for name in step.get("end", []):
            engine.release(name)
        print(f"done {step['step']}", flush=True)
    return 0
