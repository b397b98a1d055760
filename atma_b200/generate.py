"""Command line: ``python -m atma_b200.generate --model DIR --prompt 1,5,7 [--prompt 2,2] [--max-new-tokens N] ...``

Prompts and outputs are token ids (one output line per prompt).  The model class follows config.json."""

import argparse

import torch


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="python -m atma_b200.generate", description="Generate token ids with a model folder.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", action="append", required=True, help="token ids with commas between them; may be repeated")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--temperature", type=float, default=0.0, help="0 = greedy")
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=None)
    ap.add_argument("--stop", default="", help="token ids that end a sequence")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-tokens", type=int, default=32768, help="tokens that live sequences hold at most")
    ap.add_argument("--max-seqs", type=int, default=64)
    ap.add_argument("--max-step-tokens", type=int, default=8192)
    return ap.parse_args(argv)


def ids(text):
    return [int(t) for t in text.replace(",", " ").split()]


def main(argv=None):
    a = parse_args(argv)
    from .checkpoint import read_config
    from .engine import Engine, SamplingParams
    from .registry import build_kernels, load_model
    build_kernels(read_config(a.model))
    model = load_model(a.model, getattr(torch, a.dtype))
    engine = Engine(model, max_tokens=a.max_tokens, max_seqs=a.max_seqs, max_step_tokens=a.max_step_tokens)
    params = SamplingParams(a.max_new_tokens, a.temperature, a.top_k, a.top_p, tuple(ids(a.stop)), a.seed)
    for out in engine.generate([ids(p) for p in a.prompt], params):
        print(",".join(str(t) for t in out))


if __name__ == "__main__":
    main()
