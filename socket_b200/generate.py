"""Command line: greedy generation with the model of a folder (`config.json` + `model.safetensors`).

    python -m socket_b200.generate --model DIR --tokens 5,17,3 --new 32 [--dtype bfloat16|float32]
                                   [--mode MODE] [--prefill-chunk N]

Token ids in, token ids out (the framework has no tokenizer).  Several prompts of equal length, separated
by ';', run as one batch.  The architecture's CUDA libraries are built first where they are missing.
"""
from __future__ import annotations

import argparse
import sys


def parse_prompts(text: str):
    rows = [[int(t) for t in part.split(",") if t.strip()] for part in text.split(";")]
    if not rows[0] or len({len(r) for r in rows}) != 1:
        raise ValueError("prompts must be non-empty and of equal length")
    return rows


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m socket_b200.generate", description="greedy generation from token ids")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--tokens", required=True, help="prompt token ids: 5,17,3 (several prompts: 5,17,3;8,2,9)")
    ap.add_argument("--new", type=int, default=32, help="tokens to generate")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--mode", default=None, help="attention mode of models that have several (the Transformer: sparse, dense)")
    ap.add_argument("--prefill-chunk", type=int, default=8192, help="prompt tokens per portion")
    args = ap.parse_args(argv)
    prompts = parse_prompts(args.tokens)

    from . import build
    from .registry import libraries_of, load_model, read_config
    build.build(libraries=libraries_of(read_config(args.model)))
    import torch

    from .decoder import generate
    model = load_model(args.model, getattr(torch, args.dtype), "cuda")
    seq, stats = generate(model, torch.tensor(prompts), args.new, mode=args.mode, prefill_chunk=args.prefill_chunk)
    for row in seq.tolist():
        print(",".join(str(t) for t in row[len(prompts[0]):]))
    print(f"prefill {stats['prefill_time_s'] * 1e3:.1f} ms, {stats['decode_only_tokens']} decoded tokens in "
          f"{stats['decode_time_s'] * 1e3:.1f} ms", file=sys.stderr)
    return 0


if __name__ == "__main__":
    sys.exit(main())
