"""Replays a trace through a model: token ids are given step by step, logits are written to files,
nothing is sampled.  The model is driven by the entry points that generation uses: prompt portions
through `Decoder.forward_portion`, single tokens that continue a sequence through the captured decode
step.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input holds one JSON object per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every entry continues its request where the request's earlier tokens left the cache; `want` are places
among its tokens.  `DIR/<step>.f32` gets the wanted logits ([wanted, vocab] little-endian fp32) and a
line `done <step>` follows.  One request is live at a time; `end` gives its cache back.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

DTYPES = ("bfloat16", "float32")


class TraceSession:
    """One sequence slot of a decoder, fed token by token or in portions."""

    def __init__(self, model, max_tokens: int):
        self.model = model
        model.setup_caches(1, max_tokens)
        model.setup_decode(1)
        self.live, self.position = None, 0

    def run(self, request: str, tokens, want):
        """Logits [len(want), vocab] of the wanted places, or None."""
        import torch
        if self.live is None:
            self.live, self.position = request, 0
        elif self.live != request:
            raise RuntimeError(f"request {request!r} before {self.live!r} has ended")
        m = self.model
        idx = torch.tensor([list(tokens)], dtype=torch.long, device=m.device)
        start, self.position = self.position, self.position + len(tokens)
        if len(tokens) == 1 and start > 0:
            logits = m.decode_given_token(idx, start)
            return logits[[0] * len(want)] if len(want) else None
        logits = m.forward_portion(idx, start, want)
        return None if logits is None else logits[0]

    def end(self, request: str) -> None:
        if self.live == request:
            self.live, self.position = None, 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay given token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=DTYPES)
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens that live requests hold at any time")
    args = ap.parse_args(argv)

    from . import build
    from .registry import libraries_of, load_model, read_config
    build.build(libraries=libraries_of(read_config(args.model)))

    import torch
    # sums of split matrix products stay in fp32, fp32 products stay fp32
    torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
    torch.backends.cuda.matmul.allow_tf32 = False
    session = TraceSession(load_model(args.model, getattr(torch, args.dtype), "cuda"), args.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = []
        for e in step["entries"]:
            logits = session.run(e["id"], e["tokens"], e["want"])
            if logits is not None:
                parts.append(logits.float().cpu())
        for request in step.get("end", []):
            session.end(request)
        if parts:
            torch.cat(parts).contiguous().numpy().astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        else:
            torch.cuda.synchronize()
        print(f"done {step['step']}", flush=True)
    return 0
