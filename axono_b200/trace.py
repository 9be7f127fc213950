"""Replays a trace of token ids through a model, step by step, and writes the logits asked for.

Steps are read from standard input, one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}
A step brings requests their next tokens; `want` are places among them.  Their logits go to <out>/<step>.f32
(little-endian fp32, [wanted, vocab], in the order of entries and places); then "done <step>" is printed.
Requests listed under `end` give back what they hold.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=8, help="most requests alive at any time")
    args = ap.parse_args(argv)

    import torch  # first: the library then shares PyTorch's cuBLASLt

    from . import models
    from .serving import ModelRunner

    models.use_library_for(args.model)
    torch.cuda.set_device(0)
    model = models.load(args.model, getattr(torch, args.dtype))
    runner = ModelRunner(model, args.max_tokens, max_seqs=args.max_requests)
    seqs = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in seqs:
                seqs[e["id"]] = runner.open()
            entries.append((seqs[e["id"]], e["tokens"], e["want"]))
        logits = runner.step(entries) if entries else None
        data = logits.cpu().numpy().astype("<f4").tobytes() if logits is not None else None
        word = runner.error_word()
        if word:
            raise RuntimeError(f"device error word {word:#x}")
        if data is not None:
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        for name in step["end"]:
            runner.close(seqs.pop(name))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
