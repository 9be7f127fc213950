"""Greedy generation from a model folder, on token ids.

    python -m axono_b200.generate --model DIR --tokens 5,17,3 --tokens 8,8 --max-new 32
    echo "5 17 3" | python -m axono_b200.generate --model DIR --max-new 32

Every prompt becomes a request of the scheduler (axono_b200.serving.Engine); one line of token ids is printed per
prompt, in order.  --model names a folder with config.json and model.safetensors; the architecture in config.json
picks the model class.
"""
from __future__ import annotations

import argparse
import sys


def parse_prompts(tokens, stream):
    lines = tokens if tokens else [line for line in stream if line.strip()]
    return [[int(t) for t in line.replace(",", " ").split()] for line in lines]


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="axono_b200.generate", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--tokens", action="append", default=[], help="a prompt as token ids (repeatable; default: one per input line)")
    ap.add_argument("--max-new", type=int, default=16, help="tokens to generate per prompt")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-batch", type=int, default=16, help="requests that run together")
    ap.add_argument("--token-budget", type=int, default=2048, help="most tokens one step brings")
    args = ap.parse_args(argv)
    prompts = parse_prompts(args.tokens, sys.stdin)
    if not prompts or not all(prompts):
        ap.error("no prompt")

    import torch  # first: the library then shares PyTorch's cuBLASLt

    from . import models
    from .serving import ModelRunner, generate

    models.use_library_for(args.model)
    torch.cuda.set_device(0)
    model = models.load(args.model, getattr(torch, args.dtype))
    longest = max(len(p) for p in prompts) + args.max_new
    batch = min(args.max_batch, len(prompts))
    runner = ModelRunner(model, batch * longest, max_seqs=batch, max_seq_len=longest)
    for out in generate(runner, prompts, args.max_new, token_budget=args.token_budget):
        print(" ".join(map(str, out)))
    word = runner.error_word()
    if word:
        raise RuntimeError(f"device error word {word:#x}")
    return 0


if __name__ == "__main__":
    sys.exit(main())
