"""What the tests of the language models share: random tensors, a paged cache filled by hand, comparisons, and feeding a
runner in portions, and writing model folders."""
import json
import struct

import numpy as np
import torch


def rnd(shape, dtype, seed, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (scale * torch.randn(shape, generator=g)).to(dtype)


def close(got, want, t):
    got, want = got.double().cpu(), want.double().cpu()
    err = (got - want).abs().max().item() / max(1e-30, want.abs().max().item())
    assert err <= t, f"{err:.3e}"


class Pages:
    """A paged latent cache with shuffled pages, filled from contiguous rows."""

    def __init__(self, lens, row_elems, dtype, page_tokens=64, seed=0, fill=1e4):
        blocks = max(-(-n // page_tokens) for n in lens) + 1
        self.table = torch.full((len(lens), blocks), -1, dtype=torch.int32)
        perm = torch.randperm(len(lens) * blocks, generator=torch.Generator().manual_seed(seed)).to(torch.int32)
        for s, n in enumerate(lens):
            used = -(-n // page_tokens)
            self.table[s, :used] = perm[s * blocks:s * blocks + used]
        # what no sequence owns, and what lies behind a sequence's end, is large: reading it would show
        self.pool = torch.full((len(lens) * blocks, page_tokens, row_elems), fill).to(dtype)
        self.page_tokens = page_tokens

    def put(self, s, rows):
        for t in range(rows.shape[0]):
            self.pool[int(self.table[s, t // self.page_tokens]), t % self.page_tokens] = rows[t]

    def rows(self, seq, pos, max_len, segments=()):
        from axono_b200.models.layers import Rows

        return Rows(torch.tensor(seq, dtype=torch.int32).cuda(), torch.tensor(pos, dtype=torch.int32).cuda(), self.table.cuda(),
                    max_len, len(seq), list(segments))


def runner_of(cfg, w, dtype, max_tokens, **kw):
    from axono_b200 import models
    from axono_b200.serving import ModelRunner

    return ModelRunner(models.create(cfg, w, dtype), max_tokens, **kw)


def feed(runner, seq, tokens, portions):
    """All logits of `tokens` brought in portions of the given sizes (the last size repeats)."""
    out, at, sizes = [], 0, list(portions)
    while at < len(tokens):
        n = min(sizes.pop(0) if len(sizes) > 1 else sizes[0], len(tokens) - at)
        out.append(runner.step([(seq, tokens[at:at + n], list(range(n)))]).cpu().numpy())
        at += n
    assert runner.error_word() == 0
    return np.concatenate(out)


SCHEDULES = {"whole": [10000], "tokens": [1], "twos": [2], "mixed": [5, 2, 64, 1, 63, 3, 17, 65, 2, 1], "prompt_then_tokens": [120, 1]}


def position_errors(got, want):
    """Per position: rms of the difference (means taken off) over the rms of the wanted logits."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())


def write_safetensors(path, tensors, extra_header=None):
    names = {torch.bfloat16: "BF16", torch.float32: "F32", torch.int32: "I32"}
    header, data = dict(extra_header or {}), b""
    for k, t in tensors.items():
        raw = t.contiguous().view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[k] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [len(data), len(data) + len(raw)]}
        data += raw
    head = json.dumps(header).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + data)
