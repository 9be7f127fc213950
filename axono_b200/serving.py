"""Serving of registered models: the step over cached sequences, and the scheduler above it.

`ModelRunner` owns a model's cache (pages of a `KVArena`, one sequence slot per live request, and that slot's state
of recurrent layers) and runs steps: a step brings each of some sequences its next tokens - a whole prompt, a portion of one, a decoded token - and
returns the logits asked for.  `Engine` schedules requests over it: every step decodes all running requests
and fills the rest of its token budget with portions of waiting prompts; sampling is greedy (`argmax_last_dim`).
While only decoding is left and the batch does not change, the engine replays the step as a CUDA graph.
"""
from __future__ import annotations

import collections
from dataclasses import dataclass, field
from typing import List, Optional, Sequence

import numpy as np
import torch

from . import ops
from .cuda_graph import CUDAGraph
from .kv_cache import KVArena
from .models.layers import Cache, Rows


class ModelRunner:
    def __init__(self, model, max_tokens: int, max_seqs: int = 1, page_tokens: int = 64, max_seq_len: Optional[int] = None,
                 shuffle_pages: Optional[int] = None):
        """max_tokens: the most tokens that live sequences hold together; max_seq_len: the most one may hold."""
        self.model, self.max_seqs, self.page_tokens = model, max_seqs, page_tokens
        max_seq_len = max_seq_len or max_tokens
        pages = -(-max_tokens // page_tokens) + max_seqs  # each sequence's last page may be part-filled
        self.arena = KVArena.of_rows(model.cache_rows, pages, max_seqs, max_seq_len, model.dtype, page_tokens)
        if shuffle_pages is not None:
            self.arena.shuffle_free(shuffle_pages)
        self.pages = [self.arena.row_pages(c) for c in range(len(model.cache_rows))]
        self.states = [tuple(self.arena.add_state(shape, dtype) for shape, dtype in layer) for layer in model.state_shapes]
        self.cache = Cache(self.pages, self.states)
        self.block_table = self.arena.table()
        self.lengths = {}

    # -- sequences --------------------------------------------------------------------------------
    def open(self) -> int:
        seq = self.arena.alloc_seq(0)
        self.lengths[seq] = 0
        return seq

    def close(self, seq: int) -> None:
        del self.lengths[seq]
        self.arena.free_seq(seq)

    def copy_state(self, seqs):
        """The recurrent state of some sequences, for `put_state`."""
        at = torch.tensor(list(seqs), dtype=torch.int64, device=self.model.device)
        return [(t, at, t.index_select(0, at)) for layer in self.states for t in layer]

    @staticmethod
    def put_state(saved) -> None:
        for t, at, entries in saved:
            t.index_copy_(0, at, entries)

    def capacity(self) -> int:
        return self.arena.max_blocks * self.page_tokens

    # -- steps ------------------------------------------------------------------------------------
    def step(self, entries, trace=None):
        """entries: (sequence, tokens, want) - the sequence's next tokens and the places among them whose logits
        are asked for.  Returns fp32 logits (wanted, vocab), entry by entry, or None when nothing is wanted."""
        if len({e[0] for e in entries}) != len(entries):
            raise ValueError("a sequence may appear once in a step")
        for seq, tokens, want in entries:
            if seq not in self.lengths:
                raise ValueError(f"sequence {seq} is not open")
            if not len(tokens) or any(not 0 <= w < len(tokens) for w in want):
                raise ValueError("an entry needs tokens, and wanted places among them")
            self.arena.reserve(seq, self.lengths[seq] + len(tokens))
        self.arena.sync()
        # single tokens first, then portions by length: those that attend through the cache, then the long ones
        order = sorted(range(len(entries)), key=lambda i: len(entries[i][1]))
        total, wanted = sum(len(e[1]) for e in entries), sum(len(e[2]) for e in entries)
        # two copies for the step's integers: token ids and wanted rows; sequences, positions, rows before, portions
        wide, ints = np.empty(total + wanted, np.int64), np.empty((3, total), np.int32)
        first, segments, portions, latent, max_len, at = {}, [], [], 0, 1, 0
        for i in order:
            seq, tokens, _ = entries[i]
            start, n = self.lengths[seq], len(tokens)
            first[i] = at
            if n > 1:
                portions.append((seq, at, n, start))
            if self.model.takes_segment(n):
                segments.append((seq, at, n, start))
            elif segments:
                raise RuntimeError("a model that takes a portion as a segment must take every longer one")
            else:
                latent += n
                max_len = max(max_len, start + n)
            wide[at:at + n] = tokens
            ints[0, at:at + n], ints[1, at:at + n], ints[2, at:at + n] = seq, np.arange(start, start + n), np.arange(n)
            at += n
        wide[total:] = [first[i] + w for i, (_, _, places) in enumerate(entries) for w in places]
        dev, k = self.model.device, 4 * len(portions)
        packed = torch.from_numpy(np.concatenate([np.array(portions, np.int32).reshape(-1), ints.reshape(-1)])).to(dev)
        ids, (seqs, pos, back) = torch.from_numpy(wide).to(dev), packed[k:].view(3, total)
        rows = Rows(seqs, pos, self.block_table, max_len, latent, segments, total - sum(p[2] for p in portions), back, portions,
                    packed[:k].view(-1, 4))
        logits = self.model.forward(ids[:total], rows, self.cache, ids[total:], trace=trace)
        for seq, tokens, _ in entries:
            self.lengths[seq] += len(tokens)
        return logits

    def error_word(self) -> int:
        return ops.last_error()


class DecodeGraph:
    """Greedy decoding of a fixed set of sequences as one CUDA graph: token ids and positions live on the device,
    each replay appends a token to every sequence and leaves the next ones in `tokens`."""

    def __init__(self, runner: ModelRunner, seqs: Sequence[int], tokens: Sequence[int], limits: Sequence[int]):
        """limits: the length each sequence may reach."""
        self.runner, self.seqs, self.limits = runner, list(seqs), list(limits)
        dev = runner.model.device
        self.tokens = torch.tensor(list(tokens), dtype=torch.int64, device=dev)
        self.rows = Rows(torch.tensor(self.seqs, dtype=torch.int32, device=dev),
                         torch.tensor([runner.lengths[s] for s in self.seqs], dtype=torch.int32, device=dev), runner.block_table,
                         max(self.limits), len(self.seqs), singles=len(self.seqs))
        if self.room() <= 0:
            raise ValueError("DecodeGraph: no room for a token")
        for s, limit in zip(self.seqs, self.limits):  # the pages the replays will write
            runner.arena.reserve(s, limit)
        runner.arena.sync()
        saved = (self.tokens.clone(), self.rows.pos.clone())
        state = runner.copy_state(self.seqs)
        self.graph = CUDAGraph().capture(self._body)  # runs the step once before it records it
        runner.put_state(state)
        self.tokens.copy_(saved[0])
        self.rows.pos.copy_(saved[1])

    def _body(self):
        logits = self.runner.model.forward(self.tokens, self.rows, self.runner.cache, None)
        nxt = ops.argmax_last_dim(logits)
        self.tokens.copy_(nxt)
        self.rows.pos.add_(1)
        return nxt

    def room(self) -> int:
        return min(limit - self.runner.lengths[s] for s, limit in zip(self.seqs, self.limits))

    def step(self) -> torch.Tensor:
        """One token for every sequence; returns the device tensor of next ids (overwritten by the next step)."""
        if self.room() <= 0:
            raise RuntimeError("DecodeGraph: no room left")
        self.graph.replay_async()
        for s in self.seqs:
            self.runner.lengths[s] += 1
        return self.tokens


@dataclass
class Request:
    tokens: List[int]
    max_new: int
    out: List[int] = field(default_factory=list)
    seq: int = -1
    done: int = 0  # prompt tokens already in the cache

    @property
    def prompt_left(self) -> int:
        return len(self.tokens) - self.done

    @property
    def finished(self) -> bool:
        return len(self.out) >= self.max_new


def greedy(logits) -> List[int]:
    return ops.argmax_last_dim(logits).tolist()


class Engine:
    def __init__(self, runner: ModelRunner, token_budget: int = 2048, use_graphs: bool = True, sample=greedy):
        """token_budget: the most tokens one step brings (decoded tokens first, then portions of prompts); sample:
        logits (rows, vocab) -> list of ids (the graph form of decoding is greedy and only used with `greedy`)."""
        if token_budget < 1:
            raise ValueError("token_budget must be positive")
        self.runner, self.token_budget, self.sample = runner, token_budget, sample
        self.use_graphs = use_graphs and sample is greedy
        self.waiting = collections.deque()
        self.running: List[Request] = []
        self._graph: Optional[DecodeGraph] = None
        self._steady = 0  # decode-only steps since the batch last changed
        self._held = 0  # pages promised to running requests

    def submit(self, tokens: Sequence[int], max_new: int) -> Request:
        need = len(tokens) + max_new
        if not len(tokens) or max_new < 1 or need > self.runner.capacity():
            raise ValueError("a request needs tokens, room for its output and no more than the cache holds")
        req = Request(list(tokens), max_new)
        self.waiting.append(req)
        return req

    def _pages_for(self, req: Request) -> int:
        return -(-(len(req.tokens) + req.max_new) // self.runner.page_tokens)

    def _admit(self) -> None:
        total = self.runner.arena.num_pages
        while self.waiting and len(self.running) < self.runner.max_seqs and self._held + self._pages_for(self.waiting[0]) <= total:
            req = self.waiting.popleft()
            self._held += self._pages_for(req)
            req.seq = self.runner.open()
            self.running.append(req)
            self._drop_graph()
        if self.waiting and not self.running:
            raise RuntimeError("the next request does not fit the cache")

    def _drop_graph(self) -> None:
        self._graph, self._steady = None, 0

    def _retire(self) -> None:
        for req in [r for r in self.running if r.finished]:
            self.runner.close(req.seq)
            self._held -= self._pages_for(req)
            self.running.remove(req)
            self._drop_graph()

    def step(self) -> bool:
        """One step of the model; False when nothing is left to do."""
        self._admit()
        if not self.running:
            return False
        if all(r.prompt_left == 0 for r in self.running) and self._decode_by_graph():
            self._retire()
            return True
        budget, entries, reqs = self.token_budget, [], []
        for req in sorted(self.running, key=lambda r: r.prompt_left > 0):  # decoded tokens first
            n = min(req.prompt_left, budget) if req.prompt_left else min(1, budget)
            if n == 0:
                continue
            budget -= n
            if req.prompt_left:
                portion = req.tokens[req.done:req.done + n]
                last = req.done + n == len(req.tokens)
                entries.append((req.seq, portion, [n - 1] if last else []))
            else:
                entries.append((req.seq, [req.out[-1]], [0]))
                last = True
            reqs.append((req, n, last))
        logits = self.runner.step(entries)
        nxt = iter(self.sample(logits) if logits is not None else [])
        for req, n, last in reqs:
            if req.prompt_left:
                req.done += n
            if last:
                req.out.append(next(nxt))
        self._retire()
        return True

    def _decode_by_graph(self) -> bool:
        self._steady += 1
        if not self.use_graphs or self._steady < 4 or len(self.running) > self.token_budget:
            return False
        if self._graph is None:
            self._graph = DecodeGraph(self.runner, [r.seq for r in self.running], [r.out[-1] for r in self.running],
                                      [len(r.tokens) + r.max_new for r in self.running])
        for req, tok in zip(self.running, self._graph.step().tolist()):
            req.out.append(tok)
        return True

    def run(self) -> None:
        while self.step():
            pass


def generate(runner: ModelRunner, prompts: Sequence[Sequence[int]], max_new: int, **engine_options) -> List[List[int]]:
    """Greedy continuations of token-id prompts through the scheduler."""
    engine = Engine(runner, **engine_options)
    reqs = [engine.submit(p, max_new) for p in prompts]
    engine.run()
    return [r.out for r in reqs]
