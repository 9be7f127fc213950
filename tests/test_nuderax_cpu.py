"""What of the language models needs no GPU: configuration, weights, the arena of rows, the scheduler, the command
lines, and the plain evaluation against itself."""
import copy
import os
import struct
import subprocess
import sys

import pytest
import torch

import nuderax_cases as cases
import plain_nuderax as plain
from lm_helpers import write_safetensors

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_safetensors_reader(tmp_path):
    from axono_b200.models.weights import SafetensorsFile

    want = {"a": torch.randn(3, 5).to(torch.bfloat16), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, 1, 4)}
    p = str(tmp_path / "m.safetensors")
    write_safetensors(p, want, {"__metadata__": {"x": "y"}})
    with SafetensorsFile(p) as f:
        assert set(f.keys()) == set(want) and "a" in f and "d" not in f
        for k, t in want.items():
            assert f[k].dtype == t.dtype and torch.equal(f[k], t)
        with pytest.raises(KeyError):
            f["d"]
    write_safetensors(p, want)
    raw = bytearray(open(p, "rb").read())
    open(p, "wb").write(raw[:-3])  # cut short
    with SafetensorsFile(p) as f, pytest.raises(ValueError):
        f["c"]
    open(p, "wb").write(struct.pack("<Q", 1 << 40))
    with pytest.raises(ValueError):
        SafetensorsFile(p)


def test_registry_and_configuration():
    from axono_b200 import models
    from axono_b200.models.nuderax import tensor_shapes

    assert "Nuderax" in models.architectures()
    with pytest.raises(ValueError):
        models.config_of({"architecture": "Nothing"})
    assert models.config_of({"architecture": "TextTower", "hidden": 64, "mrope_section": [1, 1, 1]}).hidden == 64
    for make in (cases.odd, cases.tiles, cases.fast):
        cfg = make()
        parsed = models.config_of(cfg)
        shapes = dict(tensor_shapes(parsed))
        assert shapes == {k: tuple(v.shape) for k, v in plain.random_weights(cfg, 0).items()}
    odd = models.config_of(cases.odd())
    assert [layer.mixer.kv_from for layer in odd.layers] == [None, None, 1, 0] and odd.layers[2].mlp is None
    assert odd.layers[0].mixer.q_rank == 36 and odd.layers[0].mixer.rot_dims == 8 and odd.layers[1].mlp.shared_limit == 0.4


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="convolution"),
    lambda c: c["layers"][0]["mixer"].pop("q_rank"),
    lambda c: c["layers"][2]["mixer"].update(kv_from=3),          # a later layer
    lambda c: c["layers"][3]["mixer"].update(kv_from=2),          # one that has no latent of its own
    lambda c: c["layers"][3]["mixer"].update(kv_rank=48),         # other latent sizes
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14),     # more than rot_dim
    lambda c: c["layers"][0]["mlp"].update(kind="dense"),
])
def test_configurations_that_make_no_sense_are_refused(change):
    from axono_b200 import models

    cfg = copy.deepcopy(cases.odd())
    change(cfg)
    with pytest.raises(ValueError):
        models.config_of(cfg)


def test_arena_of_rows_bookkeeping():
    from axono_b200.kv_cache import KVArena

    a = KVArena.of_rows([160, 24], num_pages=5, max_seqs=3, max_seq_len=256, device_memory=False)
    s0, s1 = a.alloc_seq(0), a.alloc_seq(65)
    assert a.seq_pages(s1) == [0, 1] and a.seq_pages(s0) == []
    a.reserve(s0, 129)
    assert len(a.seq_pages(s0)) == 3 and a.stats()["pages_free"] == 0
    with pytest.raises(RuntimeError):
        a.reserve(s1, 129)
    a.free_seq(s0)
    a.reserve(s1, 256)
    assert len(a.seq_pages(s1)) == 4 and a.stats()["device_bytes"] == 0
    a.close()


class FakeRunner:
    """Counts what the scheduler asks for; the 'model' says that the next token is the number of tokens so far."""

    class Arena:
        num_pages = 6

    def __init__(self, max_seqs=2, page_tokens=64):
        self.arena, self.max_seqs, self.page_tokens = self.Arena(), max_seqs, page_tokens
        self.lengths, self.steps, self.free = {}, [], list(range(max_seqs))

    def capacity(self):
        return 256

    def open(self):
        s = self.free.pop(0)
        self.lengths[s] = 0
        return s

    def close(self, seq):
        del self.lengths[seq]
        self.free.append(seq)

    def step(self, entries, trace=None):
        assert len({e[0] for e in entries}) == len(entries)
        out = []
        for seq, tokens, want in entries:
            out += [self.lengths[seq] + w + 1 for w in want]
            self.lengths[seq] += len(tokens)
        self.steps.append([(seq, len(tokens)) for seq, tokens, _ in entries])
        pages = sum(-(-n // self.page_tokens) for n in self.lengths.values())
        assert pages <= self.arena.num_pages
        return out or None


def test_scheduler_portions_batches_and_slots():
    from axono_b200.serving import Engine

    r = FakeRunner()
    e = Engine(r, token_budget=50, sample=lambda logits: logits)
    reqs = [e.submit([1] * n, m) for n, m in ((120, 4), (3, 6), (60, 2), (1, 1))]
    e.run()
    assert [q.out for q in reqs] == [[120, 121, 122, 123], [3, 4, 5, 6, 7, 8], [60, 61], [1]]
    assert all(sum(n for _, n in step) <= 50 for step in r.steps)
    assert any({1} < {n for _, n in step} for step in r.steps)  # decoding beside a portion of a prompt
    assert sorted(r.free) == [0, 1] and not r.lengths


def test_scheduler_waits_for_pages_and_refuses_the_impossible():
    from axono_b200.serving import Engine

    r = FakeRunner(max_seqs=4)
    e = Engine(r, token_budget=4096, sample=lambda logits: logits)
    reqs = [e.submit([1] * 180, 10) for _ in range(4)]  # three pages each, six in all: two at a time
    e.run()
    assert all(q.out == list(range(180, 190)) for q in reqs)
    assert max(len(step) for step in r.steps) == 2
    for tokens, new in (([], 3), ([1], 0), ([1] * 250, 10)):
        with pytest.raises(ValueError):
            e.submit(tokens, new)


def test_command_lines_parse_without_a_gpu():
    for cmd in ([sys.executable, "-m", "axono_b200.generate", "--help"], [os.path.join(ROOT, "bin", "trace_run"), "--help"]):
        out = subprocess.run(cmd, capture_output=True, text=True, timeout=120, cwd=ROOT)
        assert out.returncode == 0 and "--model" in out.stdout
    from axono_b200.generate import parse_prompts

    assert parse_prompts(["5,17, 3", "8"], None) == [[5, 17, 3], [8]]
    assert parse_prompts([], ["1 2\n", "\n", "3\n"]) == [[1, 2], [3]]


# ---- the plain evaluation itself ---------------------------------------------------------------------------
def test_plain_router_closed_groups_are_not_zero():
    """All choices negative: an expert of a closed group must not win with a 0."""
    z = torch.tensor([0.0, 0.1, 0.2, 0.3, 3.0, -9.0], dtype=torch.float64)
    ids, weights = plain.route_token(z, torch.full((6,), -5.0, dtype=torch.float64), 2, 3, 1, 2.0)
    assert ids == [3, 2]  # the group of 4 and 5 has the best single expert, but the smallest sum of two
    assert weights == pytest.approx([2 / (1 + 2.718281828459045 ** -0.3), 2 / (1 + 2.718281828459045 ** -0.2)])


def test_plain_attention_is_causal_and_shares_latents():
    cfg = cases.odd()
    w = {k: v.double() for k, v in plain.random_weights(cfg, 3).items()}
    a = plain.forward(cfg, w, [5, 6, 7, 8, 9])
    b = plain.forward(cfg, w, [5, 6, 7, 100, 9])
    assert torch.allclose(a[:3], b[:3]) and not torch.allclose(a[3:], b[3:])
    w2 = dict(w)
    w2["l1.mix.dkv"] = w["l1.mix.dkv"] * torch.linspace(0.5, 2, w["l1.mix.dkv"].shape[0], dtype=torch.float64)[:, None]
    assert not torch.allclose(plain.forward(cfg, w2, [5, 6, 7]), a[:3])


def test_plain_rotation_is_relative():
    q, k = torch.randn(1, 12, dtype=torch.float64), torch.randn(1, 12, dtype=torch.float64)
    at = lambda x, p: plain.rotate_interleaved(x, torch.tensor([p]), 500.0, 8)  # noqa: E731
    assert torch.allclose(at(q, 40) @ at(k, 33).T, at(q, 7) @ at(k, 0).T)
    assert torch.equal(at(q, 40)[:, 8:], q[:, 8:]) and not torch.allclose(at(q, 40)[:, :8], q[:, :8])
