"""The Rigozen model on the GPU against the plain CPU evaluation (tests/plain_rigozen.py): whole prompts, token by token,
portions, batches, pages and slots used again, and generation through the scheduler."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_rigozen as plain
import rigozen_cases as cases
from lm_helpers import SCHEDULES, feed, position_errors, runner_of, write_safetensors

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

F32_TOL = 3e-5
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def built():
    """name -> (config, weights as stored, prompt, plain logits of the whole prompt)."""
    made = {}

    def get(name, n):
        if (name, n) not in made:
            cfg = getattr(cases, name)()
            w = plain.random_weights(cfg, seed=len(name))
            tokens = np.random.default_rng(n).integers(0, cfg["vocab"], n).tolist()
            made[(name, n)] = (cfg, w, tokens, plain.forward(cfg, {k: v.double() for k, v in w.items()}, tokens).numpy())
        return made[(name, n)]

    return get


def check(got, ref, dtype):
    """In bf16 single positions of narrow heads may be far off: an output of a few elements near zero is blown up by its
    norm."""
    err = position_errors(got, ref)
    if dtype == torch.float32:
        assert err.max() <= F32_TOL, f"worst {err.max():.2e} at {int(err.argmax())}"
    else:
        assert np.quantile(err, 0.9) <= 0.05 and err.max() <= 0.25, f"{np.quantile(err, 0.9):.3f}, worst {err.max():.3f}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("schedule", sorted(SCHEDULES))
@pytest.mark.parametrize("name", ["odd", "tiles", "recurrent"])
def test_schedules(built, name, schedule, dtype):
    cfg, w, tokens, ref = built(name, 150)
    r = runner_of(cfg, w, dtype, 192, shuffle_pages=3)
    check(feed(r, r.open(), tokens, SCHEDULES[schedule]), ref, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[10000], [390, 1], [257, 3, 130, 30], [2, 1, 63, 64, 65, 129, 1], [101]])
def test_schedules_at_tensor_core_sizes(built, sizes, dtype):
    cfg, w, tokens, ref = built("fast", 420)
    r = runner_of(cfg, w, dtype, 512, shuffle_pages=5)
    check(feed(r, r.open(), tokens, sizes), ref, dtype)


@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_residual_after_every_layer(built, name):
    cfg, w, tokens, _ = built(name, 150)
    want, got = [], []
    plain.forward(cfg, {k: v.double() for k, v in w.items()}, tokens[:90], want)
    r = runner_of(cfg, w, torch.float32, 128)
    r.step([(r.open(), tokens[:90], [])], trace=got)
    assert len(got) == len(want) == len(cfg["layers"])
    for a, b in zip(got, want):
        assert (a.cpu().double() - b).abs().max() <= 3e-5 * b.abs().max()


def test_first_tokens(built):
    cfg, w, tokens, ref = built("odd", 150)
    r = runner_of(cfg, w, torch.float32, 64)
    for n in (1, 2, 3, 4):
        for sizes in ([n], [1]):
            s = r.open()
            check(feed(r, s, tokens[:n], sizes), ref[:n], torch.float32)
            r.close(s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["tiles", "recurrent"])
def test_unequal_batch_equals_each_alone(built, name, dtype):
    """Prompts, portions and decoded tokens of different requests in the same steps."""
    cfg, w, tokens, _ = built(name, 150)
    spans = [(0, 150), (3, 83), (10, 140), (1, 2)]
    steps = [[150, 7, 0, 1], [0, 70, 100, 0], [0, 1, 1, 0], [0, 2, 29, 0]]
    r = runner_of(cfg, w, dtype, 448, max_seqs=4, shuffle_pages=1)
    seqs, at, got = [r.open() for _ in spans], [0] * 4, [[] for _ in spans]
    for step in steps:
        entries = []
        for i, n in enumerate(step):
            if n:
                lo = spans[i][0] + at[i]
                entries.append((seqs[i], tokens[lo:lo + n], list(range(n))))
        logits = r.step(entries).cpu().numpy()
        k = 0
        for i, n in enumerate(step):
            got[i].append(logits[k:k + n])
            k, at[i] = k + n, at[i] + n
    wd = {k: v.double() for k, v in w.items()}
    for i, (lo, hi) in enumerate(spans):
        assert at[i] == hi - lo
        check(np.concatenate(got[i]), plain.forward(cfg, wd, tokens[lo:hi]).numpy(), dtype)
    assert r.error_word() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["tiles", "recurrent"])
def test_pages_and_slots_used_again(built, name, dtype):
    """Freed pages and slots hold another request's rows and state; nothing of them may show."""
    cfg, w, tokens, ref = built(name, 150)
    r = runner_of(cfg, w, dtype, 192, max_seqs=2, shuffle_pages=7)
    rng = np.random.default_rng(4)
    for trial in range(3):
        s = r.open()
        feed(r, s, rng.integers(0, cfg["vocab"], 90 + 31 * trial).tolist(), [50, 1, 40])
        r.close(s)
        s = r.open()
        check(feed(r, s, tokens, [[70, 2, 1, 30], [1], [10000]][trial]), ref, dtype)
        r.close(s)
    assert r.arena.stats()["pages_free"] == r.arena.num_pages


def test_what_is_past_every_window_is_forgotten(built):
    """Only the recurrent layers remember beyond the windows: without them a far token changes nothing, with them it does."""
    cfg = dict(cases.tiles())
    w = plain.random_weights(cfg, 11)
    rng = np.random.default_rng(1)
    a = rng.integers(0, cfg["vocab"], 400).tolist()
    b = [(a[0] + 1) % cfg["vocab"]] + a[1:]
    for layers, same in (([cfg["layers"][0], cfg["layers"][2]], True), (cfg["layers"], False)):
        c = dict(cfg, layers=layers)
        own = dict(w)
        if same:  # the second layer's tensors under its new number
            own.update({"l1" + k[2:]: t for k, t in w.items() if k.startswith("l2.")})
        r = runner_of(c, own, torch.float32, 512)
        la = feed(r, r.open(), a, [300, 1])
        r = runner_of(c, own, torch.float32, 512)
        lb = feed(r, r.open(), b, [300, 1])
        reach = 70 + 65 - 2  # a layer of window n hands a token on by n - 1 places
        assert not np.array_equal(la[reach], lb[reach])
        assert np.array_equal(la[reach + 1:], lb[reach + 1:]) == same


def test_cache_overflow_is_an_error(built):
    cfg, w, tokens, _ = built("odd", 150)
    r = runner_of(cfg, w, torch.float32, 64)
    s = r.open()
    with pytest.raises(RuntimeError):
        r.step([(s, (tokens * 2)[:200], [])])


@pytest.mark.parametrize("name", ["odd", "recurrent"])
def test_greedy_generation(built, name):
    """The scheduler's tokens (portions of prompts beside decoding, then graph replays) are the plain ones."""
    from axono_b200.serving import generate

    cfg, w, tokens, _ = built(name, 150)
    wd = {k: v.double() for k, v in w.items()}
    prompts = [tokens[:5], tokens[20:90], tokens[7:8], tokens[60:75]]
    want = [plain.greedy(cfg, wd, p, 12) for p in prompts]
    for kw in (dict(token_budget=16), dict(token_budget=4096), dict(token_budget=4096, use_graphs=False)):
        r = runner_of(cfg, w, torch.float32, 384, max_seqs=3, max_seq_len=128, shuffle_pages=2)
        assert generate(r, prompts, 12, **kw) == want
        assert r.error_word() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_by_graph(built, dtype):
    """Hundreds of tokens decoded by one captured graph, over page and window borders, against the whole sequence at
    once; capturing runs a step of its own, which must leave no trace in the recurrent state."""
    from axono_b200.serving import DecodeGraph

    cfg, w, tokens, _ = built("tiles", 150)
    r = runner_of(cfg, w, dtype, 1024, max_seqs=3, max_seq_len=512, shuffle_pages=9)
    r.open()  # a slot that stays idle
    seqs = [r.open(), r.open()]
    outs = [tokens[:30], tokens[:61]]
    first = []
    for s, t in zip(seqs, outs):
        first.append(int(torch.argmax(r.step([(s, t, [len(t) - 1])]))))
    g = DecodeGraph(r, seqs, first, [400, 400])
    got = [[f] for f in first]
    for _ in range(300):
        for o, t in zip(got, g.step().tolist()):
            o.append(t)
    assert r.error_word() == 0
    for s, prompt, out in zip(seqs, outs, got):
        fresh = runner_of(cfg, w, dtype, 512)
        logits = fresh.step([(fresh.open(), prompt + out[:-1], list(range(len(prompt) - 1, len(prompt) + len(out) - 1)))])
        # a tie within rounding may go either way: the decoded token must be (nearly) the largest logit
        gap = max(float(logits[i].max() - logits[i, t]) for i, t in enumerate(out)) / float(logits.std())
        assert gap <= (2e-4 if dtype == torch.float32 else 0.3), gap


def test_command_lines_on_a_model_folder(built, tmp_path):
    """A folder with config.json and model.safetensors through the generation command line and the trace runner."""
    cfg, w, tokens, ref = built("odd", 150)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    wd = {k: v.double() for k, v in w.items()}
    prompts = [tokens[:6], tokens[40:61]]
    cmd = [sys.executable, "-m", "axono_b200.generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new", "8"]
    for p in prompts:
        cmd += ["--tokens", ",".join(map(str, p))]
    out = subprocess.run(cmd, capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert out.returncode == 0, out.stderr
    assert [[int(t) for t in line.split()] for line in out.stdout.splitlines()] == [plain.greedy(cfg, wd, p, 8) for p in prompts]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:31], "want": [0, 30]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[31:33], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[33:80], "want": [46]}, {"id": "b", "tokens": tokens[:1], "want": [0]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": tokens[:2], "want": [1]}], "end": ["a"]}]
    out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                          "--max-tokens", "160"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr
    assert [line for line in out.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(4)]
    for step, places in ((0, [0, 30]), (2, [79, 0]), (3, [1])):
        got = np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(places), cfg["vocab"])
        check(got, ref[places], torch.float32)
    assert not (tmp_path / "1.f32").exists()
