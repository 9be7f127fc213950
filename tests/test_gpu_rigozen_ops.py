"""Each mechanism of the Rigozen layers alone, on the GPU against plain fp64: norms on outputs, windows and sinks, keys
that are the values, the gated delta rule."""
import math
from types import SimpleNamespace

import pytest
import torch

import plain_rigozen as plain
from lm_helpers import Pages, close, rnd

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def tol(dtype):
    return 3e-6 if dtype == torch.float32 else 1.2e-2


# ---- the residual stream ----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [76, 256, 7168])
def test_residual_post_norm(dtype, width):
    from axono_b200 import ops

    x, y, w, f = rnd((9, width), torch.float32, 1), rnd((9, width), dtype, 2, 7.0), rnd((width,), dtype, 3, 0.3), rnd((width,), dtype, 4, 0.3)
    for offset, eps in ((1.0, 1e-3), (0.0, 30.0)):
        want = x.double() + plain.rms(y.double(), eps) * (offset + w.double())
        xd = x.cuda()
        h = ops.residual_post_norm(xd, y.cuda(), w.cuda(), eps, offset)
        close(xd, want, 1e-6)
        close(h, want, tol(dtype))
        assert h.dtype == dtype
        xd = x.cuda()
        h = ops.residual_post_norm(xd, y.cuda(), w.cuda(), eps, offset, f.cuda())
        close(xd, want, 1e-6)
        close(h, plain.rms(want, eps) * (offset + f.double()), tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
def test_embed_residual_and_bad_id(dtype):
    from axono_b200 import ops

    for width in (76, 256):
        table = rnd((50, width), dtype, 1)
        x, h = ops.embed_residual(torch.tensor([0, 49, 7, 7]).cuda(), table.cuda())
        assert torch.equal(x.cpu(), table[[0, 49, 7, 7]].float()) and torch.equal(h.cpu(), table[[0, 49, 7, 7]])
        assert ops.last_error() == 0
        ops.embed_residual(torch.tensor([-1]).cuda(), table.cuda())
        assert ops.last_error() & 8


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_mlp(dtype):
    from axono_b200.models.layers import GatedMLP

    w = {"gate": rnd((44, 76), dtype, 1, 0.3), "up": rnd((44, 76), dtype, 2, 0.3), "down": rnd((76, 44), dtype, 3, 0.2)}
    h = rnd((13, 76), dtype, 4)
    got = GatedMLP(*(w[k].cuda() for k in ("gate", "up", "down"))).forward(h.cuda())
    close(got, plain.dense({k: t.double() for k, t in w.items()}, "", h.double()), tol(dtype))


# ---- attention over cached rows ----------------------------------------------------------------------------
def plain_rows(q, keys, values, at, scale, window, sink):
    """q (heads, dim), keys and values (heads, tokens, .) -> (heads, .) of the row at position `at`."""
    return torch.stack([plain.attend_row(q[None, h].expand(at + 1, -1), keys[h], values[h], at, scale, window,
                                         None if sink is None else sink[h]) for h in range(q.shape[0])])


LATENT_SIZES = [(3, 44), (7, 160), (16, 512), (20, 256), (40, 512), (5, 64), (130, 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank", LATENT_SIZES)
def test_latent_rows_with_window_and_sink(heads, rank, dtype):
    """Rows around page and tile borders; windows of one token, around tiles, and longer than the sequence; sinks from
    negligible to dominant."""
    from axono_b200 import ops

    lens = [1, 2, 64, 65, 129, 700, 1500]
    scale = 1.3 / math.sqrt(rank)
    pages = Pages(lens, rank, dtype, seed=heads)
    ctx = [rnd((n, rank), dtype, 100 + n) for n in lens]
    for s, c in enumerate(ctx):
        pages.put(s, c)
    seq = list(range(len(lens))) + [5, 5, 6, 6, 6]
    pos = [n - 1 for n in lens] + [63, 64, 65, 1023, 1024]
    q = rnd((len(seq), heads, rank), dtype, 1)
    for window in (1, 2, 63, 64, 65, 128, 200, 1 << 20, 0):
        for sink in (None, torch.linspace(-20, 12, heads)):
            out = ops.latent_attend(q.cuda(), None, 0, 0, scale, pages.pool.cuda(), pages.rows(seq, pos, max(lens)), len(seq), window,
                                    sink.cuda() if sink is not None else None)
            assert ops.last_error() == 0
            for i, (s, at) in enumerate(zip(seq, pos)):
                c = ctx[s].double()[None].expand(heads, -1, -1)
                want = plain_rows(q[i].double(), c, c, at, scale, window, sink.double() if sink is not None else None)
                close(out[i], want, 3e-6 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank", [(3, 44), (16, 512), (24, 256)])
def test_window_edge_of_one_key(heads, rank, dtype):
    """The last key inside the window carries nearly all the weight; then it is the first one outside, and would."""
    from axono_b200 import ops

    n = 900
    base = rnd((n, rank), dtype, 5, 0.3)
    q = rnd((1, 1, rank), dtype, 1).repeat(1, heads, 1)
    direction = q[0, 0].double() / q[0, 0].double().norm()
    for window in (2, 17, 64, 127, 128, 129, 500):
        for at in (window, window + 1, 191, 192, 640, 898):
            if at < window:
                continue
            for edge in (at - window + 1, at - window):
                pages = Pages([n], rank, dtype, seed=2)
                c = base.clone()
                c[edge] = (25 * direction).to(dtype)
                pages.put(0, c)
                got = ops.latent_attend(q.cuda(), None, 0, 0, 0.1, pages.pool.cuda(), pages.rows([0], [at], n), 1, window)
                cd = c.double()[None].expand(heads, -1, -1)
                close(got[0], plain_rows(q[0].double(), cd, cd, at, 0.1, window, None), 4e-6 if dtype == torch.float32 else 1.5e-2)
    assert ops.last_error() == 0


def shared_pages(lens, kv_heads, dim, dtype, seed=0):
    """Pages for rows and factors as shared_kv_prepare leaves them."""
    from axono_b200 import ops

    return Pages(lens, ops.shared_kv_row(kv_heads, dim, dtype), dtype, seed=seed)


SHARED_SIZES = [(6, 3, 20), (10, 1, 48), (12, 2, 40), (32, 4, 128), (8, 8, 64), (40, 1, 128), (4, 2, 9), (64, 2, 256)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim", SHARED_SIZES)
def test_shared_kv_prepare_attend_gather(heads, kv_heads, dim, dtype):
    """Append with norms, then attention by rows, against grouped attention whose values are the raw keys."""
    from axono_b200 import ops

    n, eps, scale = 300, 1e-2, 1.4 / math.sqrt(dim)
    nq, nk = heads * dim, kv_heads * dim
    proj = rnd((n, nq + nk + (-(nq + nk)) % 8), dtype, 1)
    proj[:, nq:nq + nk] *= torch.linspace(0.1, 6, n).to(dtype)[:, None]  # the norm's factor differs from row to row
    qw, kw = rnd((nq,), dtype, 2) + 1, rnd((nk,), dtype, 3) + 1
    pages = shared_pages([n], kv_heads, dim, dtype, seed=dim)
    pool, rows, wd = pages.pool.cuda(), pages.rows([0] * n, list(range(n)), n), proj.cuda()
    q = ops.shared_kv_prepare(wd[:, :nq], qw.cuda(), wd[:, nq:nq + nk], kw.cuda(), pool, rows, heads, kv_heads, dim, eps)
    assert ops.last_error() == 0
    raw = proj[:, nq:nq + nk].double()
    group = heads // kv_heads
    fold = kw.double().view(kv_heads, 1, dim).expand(-1, group, -1).reshape(-1)
    want_q = plain.rms(proj[:, :nq].double(), eps) * qw.double() * fold
    close(q.view(n, -1), want_q, tol(dtype))
    keys, values = ops.shared_kv_gather(pool, rows.block_table[0], 70, 200, kv_heads, dim)
    assert torch.equal(values.cpu(), proj[70:270, nq:nq + nk])
    close(keys, plain.rms(raw, eps)[70:270], tol(dtype))
    k = plain.rms(raw, eps).view(n, kv_heads, dim).transpose(0, 1).repeat_interleave(group, 0)
    v = raw.view(n, kv_heads, dim).transpose(0, 1).repeat_interleave(group, 0)
    qd = q.cpu().double()
    picks = [0, 1, 63, 64, 65, 127, 128, 191, 256, 299]
    for window in (1, 64, 65, 130, 0):
        got = ops.latent_attend(q, None, dim, 0, scale, pool, rows, n, window, None, kv_heads, True).cpu()
        assert ops.last_error() == 0
        for i in picks:
            close(got[i], plain_rows(qd[i], k, v, i, scale, window, None), 4e-6 if dtype == torch.float32 else 1.5e-2)


def test_shared_kv_append_without_room_is_reported():
    from axono_b200 import ops

    pages = shared_pages([64], 1, 8, torch.float32)
    pool, one = pages.pool.cuda(), torch.ones(1, 8, device="cuda")
    for pos, word in ((64, 2), (64 * pages.table.shape[1], 4)):
        ops.shared_kv_prepare(one, one[0], one, one[0], pool, pages.rows([0], [pos], 256), 1, 1, 8, 1e-5)
        assert ops.last_error() == word
    assert torch.equal(pool.cpu(), pages.pool)


@pytest.mark.parametrize("heads,kv_heads,dim,rot,vdim", [(4, 4, 128, 0, 128), (6, 2, 64, 0, 64), (3, 3, 32, 0, 48), (8, 2, 48, 0, 48),
                                                         (2, 2, 72, 8, 104), (4, 4, 40, 0, 128), (2, 1, 128, 0, 64)])
def test_expanded_form_with_window_and_sink(heads, kv_heads, dim, rot, vdim):
    """Portions at several starts; a key just inside and one just outside the window of some row stand out."""
    from axono_b200 import ops

    dtype, scale, group = torch.bfloat16, 1.0 / math.sqrt(dim + rot), heads // kv_heads
    assert ops.latent_prefill_supported(heads, dim, rot, vdim, dtype)
    for n, start, window in ((2, 0, 1), (64, 0, 40), (129, 0, 128), (300, 0, 129), (257, 700, 64), (100, 63, 1000), (513, 64, 200),
                             (513, 640, 1), (400, 128, 0)):
        skv = start + n
        q, k, v = rnd((n, heads * (dim + rot) + 16), dtype, 1), rnd((skv, kv_heads * dim), dtype, 2), rnd((skv, kv_heads * vdim), dtype, 3)
        kr = rnd((skv, rot), dtype, 4) if rot else None
        qh = q[:, :heads * (dim + rot)].view(n, heads, dim + rot)
        for row in (0, n // 2, n - 1):  # a row's first key, and the one before it, point along the row's query
            for far in (start + row - window + 1, start + row - window):
                if 0 <= far < skv and window:
                    k[far] = (3.0 / scale / dim * qh[row, ::group, :dim].double()).reshape(-1).to(dtype)
        for sink in (None, torch.linspace(-9, 9, heads)):
            got = ops.latent_prefill(q.cuda(), start, k.cuda(), v.cuda(), kr.cuda() if rot else None, heads, dim, rot, vdim, scale, window,
                                     sink.cuda() if sink is not None else None, kv_heads)
            assert ops.last_error() == 0
            kd = k.view(skv, kv_heads, dim).double().repeat_interleave(group, 1)
            s = torch.einsum("nhd,khd->hnk", qh[..., :dim].double(), kd)
            if rot:
                s = s + torch.einsum("nhr,kr->hnk", qh[..., dim:].double(), kr.double())
            i, j = torch.arange(n)[:, None] + start, torch.arange(skv)[None, :]
            hidden = (j > i) | ((i - j >= window) if window else False)
            s = (s * scale).masked_fill(hidden, -math.inf)
            if sink is not None:
                s = torch.cat([s, sink.double().view(heads, 1, 1).expand(-1, n, 1)], -1)
            p = torch.softmax(s, -1)[..., :skv]
            want = torch.einsum("hnk,khv->nhv", p, v.view(skv, kv_heads, vdim).double().repeat_interleave(group, 1)).reshape(n, -1)
            close(got, want, 1.5e-2)


# ---- the gated delta rule ----------------------------------------------------------------------------------
class Mixer:
    """Random weights of one mixer, its inputs, and the plain evaluation of a whole sequence."""

    def __init__(self, heads, kv_heads, dim, vdim, taps, dtype, seed=0, decay=-1.5):
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps, self.eps, self.dtype = heads, kv_heads, dim, vdim, taps, 1e-3, dtype
        self.channels = 2 * kv_heads * dim + heads * vdim
        self.cols = self.channels + heads * vdim + 2 * heads
        r = lambda *s, k=0, scale=1.0: rnd(s, dtype, seed * 100 + k, scale)  # noqa: E731
        self.conv = rnd((taps, self.channels), torch.float32, seed * 100 + 1, 0.7)
        self.a_log, self.dt_bias = rnd((heads,), torch.float32, seed * 100 + 2) + decay, rnd((heads,), torch.float32, seed * 100 + 3)
        self.norm = r(vdim, k=4, scale=0.2) + 1

    def weights(self):
        return SimpleNamespace(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, eps=self.eps, conv=self.conv.cuda(),
                               a_log=self.a_log.cuda(), dt_bias=self.dt_bias.cuda(), norm=self.norm.cuda(), chunk_from=self.chunk_from())

    def chunk_from(self):
        from axono_b200 import ops

        return 24 if ops.delta_chunks_supported(self.dim, self.vdim, self.dtype) else 1 << 62

    def inputs(self, n, seed):
        return rnd((n, self.cols + -self.cols % 8), self.dtype, seed)

    def plain(self, proj):
        """(outputs (tokens, heads * vdim), states (heads, dim, vdim)) of a sequence's projections."""
        n, x = proj.shape[0], proj.double()
        qk = self.kv_heads * self.dim
        y = plain.causal_conv(x[:, :self.channels], self.conv.double().T)
        q = plain.unit(y[:, :qk].view(n, self.kv_heads, self.dim)) * self.dim ** -0.5
        k = plain.unit(y[:, qk:2 * qk].view(n, self.kv_heads, self.dim))
        v = y[:, 2 * qk:].view(n, self.heads, self.vdim)
        gate = plain.silu(x[:, self.channels:self.channels + self.heads * self.vdim]).view(n, self.heads, self.vdim)
        ab = x[:, self.channels + self.heads * self.vdim:self.cols]
        g = torch.exp(plain.log_decay(ab[:, :self.heads], self.a_log.double(), self.dt_bias.double()))
        beta = torch.sigmoid(ab[:, self.heads:])
        outs, states = [], []
        for h in range(self.heads):
            src = h // (self.heads // self.kv_heads)
            o, s = plain.delta_rule(q[:, src], k[:, src], v[:, h], g[:, h], beta[:, h])
            outs.append(plain.rms(o, self.eps) * self.norm.double() * gate[:, h])
            states.append(s)
        return torch.cat(outs, -1), torch.stack(states)

    def slots(self, count):
        """State and ring of `count` slots, full of what an earlier sequence might have left."""
        return (torch.full((count, self.heads, self.dim, self.vdim), 1e4, device="cuda"),
                torch.full((count, self.taps, self.channels), 1e3, device="cuda").to(self.dtype))


def run_delta(mixer, w, projs, steps, state, ring):
    """projs[s]: projections of sequence s; steps: lists of how many tokens each brings.  -> outputs per sequence."""
    from axono_b200 import ops
    from axono_b200.models.layers import GatedDelta, Rows

    at, outs = [0] * len(projs), [[] for _ in projs]
    for step in steps:
        order = sorted((i for i in range(len(projs)) if step[i]), key=lambda i: step[i])
        seq, pos, back, portions, rows = [], [], [], [], []
        for i in order:
            n = step[i]
            if n > 1:
                portions.append((i, len(seq), n, at[i]))
            seq += [i] * n
            pos += range(at[i], at[i] + n)
            back += range(n)
            rows.append(projs[i][at[i]:at[i] + n])
        ints = lambda v: torch.tensor(v, dtype=torch.int32).cuda()  # noqa: E731
        r = Rows(ints(seq), ints(pos), ints([[0]]), 1, 0, singles=sum(step[i] == 1 for i in order), back=ints(back), portions=portions,
                 portion_table=ints(portions).view(-1, 4))
        out = GatedDelta.recur(w, torch.cat(rows).cuda(), r, state, ring)
        assert ops.last_error() == 0
        k = 0
        for i in order:
            outs[i].append(out[k:k + step[i]].cpu())
            k, at[i] = k + step[i], at[i] + step[i]
    return [torch.cat(o) for o in outs]


DELTA_SIZES = [(6, 2, 20, 12, 3), (3, 3, 33, 7, 1), (4, 1, 72, 136, 4), (2, 2, 136, 40, 5), (8, 4, 128, 128, 4), (6, 2, 64, 96, 2),
               (5, 5, 32, 56, 4), (2, 1, 256, 256, 3), (3, 1, 16, 300, 7), (4, 2, 32, 64, 6), (9, 1, 64, 16, 4), (10, 2, 100, 8, 5),
               (64, 16, 32, 128, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", DELTA_SIZES)
def test_delta_in_portions_and_tokens(sizes, dtype):
    """Single tokens from the first on, portions of two and more, and whole prompts give the plain sequence and state."""
    mixer = Mixer(*sizes, dtype, seed=sizes[0])
    n = 45
    proj = mixer.inputs(n, 7)
    want, states = mixer.plain(proj)
    t = 2e-5 if dtype == torch.float32 else 2e-2
    for cut in ([1] * n, [n], [2] * 22 + [1], [1, 2, 17, 1, 1, 3, 20], [40, 1, 1, 1, 1, 1], [1, 44]):
        state, ring = mixer.slots(1)
        got, = run_delta(mixer, mixer.weights(), [proj], [[c] for c in cut], state, ring)
        close(got, want, t)
        close(state[0], states, t)
        for p in range(max(0, n - mixer.taps + 1), n):  # the ring holds the inputs as they came
            assert torch.equal(ring[0, p % mixer.taps].cpu(), proj[p, :mixer.channels])


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_unequal_batch_and_slots_used_again(dtype):
    mixer = Mixer(8, 4, 128, 128, 4, dtype, seed=3)
    w, t = mixer.weights(), 2e-5 if dtype == torch.float32 else 2e-2
    state, ring = mixer.slots(5)
    for trial in range(2):
        projs = [mixer.inputs(n, 20 + 5 * trial + i) for i, n in enumerate((60, 9, 131, 3, 1))]
        steps = [[50, 1, 64, 0, 0], [1, 0, 66, 2, 0], [1, 7, 0, 1, 1], [8, 1, 1, 0, 0]]
        for got, proj in zip(run_delta(mixer, w, projs, steps, state, ring), projs):
            close(got, mixer.plain(proj)[0], t)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decay", [-8.0, -1.5, 2.5])
def test_delta_long_memory(dtype, decay):
    """Decays near 1 (the state remembers everything) to near 0, over many chunks' lengths."""
    mixer = Mixer(3, 3, 64, 64, 4, dtype, seed=5, decay=decay)
    proj = mixer.inputs(700, 9)
    want, states = mixer.plain(proj)
    t = 3e-5 if dtype == torch.float32 else 3e-2
    for cut in ([700], [333, 1, 2, 64, 63, 65, 128, 44]):
        state, ring = mixer.slots(1)
        got, = run_delta(mixer, mixer.weights(), [proj], [[c] for c in cut], state, ring)
        close(got, want, t)
        close(state[0], states, t)


def test_delta_unit_norms_of_tiny_vectors_and_large_steps():
    """Inputs near zero (the unit norm's epsilon shows) and gates far on both sides."""
    mixer = Mixer(2, 1, 32, 32, 2, torch.float32, seed=6)
    proj = mixer.inputs(40, 3)
    proj[10:20, :2 * 32] *= 1e-3
    ab = mixer.channels + 2 * 32
    proj[:, ab:ab + 4] = torch.linspace(-40, 40, 40)[:, None]
    want, states = mixer.plain(proj)
    for cut in ([40], [1] * 40):
        state, ring = mixer.slots(1)
        got, = run_delta(mixer, mixer.weights(), [proj], [[c] for c in cut], state, ring)
        close(got, want, 3e-5)
        close(state[0], states, 3e-5)


def test_delta_slot_outside_the_pool_is_reported():
    from axono_b200 import ops
    from axono_b200.models.layers import GatedDelta, Rows

    mixer = Mixer(2, 1, 16, 16, 2, torch.float32)
    state, ring = mixer.slots(1)
    ints = lambda v: torch.tensor(v, dtype=torch.int32).cuda()  # noqa: E731
    GatedDelta.recur(mixer.weights(), mixer.inputs(1, 1).cuda(), Rows(ints([1]), ints([0]), ints([[0]]), 1, 0, singles=1), state, ring)
    assert ops.last_error() == 4
    assert float(state.min()) == 1e4
