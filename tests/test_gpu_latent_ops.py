"""Each mechanism of the latent-attention / expert-mixture models alone, on the GPU against plain torch fp64."""
import math

import numpy as np
import pytest
import torch

import plain_nuderax as plain
from lm_helpers import Pages, close, rnd

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def tol(dtype):
    return 3e-6 if dtype == torch.float32 else 1.2e-2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [76, 256, 7168])
def test_residual_layer_norm(dtype, width):
    from axono_b200 import ops

    n, top, slots = 9, 3, 31
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(1)) * 3 + 100  # a mean far from 0
    a, b, er = rnd((n, width), dtype, 2), rnd((n, width), dtype, 3), rnd((slots, width), dtype, 4)
    w1, w2 = rnd((width,), dtype, 5), rnd((width,), dtype, 6)
    slot = torch.randint(0, slots, (n, top), generator=torch.Generator().manual_seed(7), dtype=torch.int32)
    wt = torch.rand(n, top, generator=torch.Generator().manual_seed(8))
    for use in ("all", "none", "one_norm"):
        want = x.double().clone()
        if use != "none":
            want = want + a.double() + b.double() + (wt.double()[:, :, None] * er.double()[slot.long()]).sum(1)
        xd = x.cuda()
        kw = {} if use == "none" else dict(a=a.cuda(), b=b.cuda(), experts=(er.cuda(), slot.cuda(), wt.cuda()))
        h1, h2 = ops.residual_layer_norm(xd, w1.cuda(), None if use == "one_norm" else w2.cuda(), 1e-3, **kw)
        close(xd, want, 1e-6)
        # sharp on x itself; the norms see a spread of 3 around 100 in fp32
        close(h1, plain.layer_norm(want, w1.double(), 1e-3), max(tol(dtype), 3e-5))
        if use == "one_norm":
            assert h2 is None
        else:
            close(h2, plain.layer_norm(want, w2.double(), 1e-3), max(tol(dtype), 3e-5))


@pytest.mark.parametrize("dtype", DTYPES)
def test_embed_layer_norm_and_bad_id(dtype):
    from axono_b200 import ops

    table, w = rnd((50, 76), dtype, 1), rnd((76,), dtype, 2)
    ids = torch.tensor([0, 49, 7, 7], dtype=torch.int64)
    x = ops.embed_layer_norm(ids.cuda(), table.cuda(), w.cuda(), 1e-5)
    assert x.dtype == torch.float32
    close(x, plain.layer_norm(table.double()[ids], w.double(), 1e-5), 3e-6)
    assert ops.last_error() == 0
    ops.embed_layer_norm(torch.tensor([50], device="cuda"), table.cuda(), w.cuda(), 1e-5)
    assert ops.last_error() & 8


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rot,pairs,rank,q_rank", [(3, 20, 12, 4, 44, 36), (16, 128, 64, 32, 512, 1536), (5, 24, 16, 8, 136, 88),
                                                             (7, 8, 64, 20, 264, 2048)])
def test_prepare_norms_rotates_and_appends(heads, dim, rot, pairs, rank, q_rank, dtype):
    from axono_b200 import ops

    base, eps = 700.0, 1e-3
    pos = [0, 1, 63, 64, 65, 5000]
    n = len(pos)
    pages = Pages([6000], rank + rot, dtype)
    rows = pages.rows([0] * n, pos, 6000)
    inv = torch.tensor([base ** (-i / pairs) for i in range(pairs)], dtype=torch.float64).cuda()
    per = dim + rot
    wide = rnd((n, heads * per + q_rank + rank + rot + 8), dtype, 1)  # one matrix, columns side by side
    wd = wide.cuda()
    dq_w, dkv_w = rnd((q_rank,), dtype, 2), rnd((rank,), dtype, 3)
    pool = pages.pool.cuda()
    o = heads * per
    cq = ops.latent_prepare(rows, inv, rot, q=wd[:, :o], heads=heads, dim=dim, dq=wd[:, o:o + q_rank], dq_weight=dq_w.cuda(),
                            dkv=wd[:, o + q_rank:o + q_rank + rank + rot], dkv_weight=dkv_w.cuda(), pages=pool, eps=eps)
    assert ops.last_error() == 0
    p = torch.tensor(pos)
    q = wide[:, :o].double().view(n, heads, per)
    want_q = torch.cat([q[..., :dim], plain.rotate_interleaved(q[..., dim:], p, base, 2 * pairs)], -1)
    close(wd[:, :o].reshape(n, heads, per), want_q, max(tol(dtype) / 2, 1e-6))
    assert torch.equal(wd[:, :o].reshape(n, heads, per)[..., :dim].cpu(), wide[:, :o].view(n, heads, per)[..., :dim])
    assert torch.equal(wd[:, o:].cpu(), wide[:, o:])
    close(cq, plain.rms_norm(wide[:, o:o + q_rank].double(), dq_w.double(), eps), tol(dtype) / 2)
    src = wide[:, o + q_rank:o + q_rank + rank + rot].double()
    want = torch.cat([plain.rms_norm(src[:, :rank], dkv_w.double(), eps),
                      plain.rotate_interleaved(src[:, rank:], p, base, 2 * pairs)], -1)
    got = torch.stack([pool[int(pages.table[0, t // 64]), t % 64] for t in pos])
    close(got, want, tol(dtype) / 2)
    # nothing else was written
    touched = pool.cpu().clone()
    for t in pos:
        touched[int(pages.table[0, t // 64]), t % 64] = pages.pool[int(pages.table[0, t // 64]), t % 64]
    assert torch.equal(touched, pages.pool)


def test_append_without_room_is_reported():
    from axono_b200 import ops

    pages = Pages([64], 12, torch.float32)
    pool = pages.pool.cuda()
    inv = torch.ones(2, dtype=torch.float64, device="cuda")
    for pos, word in ((64, 2), (64 * pages.table.shape[1], 4)):  # a block with no page; beyond the table
        ops.latent_prepare(pages.rows([0], [pos], 256), inv, 4, dkv=torch.ones(1, 12, device="cuda"),
                           dkv_weight=torch.ones(8, device="cuda"), pages=pool)
        assert ops.last_error() == word
    assert torch.equal(pool.cpu(), pages.pool)


def plain_latent(q_lat, q_rot, rows, rank, scale):
    """(heads, rank), (heads, rot), rows (keys, rank + rot) -> (heads, rank)."""
    s = (q_lat @ rows[:, :rank].T + q_rot @ rows[:, rank:].T) * scale
    return torch.softmax(s, -1) @ rows[:, :rank]


SIZES = [(3, 20, 12, 44), (7, 40, 24, 160), (16, 128, 64, 512), (20, 64, 64, 256), (40, 128, 64, 512), (5, 16, 0, 64),
         (128, 128, 64, 512), (16, 96, 32, 384)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rot,rank", SIZES)
def test_attend(heads, dim, rot, rank, dtype):
    """Lengths around every page and tile border; rows of the same sequence at several positions."""
    from axono_b200 import ops

    lens = [1, 2, 63, 64, 65, 128, 129, 700, 1500]
    scale = 1.3 / math.sqrt(rank + rot)
    pages = Pages(lens, rank + rot, dtype, seed=heads)
    ctx = [rnd((n, rank + rot), dtype, 100 + n) for n in lens]
    for s, c in enumerate(ctx):
        pages.put(s, c)
    seq = list(range(len(lens))) + [7, 7, 8, 8, 8]
    pos = [n - 1 for n in lens] + [0, 64, 63, 1023, 1024]
    q_lat, q = rnd((len(seq), heads, rank), dtype, 1), rnd((len(seq), heads * (dim + rot) + 8), dtype, 2)
    out = ops.latent_attend(q_lat.cuda(), q.cuda(), dim, rot, scale, pages.pool.cuda(), pages.rows(seq, pos, max(lens)), len(seq))
    assert ops.last_error() == 0
    qr = q[:, :heads * (dim + rot)].view(len(seq), heads, dim + rot)[..., dim:]
    want = torch.stack([plain_latent(q_lat[i].double(), qr[i].double(), ctx[s][:p + 1].double(), rank, scale)
                        for i, (s, p) in enumerate(zip(seq, pos))])
    for i in range(len(seq)):
        close(out[i], want[i], 2e-6 if dtype == torch.float32 else 1.2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rot,rank", [(3, 20, 12, 44), (16, 128, 64, 512), (24, 64, 64, 256)])
def test_one_far_key_stands_out(heads, dim, rot, rank, dtype):
    """One key of many hundreds carries nearly all the weight, and the key just past the row's position would
    carry more: each must be seen, or not seen, exactly."""
    from axono_b200 import ops

    n = 1300
    pages = Pages([n], rank + rot, dtype, seed=1)
    ctx = rnd((n, rank + rot), dtype, 5, 0.3)
    q_lat, q = rnd((1, heads, rank), dtype, 1), rnd((1, heads * (dim + rot)), dtype, 2)
    # every head gets the same query, so that one key stands out for all of them
    q_lat[:] = q_lat[:, :1]
    qv = q.view(1, heads, dim + rot)
    qv[:] = qv[:, :1]
    direction = torch.cat([q_lat[0, 0], qv[0, 0, dim:]]).double()
    direction /= direction.norm()
    for far in (0, 1, 63, 64, 127, 128, 511, 1000):
        for at in (far, far + 1, 1198):
            if at < far or at + 1 >= n:
                continue
            c = ctx.clone()
            c[far] = (12 * direction).to(dtype)
            c[at + 1] = (40 * direction).to(dtype)  # just outside
            if at + 1 == far:
                continue
            pages.put(0, c)
            got = ops.latent_attend(q_lat.cuda(), q.cuda(), dim, rot, 0.1, pages.pool.cuda(), pages.rows([0], [at], n), 1)
            want = plain_latent(q_lat[0].double(), qv[0, :, dim:].double(), c[:at + 1].double(), rank, 0.1)
            close(got[0], want, 4e-6 if dtype == torch.float32 else 1.2e-2)
    assert ops.last_error() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_gather(dtype):
    from axono_b200 import ops

    for row in (45, 576):
        pages = Pages([5, 200], row, dtype, seed=2)
        ctx = rnd((200, row), dtype, 3)
        pages.put(1, ctx)
        got = ops.latent_gather(pages.pool.cuda(), pages.table[1].cuda(), 197)
        assert torch.equal(got.cpu(), ctx[:197])


@pytest.mark.parametrize("heads,dim,rot,vdim", [(2, 128, 64, 128), (3, 64, 64, 64), (2, 64, 32, 128), (3, 32, 24, 48), (2, 24, 16, 40),
                                                (1, 128, 64, 64), (2, 72, 8, 104)])
def test_prefill_expanded(heads, dim, rot, vdim):
    """Portions at several starts against the plain causal attention; a key just past a row's position, and one
    far before it, stand out."""
    from axono_b200 import ops

    dtype = torch.bfloat16
    if not ops.latent_prefill_supported(heads, dim, rot, vdim, dtype):
        pytest.skip("sizes outside the expanded form")
    scale = 0.9 / math.sqrt(dim + rot)
    for n, start in ((2, 0), (64, 0), (129, 0), (300, 0), (257, 700), (100, 63), (513, 64), (128, 1)):
        skv = start + n
        q, k, v = rnd((n, heads * (dim + rot) + 16), dtype, 1), rnd((skv, heads * dim), dtype, 2), rnd((skv, heads * vdim), dtype, 3)
        cached = rnd((skv, 80 + rot), dtype, 4)
        kr = cached[:, 80:]
        for far in (0, min(65, skv - 1), skv // 2, skv - 1):  # every query points along one key: the row itself may not see past it
            k[far] = (0.15 * q[:, :heads * (dim + rot)].view(n, heads, dim + rot)[..., :dim].double().sum(0)).reshape(-1).to(dtype)
        qd, cd = q.cuda(), cached.cuda()
        got = ops.latent_prefill(qd, start, k.cuda(), v.cuda(), cd[:, 80:], heads, dim, rot, vdim, scale)
        assert ops.last_error() == 0
        qh = q[:, :heads * (dim + rot)].view(n, heads, dim + rot).double()
        s = torch.einsum("nhd,khd->hnk", qh[..., :dim], k.view(skv, heads, dim).double()) + \
            torch.einsum("nhr,kr->hnk", qh[..., dim:], kr.double())
        mask = torch.arange(skv)[None, :] > torch.arange(n)[:, None] + start
        p = torch.softmax((s * scale).masked_fill(mask, -math.inf), -1)
        want = torch.einsum("hnk,khv->nhv", p, v.view(skv, heads, vdim).double()).reshape(n, -1)
        close(got, want, 1.2e-2)


@pytest.mark.parametrize("experts,groups,keep,top", [(10, 2, 1, 4), (6, 3, 2, 3), (64, 1, 1, 6), (256, 8, 4, 8), (5, 5, 3, 2), (4, 1, 1, 4), (40, 4, 4, 1)])
def test_route(experts, groups, keep, top):
    """Choices with corrections down to well below -1, so that open experts have negative choices: a closed
    group must not count as 0."""
    from axono_b200 import ops

    n, scale = 67, 1.9
    logits = torch.randn(n, experts, generator=torch.Generator().manual_seed(experts)) * 2
    for shift in (0.0, -3.0):
        corr = torch.randn(experts, generator=torch.Generator().manual_seed(1)) + shift
        ids, wts, place, counts = (t.cpu() for t in ops.moe_route(logits.cuda(), corr.cuda(), groups, keep, top, scale))
        for t in range(n):
            want, weights = plain.route_token(logits[t].double(), corr.double(), top, groups, keep, scale)
            assert ids[t].tolist() == want
            assert np.allclose(wts[t].numpy(), weights, rtol=1e-5)
        assert counts.tolist() == torch.bincount(ids.flatten().long(), minlength=experts).tolist()
        for e in range(experts):
            assert sorted(place[ids == e].tolist()) == list(range(int(counts[e])))


def test_route_many_rows():
    from axono_b200 import ops

    n, experts = 9601, 64
    logits = torch.randn(n, experts, generator=torch.Generator().manual_seed(1)) * 2
    corr = torch.randn(experts, generator=torch.Generator().manual_seed(2)) - 2
    ids, _, place, counts = (t.cpu() for t in ops.moe_route(logits.cuda(), corr.cuda(), 8, 3, 6, 1.0))
    for t in range(0, n, 37):
        assert ids[t].tolist() == plain.route_token(logits[t].double(), corr.double(), 6, 8, 3, 1.0)[0]
    assert counts.tolist() == torch.bincount(ids.flatten().long(), minlength=experts).tolist()
    for e in range(experts):
        assert sorted(place[ids == e].tolist()) == list(range(int(counts[e])))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff,experts,top,n", [(76, 44, 6, 3, 50), (200, 72, 12, 3, 9), (264, 104, 7, 2, 1), (384, 192, 16, 4, 300),
                                                    (512, 384, 4, 2, 1500), (256, 128, 8, 2, 60), (256, 128, 3, 3, 33), (128, 256, 32, 1, 40)])
def test_experts(dtype, width, ff, experts, top, n):
    """Routed and shared expert products, with gates and ups on both sides of the clamps; some experts get no row."""
    from axono_b200 import ops
    from axono_b200.models.layers import GroupedSigmoidRouter, MixtureOfExperts

    x = rnd((n, width), dtype, 1)
    gu, down = rnd((experts, 2, ff, width), dtype, 2, 1.5 / math.sqrt(width)), rnd((experts, width, ff), dtype, 3, 1 / math.sqrt(ff))
    sff = ff + (4 if n == 9 else 8)  # 4: a shared expert whose size the tensor-core form does not take beside routed ones it does
    sgu, sdown = rnd((1, 2, sff, width), dtype, 4, 1.5 / math.sqrt(width)), rnd((1, width, sff), dtype, 5, 1 / math.sqrt(sff))
    corr = torch.linspace(0, 1, experts)
    corr[0] = -9.0  # never chosen while others are left
    router = GroupedSigmoidRouter(rnd((experts, width), dtype, 6, 0.3 / math.sqrt(width)).cuda(), corr.cuda(), 1, 1, top, 1.5)
    moe = MixtureOfExperts(router, gu.cuda(), down.cuda(), 1.1, sgu.cuda(), sdown.cuda(), 0.7)
    (y, slot, wts), shared = moe.forward(x.cuda())
    ids = ops.moe_route(ops.linear(x.cuda(), router.weight, out_dtype=torch.float32), router.correction, 1, 1, top, 1.5)[0].cpu()
    assert ops.last_error() == 0

    def expert(g_u, d, limit, rows):
        w = {"gate": g_u[0].double(), "up": g_u[1].double(), "down": d.double()}
        return plain.gated_expert(w, "", rows.double(), limit)

    close(shared, expert(sgu[0], sdown[0], 0.7, x), tol(dtype))
    got, want = torch.empty(n, top, width, dtype=torch.float64), torch.empty(n, top, width, dtype=torch.float64)
    rows = y.double().cpu()[slot.cpu().long()]
    for e in range(experts):
        hit = ids == e
        if hit.any():
            at = hit.nonzero()
            want[hit] = expert(gu[e], down[e], 1.1, x[at[:, 0]])
            got[hit] = rows[hit]
    close(got, want, tol(dtype))
    assert sorted(slot.cpu().flatten().tolist()) == list(range(n * top))
