"""Layers that decoder models are put together from.  Each holds its weights in the form its kernels read
and its constants as parameters; none knows a model's configuration format.

`Rows` is what a step tells the layers about its rows: one row is one token of one sequence, a sequence's rows stand
together, sequences come in order of how many rows they bring.  For attention, the first `latent` rows (decoded
tokens, short portions) go row by row against the cache; the rest are `segments`, portions of one sequence each that
are long enough for the expanded form.  For recurrent mixers, the first `singles` rows are one token each of different
sequences, the rest `portions`.

`Cache` is what is kept for live sequences: pools of pages for what grows with them, and per-slot state for what
does not.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional, Tuple

import torch

from .. import ops


@dataclass
class Rows:
    seq: torch.Tensor          # int32 (rows): row of the block table
    pos: torch.Tensor          # int32 (rows): position in the sequence
    block_table: torch.Tensor  # int32 (max_seqs, max_blocks)
    max_len: int               # host bound of pos + 1
    latent: int                # rows [0, latent) attend through the cache
    segments: List[Tuple[int, int, int, int]] = field(default_factory=list)  # (sequence, first row, rows, start position)
    singles: int = 0
    back: Optional[torch.Tensor] = None      # int32 (rows): how many rows directly before are the same sequence's
    portions: List[Tuple[int, int, int, int]] = field(default_factory=list)  # like segments, all that are no singles
    portion_table: Optional[torch.Tensor] = None  # the portions as int32 (count, 4) on the device


@dataclass
class Cache:
    pages: List[torch.Tensor]               # per cache layer (num_pages, page_tokens, row elements)
    states: List[Tuple[torch.Tensor, ...]]  # per state layer: tensors (max_seqs, ...)


class LatentAttention:
    """Multi-head attention over a cached latent per token (and, with rot_dim, one rotated key part shared by the heads).

    Queries come from h directly (`wq`) or through a normed latent of their own (`wdq`, `dq_norm`, `wuq`).
    With `wdkv` None the layer has no latent of its own and reads the cache layer it is given.  window: how many tokens a
    row sees, itself included (0: all before it); sink: a logit per head that joins the softmax's denominator."""

    def __init__(self, heads, dim, rot_dim, vdim, kv_rank, scale, rot_base, rot_pairs, eps, wuk, wuv, wo, cache_layer,
                 wq=None, wdq=None, dq_norm=None, wuq=None, wdkv=None, dkv_norm=None, window=0, sink=None):
        self.window, self.sink = window, sink.float().contiguous() if sink is not None else None
        self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank = heads, dim, rot_dim, vdim, kv_rank
        self.scale, self.eps, self.cache_layer = float(scale), eps, cache_layer
        self.q_elems = heads * (dim + rot_dim)
        # frequencies in double: the kernels form and reduce the angle before they go to fp32
        self.inv_freq = torch.tensor([float(rot_base) ** (-i / rot_pairs) for i in range(rot_pairs)], dtype=torch.float64,
                                     device=wo.device)
        self.low_rank_q = wdq is not None
        first = wdq if self.low_rank_q else wq
        self.q_cols = first.shape[0]
        # everything that reads h is one product
        self.w_in = torch.cat([first, wdkv]).contiguous() if wdkv is not None else first.contiguous()
        self.has_latent = wdkv is not None
        self.dq_norm, self.wuq, self.dkv_norm = dq_norm, wuq, dkv_norm
        self.wuk = wuk.reshape(heads, dim, kv_rank).contiguous()
        self.wuv = wuv.reshape(heads, vdim, kv_rank).contiguous()
        self.wo = wo.contiguous()
        self.expandable = ops.latent_prefill_supported(heads, dim, rot_dim, vdim, wo.dtype) and kv_rank % 8 == 0 and scale > 0
        # a portion of n rows pays the expansion of every cached token once, (dim + vdim) * kv_rank products per
        # token and head, and saves the difference of the two forms' products per key, head and row
        saved = 2 * kv_rank - dim - vdim
        self.expand_from = max(64, -(-(dim + vdim) * kv_rank // saved)) if saved > 0 else 1 << 62

    def takes_segment(self, n: int) -> bool:
        return self.expandable and n >= self.expand_from

    def forward(self, h, rows: Rows, cache: Cache) -> torch.Tensor:
        pages = cache.pages[self.cache_layer]
        proj = ops.linear(h, self.w_in)
        head = proj[:, :self.q_cols]
        dkv = proj[:, self.q_cols:] if self.has_latent else None
        if self.low_rank_q:
            cq = ops.latent_prepare(rows, self.inv_freq, self.rot_dim, dq=head, dq_weight=self.dq_norm, dkv=dkv,
                                    dkv_weight=self.dkv_norm, pages=pages if self.has_latent else None, eps=self.eps)
            q = ops.linear(cq, self.wuq)
            if self.rot_dim:
                ops.latent_prepare(rows, self.inv_freq, self.rot_dim, q=q, heads=self.heads, dim=self.dim)
        elif self.rot_dim == 0:
            q = head
            if self.has_latent:
                ops.latent_prepare(rows, self.inv_freq, 0, dkv=dkv, dkv_weight=self.dkv_norm, pages=pages, eps=self.eps)
        else:
            q = head
            ops.latent_prepare(rows, self.inv_freq, self.rot_dim, q=q, heads=self.heads, dim=self.dim, dkv=dkv,
                               dkv_weight=self.dkv_norm, pages=pages if self.has_latent else None, eps=self.eps)
        return ops.linear(_by_form(self, q, rows, pages), self.wo)

    def _latent_form(self, q, rows, pages, m):
        per = self.dim + self.rot_dim
        q_lat = torch.empty((m, self.heads, self.kv_rank), dtype=q.dtype, device=q.device)
        ops.linear_heads(q, q.stride(0), per, self.wuk, q_lat, m, in_major=True)
        o_lat = ops.latent_attend(q_lat, q if self.rot_dim else None, self.dim, self.rot_dim, self.scale, pages, rows, m,
                                  self.window, self.sink)
        o = torch.empty((m, self.heads, self.vdim), dtype=q.dtype, device=q.device)
        ops.linear_heads(o_lat, self.heads * self.kv_rank, self.kv_rank, self.wuv, o, m, in_major=False)
        return o.view(m, self.heads * self.vdim)

    def _expanded_form(self, q, rows, pages, seq, start):
        first = _first_key(start, self.window)
        cached = ops.latent_gather(pages, rows.block_table[seq], start + q.shape[0] - first, first)
        c = cached[:, :self.kv_rank]
        k = ops.linear(c, self.wuk.view(-1, self.kv_rank))
        v = ops.linear(c, self.wuv.view(-1, self.kv_rank))
        return ops.latent_prefill(q, start - first, k, v, cached[:, self.kv_rank:] if self.rot_dim else None, self.heads, self.dim,
                                  self.rot_dim, self.vdim, self.scale, self.window, self.sink)


def _first_key(start, window):
    """The first position that rows from `start` on see, rounded down to a tile of the expanded form."""
    return max(0, start - window + 1) // 128 * 128 if window else 0


def _by_form(mixer, q, rows: Rows, pages):
    """Attention of the step's rows, each in the form its entry goes through."""
    m = rows.latent
    parts = [mixer._latent_form(q, rows, pages, m)] if m or not rows.segments else []
    parts += [mixer._expanded_form(q[r0:r0 + k], rows, pages, seq, start) for seq, r0, k, start in rows.segments]
    return parts[0] if len(parts) == 1 else torch.cat(parts)


class SharedKVAttention:
    """Grouped attention whose values are the keys as projected, with RMS norms over the whole query and key projection
    (plain weights; the value is not normed) and no rotation.  The cache holds the raw keys and one factor per token, so
    a row is read once for both uses.  window as in `LatentAttention`."""

    def __init__(self, heads, kv_heads, dim, scale, eps, wq, wk, q_norm, k_norm, wo, cache_layer, window=0):
        self.heads, self.kv_heads, self.dim, self.scale, self.eps = heads, kv_heads, dim, float(scale), eps
        self.window, self.cache_layer = window, cache_layer
        self.w_in = _padded_rows(torch.cat([wq, wk]))
        self.q_norm, self.k_norm, self.wo = q_norm, k_norm, wo
        self.row_elems = ops.shared_kv_row(kv_heads, dim, wo.dtype)
        self.expandable = ops.latent_prefill_supported(heads, dim, 0, dim, wo.dtype) and scale > 0

    def takes_segment(self, n: int) -> bool:
        return self.expandable and n >= 64

    def forward(self, h, rows: Rows, cache: Cache) -> torch.Tensor:
        pages, nq, nk = cache.pages[self.cache_layer], self.heads * self.dim, self.kv_heads * self.dim
        proj = ops.linear(h, self.w_in)
        q = ops.shared_kv_prepare(proj[:, :nq], self.q_norm, proj[:, nq:nq + nk], self.k_norm, pages, rows, self.heads,
                                  self.kv_heads, self.dim, self.eps)
        return ops.linear(_by_form(self, q, rows, pages), self.wo)

    def _latent_form(self, q, rows, pages, m):
        return ops.latent_attend(q[:m], None, self.dim, 0, self.scale, pages, rows, m, self.window, None, self.kv_heads,
                                 True).view(m, -1)

    def _expanded_form(self, q, rows, pages, seq, start):
        first = _first_key(start, self.window)
        k, v = ops.shared_kv_gather(pages, rows.block_table[seq], first, start + q.shape[0] - first, self.kv_heads, self.dim)
        return ops.latent_prefill(q.view(q.shape[0], -1), start - first, k, v, None, self.heads, self.dim, 0, self.dim, self.scale,
                                  self.window, None, self.kv_heads)


class GatedDelta:
    """The gated delta rule: short convolutions, unit queries and keys, a decaying matrix per head as fp32 state, a normed
    and gated output.  conv_* (channels, taps) with the current token's tap last."""

    def __init__(self, heads, kv_heads, dim, vdim, eps, wq, wk, wv, wg, wa, wb, conv_q, conv_k, conv_v, a_log, dt_bias, norm, wo,
                 state_layer):
        self.heads, self.kv_heads, self.dim, self.vdim, self.eps, self.state_layer = heads, kv_heads, dim, vdim, eps, state_layer
        self.w_in = _padded_rows(torch.cat([wq, wk, wv, wg, wa, wb]))  # everything that reads h is one product
        self.conv = torch.cat([conv_q, conv_k, conv_v]).float().t().contiguous()
        self.a_log, self.dt_bias = a_log.float().contiguous(), dt_bias.float().contiguous()
        self.norm, self.wo = norm, wo
        # from how many rows on a portion goes through the tensor-core form
        self.chunk_from = 24 if ops.delta_chunks_supported(dim, vdim, wo.dtype) else 1 << 62

    def state_shapes(self, dtype):
        """What one sequence keeps: (shape, dtype) of the matrices and of the convolution's last inputs."""
        return ((self.heads, self.dim, self.vdim), torch.float32), (tuple(self.conv.shape), dtype)

    def forward(self, h, rows: Rows, cache: Cache) -> torch.Tensor:
        return ops.linear(self.recur(ops.linear(h, self.w_in), rows, *cache.states[self.state_layer]), self.wo)

    def recur(self, proj, rows: Rows, state, ring) -> torch.Tensor:
        """Everything between the two products: proj (rows, >= columns of w_in) -> (rows, heads * vdim)."""
        n, m = proj.shape[0], rows.singles
        out = torch.empty((n, self.heads * self.vdim), dtype=proj.dtype, device=proj.device)
        if m:
            ops.delta_step(self, proj, rows, m, state, ring, out)
        if m < n:
            short = sum(p[2] < self.chunk_from for p in rows.portions)  # portions come by length
            c = rows.portions[short][1] if short < len(rows.portions) else n
            if short:
                qk, v, log_g, beta = ops.delta_prepare(self, proj[:c], rows, m, state, ring)
                ops.delta_scan(self, rows.portion_table[:short], m, qk, v, log_g, beta, state, out[m:c])
            if c < n:
                ops.delta_chunks(self, proj, rows.portion_table[short:], rows.portions[-1][2], c, state, ring, out[c:])
            ops.delta_finish(self, proj, rows, m, state, ring, out[m:], out[m:])
        return out


class GatedMLP:
    """W_down (silu(W_gate h) * (W_up h))."""

    def __init__(self, gate, up, down):
        self.gate_up, self.down = torch.cat([gate, up]).contiguous(), down.contiguous()

    def forward(self, h) -> torch.Tensor:
        return ops.linear(ops.silu_mul_rows(ops.linear(h, self.gate_up), self.down.shape[1]), self.down)


def _padded_rows(w):
    """w with rows of zeros up to a multiple of 8, so that the product's rows start aligned."""
    pad = -w.shape[0] % 8
    return torch.cat([w, w.new_zeros((pad, w.shape[1]))]).contiguous() if pad else w.contiguous()


class GroupedSigmoidRouter:
    """fp32 router: sigmoid scores, a correction that takes part in the choice only, expert groups of which the
    best `keep` stay open, `top` experts per token weighted by score * scale."""

    def __init__(self, weight, correction, groups, keep, top, scale):
        self.weight, self.correction = weight.contiguous(), correction
        self.groups, self.keep, self.top, self.scale = groups, keep, top, scale

    def forward(self, h):
        return ops.moe_route(ops.linear(h, self.weight, out_dtype=torch.float32), self.correction, self.groups, self.keep,
                             self.top, self.scale)


class MixtureOfExperts:
    """Routed experts and one shared expert, all of the clamped-gate form.  gate_up (experts, 2, ff, width), down
    (experts, width, ff); shared: the same with one expert."""

    def __init__(self, router, gate_up, down, limit, shared_gate_up: Optional[torch.Tensor], shared_down, shared_limit,
                 slope=1.702, offset=1.0):
        self.router, self.gate_up, self.down, self.limit = router, gate_up, down, limit
        self.shared_gate_up, self.shared_down, self.shared_limit = shared_gate_up, shared_down, shared_limit
        self.slope, self.offset = slope, offset

    def forward(self, h):
        """-> (rows, slot, weight) for `ops.residual_layer_norm`, the shared expert's output (or None)."""
        ids, weights, place, counts = self.router.forward(h)
        experts, _, ff, width = self.gate_up.shape
        tile = ops.moe_tile_rows(h.shape[0] * ids.shape[1], experts, width, ff, h.dtype)
        srt, row_of, _, tiles, n_tiles = ops.moe_sort(h, ids, place, counts, tile)
        has_shared = self.shared_gate_up is not None
        act, shared_act = ops.moe_gate_up(srt, self.gate_up, self.limit, tiles, n_tiles, tile,
                                          (h, self.shared_gate_up, self.shared_limit) if has_shared else None, self.slope,
                                          self.offset)
        y, shared = ops.moe_down(act, self.down, tiles, n_tiles, tile,
                                 (shared_act, self.shared_down) if has_shared else None)
        return (y, row_of, weights), shared
