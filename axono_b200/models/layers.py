"""Layers that decoder models are put together from.  Each holds its weights in the form its kernels read
and its constants as parameters; none knows a model's configuration format.

`Rows` is what a step tells the layers about its rows: one row is one token of one sequence.  The first
`latent` rows (decoded tokens, short portions) go through attention row by row against the cache; the rest
are `segments`, portions of one sequence each that are long enough for the expanded form.
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


class LatentAttention:
    """Multi-head attention over a cached latent per token (and one rotated key part shared by the heads).

    Queries come from h directly (`wq`) or through a normed latent of their own (`wdq`, `dq_norm`, `wuq`).
    With `wdkv` None the layer has no latent of its own and reads the cache layer it is given."""

    def __init__(self, heads, dim, rot_dim, vdim, kv_rank, scale, rot_base, rot_pairs, eps, wuk, wuv, wo, cache_layer,
                 wq=None, wdq=None, dq_norm=None, wuq=None, wdkv=None, dkv_norm=None):
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

    def forward(self, h, rows: Rows, pages) -> torch.Tensor:
        n = h.shape[0]
        proj = ops.linear(h, self.w_in)
        head = proj[:, :self.q_cols]
        dkv = proj[:, self.q_cols:] if self.has_latent else None
        if self.low_rank_q:
            cq = ops.latent_prepare(rows, self.inv_freq, self.rot_dim, dq=head, dq_weight=self.dq_norm, dkv=dkv,
                                    dkv_weight=self.dkv_norm, pages=pages if self.has_latent else None, eps=self.eps)
            q = ops.linear(cq, self.wuq)
            ops.latent_prepare(rows, self.inv_freq, self.rot_dim, q=q, heads=self.heads, dim=self.dim)
        else:
            q = head
            ops.latent_prepare(rows, self.inv_freq, self.rot_dim, q=q, heads=self.heads, dim=self.dim, dkv=dkv,
                               dkv_weight=self.dkv_norm, pages=pages if self.has_latent else None, eps=self.eps)
        m = rows.latent
        if not rows.segments:
            return ops.linear(self._latent_form(q, rows, pages, m), self.wo)
        parts = [self._latent_form(q, rows, pages, m)] if m else []
        parts += [self._expanded_form(q[r0:r0 + k], rows, pages, seq, start) for seq, r0, k, start in rows.segments]
        return ops.linear(parts[0] if len(parts) == 1 else torch.cat(parts), self.wo)

    def _latent_form(self, q, rows, pages, m):
        per = self.dim + self.rot_dim
        q_lat = torch.empty((m, self.heads, self.kv_rank), dtype=q.dtype, device=q.device)
        ops.linear_heads(q, q.stride(0), per, self.wuk, q_lat, m, in_major=True)
        o_lat = ops.latent_attend(q_lat, q, self.dim, self.rot_dim, self.scale, pages, rows, m)
        o = torch.empty((m, self.heads, self.vdim), dtype=q.dtype, device=q.device)
        ops.linear_heads(o_lat, self.heads * self.kv_rank, self.kv_rank, self.wuv, o, m, in_major=False)
        return o.view(m, self.heads * self.vdim)

    def _expanded_form(self, q, rows, pages, seq, start):
        cached = ops.latent_gather(pages, rows.block_table[seq], start + q.shape[0])
        c = cached[:, :self.kv_rank]
        k = ops.linear(c, self.wuk.view(-1, self.kv_rank))
        v = ops.linear(c, self.wuv.view(-1, self.kv_rank))
        return ops.latent_prefill(q, start, k, v, cached[:, self.kv_rank:], self.heads, self.dim, self.rot_dim, self.vdim,
                                  self.scale)


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
