"""Host-side mirror of the reference's operator API for the decode path.

Function names, argument order and meaning, and error behaviour (RuntimeError on a non-OK
status) follow the reference's Python surface:

    gqa_decode_attention(q, k, v)              axono/python/axono/gqa.py:13-33
    silu_mul(gate, up)                         axono/python/axono/fused.py:19-36
    add_rms_norm(x, residual, weight, eps)     axono/python/axono/fused.py:39-44
    rope / rope_thd / rope_with_cos_sin / mrope_cos_sin / concat
                                               axono/python/axono/core/ops/sequence.py
    rms_norm(x, weight, eps=1e-5)              axono/python/axono/core/ops/llm.py:99-109

Tensors are CUDA `torch.Tensor`s: PyTorch supplies device memory and the current stream and
nothing else - every operator is one call into the C ABI (include/axono_b200.h), and there is
no fallback when the library is missing.  Outputs are allocated here, as the reference's
binding allocates them (nanobind_module.cpp:1019).
"""
from __future__ import annotations

import torch

from . import _capi

_DTYPES = {torch.float16: _capi.FLOAT16, torch.float32: _capi.FLOAT32}
_workspaces: dict = {}
_retired: list = []  # outgrown workspaces, never freed (graphs captured earlier may still write to them)
_launches = 0  # operator calls that reached the C ABI (used to tell an empty graph capture)


def launch_count() -> int:
    return _launches


def _call(status: int, op: str) -> None:
    global _launches
    _capi.check(status, op)
    _launches += 1


def _dt(t: torch.Tensor, op: str) -> int:
    if not t.is_cuda:
        raise RuntimeError(f"{op}: expected a CUDA tensor (this package has no CPU path)")
    code = _DTYPES.get(t.dtype)
    if code is None:
        _capi.check(3, op)  # UNSUPPORTED_TYPE
    return code


def _c(t: torch.Tensor) -> torch.Tensor:
    return t if t.is_contiguous() else t.contiguous()


def _stream(t: torch.Tensor) -> int:
    return torch.cuda.current_stream(t.device).cuda_stream


def _ptr(t):
    return None if t is None else t.data_ptr()


def last_error() -> int:
    return int(_capi.lib().axb200_last_error())


def workspace(device, nbytes: int) -> torch.Tensor:
    """Scratch for the decode-attention partials, cached per device and grown on demand.
    Call once with the largest size before capturing a CUDA graph."""
    key = torch.device(device)
    if key.index is None:
        key = torch.device("cuda", torch.cuda.current_device())
    buf = _workspaces.get(key)
    if buf is None or buf.numel() < nbytes:
        if buf is not None:
            # a captured graph may have the old buffer's address baked in: keep it alive for good
            _retired.append(buf)
        buf = torch.empty(max(int(nbytes), 256), dtype=torch.uint8, device=key)
        _workspaces[key] = buf
    return buf


def gqa_workspace_bytes(batch, hq, hkv, d, max_seq_len, dtype=torch.float16) -> int:
    return int(_capi.lib().axb200_gqa_workspace_bytes(batch, hq, hkv, d, int(max_seq_len), _DTYPES[dtype]))


def decode_step_workspace_bytes(batch, hq, hkv, d, max_seq_len, dtype=torch.float16) -> int:
    """Scratch of `decode_step_paged` (the attention partials plus room for a rotated q)."""
    return int(_capi.lib().axb200_decode_step_workspace_bytes(batch, hq, hkv, d, int(max_seq_len), _DTYPES[dtype]))


def gqa_decode_attention(q, k, v):
    """q (1, n_q_heads, head_dim); k/v (seq_len, n_kv_heads, head_dim) -> (1, n_q_heads, head_dim).
    Equals scaled_dot_product_attention(q, k, v, is_causal=False); scale 1/sqrt(head_dim)."""
    op = "gqa_decode_attention"
    dt = _dt(q, op)
    if q.dim() != 3 or k.dim() != 3 or v.dim() != 3:
        _capi.check(3, op)
    if k.dtype != q.dtype or v.dtype != q.dtype:
        _capi.check(3, op)
    sq, hq, d = q.shape
    skv, hkv, dk = k.shape
    if sq != 1:
        _capi.check(1, op)
    if dk != d or tuple(v.shape) != (skv, hkv, d) or hkv == 0 or hq % hkv != 0:
        _capi.check(4, op)
    q, k, v = _c(q), _c(k), _c(v)
    out = torch.empty_like(q)
    lib = _capi.lib()
    ws_bytes = lib.axb200_gqa_workspace_bytes(1, hq, hkv, d, skv, dt)
    ws = workspace(q.device, ws_bytes)
    _call(lib.axb200_gqa_decode(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), hq, hkv, d,
                                      skv, dt, ws.data_ptr(), ws.numel(), _stream(q)), op)
    return out


def gqa_decode_attention_paged(q, k_pages, v_pages, block_table, seq_lens, max_seq_len, out=None, gather=None,
                               window: int = 0, context_parallel=None):
    """Batched decode over a paged cache (extension of the reference op to a batch).
    q (batch, hq, d); k_pages/v_pages (num_pages, hkv, page_tokens, d); block_table int32
    (batch, max_blocks); seq_lens int32 (batch) on the device; max_seq_len a host upper bound.
    gather=(PeerGather, slot): heads are sharded across ranks; the kernel writes this rank's heads into
    every rank's gathered buffer and the full (batch, hq_total, d) tensor of this rank is returned.
    window > 0: each sequence attends only its last `window` tokens.
    context_parallel=(PeerGather(kind="records"), slot): every rank caches a share of each sequence's
    tokens; the ranks exchange un-normalised partials over peer memory and all return the full result."""
    op = "gqa_decode_attention_paged"
    dt = _dt(q, op)
    batch, hq, d = q.shape
    num_pages, hkv, page_tokens, dk = k_pages.shape
    if dk != d or v_pages.shape != k_pages.shape:
        _capi.check(4, op)
    if block_table.dtype != torch.int32 or seq_lens.dtype != torch.int32:
        _capi.check(3, op)
    q = _c(q)
    lib = _capi.lib()
    ws_bytes = lib.axb200_gqa_workspace_bytes(batch, hq, hkv, d, int(max_seq_len), dt)
    ws = workspace(q.device, ws_bytes)
    if gather is not None:
        pg, slot = gather
        if pg.batch != batch or pg.d != d or pg.hq_total != hq * pg.world or pg.dtype != q.dtype:
            _capi.check(4, op)
        _call(lib.axb200_gqa_decode_paged_gather(
            q.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), block_table.data_ptr(), seq_lens.data_ptr(),
            batch, hq, hkv, d, page_tokens, block_table.shape[1], num_pages, int(max_seq_len), dt,
            ws.data_ptr(), ws.numel(), pg.out_ptrs(slot), pg.flag_ptrs, pg.state_ptr, pg.world, pg.rank,
            pg.hq_total, _stream(q)), op)
        return pg.tensor(slot)
    if out is None:
        out = torch.empty_like(q)
    if context_parallel is not None:
        pg, slot = context_parallel
        if pg.kind != "records" or pg.batch != batch or pg.d != d or pg.hq_total != hq:
            _capi.check(4, op)
        _call(lib.axb200_gqa_decode_paged_cp(
            q.data_ptr(), out.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), block_table.data_ptr(),
            seq_lens.data_ptr(), batch, hq, hkv, d, page_tokens, block_table.shape[1], num_pages,
            int(max_seq_len), dt, ws.data_ptr(), ws.numel(), pg.out_ptrs(slot), pg.flag_ptrs, pg.state_ptr,
            pg.world, pg.rank, _stream(q)), op)
        return out
    if window:
        _call(lib.axb200_gqa_decode_paged_window(
            q.data_ptr(), out.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), block_table.data_ptr(),
            seq_lens.data_ptr(), batch, hq, hkv, d, page_tokens, block_table.shape[1], num_pages,
            int(max_seq_len), int(window), dt, ws.data_ptr(), ws.numel(), _stream(q)), op)
        return out
    _call(lib.axb200_gqa_decode_paged(
        q.data_ptr(), out.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), block_table.data_ptr(),
        seq_lens.data_ptr(), batch, hq, hkv, d, page_tokens, block_table.shape[1], num_pages,
        int(max_seq_len), dt, ws.data_ptr(), ws.numel(), _stream(q)), op)
    return out


def kv_append_rope(q, k_new, v_new, k_pages, v_pages, block_table, seq_lens, pos=None, inv_freq=None,
                   theta=10000.0, mrope_section=None, rotate=True, advance=True, slot_delta=0):
    """One decode step's rope(q), rope(k) and cache append in one launch.  q (batch,hq,d) is rotated
    in place; k_new/v_new (batch,hkv,d) land in slot seq_lens[b] + slot_delta; seq_lens advances when
    asked (first layer of a step: slot_delta 0, advance; later layers: slot_delta -1, no advance).
    pos: int64 (batch), or (3,batch) with mrope_section=(t,h,w); None = the cache length."""
    op = "kv_append_rope"
    dt = _dt(k_new, op)
    batch, hkv, d = k_new.shape
    hq = q.shape[1] if q is not None else 0
    num_pages, _, page_tokens, _ = k_pages.shape
    mrope = mrope_section is not None
    h_sec, w_sec = (mrope_section[1], mrope_section[2]) if mrope else (0, 0)
    for t in (q, k_new, v_new):
        if t is not None and not t.is_contiguous():
            raise RuntimeError(f"{op}: tensors must be contiguous (q is updated in place)")
    _call(_capi.lib().axb200_kv_append_rope(
        _ptr(q), k_new.data_ptr(), v_new.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(),
        block_table.data_ptr(), seq_lens.data_ptr(), _ptr(pos), _ptr(inv_freq), float(theta),
        int(rotate), int(mrope), h_sec, w_sec, batch, hq, hkv, d, page_tokens, block_table.shape[1],
        num_pages, dt, int(slot_delta), int(advance), _stream(k_new)), op)
    return q


def decode_step_paged(q, k_new, v_new, k_pages, v_pages, block_table, seq_lens, max_seq_len, out=None, pos=None,
                      inv_freq=None, theta=10000.0, mrope_section=None, rotate=True):
    """One decode step as one operator: rope(q), rope(k_new), append of (k_new, v_new), attention of q over
    the cache including the new token.  q is read, not rotated in place; seq_lens grows by one.  One launch
    where the library's one-launch step applies (fp16, head_dim 64 or 128), else the two kernels.
    max_seq_len bounds the lengths after the append."""
    op = "decode_step_paged"
    dt = _dt(q, op)
    batch, hq, d = q.shape
    hkv = k_new.shape[1]
    num_pages, _, page_tokens, _ = k_pages.shape
    mrope = mrope_section is not None
    h_sec, w_sec = (mrope_section[1], mrope_section[2]) if mrope else (0, 0)
    for t in (q, k_new, v_new):
        if not t.is_contiguous():
            raise RuntimeError(f"{op}: tensors must be contiguous")
    if out is None:
        out = torch.empty_like(q)
    lib = _capi.lib()
    ws = workspace(q.device, lib.axb200_decode_step_workspace_bytes(batch, hq, hkv, d, int(max_seq_len), dt))
    _call(lib.axb200_decode_step_paged(
        q.data_ptr(), k_new.data_ptr(), v_new.data_ptr(), out.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(),
        block_table.data_ptr(), seq_lens.data_ptr(), _ptr(pos), _ptr(inv_freq), float(theta), int(rotate), int(mrope),
        h_sec, w_sec, batch, hq, hkv, d, page_tokens, block_table.shape[1], num_pages, int(max_seq_len), dt,
        ws.data_ptr(), ws.numel(), _stream(q)), op)
    return out


def kv_prefill_write(q, k, v, k_pages, v_pages, block_row, start=0, pos=None, inv_freq=None, theta=10000.0,
                     mrope_section=None, rotate=True):
    """Writes the n tokens k, v (n,hkv,d) of one sequence into its pages at slots start.., rotating k (and
    q (n,hq,d) in place when given) with each token's position: pos int64 (n) / (3,n) / None = start+i."""
    op = "kv_prefill_write"
    dt = _dt(k, op)
    n, hkv, d = k.shape
    num_pages, _, page_tokens, _ = k_pages.shape
    mrope = mrope_section is not None
    h_sec, w_sec = (mrope_section[1], mrope_section[2]) if mrope else (0, 0)
    for t in (q, k, v):
        if t is not None and not t.is_contiguous():
            raise RuntimeError(f"{op}: tensors must be contiguous")
    _call(_capi.lib().axb200_kv_prefill_write(
        _ptr(q), k.data_ptr(), v.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(), block_row.data_ptr(),
        _ptr(pos), _ptr(inv_freq), float(theta), int(rotate), int(mrope), h_sec, w_sec, n,
        q.shape[1] if q is not None else 0, hkv, d, page_tokens, block_row.numel(), num_pages, int(start), dt,
        _stream(k)), op)
    return q


def qkv_norm_rope_append(qkv, n_q_heads, q_norm_weight, k_norm_weight, eps, k_pages, v_pages, block_table, seq_lens,
                         pos=None, inv_freq=None, theta=10000.0, mrope_section=None, rotate=True, advance=True,
                         slot_delta=0):
    """Per-head rms_norm(q), rms_norm(k), rope on both and the cache append, straight from the QKV
    projection output qkv (batch, (hq + 2*hkv) * d) (rows may be strided).  Returns the normed, rotated
    q as a new (batch, hq, d) tensor."""
    op = "qkv_norm_rope_append"
    dt = _dt(qkv, op)
    if qkv.dim() != 2 or qkv.stride(1) != 1:
        _capi.check(4, op)
    num_pages, hkv, page_tokens, d = k_pages.shape
    batch = qkv.shape[0]
    if qkv.shape[1] != (n_q_heads + 2 * hkv) * d:
        _capi.check(4, op)
    for w in (q_norm_weight, k_norm_weight):
        if w is not None and (w.dtype != qkv.dtype or tuple(w.shape) != (d,) or not w.is_contiguous()):
            _capi.check(4, op)
    mrope = mrope_section is not None
    h_sec, w_sec = (mrope_section[1], mrope_section[2]) if mrope else (0, 0)
    q_out = torch.empty((batch, n_q_heads, d), dtype=qkv.dtype, device=qkv.device)
    _call(_capi.lib().axb200_qkv_norm_rope_append(
        qkv.data_ptr(), qkv.stride(0), _ptr(q_norm_weight), _ptr(k_norm_weight), float(eps), q_out.data_ptr(),
        k_pages.data_ptr(), v_pages.data_ptr(), block_table.data_ptr(), seq_lens.data_ptr(), _ptr(pos),
        _ptr(inv_freq), float(theta), int(rotate), int(mrope), h_sec, w_sec, batch, n_q_heads, hkv, d,
        page_tokens, block_table.shape[1], num_pages, dt, int(slot_delta), int(advance), _stream(qkv)), op)
    return q_out


def qkv_decode_step_paged(qkv, n_q_heads, q_norm_weight, k_norm_weight, eps, k_pages, v_pages, block_table, seq_lens,
                          max_seq_len, out=None, pos=None, inv_freq=None, theta=10000.0, mrope_section=None, rotate=True,
                          advance=True, slot_delta=0, gather=None):
    """`qkv_norm_rope_append` followed by `gqa_decode_attention_paged` as one operator (one launch for fp16
    with head_dim 64 / 128): the tower layer's step straight from the QKV projection output qkv
    (batch, (hq + 2*hkv) * d), rows may be strided.  Returns the attention output (batch, hq, d), or with
    gather=(PeerGather, slot) this rank's gathered (batch, hq_total, d)."""
    op = "qkv_decode_step_paged"
    dt = _dt(qkv, op)
    if qkv.dim() != 2 or qkv.stride(1) != 1:
        _capi.check(4, op)
    num_pages, hkv, page_tokens, d = k_pages.shape
    batch = qkv.shape[0]
    if qkv.shape[1] != (n_q_heads + 2 * hkv) * d:
        _capi.check(4, op)
    for w in (q_norm_weight, k_norm_weight):
        if w is not None and (w.dtype != qkv.dtype or tuple(w.shape) != (d,) or not w.is_contiguous()):
            _capi.check(4, op)
    mrope = mrope_section is not None
    h_sec, w_sec = (mrope_section[1], mrope_section[2]) if mrope else (0, 0)
    lib = _capi.lib()
    ws = workspace(qkv.device, lib.axb200_decode_step_workspace_bytes(batch, n_q_heads, hkv, d, int(max_seq_len), dt))
    if gather is not None:
        pg, slot = gather
        if pg.batch != batch or pg.d != d or pg.hq_total != n_q_heads * pg.world or pg.dtype != qkv.dtype:
            _capi.check(4, op)
        peers, out_ptr = (pg.out_ptrs(slot), pg.flag_ptrs, pg.state_ptr, pg.world, pg.rank, pg.hq_total), None
    else:
        if out is None:
            out = torch.empty((batch, n_q_heads, d), dtype=qkv.dtype, device=qkv.device)
        peers, out_ptr = (None, None, None, 0, 0, n_q_heads), out.data_ptr()
    _call(lib.axb200_qkv_decode_step_paged(
        qkv.data_ptr(), qkv.stride(0), _ptr(q_norm_weight), _ptr(k_norm_weight), float(eps), out_ptr, k_pages.data_ptr(),
        v_pages.data_ptr(), block_table.data_ptr(), seq_lens.data_ptr(), _ptr(pos), _ptr(inv_freq), float(theta),
        int(rotate), int(mrope), h_sec, w_sec, batch, n_q_heads, hkv, d, page_tokens, block_table.shape[1], num_pages,
        int(max_seq_len), dt, int(slot_delta), int(advance), ws.data_ptr(), ws.numel(), *peers, _stream(qkv)), op)
    return pg.tensor(slot) if gather is not None else out


def silu_mul_rows(gate_up, n: int):
    """silu(gate) * up for gate = gate_up[:, :n], up = gate_up[:, n:2n] (one fused gate|up projection
    output, rows may be strided) -> (rows, n)."""
    op = "silu_mul_rows"
    dt = _capi.BFLOAT16 if gate_up.is_cuda and gate_up.dtype == torch.bfloat16 else _dt(gate_up, op)
    if gate_up.dim() != 2 or gate_up.stride(1) != 1 or gate_up.shape[1] != 2 * n:
        _capi.check(4, op)
    out = torch.empty((gate_up.shape[0], n), dtype=gate_up.dtype, device=gate_up.device)
    _call(_capi.lib().axb200_silu_mul_rows(gate_up.data_ptr(), gate_up.stride(0), n, gate_up.shape[0],
                                           out.data_ptr(), dt, _stream(gate_up)), op)
    return out


def decode_step_host(q_host, k_new_host, v_new_host, out_host, staging, k_pages, v_pages, block_table, seq_lens,
                     max_seq_len, theta=10000.0, pos=None, inv_freq=None, mrope_section=None, rotate=True):
    """One decode step whose activations live on the host: q/k_new/v_new/out are CPU tensors (pinned for
    asynchronous copies), `staging` = (q_dev, k_dev, v_dev, out_dev) device buffers of the same shapes.
    Copies in, rope + append, paged decode attention, copies out and waits; a single C-ABI call."""
    op = "decode_step_host"
    q_dev, k_dev, v_dev, out_dev = staging
    dt = _dt(q_dev, op)
    for t in (q_host, k_new_host, v_new_host, out_host):
        if t.is_cuda or not t.is_contiguous() or t.dtype != q_dev.dtype:
            _capi.check(1, op)
    batch, hq, d = q_dev.shape
    num_pages, hkv, page_tokens, _ = k_pages.shape
    mrope = mrope_section is not None
    h_sec, w_sec = (mrope_section[1], mrope_section[2]) if mrope else (0, 0)
    lib = _capi.lib()
    ws_bytes = lib.axb200_gqa_workspace_bytes(batch, hq, hkv, d, int(max_seq_len), dt)
    ws = workspace(q_dev.device, ws_bytes)
    _call(lib.axb200_decode_step_host(
        q_host.data_ptr(), k_new_host.data_ptr(), v_new_host.data_ptr(), out_host.data_ptr(), q_dev.data_ptr(),
        k_dev.data_ptr(), v_dev.data_ptr(), out_dev.data_ptr(), k_pages.data_ptr(), v_pages.data_ptr(),
        block_table.data_ptr(), seq_lens.data_ptr(), _ptr(pos), _ptr(inv_freq), float(theta), int(rotate),
        int(mrope), h_sec, w_sec, batch, hq, hkv, d, page_tokens, block_table.shape[1], num_pages,
        int(max_seq_len), dt, ws.data_ptr(), ws.numel(), _stream(q_dev)), op)
    return out_host


def rope(x, pos_ids, theta: float = 10000.0):
    op = "rope"
    dt = _dt(x, op)
    if x.dim() != 3:
        _capi.check(3, op)
    rows, heads, dim = x.shape
    if pos_ids.dtype != torch.int64 or pos_ids.numel() != rows:
        _capi.check(3, op)
    x = _c(x)
    out = torch.empty_like(x)
    _call(_capi.lib().axb200_rope(x.data_ptr(), _c(pos_ids).data_ptr(), float(theta), out.data_ptr(),
                                        rows, heads, dim, dt, _stream(x)), op)
    return out


def rope_thd(x, pos, inv_freq, mrope_section):
    op = "rope_thd"
    dt = _dt(x, op)
    if x.dim() != 3:
        _capi.check(3, op)
    rows, heads, dim = x.shape
    if pos.dtype != torch.int64 or tuple(pos.shape) != (3, rows):
        _capi.check(4, op)
    if inv_freq.dtype != torch.float32 or tuple(inv_freq.shape) != (dim // 2,):
        _capi.check(4, op)
    x = _c(x)
    out = torch.empty_like(x)
    t, h, w = mrope_section
    _call(_capi.lib().axb200_rope_thd(x.data_ptr(), _c(pos).data_ptr(), _c(inv_freq).data_ptr(), t, h, w,
                                            out.data_ptr(), rows, heads, dim, dt, _stream(x)), op)
    return out


def rope_with_cos_sin(x, cos, sin):
    op = "rope_with_cos_sin"
    dt = _dt(x, op)
    rows, heads, dim = x.shape
    if tuple(cos.shape) != (rows, dim) or tuple(sin.shape) != (rows, dim) or cos.dtype != torch.float32:
        _capi.check(4, op)
    x = _c(x)
    out = torch.empty_like(x)
    _call(_capi.lib().axb200_rope_with_cos_sin(x.data_ptr(), _c(cos).data_ptr(), _c(sin).data_ptr(),
                                                     out.data_ptr(), rows, heads, dim, dt, _stream(x)), op)
    return out


def mrope_cos_sin(pos, inv_freq, h_sec: int, w_sec: int):
    op = "mrope_cos_sin"
    if pos.dim() != 2 or pos.shape[0] != 3 or pos.dtype != torch.int64:
        _capi.check(4, op)
    rows, half = pos.shape[1], inv_freq.shape[0]
    cos = torch.empty((rows, 2 * half), dtype=torch.float32, device=pos.device)
    sin = torch.empty_like(cos)
    _call(_capi.lib().axb200_mrope_cos_sin(_c(pos).data_ptr(), _c(inv_freq).data_ptr(), h_sec, w_sec,
                                                 cos.data_ptr(), sin.data_ptr(), rows, half, _stream(pos)), op)
    return cos, sin


def add_rms_norm(x, residual, weight, eps: float = 1e-6):
    """y = x + residual; out = y * rsqrt(mean(y^2) + eps) * weight.  Returns (y, out)."""
    op = "add_rms_norm"
    dt = _dt(x, op)
    if x.shape != residual.shape or x.dtype != residual.dtype:
        _capi.check(4, op)
    hidden = x.shape[-1]
    if weight.dim() != 1 or weight.shape[0] != hidden or weight.dtype != x.dtype:
        _capi.check(4, op)
    x, residual, weight = _c(x), _c(residual), _c(weight)
    y = torch.empty_like(x)
    out = torch.empty_like(x)
    _call(_capi.lib().axb200_add_rms_norm(x.data_ptr(), residual.data_ptr(), weight.data_ptr(), float(eps),
                                                y.data_ptr(), out.data_ptr(), x.numel() // hidden, hidden, dt,
                                                _stream(x)), op)
    return y, out


def silu_mul(gate, up):
    op = "silu_mul"
    dt = _dt(gate, op)
    if gate.shape != up.shape or gate.dtype != up.dtype:
        _capi.check(4, op)
    gate, up = _c(gate), _c(up)
    out = torch.empty_like(gate)
    _call(_capi.lib().axb200_silu_mul(gate.data_ptr(), up.data_ptr(), out.data_ptr(), gate.numel(), dt,
                                            _stream(gate)), op)
    return out


def rms_norm(x, weight, eps: float = 1e-5):
    op = "rms_norm"
    dt = _dt(x, op)
    cols = x.shape[-1]
    has_w = weight is not None and weight.numel() != 0
    if has_w and (weight.dim() != 1 or weight.shape[0] != cols or weight.dtype != x.dtype):
        _capi.check(4, op)
    x = _c(x)
    out = torch.empty_like(x)
    _call(_capi.lib().axb200_rms_norm(x.data_ptr(), _c(weight).data_ptr() if has_w else None, float(eps),
                                            out.data_ptr(), x.numel() // cols, cols, dt, _stream(x)), op)
    return out


def linear_nobias(x, weight):
    """x (rows, in) . weight (out, in)^T -> (rows, out): one cuBLASLt call whose algorithm is timed and
    chosen on the first use of a shape (so call it once eagerly before capturing it)."""
    op = "linear_nobias"
    dt = _dt(x, op)
    if x.dim() != 2 or weight.dim() != 2 or x.shape[1] != weight.shape[1] or weight.dtype != x.dtype:
        _capi.check(4, op)  # SHAPE_MISMATCH
    x, weight = _c(x), _c(weight)
    out = torch.empty((x.shape[0], weight.shape[0]), dtype=x.dtype, device=x.device)
    _call(_capi.lib().axb200_linear_nobias(x.data_ptr(), weight.data_ptr(), out.data_ptr(), x.shape[0], weight.shape[0],
                                           x.shape[1], dt, _stream(x)), op)
    return out


def cast(x, dtype):
    """Tensor.cast_to on the device (src/core/cuda/tensor/kernel.cu:175-193): float16 <-> float32."""
    op = "cast"
    src = _dt(x, op)
    if dtype == x.dtype:
        return x
    if {x.dtype, dtype} != {torch.float16, torch.float32}:
        raise RuntimeError(f"{op}: only float16 <-> float32")
    if not x.is_contiguous():
        raise RuntimeError(f"{op}: tensor must be contiguous")
    out = torch.empty(x.shape, dtype=dtype, device=x.device)
    dst = _DTYPES[dtype]
    _call(_capi.lib().axb200_cast(x.data_ptr(), src, out.data_ptr(), dst, x.numel(), _stream(x)), op)
    return out


def concat(a, b, axis: int):
    op = "concat"
    if a.dim() < 1 or a.dim() != b.dim() or a.dtype != b.dtype:
        _capi.check(1, op)
    nd = a.dim()
    ax = axis + nd if axis < 0 else axis
    if ax < 0 or ax >= nd:
        _capi.check(1, op)
    for i in range(nd):
        if i != ax and a.shape[i] != b.shape[i]:
            _capi.check(4, op)
    a, b = _c(a), _c(b)
    shape = list(a.shape)
    shape[ax] += b.shape[ax]
    out = torch.empty(shape, dtype=a.dtype, device=a.device)
    outer = 1
    for i in range(ax):
        outer *= a.shape[i]
    es = a.element_size()
    a_bytes = (a.numel() // max(outer, 1)) * es
    b_bytes = (b.numel() // max(outer, 1)) * es
    _call(_capi.lib().axb200_concat(a.data_ptr(), b.data_ptr(), out.data_ptr(), outer, a_bytes, b_bytes,
                                          _stream(a)), op)
    return out


def embedding(ids, table):
    """table[ids]: ids int32/int64 of any shape, table (vocab, hidden) -> ids.shape + (hidden,)."""
    op = "embedding"
    dt = _capi.BFLOAT16 if table.is_cuda and table.dtype == torch.bfloat16 else _dt(table, op)
    if table.dim() != 2 or ids.dim() < 1:
        _capi.check(1, op)
    code = {torch.int64: _capi.INT64, torch.int32: _capi.INT32}.get(ids.dtype)
    if code is None:
        _capi.check(3, op)
    ids, table = _c(ids), _c(table)
    out = torch.empty(tuple(ids.shape) + (table.shape[1],), dtype=table.dtype, device=table.device)
    _call(_capi.lib().axb200_embedding(ids.data_ptr(), code, table.data_ptr(), out.data_ptr(), ids.numel(),
                                       table.shape[0], table.shape[1], dt, _stream(table)), op)
    return out


def argmax_last_dim(x):
    """Index of the first maximum along the last dim -> int64 tensor of shape x.shape[:-1]."""
    op = "argmax_last_dim"
    dt = _dt(x, op)
    if x.dim() < 1:
        _capi.check(1, op)
    x = _c(x)
    cols = x.shape[-1]
    out = torch.empty(x.shape[:-1], dtype=torch.int64, device=x.device)
    _call(_capi.lib().axb200_argmax_last_dim(x.data_ptr(), out.data_ptr(), x.numel() // cols, cols, dt, _stream(x)), op)
    return out


def scaled_dot_product_attention(q, k, v, is_causal: bool = False):
    """q (sq, hq, d), k/v (skv, hkv, d) -> (sq, hq, d); with is_causal row t sees keys [0, t]
    (axono/python/axono/core/ops/sequence.py scaled_dot_product_attention of the reference)."""
    op = "scaled_dot_product_attention"
    dt = _dt(q, op)
    if q.dim() != 3 or k.dim() != 3 or v.dim() != 3:
        _capi.check(1, op)
    if k.dtype != q.dtype or v.dtype != q.dtype:
        _capi.check(3, op)
    sq, hq, d = q.shape
    skv, hkv, dk = k.shape
    if dk != d or tuple(v.shape) != (skv, hkv, d) or hkv == 0 or hq % hkv != 0:
        _capi.check(4, op)
    q, k, v = _c(q), _c(k), _c(v)
    out = torch.empty_like(q)
    lib = _capi.lib()
    ws = workspace(q.device, lib.axb200_sdpa_workspace_bytes(sq, hq, hkv, d, skv, dt))
    _call(lib.axb200_sdpa(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), sq, hq, hkv, d, skv,
                          int(bool(is_causal)), dt, ws.data_ptr(), ws.numel(), _stream(q)), op)
    return out


# ---- operators of the language models (fp32 or bf16; residual, scores, norms and routers in fp32) -----------
_LM_DTYPES = {torch.bfloat16: _capi.BFLOAT16, torch.float32: _capi.FLOAT32}


def _lm_dt(t: torch.Tensor, op: str) -> int:
    if not t.is_cuda:
        raise RuntimeError(f"{op}: expected a CUDA tensor (this package has no CPU path)")
    code = _LM_DTYPES.get(t.dtype)
    if code is None:
        _capi.check(3, op)  # UNSUPPORTED_TYPE
    return code


def linear(x, weight, out_dtype=None):
    """x (rows, in), rows may be strided, . weight (out, in)^T -> (rows, out) of out_dtype (x's type or fp32)."""
    op = "linear"
    dt = _lm_dt(x, op)
    if x.dim() != 2 or weight.dim() != 2 or x.shape[1] != weight.shape[1] or weight.dtype != x.dtype or x.stride(1) != 1:
        _capi.check(4, op)
    rows, k = x.shape
    n = weight.shape[0]
    out = torch.empty((rows, n), dtype=out_dtype or x.dtype, device=x.device)
    if rows:
        _call(_capi.lib().axb200_linear_strided(x.data_ptr(), weight.data_ptr(), out.data_ptr(), rows, n, k, x.stride(0),
                                                weight.stride(0), n, 1, 0, 0, 0, 0, dt, _LM_DTYPES[out.dtype], _stream(x)), op)
    return out


def linear_heads(x, x_ld, x_stride, weight, out, rows, in_major):
    """One product per head: out[:, h] (rows, heads, n) = x_h . weight[h]^T, where x_h (rows, k) starts
    h * x_stride elements into x with row stride x_ld; weight (heads, n, k), or (heads, k, n) with in_major."""
    op = "linear_heads"
    dt = _lm_dt(x, op)
    heads, n = out.shape[1], out.shape[2]
    k = weight.shape[1] if in_major else weight.shape[2]
    if weight.shape[0] != heads or weight.shape[2 if in_major else 1] != n or out.dtype != x.dtype:
        _capi.check(4, op)
    if rows:
        _call(_capi.lib().axb200_linear_strided(
            x.data_ptr(), weight.data_ptr(), out.data_ptr(), rows, n, k, x_ld, weight.shape[2], heads * n, heads, x_stride,
            n * k, n, int(in_major), dt, dt, _stream(x)), op)
    return out


def embed_layer_norm(ids, table, weight, eps):
    """layer_norm(table[ids]) * weight as the fp32 residual stream (n, width)."""
    op = "embed_layer_norm"
    dt = _lm_dt(table, op)
    if ids.dtype != torch.int64 or weight.dtype != table.dtype:
        _capi.check(3, op)
    x = torch.empty((ids.numel(), table.shape[1]), dtype=torch.float32, device=table.device)
    _call(_capi.lib().axb200_embed_layer_norm(ids.data_ptr(), table.data_ptr(), weight.data_ptr(), float(eps), x.data_ptr(),
                                              ids.numel(), table.shape[0], table.shape[1], dt, _stream(table)), op)
    return x


def residual_layer_norm(x, w1, w2, eps, a=None, b=None, experts=None):
    """x (rows, width) fp32 += a + b + sum of the routed experts' rows, in place; returns (h1, h2), the layer norm of
    the new x times w1 and w2 (None where the weight is None).  experts = (rows, slot, weight) of `MoE`."""
    op = "residual_layer_norm"
    dt = _lm_dt(w1 if w1 is not None else w2, op)
    dtype = (w1 if w1 is not None else w2).dtype
    for t in (a, b, w2, experts[0] if experts is not None else None):
        if t is not None and (t.dtype != dtype or not t.is_contiguous()):
            _capi.check(3, op)
    h1 = torch.empty(x.shape, dtype=dtype, device=x.device) if w1 is not None else None
    h2 = torch.empty(x.shape, dtype=dtype, device=x.device) if w2 is not None else None
    er, slot, weight = experts if experts is not None else (None, None, None)
    _call(_capi.lib().axb200_residual_layer_norm(
        x.data_ptr(), _ptr(a), _ptr(b), _ptr(er), _ptr(slot), _ptr(weight), slot.shape[1] if slot is not None else 0, _ptr(w1),
        _ptr(h1), _ptr(w2), _ptr(h2), float(eps), x.shape[0], x.shape[1], dt, _stream(x)), op)
    return h1, h2


def embed_residual(ids, table):
    """(x, h): table[ids] as the fp32 residual stream (n, width) and in the table's type (x itself when that is fp32)."""
    op = "embed_residual"
    dt = _lm_dt(table, op)
    if ids.dtype != torch.int64:
        _capi.check(3, op)
    x = torch.empty((ids.numel(), table.shape[1]), dtype=torch.float32, device=table.device)
    h = x if table.dtype == torch.float32 else torch.empty(x.shape, dtype=table.dtype, device=table.device)
    _call(_capi.lib().axb200_embed_residual(ids.data_ptr(), table.data_ptr(), x.data_ptr(), None if h is x else h.data_ptr(),
                                            ids.numel(), table.shape[0], table.shape[1], dt, _stream(table)), op)
    return x, h


def residual_post_norm(x, y, weight, eps, offset=0.0, final=None):
    """x (rows, width) fp32 += rms_norm(y) * (offset + weight), in place; returns x in y's type (x itself when that is
    fp32), or with `final` its rms norm times (offset + final)."""
    op = "residual_post_norm"
    dt = _lm_dt(y, op)
    if x.dtype != torch.float32 or x.shape != y.shape or not y.is_contiguous() or weight.dtype != y.dtype or \
            (final is not None and final.dtype != y.dtype):
        _capi.check(4, op)
    h = x if final is None and y.dtype == torch.float32 else torch.empty(x.shape, dtype=y.dtype, device=y.device)
    _call(_capi.lib().axb200_residual_post_norm(x.data_ptr(), y.data_ptr(), weight.data_ptr(), float(offset), float(eps),
                                                _ptr(final), None if h is x else h.data_ptr(), x.shape[0], x.shape[1], dt,
                                                _stream(y)), op)
    return h


def latent_prepare(rows, inv_freq, rot_dim, q=None, heads=0, dim=0, dq=None, dq_weight=None, dkv=None, dkv_weight=None,
                   pages=None, eps=1e-5):
    """The step's norms, rotation and append of latent attention in one launch; each of q (rows, >= heads *
    (dim + rot_dim)), dq (rows, q_rank) and dkv (rows, kv_rank + rot_dim) is optional and may be a column slice of
    a wider matrix.  q is rotated in place; returns the normed query latent (or None)."""
    op = "latent_prepare"
    ref = next(t for t in (q, dq, dkv) if t is not None)
    dt = _lm_dt(ref, op)
    for t in (q, dq, dkv):
        if t is not None and (t.dim() != 2 or t.stride(1) != 1 or t.dtype != ref.dtype):
            _capi.check(4, op)
    n = ref.shape[0]
    cq = torch.empty((n, dq.shape[1]), dtype=ref.dtype, device=ref.device) if dq is not None else None
    ld = lambda t: t.stride(0) if t is not None else 0  # noqa: E731
    geo = (pages.shape[1], rows.block_table.shape[1], pages.shape[0]) if pages is not None else (1, 1, 1)
    _call(_capi.lib().axb200_latent_prepare(
        _ptr(q), ld(q), heads, dim, _ptr(dq), ld(dq), dq.shape[1] if dq is not None else 0, _ptr(dq_weight), _ptr(cq),
        _ptr(dkv), ld(dkv), dkv.shape[1] - rot_dim if dkv is not None else 0, _ptr(dkv_weight), float(eps), _ptr(pages),
        rows.block_table.data_ptr(), rows.seq.data_ptr(), rows.pos.data_ptr(), inv_freq.data_ptr(), rot_dim,
        inv_freq.numel(), n, *geo, rows.block_table.shape[0], dt, _stream(ref)), op)
    return cq


def latent_attend(q_lat, q, dim, rot_dim, scale, pages, rows, n, window=0, sink=None, kv_heads=1, key_scale=False):
    """Latent attention of the first n rows: q_lat (n, heads, kv_rank), the rotated query parts inside q (strided
    rows of heads x (dim + rot_dim); None without them) -> (n, heads, kv_rank).  window: keys a row sees (0: all); sink
    (heads) fp32: logit in the denominator; kv_heads rows per
    cached token; key_scale: pages end with a factor per token (`shared_kv_prepare`)."""
    op = "latent_attend"
    if sink is not None and (sink.dtype != torch.float32 or sink.numel() != q_lat.shape[1]):
        _capi.check(4, op)
    elems = kv_heads * q_lat.shape[2] + rot_dim + (4 // pages.element_size() if key_scale else 0)
    if not q_lat.is_contiguous() or q_lat.dtype != pages.dtype or pages.shape[2] != elems:
        _capi.check(4, op)
    dt = _lm_dt(q_lat, op)
    heads, rank = q_lat.shape[1], q_lat.shape[2]
    out = torch.empty_like(q_lat)
    lib = _capi.lib()
    ws = workspace(q_lat.device, lib.axb200_latent_attend_workspace_bytes(n, heads // kv_heads, rank, rot_dim, rows.max_len, dt))
    _call(lib.axb200_latent_attend(
        q_lat.data_ptr(), _ptr(q), q.stride(0) if q is not None else 0, dim, out.data_ptr(), pages.data_ptr(),
        rows.block_table.data_ptr(), rows.seq.data_ptr(), rows.pos.data_ptr(), _ptr(sink), n, heads, kv_heads, rank, rot_dim,
        int(key_scale), int(window), float(scale), pages.shape[1], rows.block_table.shape[1], pages.shape[0],
        rows.block_table.shape[0], int(rows.max_len), dt, ws.data_ptr(), ws.numel(), _stream(q_lat)), op)
    return out


def latent_gather(pages, block_row, n, first=0):
    """The n cached rows from position `first` on of the sequence whose block-table row is block_row, contiguous."""
    op = "latent_gather"
    out = torch.empty((n, pages.shape[2]), dtype=pages.dtype, device=pages.device)
    _call(_capi.lib().axb200_latent_gather(pages.data_ptr(), block_row.data_ptr(), out.data_ptr(), int(first), n, pages.shape[2],
                                           pages.shape[1], block_row.numel(), pages.shape[0], _lm_dt(pages, op), _stream(pages)), op)
    return out


def latent_prefill_supported(heads, dim, rot_dim, vdim, dtype) -> bool:
    return bool(_capi.lib().axb200_latent_prefill_supported(heads, dim, rot_dim, vdim, _LM_DTYPES[dtype]))


def latent_prefill(q, start, k, v, rot, heads, dim, rot_dim, vdim, scale, window=0, sink=None, kv_heads=None):
    """Expanded form of one sequence's portion: q (n, >= heads * (dim + rot_dim)) at positions start.., k (start + n,
    kv_heads * dim), v (start + n, kv_heads * vdim), rot (start + n, rot_dim) with strided rows (None without a rotated
    part) -> (n, heads * vdim).  kv_heads defaults to heads; window and sink as in `latent_attend`."""
    op = "latent_prefill"
    dt = _lm_dt(q, op)
    n = q.shape[0]
    kv_heads = kv_heads or heads
    if k.shape != (start + n, kv_heads * dim) or v.shape != (start + n, kv_heads * vdim) or not (k.is_contiguous() and v.is_contiguous()) \
            or (rot is None) != (rot_dim == 0) or (rot is not None and rot.shape[0] != start + n):
        _capi.check(4, op)
    if sink is not None and (sink.dtype != torch.float32 or sink.numel() != heads):
        _capi.check(4, op)
    out = torch.empty((n, heads * vdim), dtype=q.dtype, device=q.device)
    _call(_capi.lib().axb200_latent_prefill(q.data_ptr(), q.stride(0), k.data_ptr(), v.data_ptr(), _ptr(rot),
                                            rot.stride(0) if rot is not None else 0, _ptr(sink), out.data_ptr(), n, int(start),
                                            heads, kv_heads, dim, rot_dim, vdim, int(window), float(scale), dt, _stream(q)), op)
    return out


def shared_kv_row(kv_heads, dim, dtype):
    """Elements a token takes in the cache of raw keys: its rows and its share of the page's factors."""
    return kv_heads * dim + 4 // torch.empty((), dtype=dtype).element_size()


def shared_kv_factors(pages):
    """The factors (num_pages, page_tokens) at the end of each page."""
    per = 4 // pages.element_size()
    return pages.view(pages.shape[0], -1)[:, pages.shape[1] * (pages.shape[2] - per):].view(torch.float32)


def shared_kv_prepare(q, q_weight, k, k_weight, pages, rows, heads, kv_heads, dim, eps):
    """Norms q (rows, heads * dim) over the whole row with both weights folded in -> (rows, heads, dim), and appends the
    raw k (rows, kv_heads * dim) with its factor; both may be column slices of a wider matrix."""
    op = "shared_kv_prepare"
    dt = _lm_dt(q, op)
    n = q.shape[0]
    if k.dtype != q.dtype or k.shape[0] != n or q.stride(1) != 1 or k.stride(1) != 1 or q.shape[1] != heads * dim or \
            k.shape[1] != kv_heads * dim or pages.dtype != q.dtype or pages.shape[2] != shared_kv_row(kv_heads, dim, q.dtype) or q_weight.dtype != q.dtype or k_weight.dtype != q.dtype:
        _capi.check(4, op)
    out = torch.empty((n, heads, dim), dtype=q.dtype, device=q.device)
    _call(_capi.lib().axb200_shared_kv_prepare(
        q.data_ptr(), q.stride(0), q_weight.data_ptr(), out.data_ptr(), k.data_ptr(), k.stride(0), k_weight.data_ptr(), float(eps),
        pages.data_ptr(), rows.block_table.data_ptr(), rows.seq.data_ptr(), rows.pos.data_ptr(), n, heads, kv_heads, dim,
        pages.shape[1], rows.block_table.shape[1], pages.shape[0], rows.block_table.shape[0], dt, _stream(q)), op)
    return out


def shared_kv_gather(pages, block_row, first, n, kv_heads, dim):
    """Cached rows first .. first + n - 1 of a sequence -> normed keys (without their weight), values; (n, kv_heads * dim)."""
    op = "shared_kv_gather"
    keys = torch.empty((n, kv_heads * dim), dtype=pages.dtype, device=pages.device)
    values = torch.empty_like(keys)
    _call(_capi.lib().axb200_shared_kv_gather(
        pages.data_ptr(), block_row.data_ptr(), keys.data_ptr(), values.data_ptr(), int(first), n, kv_heads, dim,
        pages.shape[1], block_row.numel(), pages.shape[0], _lm_dt(pages, op), _stream(pages)), op)
    return keys, values


def _delta_args(m, proj, state, ring):
    """(weights, sizes) shared by the operators of the gated delta rule; m holds conv (taps, channels), a_log, dt_bias, norm
    and the sizes."""
    if state.dtype != torch.float32 or ring.dtype != proj.dtype or proj.stride(1) != 1 or m.norm.dtype != proj.dtype:
        _capi.check(3, "delta")
    if tuple(state.shape[1:]) != (m.heads, m.dim, m.vdim) or tuple(ring.shape) != (state.shape[0],) + tuple(m.conv.shape):
        _capi.check(4, "delta")
    return ((m.conv.data_ptr(), m.a_log.data_ptr(), m.dt_bias.data_ptr(), m.norm.data_ptr(), ring.data_ptr(), state.data_ptr()),
            (m.heads, m.kv_heads, m.dim, m.vdim, m.conv.shape[0], state.shape[0], float(m.eps)))


def delta_step(m, proj, rows, n, state, ring, out):
    """The gated delta rule for the first n rows, tokens of different sequences, into out[:n]."""
    op = "delta_step"
    weights, sizes = _delta_args(m, proj, state, ring)
    _call(_capi.lib().axb200_delta_step(proj.data_ptr(), proj.stride(0), rows.seq.data_ptr(), rows.pos.data_ptr(), n, *weights,
                                        out.data_ptr(), *sizes, _lm_dt(proj, op), _stream(proj)), op)


def delta_prepare(m, proj, rows, first, state, ring):
    """Rows first.. of a step: (qk fp32, v, log_g, beta) of axb200_delta_prepare."""
    op = "delta_prepare"
    weights, sizes = _delta_args(m, proj, state, ring)
    n = proj.shape[0] - first
    f32 = lambda cols: torch.empty((n, cols), dtype=torch.float32, device=proj.device)  # noqa: E731
    qk, log_g, beta = f32(2 * m.kv_heads * m.dim), f32(m.heads), f32(m.heads)
    v = torch.empty((n, m.heads * m.vdim), dtype=proj.dtype, device=proj.device)
    _call(_capi.lib().axb200_delta_prepare(
        proj.data_ptr(), proj.stride(0), rows.seq.data_ptr(), rows.pos.data_ptr(), rows.back.data_ptr(), first, proj.shape[0],
        *weights, qk.data_ptr(), v.data_ptr(), log_g.data_ptr(), beta.data_ptr(), *sizes, _lm_dt(proj, op), _stream(proj)), op)
    return qk, v, log_g, beta


def delta_scan(m, portions, first, qk, v, log_g, beta, state, out):
    """The recurrence of the portions (int32 (count, 4)), token by token, into out (rows - first, heads * vdim)."""
    op = "delta_scan"
    _call(_capi.lib().axb200_delta_scan(
        portions.data_ptr(), portions.shape[0], first, qk.data_ptr(), v.data_ptr(), log_g.data_ptr(), beta.data_ptr(),
        state.data_ptr(), out.data_ptr(), m.heads, m.kv_heads, m.dim, m.vdim, state.shape[0], _lm_dt(v, op), _stream(v)), op)


def delta_chunks_supported(dim, vdim, dtype) -> bool:
    return bool(_capi.lib().axb200_delta_chunks_supported(dim, vdim, _LM_DTYPES[dtype]))


def delta_chunks(m, proj, portions, longest, first, state, ring, out):
    """`delta_prepare` and `delta_scan` of the portions (int32 (count, 4), rows first..) in chunks of 64 tokens, bf16."""
    op = "delta_chunks"
    (conv, a_log, dt_bias, _, ring_ptr, state_ptr), sizes = _delta_args(m, proj, state, ring)
    lib = _capi.lib()
    n = proj.shape[0] - first
    # not the shared workspace: it grows with the prompt
    ws = torch.empty(lib.axb200_delta_chunks_workspace_bytes(n, portions.shape[0], m.heads, m.kv_heads, m.dim, m.vdim),
                     dtype=torch.uint8, device=proj.device)
    _call(lib.axb200_delta_chunks(
        proj.data_ptr(), proj.stride(0), first, proj.shape[0], conv, a_log, dt_bias, ring_ptr, state_ptr, portions.data_ptr(),
        portions.shape[0], int(longest), out.data_ptr(), *sizes[:-1], _lm_dt(proj, op), ws.data_ptr(), ws.numel(), _stream(proj)), op)


def delta_finish(m, proj, rows, first, state, ring, o, out):
    """Norm and gate of the recurrence's output o (rows - first, heads * vdim) into out (may be o), and the ring."""
    op = "delta_finish"
    weights, sizes = _delta_args(m, proj, state, ring)
    _call(_capi.lib().axb200_delta_finish(
        proj.data_ptr(), proj.stride(0), rows.seq.data_ptr(), rows.pos.data_ptr(), rows.back.data_ptr(), first, proj.shape[0],
        *weights, o.data_ptr(), out.data_ptr(), *sizes, _lm_dt(proj, op), _stream(proj)), op)


def moe_route(logits, correction, groups, keep, top, scale):
    """Grouped top-k routing over sigmoid scores: (ids, weights, place, counts) of axb200_moe_route."""
    op = "moe_route"
    n, experts = logits.shape
    ids = torch.empty((n, top), dtype=torch.int32, device=logits.device)
    place = torch.empty_like(ids)
    weights = torch.empty((n, top), dtype=torch.float32, device=logits.device)
    counts = torch.empty((experts,), dtype=torch.int32, device=logits.device)
    if logits.dtype != torch.float32 or (correction is not None and correction.dtype != torch.float32):
        _capi.check(3, op)
    _call(_capi.lib().axb200_moe_route(logits.data_ptr(), _ptr(correction), ids.data_ptr(), weights.data_ptr(), place.data_ptr(),
                                       counts.data_ptr(), n, experts, groups, keep, top, float(scale), _stream(logits)), op)
    return ids, weights, place, counts


def moe_tile_rows(rows, experts, width, ff, dtype) -> int:
    return int(_capi.lib().axb200_moe_tile_rows(rows, experts, width, ff, _LM_DTYPES[dtype]))


def moe_sort(x, ids, place, counts, tile_rows):
    """Rows of x once per chosen expert, in expert order: (sorted, row_of, offsets, tiles, n_tiles)."""
    op = "moe_sort"
    n, top = ids.shape
    experts = counts.numel()
    srt = torch.empty((n * top, x.shape[1]), dtype=x.dtype, device=x.device)
    row_of = torch.empty_like(ids)
    ints = lambda *s: torch.empty(s, dtype=torch.int32, device=x.device)  # noqa: E731
    offsets, tiles, n_tiles = ints(experts + 1), ints(n * top // tile_rows + min(experts, n * top), 4), ints(1)
    _call(_capi.lib().axb200_moe_sort(x.data_ptr(), srt.data_ptr(), ids.data_ptr(), place.data_ptr(), counts.data_ptr(),
                                      row_of.data_ptr(), offsets.data_ptr(), tiles.data_ptr(), n_tiles.data_ptr(), n, experts, top,
                                      tile_rows, x.shape[1], _lm_dt(x, op), _stream(x)), op)
    return srt, row_of, offsets, tiles, n_tiles


def moe_gate_up(x, weight, limit, tiles, n_tiles, tile_rows, shared=None, slope=1.702, offset=1.0):
    """Gate, up and clamped-gate activation of every routed row's expert: weight (experts, 2, ff, width) -> (rows, ff).
    shared = (x, weight (1, 2, ff, width), limit): one more expert over all rows of its x, in the same launch; returns
    (routed, shared) activations."""
    op = "moe_gate_up"
    experts, _, ff, width = weight.shape
    sx, sw, slimit = shared if shared is not None else (None, None, 0.0)
    new = lambda n, f: torch.empty((n, f), dtype=x.dtype, device=x.device)  # noqa: E731
    act, sact = new(x.shape[0], ff), new(sx.shape[0], sw.shape[2]) if sx is not None else None
    _call(_capi.lib().axb200_moe_gate_up(
        x.data_ptr(), weight.data_ptr(), act.data_ptr(), _ptr(tiles), _ptr(n_tiles), x.shape[0], experts, ff, float(limit),
        _ptr(sx), _ptr(sw), _ptr(sact), sx.shape[0] if sx is not None else 0, sw.shape[2] if sw is not None else 0, float(slimit),
        width, tile_rows, float(slope), float(offset), _lm_dt(x, op), _stream(x)), op)
    return act, sact


def moe_down(act, weight, tiles, n_tiles, tile_rows, shared=None):
    """Down product of every routed row's expert: weight (experts, width, ff) -> (rows, width).  shared = (act, weight
    (1, width, ff)) as in `moe_gate_up`; returns (routed, shared)."""
    op = "moe_down"
    experts, width, ff = weight.shape
    sact, sw = shared if shared is not None else (None, None)
    new = lambda n: torch.empty((n, width), dtype=act.dtype, device=act.device)  # noqa: E731
    y, sy = new(act.shape[0]), new(sact.shape[0]) if sact is not None else None
    _call(_capi.lib().axb200_moe_down(
        act.data_ptr(), weight.data_ptr(), y.data_ptr(), _ptr(tiles), _ptr(n_tiles), act.shape[0], experts, ff, _ptr(sact),
        _ptr(sw), _ptr(sy), sact.shape[0] if sact is not None else 0, sw.shape[2] if sw is not None else 0, width, tile_rows,
        _lm_dt(act, op), _stream(act)), op)
    return y, sy
