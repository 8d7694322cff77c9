"""Latent attention over paged rows ``[c | rotated key part]``, one row a token for all heads (see csrc/attention_latent.cu).

Pages are ``[blocks, 16, 1, Rp]`` in the activation dtype: the normed latent padded to ``Cp`` channels, then the rotated part.
``w_key [H, dqp, Rp]`` makes a head's whole key from a row: W_uk beside an identity for the rotated part, so that the same
weight expands rows into keys (``K = rows w_key^T``) and moves queries into the latent space (``q w_key``).
``w_value [H, dvp, Cp]`` likewise for values."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _native as nv
from .gemm import gemm
from .paged_rows import _split, decode_attention
from .portions import Portions

MAX_EXPANDED_BYTES = 4 << 30     # keys and values of long portions' contexts, made at once


def _turn(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """fp32, pairs of neighbours over the last dimension; one angle per row and pair."""
    u, v = x[..., 0::2].float(), x[..., 1::2].float()
    s = (slice(None),) + (None,) * (x.dim() - 2)
    return torch.stack([u * cos[s] - v * sin[s], v * cos[s] + u * sin[s]], -1).flatten(-2)


def latent_store(q: Optional[torch.Tensor], c: torch.Tensor, kr: torch.Tensor, pages: torch.Tensor, p: Portions, H: int, dim: int,
                 rank: int, rot: int, w: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, eps: float,
                 cq: Optional[torch.Tensor] = None, wq: Optional[torch.Tensor] = None, q_rank: int = 0) -> None:
    """``q [M, H*dqp]``, ``c [M, Cp]``, ``kr [M, Rp - Cp]`` are column slices of one matrix.  The rotated part of every head of
    ``q`` (channels ``dim .. dim + rot - 1``, pairs of neighbours) is turned in place; ``rms(c) w`` and the turned ``kr``
    go to the rows' pages.  ``cq [M, Qp]`` (a slice of the same matrix): the latent that the queries are made from, ``rms(cq) wq``
    over ``q_rank`` channels in place; ``q`` is None then."""
    M, Cp, Rp = c.shape[0], c.shape[1], pages.shape[-1]
    dqp = 0 if q is None else q.shape[1] // H
    if not c.is_cuda:
        def rms(x, g, n):
            x = x.float()
            return x * torch.rsqrt((x * x).sum(-1, keepdim=True) / n + eps) * g.float()
        if q is not None:
            part = q.unflatten(1, (H, dqp))[:, :, dim:dim + rot]
            part.copy_(_turn(part, cos, sin).to(q.dtype))
        if cq is not None:
            cq.copy_(rms(cq, wq, q_rank).to(cq.dtype))
        row = torch.cat([rms(c, w, rank), torch.nn.functional.pad(_turn(kr[:, :rot], cos, sin), (0, Rp - Cp - rot))], 1).to(pages.dtype)
        for r, (s, pos) in enumerate(zip(p.row_seq.tolist(), p.positions.tolist())):
            if int(p.slots[s]) >= 0:
                pages[int(p.block_tables[s, pos // 16]), pos % 16, 0] = row[r]
        return
    assert all(t is None or t.stride(0) == c.stride(0) for t in (q, cq, kr)) and pages.shape[1] == 16
    nv.check(nv.lib().b2_latent_store(
        nv.ptr(q), nv.ptr(cq), nv.ptr(c), nv.ptr(kr), nv.ctypes.c_longlong(c.stride(0)), nv.ptr(pages), nv.ptr(w), nv.ptr(wq),
        nv.ptr(p.block_tables), nv.ptr(p.row_seq), nv.ptr(p.positions), nv.ptr(p.slots), nv.ptr(cos), nv.ptr(sin), M,
        p.block_tables.shape[1], H, dim, dqp, rank, Cp, Rp, rot, q_rank, 0 if cq is None else cq.shape[1], nv.ctypes.c_float(eps),
        int(c.dtype == torch.float32), nv.stream_ptr()), "latent_store")
    nv.count_launch()


def latent_turn(q: torch.Tensor, H: int, dim: int, cos: torch.Tensor, sin: torch.Tensor) -> None:
    """The rotated part of every head of ``q [M, H*dqp]`` (pairs of neighbours from channel ``dim`` on), in place; ``cos``, ``sin``
    ``[M, rot / 2]``."""
    dqp, rot = q.shape[1] // H, 2 * cos.shape[1]
    if not q.is_cuda:
        part = q.unflatten(1, (H, dqp))[:, :, dim:dim + rot]
        part.copy_(_turn(part, cos, sin).to(q.dtype))
        return
    nv.check(nv.lib().b2_latent_turn(nv.ptr(q), nv.ctypes.c_longlong(q.stride(0)), nv.ptr(cos), nv.ptr(sin), q.shape[0], H, dim, dqp, rot,
                                     int(q.dtype == torch.float32), nv.stream_ptr()), "latent_turn")
    nv.count_launch()


def head_linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, transposed: bool = False, turn=None,
                gate: Optional[torch.Tensor] = None) -> None:
    """``out[:, h] = W_h x[:, h]`` for every head: ``x [M, H*K]`` and ``out [M, H*N]`` (column slices), ``w [H, N, K]``, or
    ``[H, K, N]`` when ``transposed``.  On the 32-bit result: ``turn = (cos, sin, first)`` (``[M, rot / 2]`` each) turns the
    columns from ``first`` on of every head in pairs of neighbours, ``gate [M, H]`` multiplies a head by ``sigmoid(gate)``."""
    H = w.shape[0]
    K, N = (w.shape[1], w.shape[2]) if transposed else (w.shape[2], w.shape[1])
    if not x.is_cuda:
        y = torch.einsum("mhk,hkn->mhn" if transposed else "mhk,hnk->mhn", x.reshape(-1, H, K).float(), w.float())
        if turn is not None:
            cos, sin, first = turn
            part = y[:, :, first:first + 2 * cos.shape[1]]
            part.copy_(_turn(part, cos, sin))
        if gate is not None:
            y = y * torch.sigmoid(gate.float())[:, :, None]
        out.copy_(y.reshape(-1, H * N).to(out.dtype))
        return
    cos, sin, first = turn if turn is not None else (None, None, 0)
    assert w.is_contiguous() and x.shape[1] == H * K and out.shape[1] == H * N
    nv.check(nv.lib().b2_head_linear(
        nv.ptr(x), nv.ptr(w), nv.ptr(out), nv.ctypes.c_longlong(x.stride(0)), nv.ctypes.c_longlong(out.stride(0)), x.shape[0], H, N, K,
        K, N, int(transposed), nv.ptr(cos), nv.ptr(sin), first, 0 if cos is None else cos.shape[1], nv.ptr(gate),
        nv.ctypes.c_longlong(0 if gate is None else gate.stride(0)), int(x.dtype == torch.float32), 0, nv.stream_ptr()), "head_linear")
    nv.count_launch()


def latent_attention(q: torch.Tensor, pages: torch.Tensor, out: torch.Tensor, p: Portions, w_key: torch.Tensor,
                     w_value: torch.Tensor, scale: float, sink: Optional[torch.Tensor] = None, window: int = 0,
                     gate: Optional[torch.Tensor] = None, turn=None) -> None:
    """``out [M, H*dvp]`` (a column slice): causal softmax attention of every row over its sequence's cached rows (``window > 0``:
    over the last ``window`` of them).  ``q [M, H*dqp]`` with its rotated part turned; ``turn = (cos, sin, dim)``: it is not yet, and
    ``q`` may be overwritten.  ``sink [H]``: ``exp(sink)`` joins the denominator.  ``gate [M, H]``: a head's output times
    ``sigmoid(gate)``."""
    H, dqp, Rp = w_key.shape
    dvp, Cp = w_value.shape[1:]
    if not q.is_cuda:
        if turn is not None:
            latent_turn(q, H, turn[2], *turn[:2])
        slots = p.slots.tolist()
        for r, (s, pos) in enumerate(zip(p.row_seq.tolist(), p.positions.tolist())):
            if slots[s] < 0:
                out[r] = 0
                continue
            j = torch.arange(max(0, pos - window + 1) if window > 0 else 0, pos + 1)
            rows = pages[p.block_tables[s, j // 16].long(), j % 16, 0].float()
            K = torch.einsum("nr,hdr->nhd", rows, w_key.float())
            V = torch.einsum("nc,hdc->nhd", rows[:, :Cp], w_value.float())
            sc = torch.einsum("hd,nhd->hn", q[r].reshape(H, dqp).float(), K) * scale
            if sink is not None:
                sc = torch.cat([sc, sink.float()[:, None]], 1)
            w = sc.softmax(-1)[:, :j.numel()]
            o = torch.einsum("hn,nhd->hd", w, V)
            if gate is not None:
                o = o * torch.sigmoid(gate[r].float())[:, None]
            out[r] = o.reshape(-1).to(out.dtype)
        return
    lead, ns = p.rows, p.num_short
    if p.nseq > ns and q.dtype == torch.bfloat16 and dqp <= 192 and dvp <= 128:
        row_bytes = H * (dqp + dvp) * 2
        if max(p.context(window).counts) * 16 * row_bytes <= MAX_EXPANDED_BYTES:
            lead = p.short_rows
            if turn is not None:
                latent_turn(q[lead:], H, turn[2], turn[0][lead:], turn[1][lead:])
            _expanded(q, pages, out, p, w_key, w_value, scale, sink, MAX_EXPANDED_BYTES // (16 * row_bytes), window, gate)
    if lead == 0:
        return
    ql = torch.empty((lead, H * Rp), device=q.device, dtype=q.dtype)
    # the identity beside W_uk puts a head's rotated part behind the latent's channels
    head_linear(q[:lead], w_key, ql, transposed=True, turn=None if turn is None else (turn[0], turn[1], Cp))
    ol = torch.empty((lead, H * Cp), device=q.device, dtype=q.dtype)
    latent_rows(ql, pages, ol, p, H, Cp, scale, sink, window)
    head_linear(ol, w_value, out[:lead], gate=gate)


def latent_rows(q: torch.Tensor, pages: torch.Tensor, out: torch.Tensor, p: Portions, H: int, Cp: int, scale: float,
                sink: Optional[torch.Tensor], window: int = 0) -> None:
    """Attention of the first rows of the step in the latent space: ``q [m, H*Rp]`` -> ``out [m, H*Cp]``."""
    m, Rp = q.shape[0], pages.shape[-1]
    if q.dtype == torch.bfloat16 and decode_attention(q, pages, None, out, p, m, H, 1, Rp, Cp, scale, sink, window=window):
        return
    part, nsplit = _split(m * H, 1, 1, min(p.max_keys, window or p.max_keys))
    po = pm = None
    if nsplit > 1:
        po = torch.empty((m, H, nsplit, Cp), device=q.device, dtype=torch.float32)
        pm = torch.empty((m, H, nsplit, 2), device=q.device, dtype=torch.float32)
    nv.check(nv.lib().b2_latent_rows(
        nv.ptr(q), nv.ptr(pages), nv.ptr(p.block_tables), nv.ptr(p.row_seq), nv.ptr(p.positions), nv.ptr(p.slots), nv.ptr(sink),
        nv.ptr(out), nv.ptr(po), nv.ptr(pm), m, p.block_tables.shape[1], H, Rp, Cp, part, nsplit, window, nv.ctypes.c_float(scale),
        int(q.dtype == torch.float32), nv.stream_ptr()), "latent_rows")
    nv.count_launch(2 if nsplit > 1 else 1)


def _expanded(q, pages, out, p: Portions, w_key, w_value, scale, sink, max_pages: int, window: int = 0, gate=None) -> None:
    """The long portions: their contexts' rows in token order, keys and values of all heads from them, tensor-core attention."""
    H, dqp, Rp = w_key.shape
    dvp, Cp = w_value.shape[1:]
    ctx = p.context(window)
    counts, a, first = ctx.counts, 0, 0
    assert out.stride(0) % 8 == 0 and pages.is_contiguous()
    while a < len(counts):
        b, n = a, 0
        while b < len(counts) and (n == 0 or n + counts[b] <= max_pages):
            n += counts[b]
            b += 1
        rows = torch.empty((n * 16, Rp), device=q.device, dtype=q.dtype)
        gather(pages, ctx.pages[first:first + n], rows)
        k = gemm(rows, w_key.view(H * dqp, Rp))
        v = gemm(rows[:, :Cp], w_value.view(H * dvp, Cp))
        tables = ctx.tables[a:b] if first == 0 else ctx.tables[a:b] - first
        expanded_attention(q, k, v, out, p, H, dqp, dvp, scale, sink, a, b, tables, window, gate)
        a, first = b, first + n


def gather(pages: torch.Tensor, ids: torch.Tensor, rows: torch.Tensor) -> None:
    """Pages ``ids`` of the pool one after the other: ``rows [16 n, Rp]``."""
    nv.check(nv.lib().b2_latent_gather(nv.ptr(pages), nv.ptr(ids), nv.ptr(rows), ids.numel(), 16 * rows.shape[1] * rows.element_size(),
                                       nv.stream_ptr()), "latent_gather")
    nv.count_launch()


def expanded_attention(q, k, v, out, p: Portions, H: int, dqp: int, dvp: int, scale: float, sink, a: int, b: int, tables, window: int = 0,
                       gate=None) -> None:
    """Long portions ``a .. b - 1`` over keys and values laid out by ``tables`` in pages of 16 rows."""
    ns, cf, cl = p.num_short, nv.ctypes.c_float, nv.ctypes.c_longlong
    nv.check(nv.lib().b2_attn_fwd_paged_ext(
        nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ptr(out), cl(out.stride(0)), b - a, H, H, dqp, dvp, k.shape[0] // 16, cf(scale),
        nv.ptr(p.cu[ns + a:]), nv.ptr(p.starts[ns + a:]), nv.ptr(tables), tables.shape[1], p.max_long, p.rows, 0, None, None, 0,
        nv.ptr(sink), nv.ptr(gate), cl(0 if gate is None else gate.stride(0)), cl(q.stride(0)), window, cf(0.0), 1, None, cf(0.0), cf(0.0), 0, None, nv.stream_ptr()),
        "attn_fwd_paged_ext")
    nv.count_launch()
