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


def latent_store(q: torch.Tensor, c: torch.Tensor, kr: torch.Tensor, pages: torch.Tensor, p: Portions, H: int, dim: int,
                 rank: int, rot: int, w: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, eps: float) -> None:
    """``q [M, H*dqp]``, ``c [M, Cp]``, ``kr [M, Rp - Cp]`` are column slices of one matrix.  The rotated part of every head of
    ``q`` (channels ``dim .. dim + rot - 1``, pairs of neighbours) is turned in place; ``rms(c) w`` and the turned ``kr``
    go to the rows' pages."""
    M, Cp, Rp = q.shape[0], c.shape[1], pages.shape[-1]
    dqp = q.shape[1] // H
    if not q.is_cuda:
        def turn(x):
            u, v = x[..., 0::2].float(), x[..., 1::2].float()
            s = (slice(None),) + (None,) * (x.dim() - 2)
            return torch.stack([u * cos[s] - v * sin[s], v * cos[s] + u * sin[s]], -1).flatten(-2)
        part = q.unflatten(1, (H, dqp))[:, :, dim:dim + rot]
        part.copy_(turn(part).to(q.dtype))
        cf = c.float()
        cf = cf * torch.rsqrt((cf * cf).sum(-1, keepdim=True) / rank + eps) * w.float()
        row = torch.cat([cf, torch.nn.functional.pad(turn(kr[:, :rot]), (0, Rp - Cp - rot))], 1).to(pages.dtype)
        for r, (s, pos) in enumerate(zip(p.row_seq.tolist(), p.positions.tolist())):
            if int(p.slots[s]) >= 0:
                pages[int(p.block_tables[s, pos // 16]), pos % 16, 0] = row[r]
        return
    assert q.stride(0) == c.stride(0) == kr.stride(0) and pages.shape[1] == 16
    nv.check(nv.lib().b2_latent_store(
        nv.ptr(q), nv.ptr(c), nv.ptr(kr), nv.ctypes.c_longlong(q.stride(0)), nv.ptr(pages), nv.ptr(w), nv.ptr(p.block_tables),
        nv.ptr(p.row_seq), nv.ptr(p.positions), nv.ptr(p.slots), nv.ptr(cos), nv.ptr(sin), M, p.block_tables.shape[1], H, dim, dqp,
        rank, Cp, Rp, rot, nv.ctypes.c_float(eps), int(q.dtype == torch.float32), nv.stream_ptr()), "latent_store")
    nv.count_launch()


def head_linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, transposed: bool = False) -> None:
    """``out[:, h] = W_h x[:, h]`` for every head: ``x [M, H*K]`` and ``out [M, H*N]`` (column slices), ``w [H, N, K]``, or
    ``[H, K, N]`` when ``transposed``."""
    H = w.shape[0]
    K, N = (w.shape[1], w.shape[2]) if transposed else (w.shape[2], w.shape[1])
    if not x.is_cuda:
        y = torch.einsum("mhk,hkn->mhn" if transposed else "mhk,hnk->mhn", x.reshape(-1, H, K).float(), w.float())
        out.copy_(y.reshape(-1, H * N).to(out.dtype))
        return
    assert w.is_contiguous() and x.shape[1] == H * K and out.shape[1] == H * N
    nv.check(nv.lib().b2_head_linear(
        nv.ptr(x), nv.ptr(w), nv.ptr(out), nv.ctypes.c_longlong(x.stride(0)), nv.ctypes.c_longlong(out.stride(0)), x.shape[0], H, N, K,
        K, N, int(transposed), int(x.dtype == torch.float32), 0, nv.stream_ptr()), "head_linear")
    nv.count_launch()


def latent_attention(q: torch.Tensor, pages: torch.Tensor, out: torch.Tensor, p: Portions, w_key: torch.Tensor,
                     w_value: torch.Tensor, scale: float, sink: Optional[torch.Tensor] = None) -> None:
    """``out [M, H*dvp]`` (a column slice): causal softmax attention of every row over its sequence's cached rows.
    ``q [M, H*dqp]`` with its rotated part turned.  ``sink [H]``: ``exp(sink)`` joins the denominator."""
    H, dqp, Rp = w_key.shape
    dvp, Cp = w_value.shape[1:]
    if not q.is_cuda:
        slots = p.slots.tolist()
        for r, (s, pos) in enumerate(zip(p.row_seq.tolist(), p.positions.tolist())):
            if slots[s] < 0:
                out[r] = 0
                continue
            j = torch.arange(pos + 1)
            rows = pages[p.block_tables[s, j // 16].long(), j % 16, 0].float()
            K = torch.einsum("nr,hdr->nhd", rows, w_key.float())
            V = torch.einsum("nc,hdc->nhd", rows[:, :Cp], w_value.float())
            sc = torch.einsum("hd,nhd->hn", q[r].reshape(H, dqp).float(), K) * scale
            if sink is not None:
                sc = torch.cat([sc, sink.float()[:, None]], 1)
            w = sc.softmax(-1)[:, :j.numel()]
            out[r] = torch.einsum("hn,nhd->hd", w, V).reshape(-1).to(out.dtype)
        return
    lead, ns = p.rows, p.num_short
    if p.nseq > ns and q.dtype == torch.bfloat16 and dqp <= 192 and dvp <= 128:
        row_bytes = H * (dqp + dvp) * 2
        if max(p.ctx_counts) * 16 * row_bytes <= MAX_EXPANDED_BYTES:
            lead = p.short_rows
            _expanded(q, pages, out, p, w_key, w_value, scale, sink, MAX_EXPANDED_BYTES // (16 * row_bytes))
    if lead == 0:
        return
    ql = torch.empty((lead, H * Rp), device=q.device, dtype=q.dtype)
    head_linear(q[:lead], w_key, ql, transposed=True)
    ol = torch.empty((lead, H * Cp), device=q.device, dtype=q.dtype)
    latent_rows(ql, pages, ol, p, H, Cp, scale, sink)
    head_linear(ol, w_value, out[:lead])


def latent_rows(q: torch.Tensor, pages: torch.Tensor, out: torch.Tensor, p: Portions, H: int, Cp: int, scale: float,
                sink: Optional[torch.Tensor]) -> None:
    """Attention of the first rows of the step in the latent space: ``q [m, H*Rp]`` -> ``out [m, H*Cp]``."""
    m, Rp = q.shape[0], pages.shape[-1]
    if q.dtype == torch.bfloat16 and decode_attention(q, pages, None, out, p, m, H, 1, Rp, Cp, scale, sink):
        return
    part, nsplit = _split(m * H, 1, 1, p.max_keys)
    po = pm = None
    if nsplit > 1:
        po = torch.empty((m, H, nsplit, Cp), device=q.device, dtype=torch.float32)
        pm = torch.empty((m, H, nsplit, 2), device=q.device, dtype=torch.float32)
    nv.check(nv.lib().b2_latent_rows(
        nv.ptr(q), nv.ptr(pages), nv.ptr(p.block_tables), nv.ptr(p.row_seq), nv.ptr(p.positions), nv.ptr(p.slots), nv.ptr(sink),
        nv.ptr(out), nv.ptr(po), nv.ptr(pm), m, p.block_tables.shape[1], H, Rp, Cp, part, nsplit, nv.ctypes.c_float(scale),
        int(q.dtype == torch.float32), nv.stream_ptr()), "latent_rows")
    nv.count_launch(2 if nsplit > 1 else 1)


def _expanded(q, pages, out, p: Portions, w_key, w_value, scale, sink, max_pages: int) -> None:
    """The long portions: their contexts' rows in token order, keys and values of all heads from them, tensor-core attention."""
    H, dqp, Rp = w_key.shape
    dvp, Cp = w_value.shape[1:]
    counts, a, first = p.ctx_counts, 0, 0
    assert out.stride(0) % 8 == 0 and pages.is_contiguous()
    while a < len(counts):
        b, n = a, 0
        while b < len(counts) and (n == 0 or n + counts[b] <= max_pages):
            n += counts[b]
            b += 1
        rows = torch.empty((n * 16, Rp), device=q.device, dtype=q.dtype)
        gather(pages, p.ctx_pages[first:first + n], rows)
        k = gemm(rows, w_key.view(H * dqp, Rp))
        v = gemm(rows[:, :Cp], w_value.view(H * dvp, Cp))
        tables = p.ctx_tables[a:b] if first == 0 else p.ctx_tables[a:b] - first
        expanded_attention(q, k, v, out, p, H, dqp, dvp, scale, sink, a, b, tables)
        a, first = b, first + n


def gather(pages: torch.Tensor, ids: torch.Tensor, rows: torch.Tensor) -> None:
    """Pages ``ids`` of the pool one after the other: ``rows [16 n, Rp]``."""
    nv.check(nv.lib().b2_latent_gather(nv.ptr(pages), nv.ptr(ids), nv.ptr(rows), ids.numel(), 16 * rows.shape[1] * rows.element_size(),
                                       nv.stream_ptr()), "latent_gather")
    nv.count_launch()


def expanded_attention(q, k, v, out, p: Portions, H: int, dqp: int, dvp: int, scale: float, sink, a: int, b: int, tables) -> None:
    """Long portions ``a .. b - 1`` over keys and values laid out by ``tables`` in pages of 16 rows."""
    ns, cf, cl = p.num_short, nv.ctypes.c_float, nv.ctypes.c_longlong
    nv.check(nv.lib().b2_attn_fwd_paged_ext(
        nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ptr(out), cl(out.stride(0)), b - a, H, H, dqp, dvp, k.shape[0] // 16, cf(scale),
        nv.ptr(p.cu[ns + a:]), nv.ptr(p.starts[ns + a:]), nv.ptr(tables), tables.shape[1], p.max_long, p.rows, 0, None, None, 0,
        nv.ptr(sink), None, cl(0), cl(q.stride(0)), 0, cf(0.0), 1, None, cf(0.0), cf(0.0), 0, None, nv.stream_ptr()),
        "attn_fwd_paged_ext")
    nv.count_launch()
