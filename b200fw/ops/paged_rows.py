"""Paged attention for any head sizes with the options other designs add to the causal form: chunked visibility, a learned
distance bias, a softmax sink, an output gate; and the per-head norm + cache store before it.

K pages are ``[blocks, 16, G, dkp]``, V pages ``[blocks, 16, G, dvp]`` in the activation dtype (head sizes padded to a
multiple of eight)."""
from __future__ import annotations

import math
from typing import Optional

import torch

from .. import _native as nv
from .portions import Portions


def distance_buckets(rows: int, far: float, length: int, device=None) -> torch.Tensor:
    """int32 bucket of every distance ``0 .. length-1``: one per distance below ``rows / 2``, then logarithmic up to
    ``far``.  A distance that falls exactly on an edge belongs to the upper bucket (the tolerance only absorbs the rounding
    of the two logarithms)."""
    half, out = rows // 2, []
    for n in range(length):
        if n < half:
            out.append(n)
        elif far <= half:
            out.append(rows - 1)
        else:
            out.append(min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9)))
    return torch.tensor(out, dtype=torch.int32, device=device)


def qk_norm_store(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                  p: Portions, H: int, dk: int, norm: bool, eps: float, wq: Optional[torch.Tensor] = None,
                  wk: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Per-head RMS norm of q and k (``norm``; optional weights ``[dk]``), k and v stored into their sequences' pages.
    ``q, k, v`` are column slices of one matrix; returns the normed q ``[M, H*dkp]``."""
    nblk, bs, G, dkp = k_cache.shape
    dvp, M = v_cache.shape[-1], q.shape[0]
    if not q.is_cuda:
        def n(x, w):
            x = x.float()
            if norm:
                x = x * torch.rsqrt((x * x).sum(-1, keepdim=True) / dk + eps)
                if w is not None:
                    x = x * torch.nn.functional.pad(w.float(), (0, dkp - dk))
            return x
        kf = n(k.reshape(M, G, dkp), wk).to(k_cache.dtype)
        vf = v.reshape(M, G, dvp).to(v_cache.dtype)
        for r, (s, pos) in enumerate(zip(p.row_seq.tolist(), p.positions.tolist())):
            if int(p.slots[s]) < 0:
                continue
            blk = int(p.block_tables[s, pos // bs])
            k_cache[blk, pos % bs], v_cache[blk, pos % bs] = kf[r], vf[r]
        return n(q.reshape(M, H, dkp), wq).reshape(M, H * dkp).to(q.dtype)
    assert bs == 16 and q.stride(0) == k.stride(0) == v.stride(0)
    out = torch.empty((M, H * dkp), device=q.device, dtype=q.dtype)
    nv.check(nv.lib().b2_qk_norm_store(
        nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ctypes.c_longlong(q.stride(0)), nv.ptr(out), nv.ptr(k_cache), nv.ptr(v_cache),
        nv.ptr(p.block_tables), nv.ptr(p.row_seq), nv.ptr(p.positions), nv.ptr(p.slots), M, p.block_tables.shape[1], H, G, dk,
        dkp, dvp, nv.ptr(wq), nv.ptr(wk), int(norm), nv.ctypes.c_float(eps), int(q.dtype == torch.float32), nv.stream_ptr()),
        "qk_norm_store")
    nv.count_launch()
    return out


def paged_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor, p: Portions, H: int,
                    scale: float, chunk: int = 0, rel: Optional[torch.Tensor] = None, bucket: Optional[torch.Tensor] = None,
                    sink: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None) -> None:
    """``out [M, H*dvp]`` (a column slice) = softmax attention of every row over its sequence's pages.

    ``chunk > 0``: a row at position i sees keys ``i // chunk * chunk .. i`` (0: all keys up to i).  ``rel [buckets, H]``
    with ``bucket`` (int32, distance -> bucket, the last entry for every larger distance) adds a bias to the scaled score.
    ``sink [H]``: ``exp(sink)`` joins the denominator.  ``gate [M, H]``: the head's output times ``sigmoid(gate)``."""
    nblk, bs, G, dkp = k_cache.shape
    dvp, M = v_cache.shape[-1], q.shape[0]
    if not q.is_cuda:
        slots, per = p.slots.tolist(), H // G
        for r, (s, pos) in enumerate(zip(p.row_seq.tolist(), p.positions.tolist())):
            if slots[s] < 0:
                out[r] = 0
                continue
            j = torch.arange(pos // chunk * chunk if chunk else 0, pos + 1)
            blk = p.block_tables[s, j // bs].long()
            K = k_cache[blk, j % bs].float().repeat_interleave(per, 1)
            V = v_cache[blk, j % bs].float().repeat_interleave(per, 1)
            sc = torch.einsum("hd,nhd->hn", q[r].reshape(H, dkp).float(), K) * scale
            if rel is not None:
                sc = sc + rel.float()[bucket[(pos - j).clamp(max=bucket.numel() - 1)].long()].t()
            if sink is not None:
                sc = torch.cat([sc, sink.float()[:, None]], 1)
            w = sc.softmax(-1)[:, :j.numel()]
            o = torch.einsum("hn,nhd->hd", w, V)
            if gate is not None:
                o = o * torch.sigmoid(gate[r].float())[:, None]
            out[r] = o.reshape(-1).to(out.dtype)
        return
    lead = M
    if p.nseq > p.num_short and dkp <= 128 and dvp <= 128 and (bucket is None or bucket.numel() <= 7680):
        lead, ns = p.short_rows, p.num_short          # the long portions: tensor-core tiles straight over the pages
        assert out.stride(0) % 8 == 0 and k_cache.is_contiguous() and v_cache.is_contiguous()
        nv.check(nv.lib().b2_attn_fwd_paged_ext(
            nv.ptr(q), nv.ptr(k_cache), nv.ptr(v_cache), nv.ptr(out), nv.ctypes.c_longlong(out.stride(0)), p.nseq - ns, H, G, dkp,
            dvp, nblk, nv.ctypes.c_float(scale), nv.ptr(p.cu[ns:]), nv.ptr(p.starts[ns:]), nv.ptr(p.block_tables[ns:]),
            p.block_tables.shape[1], p.max_long, M, chunk, nv.ptr(rel), nv.ptr(bucket), 0 if bucket is None else bucket.numel(),
            nv.ptr(sink), nv.ptr(gate), nv.ctypes.c_longlong(0 if gate is None else gate.stride(0)), nv.stream_ptr()),
            "attn_fwd_paged_ext")
        nv.count_launch()
    if lead == 0:
        return
    keys = p.max_keys if chunk <= 0 else min(p.max_keys, chunk)
    groups = (H // G + 3) // 4
    part, nsplit = _split(lead, G * groups, -(-(H // G) // groups), keys)
    po = pm = None
    if nsplit > 1:
        po = torch.empty((lead, H, nsplit, dvp), device=q.device, dtype=torch.float32)
        pm = torch.empty((lead, H, nsplit, 2), device=q.device, dtype=torch.float32)
    nv.check(nv.lib().b2_attn_rows(
        nv.ptr(q), nv.ptr(k_cache), nv.ptr(v_cache), nv.ptr(p.block_tables), nv.ptr(p.row_seq), nv.ptr(p.positions),
        nv.ptr(p.slots), nv.ptr(gate), nv.ctypes.c_longlong(0 if gate is None else gate.stride(0)), nv.ptr(sink), nv.ptr(rel),
        nv.ptr(bucket), 0 if bucket is None else bucket.numel(), nv.ptr(out), nv.ctypes.c_longlong(out.stride(0)), nv.ptr(po),
        nv.ptr(pm), lead, p.block_tables.shape[1], H, G, dkp, dvp, chunk, part, nsplit, nv.ctypes.c_float(scale),
        int(q.dtype == torch.float32), nv.stream_ptr()), "attn_rows")
    nv.count_launch(2 if nsplit > 1 else 1)


def _split(rows: int, groups_per_row: int, heads: int, keys: int):
    """Keys per split and number of splits (measured at 8 to 256 rows): one wave of resident CTAs when the rows alone are
    fewer than that, else three or four splits so that the last wave is short; 128 to 2048 keys each.  ``heads``: query heads
    of a CTA (three or four leave registers for three CTAs per SM instead of four)."""
    ctas, resident, few = max(1, rows * groups_per_row), 148 * (3 if heads > 2 else 4), 3 if heads > 2 else 4
    n = 1 if ctas > 8 * resident else min((keys + 127) // 128, max(resident // ctas, few))
    n = max(n, (keys + 2047) // 2048)
    if n <= 1:
        return max(1, keys), 1
    part = ((keys + n - 1) // n + 63) // 64 * 64
    return part, (keys + part - 1) // part
