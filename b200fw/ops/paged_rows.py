"""Paged attention for any head sizes with the options other designs add to the causal form: chunked visibility or a sliding
window, a soft cap on the scores, a learned distance bias, a softmax sink, an output gate, differential heads; and the per-head
bias + norm + rotation + cache store before it.

K pages are ``[blocks, 16, G, dkp]``, V pages ``[blocks, 16, G, dvp]`` in the activation dtype (head sizes padded to a
multiple of eight)."""
from __future__ import annotations

import functools
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


def qk_norm_store(q: torch.Tensor, k: Optional[torch.Tensor], v: Optional[torch.Tensor], k_cache: torch.Tensor, v_cache: torch.Tensor,
                  p: Portions, H: int, dk: int, norm: bool, eps: float, wq: Optional[torch.Tensor] = None,
                  wk: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None, cos: Optional[torch.Tensor] = None,
                  sin: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``bias`` (one vector over the columns of q, k and v) added, per-head RMS norm of q and k (``norm``; optional weights
    ``[dkp]``), rotary positions of q and k on channel pairs (2 i, 2 i + 1) (``cos, sin [M, dims/2]``), k and v stored into their
    sequences' pages.  ``q, k, v`` are column slices of one matrix; returns the new q ``[M, H*dkp]``.  K and V pages may have
    different head counts (two key rows over one value row).  ``k`` and ``v`` None: queries alone, over pages another layer fills."""
    nblk, bs, G, dkp = k_cache.shape
    Gv, dvp, M = v_cache.shape[2], v_cache.shape[3], q.shape[0]
    if k is None:
        G = Gv = 0
    bq = bk = bv = None
    if bias is not None:
        bq, bk, bv = bias[:H * dkp], bias[H * dkp:(H + G) * dkp], bias[(H + G) * dkp:]
        if k is None:
            bk = bv = bq
    if not q.is_cuda:
        if bias is not None:
            q = q.float() + bq.float()
            if k is not None:
                k, v = k.float() + bk.float(), v.float() + bv.float()

        def n(x, w):
            x = x.float()
            if norm:
                x = x * torch.rsqrt((x * x).sum(-1, keepdim=True) / dk + eps)
                if w is not None:
                    x = x * w.float()
            if cos is not None:
                rot = 2 * cos.shape[1]
                u, z, c, s = x[..., 0:rot:2], x[..., 1:rot:2], cos[:, None, :], sin[:, None, :]
                x = torch.cat([torch.stack([u * c - z * s, z * c + u * s], -1).flatten(-2), x[..., rot:]], -1)
            return x
        qf = n(q.reshape(M, H, dkp), wq).reshape(M, H * dkp).to(k_cache.dtype)
        if k is None:
            return qf
        kf = n(k.reshape(M, G, dkp), wk).to(k_cache.dtype)
        vf = v.reshape(M, Gv, dvp).to(v_cache.dtype)
        for r, (s, pos) in enumerate(zip(p.row_seq.tolist(), p.positions.tolist())):
            if int(p.slots[s]) < 0:
                continue
            blk = int(p.block_tables[s, pos // bs])
            k_cache[blk, pos % bs], v_cache[blk, pos % bs] = kf[r], vf[r]
        return qf
    assert bs == 16 and (k is None or q.stride(0) == k.stride(0) == v.stride(0))
    out = torch.empty((M, H * dkp), device=q.device, dtype=q.dtype)
    nv.check(nv.lib().b2_qk_norm_store(
        nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ctypes.c_longlong(q.stride(0)), nv.ptr(out), nv.ptr(k_cache), nv.ptr(v_cache),
        nv.ptr(p.block_tables), nv.ptr(p.row_seq), nv.ptr(p.positions), nv.ptr(p.slots), M, p.block_tables.shape[1], H, G, Gv, dk,
        dkp, dvp, nv.ptr(wq), nv.ptr(wk), int(norm), nv.ctypes.c_float(eps), nv.ptr(bq), nv.ptr(bk), nv.ptr(bv), nv.ptr(cos),
        nv.ptr(sin), 0 if cos is None else 2 * cos.shape[1], int(q.dtype == torch.float32), nv.stream_ptr()),
        "qk_norm_store")
    nv.count_launch()
    return out


@functools.lru_cache(maxsize=None)
def _sms(device: torch.device) -> int:
    return torch.cuda.get_device_properties(device).multi_processor_count


def _visible(pos: int, chunk: int, window: int) -> int:
    """First key the row at ``pos`` sees."""
    return pos // chunk * chunk if chunk else max(0, pos - window + 1) if window else 0


def paged_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor, p: Portions, H: int,
                    scale: float, chunk: int = 0, rel: Optional[torch.Tensor] = None, bucket: Optional[torch.Tensor] = None,
                    sink: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None, window: int = 0,
                    softcap: float = 0.0) -> None:
    """``out [M, H*dvp]`` (a column slice) = softmax attention of every row over its sequence's pages.

    ``chunk > 0``: a row at position i sees keys ``i // chunk * chunk .. i``; ``window > 0``: keys ``i - window + 1 .. i`` (both 0:
    all keys up to i).  ``softcap > 0``: scores become ``softcap * tanh(score / softcap)``.  ``rel [buckets, H]`` with ``bucket``
    (int32, distance -> bucket, the last entry for every larger distance) adds a bias to the scaled score.  ``sink [H]``:
    ``exp(sink)`` joins the denominator.  ``gate [M, H]``: the head's output times ``sigmoid(gate)``."""
    if not q.is_cuda:
        o = _attention_cpu(q, k_cache, v_cache, p, H, scale, chunk, rel, bucket, sink, window, softcap)
        if gate is not None:
            o = o * torch.sigmoid(gate.float())[:, :, None]
        out.copy_(o.reshape(out.shape).to(out.dtype))
        return
    _attention(q, k_cache, v_cache, out, p, H, scale, chunk, rel, bucket, sink, gate, window, softcap, None, 0.0, 0.0, 0)


def differential_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor, p: Portions, H: int,
                           scale: float, lam: torch.Tensor, lam_init: float, dv: int, eps: float,
                           gate: Optional[torch.Tensor] = None, window: int = 0, softcap: float = 0.0) -> None:
    """Differential heads: ``q [M, H, 2, dkp]`` and K pages ``[blocks, 16, 2 G, dkp]`` (map 1, map 2 of every head) over V pages
    ``[blocks, 16, G, dvp]``.  With a1, a2 the two maps' attentions and ``lambda = exp(l0 . l1) - exp(l2 . l3) + lam_init`` from
    ``lam [4, dkp]``: ``out [M, H*dvp] = rms(a1 - lambda a2) (1 - lam_init) sigmoid(gate)``, the norm over a head's ``dv``
    channels, ``gate [M, H*dvp]``."""
    if not q.is_cuda:
        dvp = v_cache.shape[-1]
        o = _attention_cpu(q, k_cache, v_cache.repeat_interleave(2, 2), p, 2 * H, scale, 0, None, None, None, window, softcap,
                           lambda h, per: 2 * (h // (2 * per)) + h % 2)
        l4 = lam.float()
        full = (l4[0] * l4[1]).sum().exp() - (l4[2] * l4[3]).sum().exp() + lam_init
        o = o[:, 0::2] - full * o[:, 1::2]
        o = o * torch.rsqrt((o * o).sum(-1, keepdim=True) / dv + eps) * (1.0 - lam_init)
        if gate is not None:
            o = o * torch.sigmoid(gate.float()).reshape(-1, H, dvp)
        out.copy_(o.reshape(out.shape).to(out.dtype))
        return
    _attention(q, k_cache, v_cache, out, p, H, scale, 0, None, None, None, gate, window, softcap, lam, lam_init, eps, dv)


def _attention_cpu(q, k_cache, v_cache, p, H, scale, chunk, rel, bucket, sink, window, softcap, key_of=lambda h, per: h // per):
    """fp32 ``[M, H, dvp]``; query head h reads key and value head ``key_of(h, query heads per key head)``."""
    nblk, bs, G, dkp = k_cache.shape
    slots, of = p.slots.tolist(), torch.tensor([key_of(h, H // G) for h in range(H)])
    out = torch.zeros(q.shape[0], H, v_cache.shape[-1])
    for r, (s, pos) in enumerate(zip(p.row_seq.tolist(), p.positions.tolist())):
        if slots[s] < 0:
            continue
        j = torch.arange(_visible(pos, chunk, window), pos + 1)
        blk = p.block_tables[s, j // bs].long()
        K, V = k_cache[blk, j % bs].float()[:, of], v_cache[blk, j % bs].float()[:, of]
        sc = torch.einsum("hd,nhd->hn", q[r].reshape(H, dkp).float(), K) * scale
        if softcap:
            sc = softcap * torch.tanh(sc / softcap)
        if rel is not None:
            sc = sc + rel.float()[bucket[(pos - j).clamp(max=bucket.numel() - 1)].long()].t()
        if sink is not None:
            sc = torch.cat([sc, sink.float()[:, None]], 1)
        out[r] = torch.einsum("hn,nhd->hd", sc.softmax(-1)[:, :j.numel()], V)
    return out


def _attention(q, k_cache, v_cache, out, p, H, scale, chunk, rel, bucket, sink, gate, window, softcap, lam, lam_init, eps, dv):
    nblk, bs, G, dvp = v_cache.shape
    dkp, M, maps = k_cache.shape[-1], q.shape[0], 2 if lam is not None else 1
    cf, cl = nv.ctypes.c_float, nv.ctypes.c_longlong
    ld_gate = cl(0 if gate is None else gate.stride(0))
    nbucket = 0 if bucket is None else bucket.numel()
    lead = M
    if p.nseq > p.num_short and q.dtype == torch.bfloat16 and dkp <= 128 and dvp <= 128 and nbucket <= 7680:
        lead, ns = p.short_rows, p.num_short          # the long portions: tensor-core tiles straight over the pages
        assert out.stride(0) % 8 == 0 and k_cache.is_contiguous() and v_cache.is_contiguous()
        scratch = torch.empty(_sms(q.device) * 256 * 64, device=q.device, dtype=torch.float32) if maps == 2 else None
        nv.check(nv.lib().b2_attn_fwd_paged_ext(
            nv.ptr(q), nv.ptr(k_cache), nv.ptr(v_cache), nv.ptr(out), cl(out.stride(0)), p.nseq - ns, H, G, dkp, dvp, nblk, cf(scale),
            nv.ptr(p.cu[ns:]), nv.ptr(p.starts[ns:]), nv.ptr(p.block_tables[ns:]), p.block_tables.shape[1], p.max_long, M, chunk,
            nv.ptr(rel), nv.ptr(bucket), nbucket, nv.ptr(sink), nv.ptr(gate), ld_gate, cl(q.stride(0)), window, cf(softcap), maps,
            nv.ptr(lam), cf(lam_init), cf(eps), dv, nv.ptr(scratch), nv.stream_ptr()), "attn_fwd_paged_ext")
        nv.count_launch()
    if lead == 0:
        return
    plain = lam is None and gate is None and rel is None and chunk == 0
    if q.dtype == torch.bfloat16 and (plain or lam is not None) and decode_attention(
            q, k_cache, v_cache, out, p, lead, H, G, maps * dkp, dvp, scale, sink, gate, window, softcap, lam, lam_init, eps, dv):
        return
    assert q.is_contiguous()
    keys = min(p.max_keys, chunk or window or p.max_keys)
    most = 4 // maps
    groups = (H // G + most - 1) // most
    part, nsplit = _split(lead, G * groups, -(-(H // G) // groups) * maps, keys)
    po = pm = None
    if nsplit > 1:
        po = torch.empty((lead, H * maps, nsplit, dvp), device=q.device, dtype=torch.float32)
        pm = torch.empty((lead, H * maps, nsplit, 2), device=q.device, dtype=torch.float32)
    nv.check(nv.lib().b2_attn_rows(
        nv.ptr(q), nv.ptr(k_cache), nv.ptr(v_cache), nv.ptr(p.block_tables), nv.ptr(p.row_seq), nv.ptr(p.positions),
        nv.ptr(p.slots), nv.ptr(gate), ld_gate, nv.ptr(sink), nv.ptr(rel), nv.ptr(bucket), nbucket, nv.ptr(out), cl(out.stride(0)),
        nv.ptr(po), nv.ptr(pm), lead, p.block_tables.shape[1], H, G, dkp, dvp, chunk, part, nsplit, cf(scale), window, cf(softcap),
        nv.ptr(lam), cf(lam_init), cf(eps), dv, int(q.dtype == torch.float32), nv.stream_ptr()), "attn_rows")
    nv.count_launch(2 if nsplit > 1 else 1)


def decode_attention(q, k_cache, v_cache, out, p: Portions, rows: int, H: int, G: int, R: int, C: int, scale: float, sink, gate=None,
                     window: int = 0, softcap: float = 0.0, lam=None, lam_init: float = 0.0, eps: float = 0.0, dv: int = 0) -> bool:
    """The first ``rows`` rows of the step, one query token each, on the tensor cores with the work split evenly over the SMs
    (csrc/attention_decode.cu).  ``v_cache`` None: a value is the first ``C`` channels of its key row.  False, with nothing done,
    for sizes the kernel has no form for."""
    tile = nv.lib().b2_decode_tile(R, C, int(v_cache is not None))
    if tile == 0:
        return False
    key = (rows, window, tile)
    if key not in p.plans:
        p.plans[key] = torch.empty(rows + 1, device=q.device, dtype=torch.int32)
        nv.check(nv.lib().b2_decode_plan(nv.ptr(p.positions), nv.ptr(p.row_seq), nv.ptr(p.slots), nv.ptr(p.plans[key]), rows, window,
                                         tile, nv.stream_ptr()), "decode_plan")
        nv.count_launch()
    n = _sms(q.device)
    po = torch.empty((n, 2, 16, C), device=q.device, dtype=torch.float32)
    pm = torch.empty((n, 2, 16, 2), device=q.device, dtype=torch.float32)
    cf, cl = nv.ctypes.c_float, nv.ctypes.c_longlong
    nv.check(nv.lib().b2_decode_attention(
        nv.ptr(q), nv.ptr(k_cache), nv.ptr(v_cache), nv.ptr(p.block_tables), nv.ptr(p.row_seq), nv.ptr(p.positions),
        nv.ptr(p.plans[key]), nv.ptr(sink), nv.ptr(gate), nv.ptr(lam), nv.ptr(out), nv.ptr(po), nv.ptr(pm), cl(q.stride(0)),
        cl(0 if gate is None else gate.stride(0)), cl(out.stride(0)), rows, k_cache.shape[0], p.block_tables.shape[1], H, G, R, C, window, dv, cf(scale),
        cf(softcap), cf(lam_init), cf(eps), nv.stream_ptr()), "decode_attention")
    nv.count_launch(2)
    return True


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
