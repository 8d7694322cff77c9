"""Ops around a 32-bit residual stream: embedding into it (of tokens, or of tokens and pairs of neighbours), RMS norm or layer norm
out of it, normed branches added to it, gated activations over column slices or with a table of per-token vectors, rotary tables for
a batch's positions.

Activations and residual rows are padded to a multiple of eight columns (:func:`pad8`); the padding is zero."""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch

from .. import _native as nv
from .portions import Portions


def _f32(t: torch.Tensor) -> int:
    return int(t.dtype == torch.float32)


def embedding_f32(ids: torch.Tensor, table: torch.Tensor, vocab: Optional[int] = None, scale: float = 1.0, h: bool = False):
    """Rows of ``table`` times ``scale`` as fp32; an id outside ``[0, vocab)`` (padding rows of a graph batch) gives zeros on a
    GPU.  ``h``: returns ``(x, x in the table's dtype)``."""
    if not table.is_cuda:
        x = table[ids].float() * scale
        return (x, x.to(table.dtype)) if h else x
    x = torch.empty((ids.numel(), table.shape[1]), device=table.device, dtype=torch.float32)
    low = torch.empty(x.shape, device=x.device, dtype=table.dtype) if h and table.dtype != torch.float32 else None
    nv.check(nv.lib().b2_embed_f32(nv.ptr(ids), nv.ptr(table), nv.ptr(x), nv.ptr(low), ids.numel(), table.shape[1],
                                   table.shape[0] if vocab is None else vocab, nv.ctypes.c_float(scale), _f32(table),
                                   nv.stream_ptr()), "embed_f32")
    nv.count_launch()
    return (x, x if low is None else low) if h else x


def rmsnorm_f32(x: torch.Tensor, w: torch.Tensor, n: int, eps: float, rows: Optional[torch.Tensor] = None,
                scale: float = 1.0) -> torch.Tensor:
    """``x[rows] / sqrt(mean(x^2) + eps) * w * scale`` in ``w``'s dtype; ``n`` real columns, ``w`` zero past them.  ``rows``
    (int64) selects and orders the rows of ``x``."""
    if not x.is_cuda:
        xs = x if rows is None else x[rows]
        r = scale * torch.rsqrt((xs[:, :n] * xs[:, :n]).mean(-1, keepdim=True) + eps)
        return (xs * r * w.float()).to(w.dtype)
    M = x.shape[0] if rows is None else rows.numel()
    h = torch.empty((M, x.shape[1]), device=x.device, dtype=w.dtype)
    nv.check(nv.lib().b2_rmsnorm_f32(nv.ptr(x), nv.ptr(w), nv.ptr(h), nv.ptr(rows), M, x.shape[1], n,
                                     nv.ctypes.c_float(eps), nv.ctypes.c_float(scale), _f32(w), nv.stream_ptr()), "rmsnorm_f32")
    nv.count_launch()
    return h


def merge_norm_add(x: torch.Tensor, a: torch.Tensor, b: torch.Tensor, wa: torch.Tensor, wb: torch.Tensor, coef: float,
                   n: int, eps: float, w_next: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """In place ``x += coef * (rms(a) wa + rms(b) wb)`` (``a``, ``b``, ``x`` fp32); returns ``rms(x) w_next`` when the
    next norm's weight is given."""
    if not x.is_cuda:
        def rms(t):
            return t * torch.rsqrt((t[:, :n] * t[:, :n]).mean(-1, keepdim=True) + eps)
        x += coef * (rms(a) * wa.float() + rms(b) * wb.float())
        return None if w_next is None else (rms(x) * w_next.float()).to(w_next.dtype)
    h = None if w_next is None else torch.empty(x.shape, device=x.device, dtype=w_next.dtype)
    nv.check(nv.lib().b2_merge_norm_add(nv.ptr(x), nv.ptr(a), nv.ptr(b), nv.ptr(wa), nv.ptr(wb), nv.ptr(w_next), nv.ptr(h),
                                        x.shape[0], x.shape[1], n, nv.ctypes.c_float(coef), nv.ctypes.c_float(eps),
                                        _f32(wa), nv.stream_ptr()), "merge_norm_add")
    nv.count_launch()
    return h


def post_norm(x: torch.Tensor, y: torch.Tensor, w: torch.Tensor, alpha: float, n: int, eps: float,
              bias: Optional[torch.Tensor] = None, sumsq: Optional[torch.Tensor] = None, sumsq_n: int = 0) -> torch.Tensor:
    """In place ``x = rms(alpha * x + y + bias) * w`` (``x``, ``y`` fp32); returns the new ``x`` in ``w``'s dtype (``x``
    itself in 32-bit).  ``sumsq [rows, parts]``: ``y`` is first divided by the root mean square (over ``sumsq_n`` channels) of
    the input it was projected from, whose sums of squares these are."""
    if not x.is_cuda:
        if sumsq is not None:
            y = y * torch.rsqrt(sumsq.sum(-1, keepdim=True) / sumsq_n + eps)
        t = alpha * x + y
        if bias is not None:
            t = t + bias.float()
        x.copy_(t * torch.rsqrt((t[:, :n] * t[:, :n]).mean(-1, keepdim=True) + eps) * w.float())
        return x if w.dtype == torch.float32 else x.to(w.dtype)
    h = None if w.dtype == torch.float32 else torch.empty(x.shape, device=x.device, dtype=w.dtype)
    nv.check(nv.lib().b2_post_norm(nv.ptr(x), nv.ptr(y), nv.ptr(w), nv.ptr(bias), nv.ptr(sumsq), 0 if sumsq is None else sumsq.shape[1],
                                   sumsq_n, nv.ptr(h), x.shape[0], x.shape[1], n, nv.ctypes.c_float(alpha), nv.ctypes.c_float(eps),
                                   _f32(w), nv.stream_ptr()), "post_norm")
    nv.count_launch()
    return x if h is None else h


def norm_add(x: torch.Tensor, y: torch.Tensor, w: torch.Tensor, coef: float, n: int, eps: float, y_scale: float = 1.0) -> torch.Tensor:
    """In place ``x += coef * rms(y_scale * y) * w`` (``x``, ``y`` fp32); returns the new ``x`` in ``w``'s dtype (``x`` itself in
    32-bit)."""
    if not x.is_cuda:
        t = y_scale * y
        x += coef * t * torch.rsqrt((t[:, :n] * t[:, :n]).mean(-1, keepdim=True) + eps) * w.float()
        return x if w.dtype == torch.float32 else x.to(w.dtype)
    h = None if w.dtype == torch.float32 else torch.empty(x.shape, device=x.device, dtype=w.dtype)
    nv.check(nv.lib().b2_norm_add(nv.ptr(x), nv.ptr(y), nv.ptr(w), nv.ptr(h), x.shape[0], x.shape[1], n, nv.ctypes.c_float(coef),
                                  nv.ctypes.c_float(eps), nv.ctypes.c_float(y_scale), _f32(w), nv.stream_ptr()), "norm_add")
    nv.count_launch()
    return x if h is None else h


Norm = Tuple[torch.Tensor, torch.Tensor]      # weight and bias of a layer norm, zero past the real columns


def _layer_norm(x: torch.Tensor, w: Norm, n: int, eps: float) -> torch.Tensor:
    """fp32 rows ``x [M, ld]``, zero past ``n``."""
    d = x - x[:, :n].mean(-1, keepdim=True)
    return d * torch.rsqrt((d[:, :n] * d[:, :n]).mean(-1, keepdim=True) + eps) * w[0].float() + w[1].float()


def layernorm_f32(x: torch.Tensor, w: Norm, n: int, eps: float, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Layer norm of ``x[rows]`` (``rows`` int64 selects and orders) over its ``n`` real columns, in the weight's dtype."""
    if not x.is_cuda:
        return _layer_norm(x if rows is None else x[rows], w, n, eps).to(w[0].dtype)
    M = x.shape[0] if rows is None else rows.numel()
    h = torch.empty((M, x.shape[1]), device=x.device, dtype=w[0].dtype)
    nv.check(nv.lib().b2_layernorm_f32(nv.ptr(x), nv.ptr(w[0]), nv.ptr(w[1]), nv.ptr(h), nv.ptr(rows), M, x.shape[1], n, nv.ctypes.c_float(eps),
                                       _f32(h), nv.stream_ptr()), "layernorm_f32")
    nv.count_launch()
    return h


def embedding_pairs(ids: torch.Tensor, table: torch.Tensor, pairs: torch.Tensor, last: torch.Tensor, p: Portions, vocab: int,
                    mul_prev: int, mul_cur: int, w: Norm, n: int, eps: float, next_norm: Norm) -> Tuple[torch.Tensor, torch.Tensor]:
    """Layer norm of ``table[id] + pairs[(before * mul_prev + id * mul_cur) mod buckets]``, ``before`` being the sequence's token before
    this one; the first token of a sequence takes the last of the ``buckets + 1`` rows.  ``last [slots]`` int32 keeps every sequence's
    last token between steps.  Returns the rows in 32-bit and their layer norm with ``next_norm`` in the table's dtype."""
    buckets = pairs.shape[0] - 1
    if not table.is_cuda:
        cu, slots, row = p.cu.tolist(), p.slots.tolist(), torch.full((ids.numel(),), buckets)
        for s, start in enumerate(p.starts.tolist()):
            a, e = cu[s], cu[s + 1]
            if e > a and slots[s] >= 0:
                before = torch.cat([last[slots[s]].reshape(1).long(), ids[a:e - 1].long()])
                row[a:e] = (before * mul_prev + ids[a:e].long() * mul_cur) % buckets
                if start == 0:
                    row[a] = buckets
                last[slots[s]] = ids[e - 1]
        x = _layer_norm(table[ids].float() + pairs[row].float(), w, n, eps)
        return x, _layer_norm(x, next_norm, n, eps).to(table.dtype)
    x = torch.empty((ids.numel(), table.shape[1]), device=table.device, dtype=torch.float32)
    h = torch.empty(x.shape, device=x.device, dtype=table.dtype)
    cl = nv.ctypes.c_longlong
    nv.check(nv.lib().b2_embed_pairs(
        nv.ptr(ids), nv.ptr(table), nv.ptr(pairs), nv.ptr(last), nv.ptr(p.cu), nv.ptr(p.row_seq), nv.ptr(p.positions), nv.ptr(p.slots),
        nv.ptr(w[0]), nv.ptr(w[1]), nv.ptr(next_norm[0]), nv.ptr(next_norm[1]), nv.ptr(x), nv.ptr(h), ids.numel(), x.shape[1], n, vocab,
        cl(buckets), cl(mul_prev), cl(mul_cur), nv.ctypes.c_float(eps), _f32(table), nv.stream_ptr()), "embed_pairs")
    nv.count_launch()
    return x, h


def branch_add(x: torch.Tensor, y, w: Norm, n: int, eps: float, gate: Optional[torch.Tensor] = None, gate_bias: Optional[torch.Tensor] = None,
               scale: Optional[torch.Tensor] = None, next_norm: Optional[Norm] = None) -> Optional[torch.Tensor]:
    """In place ``x += scale * norm(y * sigmoid(gate + gate_bias))``, the layer norm having weight and bias ``w``; returns the layer norm
    of the new ``x`` with ``next_norm`` in the weights' dtype when that is given.  ``y``: fp32 ``[M, ld]``, or ``(rows, routing)``: the
    weighted sum of every token's expert rows.  ``gate [M, ld]`` (a column slice, fp32 or the weights' dtype), ``gate_bias`` and
    ``scale [ld]`` are optional."""
    rows, r = y if isinstance(y, tuple) else (None, None)
    if not x.is_cuda:
        t = y if r is None else (rows[r.place.long()].float() * r.weights[:, :, None]).sum(1)
        if gate is not None:
            t = t * torch.sigmoid(gate.float() + gate_bias.float())
        t = _layer_norm(t, w, n, eps)
        x += t if scale is None else scale.float() * t
        return None if next_norm is None else _layer_norm(x, next_norm, n, eps).to(w[0].dtype)
    h = None if next_norm is None else torch.empty(x.shape, device=x.device, dtype=w[0].dtype)
    nw, nb = (None, None) if next_norm is None else next_norm
    assert gate is None or (gate.stride(1) == 1 and gate.dtype in (torch.float32, w[0].dtype))
    nv.check(nv.lib().b2_branch_add(
        nv.ptr(x), nv.ptr(None if r is not None else y), nv.ptr(rows), nv.ptr(None if r is None else r.place),
        nv.ptr(None if r is None else r.weights), 0 if r is None else r.place.shape[1], 0 if r is None else rows.shape[0], nv.ptr(gate),
        nv.ctypes.c_longlong(0 if gate is None else gate.stride(0)), int(gate is not None and gate.dtype == torch.float32),
        nv.ptr(gate_bias), nv.ptr(w[0]), nv.ptr(w[1]), nv.ptr(scale), nv.ptr(nw), nv.ptr(nb), nv.ptr(h), x.shape[0], x.shape[1], n,
        nv.ctypes.c_float(eps), _f32(w[0]), nv.stream_ptr()), "branch_add")
    nv.count_launch()
    return h


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return torch.nn.functional.gelu(z, approximate="tanh")


def gelu_times_token(gate: torch.Tensor, table: torch.Tensor, ids: torch.Tensor, first: int, vocab: int) -> torch.Tensor:
    """``gelu_tanh(gate) * table[ids, first : first + n]`` with ``gate [M, n]``; ids outside ``[0, vocab)`` give zeros on a GPU."""
    M, n = gate.shape
    if not gate.is_cuda:
        return (gelu_tanh(gate.float()) * table[ids, first:first + n].float()).to(gate.dtype)
    out = torch.empty((M, n), device=gate.device, dtype=gate.dtype)
    assert gate.stride(1) == 1 and table.stride(1) == 1
    nv.check(nv.lib().b2_gelu_token(nv.ptr(gate), nv.ptr(table), nv.ptr(ids), nv.ptr(out), M, n, gate.stride(0),
                                    nv.ctypes.c_longlong(table.stride(0)), first, vocab, _f32(gate), nv.stream_ptr()), "gelu_token")
    nv.count_launch()
    return out


def glu(gate: torch.Tensor, up: torch.Tensor, out: torch.Tensor) -> None:
    """``out = silu(gate) * up``; the three are column slices (``gate`` and ``up`` of one matrix)."""
    if not gate.is_cuda:
        g = gate.float()
        out.copy_((g * torch.sigmoid(g) * up.float()).to(out.dtype))
        return
    assert gate.stride(0) == up.stride(0)
    nv.check(nv.lib().b2_glu(nv.ptr(gate), nv.ptr(up), nv.ptr(out), gate.shape[0], gate.shape[1], gate.stride(0),
                             out.stride(0), _f32(gate), nv.stream_ptr()), "glu")
    nv.count_launch()


def rope_turns(base: float, dims: int, device, stretch: Optional[Tuple[float, float, float, float]] = None) -> torch.Tensor:
    """Turns per position ``base^(-2 i / dims) / (2 pi)`` for i < dims / 2, in double precision.

    ``stretch = (factor, low, high, original)`` slows the low frequencies for contexts longer than ``original``: a pair that turns
    fewer than ``low`` times over ``original`` positions is slowed by ``factor``, one that turns more than ``high`` times is kept,
    and between the two the frequency is blended linearly."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims) / (2.0 * math.pi)
        if stretch is not None:
            factor, low, high, original = stretch
            turns = original * f
            if turns < low:
                f /= factor
            elif turns <= high:
                s = (turns - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64, device=device)


def rope_rows(positions: torch.Tensor, turns: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """fp32 ``cos`` / ``sin`` ``[rows, dims/2]`` of every row's position: no table bounds the context length."""
    M, half = positions.numel(), turns.numel()
    if not positions.is_cuda:
        a = positions.double()[:, None] * turns[None, :] * (2.0 * math.pi)
        return a.cos().float(), a.sin().float()
    cs = torch.empty((M, half), device=positions.device, dtype=torch.float32)
    sn = torch.empty_like(cs)
    nv.check(nv.lib().b2_rope_rows(nv.ptr(positions), nv.ptr(turns), nv.ptr(cs), nv.ptr(sn), M, half, nv.stream_ptr()),
             "rope_rows")
    nv.count_launch()
    return cs, sn
