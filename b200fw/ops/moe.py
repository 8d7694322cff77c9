"""Mixture of experts: sigmoid or softmax scores, a choice limited to the best groups of experts, grouped products over the rows each
expert was given, and the weighted sum of a token's experts (with a gated shared expert) added to the residual through a norm
(:func:`b200fw.ops.branch_add` does the same through a layer norm, with a gate per channel)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from .. import _native as nv
from .gemm import gemm, linear
from .residual import _f32, gelu_times_token, glu


@dataclass
class Routing:
    """Which experts every token uses.  The step's (token, choice) pairs are laid out expert after expert: pair ``(t, c)`` is row
    ``place[t, c]``, and expert e owns rows ``offsets[e] : offsets[e+1]``."""
    weights: torch.Tensor        # fp32 [M, top]
    place: torch.Tensor          # int32 [M, top]
    token: torch.Tensor          # int32 [M * top] token of every row
    offsets: torch.Tensor        # int32 [E + 1]


def route(logits: torch.Tensor, correction: Optional[torch.Tensor], top: int, groups: int, keep: int, scale: float,
          joint: Optional[torch.Tensor] = None, score: str = "sigmoid", experts: int = 0) -> Routing:
    """``logits [M, >= E]`` fp32, ``correction [E]`` (None: zero, ``experts`` then says how many there are): scores ``s =
    sigmoid(logits)``, or their ``softmax`` over all experts; the experts are ``groups`` equal groups of neighbours, a group counts by
    the sum of its two largest ``s + correction``, and the ``top`` largest ``s + correction`` of the ``keep`` best groups are chosen,
    with weight ``s * scale``.  Ties go to the lower index."""
    M, E = logits.shape[0], experts if correction is None else correction.numel()
    assert score in ("sigmoid", "softmax") and E > 0
    if not logits.is_cuda:
        z = logits[:, :E]
        s = torch.softmax(z, -1) if score == "softmax" else torch.sigmoid(z)
        c = s + correction.float() if correction is not None else z if keep == groups else s
        if keep < groups:
            per = E // groups
            gs = c.reshape(M, groups, per).topk(min(2, per), -1).values.sum(-1)
            best = gs.sort(dim=-1, descending=True, stable=True).indices[:, :keep]
            open_ = torch.zeros(M, groups, dtype=torch.bool).scatter_(1, best, True)
            c = c.masked_fill(~open_.repeat_interleave(per, 1), float("-inf"))
        ids = c.sort(dim=-1, descending=True, stable=True).indices[:, :top]
        weights = s.gather(1, ids) * scale
        if joint is not None:
            ids, weights = torch.cat([ids, torch.full((M, 1), E)], 1), torch.cat([weights, torch.sigmoid(joint)[:, None]], 1)
            E, top = E + 1, top + 1
        flat = ids.reshape(-1)
        order = flat.sort(stable=True).indices
        place = torch.empty(M * top, dtype=torch.int32)
        place[order] = torch.arange(M * top, dtype=torch.int32)
        offsets = torch.zeros(E + 1, dtype=torch.int32)
        offsets[1:] = torch.bincount(flat, minlength=E).cumsum(0)
        return Routing(weights, place.reshape(M, top), (order // top).to(torch.int32), offsets)
    more = int(joint is not None)
    r, work = _routing(M, E + more, top + more, logits.device)
    nv.check(nv.lib().b2_moe_route(
        nv.ptr(logits), nv.ctypes.c_longlong(logits.stride(0)), nv.ptr(joint), nv.ctypes.c_longlong(joint.stride(0) if more else 0), more,
        nv.ptr(correction), nv.ptr(r.weights), nv.ptr(r.place), nv.ptr(r.token),
        nv.ptr(r.offsets), nv.ptr(work), M, E, top, groups, keep, nv.ctypes.c_float(scale), int(score == "softmax"),
        int(correction is not None and correction.dtype == torch.float32), nv.stream_ptr()), "moe_route")
    nv.count_launch(2 if M * (top + more) <= 16384 else 3)
    return r


def _routing(M: int, E: int, top: int, dev):
    r = Routing(torch.empty((M, top), device=dev, dtype=torch.float32), torch.empty((M, top), device=dev, dtype=torch.int32),
                torch.empty(M * top, device=dev, dtype=torch.int32), torch.empty(E + 1, device=dev, dtype=torch.int32))
    return r, torch.empty(E + M * top, device=dev, dtype=torch.int32)      # rows per expert, then the expert of every pair


def router(h: torch.Tensor, w: torch.Tensor, shared_row: int, correction: torch.Tensor, top: int, groups: int, keep: int, scale: float,
           joint: bool = False):
    """Router product in 32-bit and :func:`route`: ``h [M, K]``, ``w [>= E, K]`` with the experts' rows first; ``shared_row >= 0``: that
    row's product is the shared expert's gate, ``joint``: of a shared expert that is expert E.  Returns ``(Routing, gate [M])``, the gate
    None without a shared expert and with a joint one."""
    M, E, N = h.shape[0], correction.numel(), w.shape[0]
    if not h.is_cuda or h.dtype != torch.bfloat16 or N > SKINNY:
        z = linear_fp32(h, w)
        gate = None if shared_row < 0 else z[:, shared_row]
        return route(z, correction, top, groups, keep, scale, gate if joint else None), None if joint else gate
    more = int(joint)
    r, work = _routing(M, E + more, top + more, h.device)
    gate = torch.empty(M, device=h.device, dtype=torch.float32) if shared_row >= 0 and not joint else None
    cl = nv.ctypes.c_longlong
    nv.check(nv.lib().b2_moe_router(
        nv.ptr(h), cl(h.stride(0)), nv.ptr(w), cl(w.stride(0)), N, h.shape[1], shared_row, nv.ptr(gate), more,
        nv.ptr(correction), nv.ptr(r.weights), nv.ptr(r.place), nv.ptr(r.token), nv.ptr(r.offsets), nv.ptr(work), M, E, top, groups, keep,
        nv.ctypes.c_float(scale), 0, nv.stream_ptr()), "moe_router")
    nv.count_launch(2 if M * (top + more) <= 16384 else 3)
    return r, gate


GATHER_ROWS = 16  # rows per expert (on average) from which they are laid out before the product
SKINNY = 72      # outputs of a product that take the kernel for few of them


def linear_fp32(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``x [M, K] w [N, K]^T`` with a 32-bit result."""
    z = torch.empty((x.shape[0], w.shape[0]), dtype=torch.float32, device=x.device)
    if not x.is_cuda or x.dtype != torch.bfloat16 or w.shape[0] > SKINNY:
        return gemm(x, w, out=z)
    cl = nv.ctypes.c_longlong
    nv.check(nv.lib().b2_skinny(nv.ptr(x), cl(x.stride(0)), nv.ptr(w), cl(w.stride(0)), nv.ptr(z), cl(z.stride(0)), x.shape[0], w.shape[0],
                                x.shape[1], nv.stream_ptr()), "skinny")
    nv.count_launch()
    return z


def token_gate(h: torch.Tensor, w: torch.Tensor, table: torch.Tensor, ids: torch.Tensor, first: int, vocab: int) -> torch.Tensor:
    """``gelu_tanh(h w^T) * table[ids, first : first + N]``, ``w [N, K]``."""
    M, N = h.shape[0], w.shape[0]
    if not h.is_cuda or h.dtype != torch.bfloat16 or M > 1024:
        return gelu_times_token(linear(h, w), table, ids, first, vocab)
    out = torch.empty((M, N), device=h.device, dtype=h.dtype)
    cl = nv.ctypes.c_longlong
    nv.check(nv.lib().b2_token_gate(nv.ptr(h), cl(h.stride(0)), nv.ptr(w), cl(w.stride(0)), nv.ptr(table), cl(table.stride(0)), nv.ptr(ids),
                                    nv.ptr(out), M, N, h.shape[1], first, vocab, nv.stream_ptr()), "token_gate")
    nv.count_launch()
    return out


def glu_linear(h: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """``out [M, F] = silu(W_gate h) * (W_up h)`` with ``w [2 F, K]``: gate rows, then up rows."""
    F = out.shape[1]
    if not h.is_cuda or h.dtype != torch.bfloat16:
        y = linear(h, w)
        return glu(y[:, :F], y[:, F:], out)
    assert w.is_contiguous() and w.shape[0] == 2 * F and h.stride(1) == 1
    cl = nv.ctypes.c_longlong
    nv.check(nv.lib().b2_rows_glu(nv.ptr(h), cl(h.stride(0)), nv.ptr(w), nv.ptr(out), cl(out.stride(0)), h.shape[0], F, h.shape[1],
                                  nv.stream_ptr()), "rows_glu")
    nv.count_launch()


def expert_glu(h: torch.Tensor, w: torch.Tensor, r: Routing, clamped: Optional[Tuple[float, float]] = None) -> torch.Tensor:
    """``silu(W_gate h) * (W_up h)`` of every (token, choice) pair in the routing's row order; ``h [M, K]``, ``w [E, 2, F, K]``
    (gate, up): ``[M * top, F]``.  ``clamped = (alpha, limit)``: with ``g = min(W_gate h, limit)`` and ``u = clamp(W_up h, -limit,
    limit)`` it is ``g sigmoid(alpha g) (u + 1)`` instead."""
    E, _, F, K = w.shape
    P = r.token.numel()
    out = torch.empty((P, F), device=h.device, dtype=h.dtype)
    if not h.is_cuda:
        off = r.offsets.tolist()
        for e in range(E):
            x = h[r.token[off[e]:off[e + 1]].long()].float()
            g, u = x @ w[e, 0].float().t(), x @ w[e, 1].float().t()
            if clamped is not None:
                alpha, limit = clamped
                g, u = g.clamp(max=limit), u.clamp(-limit, limit)
                y = g * torch.sigmoid(alpha * g) * (u + 1.0)
            else:
                y = torch.nn.functional.silu(g) * u
            out[off[e]:off[e + 1]] = y.to(h.dtype)
        return out
    alpha, limit = clamped if clamped is not None else (0.0, 0.0)
    assert h.stride(1) == 1 and w.is_contiguous()
    rows = torch.empty((P, K), device=h.device, dtype=h.dtype) if h.dtype == torch.bfloat16 and P >= GATHER_ROWS * E else None
    nv.check(nv.lib().b2_moe_glu(nv.ptr(h), nv.ctypes.c_longlong(h.stride(0)), nv.ptr(w), nv.ptr(r.token), nv.ptr(r.offsets), nv.ptr(rows),
                                 nv.ptr(out), h.shape[0], P, E, F, K, int(clamped is not None), nv.ctypes.c_float(alpha),
                                 nv.ctypes.c_float(limit), _f32(h), nv.stream_ptr()), "moe_glu")
    nv.count_launch(1 if rows is None else 2)
    return out


def expert_down(a: torch.Tensor, w: torch.Tensor, r: Routing) -> torch.Tensor:
    """``W_e a`` of every row, ``a [P, F]``, ``w [E, N, F]``: ``[P, N]`` in ``a``'s dtype."""
    E, N, F = w.shape
    P = a.shape[0]
    out = torch.empty((P, N), device=a.device, dtype=a.dtype)
    if not a.is_cuda:
        off = r.offsets.tolist()
        for e in range(E):
            out[off[e]:off[e + 1]] = (a[off[e]:off[e + 1]].float() @ w[e].float().t()).to(a.dtype)
        return out
    assert a.is_contiguous() and w.is_contiguous()
    nv.check(nv.lib().b2_moe_down(nv.ptr(a), nv.ptr(w), nv.ptr(r.offsets), nv.ptr(out), P, E, N, F, _f32(a), nv.stream_ptr()), "moe_down")
    nv.count_launch()
    return out


def moe_norm_add(x: torch.Tensor, rows: torch.Tensor, r: Routing, shared: Optional[torch.Tensor], shared_gate: Optional[torch.Tensor],
                 w: torch.Tensor, coef: float, n: int, eps: float) -> torch.Tensor:
    """With ``y = sum_c weights[t, c] rows[place[t, c]] + sigmoid(shared_gate) shared`` (``shared [M, N]`` fp32, ``shared_gate [M]``
    fp32): in place ``x += coef * rms(y) * w``; returns the new ``x`` in ``w``'s dtype (``x`` itself in 32-bit)."""
    if not x.is_cuda:
        y = (rows[r.place.long()].float() * r.weights[:, :, None]).sum(1)
        if shared is not None:
            y = y + torch.sigmoid(shared_gate)[:, None] * shared
        x += coef * y * torch.rsqrt((y[:, :n] * y[:, :n]).mean(-1, keepdim=True) + eps) * w.float()
        return x if w.dtype == torch.float32 else x.to(w.dtype)
    h = None if w.dtype == torch.float32 else torch.empty(x.shape, device=x.device, dtype=w.dtype)
    nv.check(nv.lib().b2_moe_norm_add(
        nv.ptr(x), nv.ptr(rows), nv.ptr(r.place), nv.ptr(r.weights), r.place.shape[1], rows.shape[0], nv.ptr(shared), nv.ptr(shared_gate),
        0 if shared_gate is None else shared_gate.stride(0), nv.ptr(w), nv.ptr(h), x.shape[0], x.shape[1], n, nv.ctypes.c_float(coef),
        nv.ctypes.c_float(eps), _f32(w), nv.stream_ptr()), "moe_norm_add")
    nv.count_launch()
    return x if h is None else h
