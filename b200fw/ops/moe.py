"""Mixture of experts: sigmoid scores, a choice limited to the best groups of experts, grouped products over the rows each expert
was given, and the weighted sum of a token's experts (with a gated shared expert) added to the residual through a norm."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _native as nv
from .residual import _f32


@dataclass
class Routing:
    """Which experts every token uses.  The step's (token, choice) pairs are laid out expert after expert: pair ``(t, c)`` is row
    ``place[t, c]``, and expert e owns rows ``offsets[e] : offsets[e+1]``."""
    weights: torch.Tensor        # fp32 [M, top]
    place: torch.Tensor          # int32 [M, top]
    token: torch.Tensor          # int32 [M * top] token of every row
    offsets: torch.Tensor        # int32 [E + 1]

    @property
    def experts(self) -> int:
        return self.offsets.numel() - 1


def route(logits: torch.Tensor, correction: torch.Tensor, top: int, groups: int, keep: int, scale: float) -> Routing:
    """``logits [M, >= E]`` fp32, ``correction [E]``: scores ``s = sigmoid(logits)``; the experts are ``groups`` equal groups of
    neighbours, a group counts by the sum of its two largest ``s + correction``, and the ``top`` largest ``s + correction`` of the
    ``keep`` best groups are chosen, with weight ``s * scale``.  Ties go to the lower index."""
    M, E = logits.shape[0], correction.numel()
    if not logits.is_cuda:
        s = torch.sigmoid(logits[:, :E])
        c = s + correction.float()
        if keep < groups:
            per = E // groups
            gs = c.reshape(M, groups, per).topk(min(2, per), -1).values.sum(-1)
            best = gs.sort(dim=-1, descending=True, stable=True).indices[:, :keep]
            open_ = torch.zeros(M, groups, dtype=torch.bool).scatter_(1, best, True)
            c = c.masked_fill(~open_.repeat_interleave(per, 1), float("-inf"))
        ids = c.sort(dim=-1, descending=True, stable=True).indices[:, :top]
        flat = ids.reshape(-1)
        order = flat.sort(stable=True).indices
        place = torch.empty(M * top, dtype=torch.int32)
        place[order] = torch.arange(M * top, dtype=torch.int32)
        offsets = torch.zeros(E + 1, dtype=torch.int32)
        offsets[1:] = torch.bincount(flat, minlength=E).cumsum(0)
        return Routing(s.gather(1, ids) * scale, place.reshape(M, top), (order // top).to(torch.int32), offsets)
    dev = logits.device
    r = Routing(torch.empty((M, top), device=dev, dtype=torch.float32), torch.empty((M, top), device=dev, dtype=torch.int32),
                torch.empty(M * top, device=dev, dtype=torch.int32), torch.empty(E + 1, device=dev, dtype=torch.int32))
    work = torch.empty(E + M * top, device=dev, dtype=torch.int32)      # rows per expert, then (expert, rank) of every pair
    nv.check(nv.lib().b2_moe_route(
        nv.ptr(logits), nv.ctypes.c_longlong(logits.stride(0)), nv.ptr(correction), nv.ptr(r.weights), nv.ptr(r.place), nv.ptr(r.token),
        nv.ptr(r.offsets), nv.ptr(work), M, E, top, groups, keep, nv.ctypes.c_float(scale), _f32(correction), nv.stream_ptr()), "moe_route")
    nv.count_launch(2)
    return r


def expert_glu(h: torch.Tensor, w: torch.Tensor, r: Routing) -> torch.Tensor:
    """``silu(W_gate h) * (W_up h)`` of every (token, choice) pair in the routing's row order; ``h [M, K]``, ``w [E, 2, F, K]``
    (gate, up): ``[M * top, F]``."""
    E, _, F, K = w.shape
    P = r.token.numel()
    out = torch.empty((P, F), device=h.device, dtype=h.dtype)
    if not h.is_cuda:
        off = r.offsets.tolist()
        for e in range(E):
            x = h[r.token[off[e]:off[e + 1]].long()].float()
            out[off[e]:off[e + 1]] = (torch.nn.functional.silu(x @ w[e, 0].float().t()) * (x @ w[e, 1].float().t())).to(h.dtype)
        return out
    assert h.stride(1) == 1 and w.is_contiguous()
    nv.check(nv.lib().b2_moe_glu(nv.ptr(h), nv.ctypes.c_longlong(h.stride(0)), nv.ptr(w), nv.ptr(r.token), nv.ptr(r.offsets), nv.ptr(out), h.shape[0], P, E, F,
                                 K, _f32(h), nv.stream_ptr()), "moe_glu")
    nv.count_launch()
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
        nv.ptr(x), nv.ptr(rows), nv.ptr(r.place), nv.ptr(r.weights), r.place.shape[1], nv.ptr(shared), nv.ptr(shared_gate),
        0 if shared_gate is None else shared_gate.stride(0), nv.ptr(w), nv.ptr(h), x.shape[0], x.shape[1], n, nv.ctypes.c_float(coef),
        nv.ctypes.c_float(eps), _f32(w), nv.stream_ptr()), "moe_norm_add")
    nv.count_launch()
    return x if h is None else h
