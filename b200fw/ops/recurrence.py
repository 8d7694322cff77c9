"""Gated linear recurrence with one state per channel: a short causal convolution, block-diagonal input and recurrence gates, and

    log a = -8 r softplus(lam),   S <- a S + sqrt(1 - a^2) i u,   out = S gelu(y)

Channels are laid out in blocks padded to a multiple of eight (``np`` channels each); padding channels stay zero."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _native as nv
from .linear_state import _cpu_sequences
from .portions import Portions
from .residual import _f32, gelu_tanh

DECAY_RATE = 8.0      # a = sigmoid-gated exp(-DECAY_RATE softplus(lam))


def causal_conv(x: torch.Tensor, x_bias: Optional[torch.Tensor], taps: torch.Tensor, bias: Optional[torch.Tensor],
                conv_state: torch.Tensor, p: Portions, add_input: bool = False) -> torch.Tensor:
    """Per channel ``sum_j taps[:, K-1-j] (x + x_bias)[t - j] + bias``, zeros before the sequence's start; ``add_input``: and the
    input itself, ``(x + x_bias)[t]``.  ``x [M, C]`` (a column slice), ``taps [C, K]``; the K - 1 inputs before the portion come from
    ``conv_state [slots, C, K-1]``, which is replaced."""
    M, C = x.shape
    K = taps.shape[1]
    if not x.is_cuda:
        xf, tf = x.float() + (0 if x_bias is None else x_bias.float()), taps.float()
        u = torch.zeros(M, C)
        for a, e, start, slot in _cpu_sequences(p):
            past = torch.zeros(K - 1, C) if start == 0 else conv_state[slot].t()
            full = torch.cat([past, xf[a:e]], 0)
            for j in range(K):
                u[a:e] += tf[:, j] * full[j:j + e - a]
            if bias is not None:
                u[a:e] += bias.float()
            if add_input:
                u[a:e] += xf[a:e]
            conv_state[slot] = full[full.shape[0] - (K - 1):].t()
        return u.to(x.dtype)
    u = torch.empty((M, C), device=x.device, dtype=x.dtype)
    nv.check(nv.lib().b2_causal_conv(
        nv.ptr(x), nv.ctypes.c_longlong(x.stride(0)), nv.ptr(x_bias), nv.ptr(taps), nv.ptr(bias), nv.ptr(conv_state), nv.ptr(u),
        nv.ptr(p.cu), nv.ptr(p.starts), nv.ptr(p.slots), nv.ptr(p.tiles), p.tiles.shape[0], C, K, int(add_input), _f32(x),
        nv.stream_ptr()), "causal_conv")
    nv.count_launch()
    return u


def block_gates(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``w [B, 2*np, np]`` (recurrence gate over input gate) times every block of ``u [M, B*np]``: fp32 ``[M, B*2*np]``."""
    B, n2, n = w.shape
    if not u.is_cuda:
        return torch.einsum("mbk,bnk->mbn", u.reshape(-1, B, n).float(), w.float()).reshape(-1, B * n2)
    out = torch.empty((u.shape[0], B * n2), device=u.device, dtype=torch.float32)
    nv.check(nv.lib().b2_head_linear(
        nv.ptr(u), nv.ptr(w), nv.ptr(out), nv.ctypes.c_longlong(u.stride(0)), nv.ctypes.c_longlong(out.stride(0)), u.shape[0], B, n2, n,
        n, n2, 0, None, None, 0, 0, None, nv.ctypes.c_longlong(0), _f32(u), 1, nv.stream_ptr()), "head_linear")
    nv.count_launch()
    return out


def linear_recurrence(u: torch.Tensor, z: torch.Tensor, z_bias: torch.Tensor, lam: torch.Tensor, y: torch.Tensor, y_bias: torch.Tensor,
                      out: torch.Tensor, state: torch.Tensor, p: Portions, block: int, short_only: bool = False) -> None:
    """The recurrence over ``u [M, C]`` with gates ``r, i = sigmoid(z + z_bias)`` (``z`` as :func:`block_gates` gives it, ``z_bias``
    in its order, ``block`` = np) and ``out [M, C] = S gelu_tanh(y + y_bias)``; ``y`` and ``out`` are column slices.  ``state
    [slots, C]`` fp32.  ``short_only``: the rows of the short portions alone (``z`` may end there)."""
    M, C = u.shape
    if not u.is_cuda:
        zz = (z + z_bias.float()).reshape(M, C // block, 2, block)
        r, i = torch.sigmoid(zz[:, :, 0]).reshape(M, C), torch.sigmoid(zz[:, :, 1]).reshape(M, C)
        log_a = -DECAY_RATE * r * torch.nn.functional.softplus(lam.float())
        a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u.float()
        s = torch.zeros(M, C)
        for lo, hi, start, slot in _cpu_sequences(p):
            S = torch.zeros(C) if start == 0 else state[slot].clone()
            for t in range(lo, hi):
                S = a[t] * S + b[t]
                s[t] = S
            state[slot] = S
        out.copy_((s * gelu_tanh(y.float() + y_bias.float())).to(out.dtype))
        return
    cl = nv.ctypes.c_longlong
    for lo, cnt in ((0, p.num_short), (p.num_short, p.nseq - p.num_short)):
        if cnt <= 0 or (short_only and lo > 0):
            continue
        chunks = p.chunks64 if lo == p.num_short else None
        n = 0 if chunks is None else chunks.shape[0]
        ws = torch.empty((n, 2, 2, C), device=u.device, dtype=torch.float32) if n else None
        nv.check(nv.lib().b2_linear_recurrence(
            nv.ptr(u), cl(u.stride(0)), nv.ptr(z), cl(z.stride(0)), nv.ptr(z_bias), nv.ptr(lam), nv.ptr(y), cl(y.stride(0)), nv.ptr(y_bias),
            nv.ptr(out), cl(out.stride(0)), nv.ptr(state), nv.ptr(ws), nv.ptr(p.cu), nv.ptr(p.starts), nv.ptr(p.slots),
            nv.ptr(chunks), nv.ptr(p.first64 if n else None), n, lo, cnt, C, block, _f32(u), nv.stream_ptr()), "linear_recurrence")
        nv.count_launch(3 if n else 1)


def gated_recurrence(y: torch.Tensor, x: torch.Tensor, y_bias: torch.Tensor, x_bias: torch.Tensor, taps: torch.Tensor,
                     conv_bias: torch.Tensor, w_gates: torch.Tensor, gate_bias: torch.Tensor, lam: torch.Tensor, out: torch.Tensor,
                     state: torch.Tensor, conv_state: torch.Tensor, p: Portions) -> None:
    """Convolution, gates and recurrence of a step: ``x``, ``y`` and ``out [M, C]`` are column slices, ``w_gates [B, 2, np, np]`` and
    ``gate_bias [B, 2, np]`` hold the recurrence gate, then the input gate of every block."""
    B, _, n, _ = w_gates.shape
    u = causal_conv(x, x_bias, taps, conv_bias, conv_state, p)
    tiled = u.is_cuda and u.dtype == torch.bfloat16 and p.nseq > p.num_short and n <= 256
    if tiled:          # the long portions: gates inside the passes over them
        ns, nc, cl = p.num_short, p.chunks128.shape[0], nv.ctypes.c_longlong
        C = u.shape[1]
        ws = torch.empty((nc, 4, 2, C), device=u.device, dtype=torch.float32)
        nv.check(nv.lib().b2_gated_recurrence(
            nv.ptr(u), nv.ptr(w_gates), nv.ptr(gate_bias), nv.ptr(lam), nv.ptr(y), cl(y.stride(0)), nv.ptr(y_bias), nv.ptr(out),
            cl(out.stride(0)), nv.ptr(state), nv.ptr(ws), nv.ptr(p.starts), nv.ptr(p.slots), nv.ptr(p.chunks128), nv.ptr(p.first128), nc,
            ns, p.nseq - ns, u.shape[0], C, n, nv.stream_ptr()), "gated_recurrence")
        nv.count_launch(3)
        if ns == 0:
            return
    z = block_gates(u[:p.short_rows] if tiled else u, w_gates.view(B, 2 * n, n))
    linear_recurrence(u, z, gate_bias.view(-1), lam, y, y_bias, out, state, p, n, tiled)
