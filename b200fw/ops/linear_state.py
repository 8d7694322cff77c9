"""Linear-attention recurrences over per-sequence state slots: retention (one fixed decay per head), the gated delta rule
(one learned decay per head and key channel), with the delta rule's input stage, and matrix memory (exponential input and
forget gates per head, normalised).

All head sizes are stored padded to a multiple of eight (``dkp``, ``dvp``); ``dk``, ``dv`` are the real ones.  States are
fp32 ``[slots, H, dkp, dvp]``; a sequence whose portion starts at position 0 starts from zero whatever its slot holds."""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from .. import _native as nv
from .portions import Portions, pad8


def _sub(p: Portions, lo: int):
    """Pointers to the per-sequence arrays from sequence ``lo`` on (row numbers stay absolute)."""
    return nv.ptr(p.cu[lo:]), nv.ptr(p.starts[lo:]), nv.ptr(p.slots[lo:])


def _cpu_sequences(p: Portions):
    cu, starts, slots = p.cu.tolist(), p.starts.tolist(), p.slots.tolist()
    for s in range(p.nseq):
        if slots[s] >= 0 and cu[s + 1] > cu[s]:
            yield cu[s], cu[s + 1], starts[s], slots[s]


def _head_rms(o: torch.Tensor, dv: int, eps: float) -> torch.Tensor:
    return o * torch.rsqrt((o * o).sum(-1, keepdim=True) / dv + eps)


def retention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: torch.Tensor, out: torch.Tensor, state: torch.Tensor,
              p: Portions, decay: torch.Tensor, dk: int, dv: int, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor],
              k_scale: float, eps: float, norm_w: Optional[torch.Tensor] = None, sumsq: Optional[torch.Tensor] = None) -> None:
    """``S <- decay_h S + k v^T``, ``o = S^T q`` with rotary positions on q and k and ``k_scale`` on the rotated k; then
    ``out = o / rms(o) * silu(gate)`` per head.  ``q, k [M, H*dkp]``, ``v, gate, out [M, H*dvp]`` are column slices
    (the first four of one matrix).

    ``sumsq [M, H]`` (fp32, written): the heads are normed together, by whoever reads ``out``'s projection; then
    ``out = o * norm_w * sigmoid(gate)`` with ``norm_w [H*dvp]``, and ``sumsq`` holds every head's ``sum(o^2)``."""
    H, dkp, dvp = state.shape[1:]
    rot = 0 if cos is None else 2 * cos.shape[1]
    if not q.is_cuda:
        M = q.shape[0]
        qf, kf = q.reshape(M, H, dkp).float(), k.reshape(M, H, dkp).float()
        if rot:
            h = rot // 2
            c, s = cos[:, None, :], sin[:, None, :]

            def turn(x):
                u, w = x[..., :h], x[..., h:rot]
                return torch.cat([u * c - w * s, w * c + u * s, x[..., rot:]], -1)
            qf, kf = turn(qf), turn(kf)
        kf = kf * k_scale
        vf, gf = v.reshape(M, H, dvp).float(), gate.reshape(M, H, dvp).float()
        o = torch.zeros(M, H, dvp)
        for a, b, start, slot in _cpu_sequences(p):
            S = torch.zeros(H, dkp, dvp) if start == 0 else state[slot].clone()
            for t in range(a, b):
                S = decay[:, None, None] * S + kf[t, :, :, None] * vf[t, :, None, :]
                o[t] = (S * qf[t, :, :, None]).sum(1)
            state[slot] = S
        if sumsq is not None:
            sumsq.copy_((o * o).sum(-1))
            out.copy_((o * norm_w.float().reshape(H, dvp) * torch.sigmoid(gf)).reshape(M, H * dvp).to(out.dtype))
            return
        out.copy_((_head_rms(o, dv, eps) * gf * torch.sigmoid(gf)).reshape(M, H * dvp).to(out.dtype))
        return
    assert q.stride(0) == k.stride(0) == v.stride(0) == gate.stride(0)
    ns = p.num_short
    if ns:
        cu, st, sl = _sub(p, 0)
        nv.check(nv.lib().b2_retention_serial(
            nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ptr(gate), nv.ptr(out), nv.ptr(state), nv.ptr(decay), nv.ptr(cos), nv.ptr(sin),
            cu, st, sl, ns, p.max_short, H, dk, dkp, dv, dvp, rot, nv.ctypes.c_longlong(q.stride(0)),
            nv.ctypes.c_longlong(out.stride(0)), nv.ctypes.c_float(k_scale), nv.ctypes.c_float(eps), nv.ptr(norm_w), nv.ptr(sumsq),
            int(q.dtype == torch.float32), nv.stream_ptr()), "retention_serial")
        nv.count_launch()
    if p.nseq > ns:
        nlong, n = p.nseq - ns, p.chunks128.shape[0]
        if q.dtype == torch.bfloat16 and dkp <= 128 and dvp <= 128:
            ws = torch.empty((n, H, dkp, dvp), device=q.device, dtype=torch.float32)
            nv.check(nv.lib().b2_retention_chunk(
                nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ptr(gate), nv.ptr(out), nv.ptr(ws), nv.ptr(state), nv.ptr(decay), nv.ptr(cos),
                nv.ptr(sin), nv.ptr(p.chunks128), nv.ptr(p.first128), nv.ptr(p.starts), nv.ptr(p.slots), n, ns, nlong, H, dk, dkp,
                dv, dvp, rot, nv.ctypes.c_longlong(q.stride(0)), nv.ctypes.c_longlong(out.stride(0)),
                nv.ctypes.c_float(k_scale), nv.ctypes.c_float(eps), nv.ptr(norm_w), nv.ptr(sumsq), nv.stream_ptr()), "retention_chunk")
            nv.count_launch(3)
            return
        cu, st, sl = _sub(p, ns)
        nv.check(nv.lib().b2_retention_serial(
            nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ptr(gate), nv.ptr(out), nv.ptr(state), nv.ptr(decay), nv.ptr(cos), nv.ptr(sin),
            cu, st, sl, nlong, p.max_long, H, dk, dkp, dv, dvp, rot, nv.ctypes.c_longlong(q.stride(0)),
            nv.ctypes.c_longlong(out.stride(0)), nv.ctypes.c_float(k_scale), nv.ctypes.c_float(eps), nv.ptr(norm_w), nv.ptr(sumsq),
            int(q.dtype == torch.float32), nv.stream_ptr()), "retention_serial")
        nv.count_launch()


def delta_inputs(x: torch.Tensor, taps: torch.Tensor, b: torch.Tensor, a2: torch.Tensor, A_log: torch.Tensor,
                 dt_bias: torch.Tensor, conv_state: torch.Tensor, p: Portions, G: int, dk: int, dv: int, q_scale: float,
                 unit_eps: float = 1e-6) -> Tuple[torch.Tensor, ...]:
    """Input stage of the gated delta rule.  ``x [M, C]`` = projected ``q (G heads) | k (G heads) | v (H heads)``; every
    channel passes a causal convolution over time (``taps [C, K]``, last column = current token; the K - 1 inputs before
    the portion come from ``conv_state [slots, C, K-1]``, which is replaced) and silu; q and k become unit vectors per
    head, q times ``q_scale``; ``beta = sigmoid(b)``; log decays ``-exp(A_log) softplus(a2 + dt_bias)``.
    Returns ``q, k [M, G*dkp]`` fp32, ``v [M, H*dvp]``, ``log_decay [M, H*dkp]`` fp32, ``beta [M, H]`` fp32."""
    M, C = x.shape
    K, H = taps.shape[1], A_log.numel()
    dkp, dvp = pad8(dk), pad8(dv)
    assert C == 2 * G * dkp + H * dvp == taps.shape[0]
    if not x.is_cuda:
        xf, tf = x.float(), taps.float()
        y = torch.zeros(M, C)
        for a, e, start, slot in _cpu_sequences(p):
            past = torch.zeros(K - 1, C) if start == 0 else conv_state[slot].t()
            full = torch.cat([past, xf[a:e]], 0)
            for j in range(K):
                y[a:e] += tf[:, j] * full[j:j + e - a]
            conv_state[slot] = full[full.shape[0] - (K - 1):].t()
        y = y * torch.sigmoid(y)

        def unit(t):
            return t * torch.rsqrt((t * t).sum(-1, keepdim=True) + unit_eps)
        w = G * dkp
        q = unit(y[:, :w].reshape(M, G, dkp)).reshape(M, w) * q_scale
        k = unit(y[:, w:2 * w].reshape(M, G, dkp)).reshape(M, w)
        v = y[:, 2 * w:].to(x.dtype)
        z = a2.float() + dt_bias.float()
        g = (-A_log.float().exp())[None, :, None] * torch.nn.functional.softplus(z).reshape(M, H, dkp)
        return q, k, v, g.reshape(M, H * dkp), torch.sigmoid(b.float())
    dev = x.device
    q = torch.empty((M, G * dkp), device=dev, dtype=torch.float32)
    k = torch.empty_like(q)
    v = torch.empty((M, H * dvp), device=dev, dtype=x.dtype)
    g = torch.empty((M, H * dkp), device=dev, dtype=torch.float32)
    beta = torch.empty((M, H), device=dev, dtype=torch.float32)
    assert b.stride(0) == x.stride(0)
    nv.check(nv.lib().b2_delta_prep(
        nv.ptr(x), nv.ptr(taps), nv.ptr(b), nv.ptr(a2), nv.ptr(A_log), nv.ptr(dt_bias), nv.ptr(conv_state), nv.ptr(q), nv.ptr(k),
        nv.ptr(v), nv.ptr(g), nv.ptr(beta), nv.ptr(p.cu), nv.ptr(p.starts), nv.ptr(p.slots), nv.ptr(p.tiles), p.tiles.shape[0],
        H, G, dk, dkp, dv, dvp, K, nv.ctypes.c_longlong(x.stride(0)), nv.ctypes.c_longlong(a2.stride(0)),
        nv.ctypes.c_float(q_scale), nv.ctypes.c_float(unit_eps), int(x.dtype == torch.float32), nv.stream_ptr()), "delta_prep")
    nv.count_launch()
    return q, k, v, g, beta


def gated_delta(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, log_decay: torch.Tensor, beta: torch.Tensor,
                gate: torch.Tensor, norm_w: Optional[torch.Tensor], out: torch.Tensor, state: torch.Tensor, p: Portions,
                G: int, dk: int, dv: int, eps: float) -> None:
    """``S <- exp(log_decay) . S``, ``u = beta (v - S^T k)``, ``S <- S + k u^T``, ``o = S^T q``; then
    ``out = o / rms(o) * norm_w * sigmoid(gate)`` per head.  Inputs as :func:`delta_inputs` returns them; ``gate`` is
    fp32 ``[M, H*dvp]`` (may be a column slice), ``out [M, H*dvp]``.  Head h uses q / k head ``h // (H / G)``."""
    H, dkp, dvp = state.shape[1:]
    if not v.is_cuda:
        M = v.shape[0]
        of = torch.arange(H) // (H // G)
        qf, kf = q.reshape(M, G, dkp)[:, of], k.reshape(M, G, dkp)[:, of]
        vf, g = v.reshape(M, H, dvp).float(), log_decay.reshape(M, H, dkp).exp()
        o = torch.zeros(M, H, dvp)
        for a, b, start, slot in _cpu_sequences(p):
            S = torch.zeros(H, dkp, dvp) if start == 0 else state[slot].clone()
            for t in range(a, b):
                S = g[t, :, :, None] * S
                u = beta[t, :, None] * (vf[t] - (S * kf[t, :, :, None]).sum(1))
                S = S + kf[t, :, :, None] * u[:, None, :]
                o[t] = (S * qf[t, :, :, None]).sum(1)
            state[slot] = S
        o = _head_rms(o, dv, eps)
        if norm_w is not None:
            o = o * norm_w.float()
        out.copy_((o.reshape(M, H * dvp) * torch.sigmoid(gate)).to(out.dtype))
        return
    assert gate.dtype == torch.float32
    for lo, n, longest in ((0, p.num_short, p.max_short), (p.num_short, p.nseq - p.num_short, p.max_long)):
        if n <= 0:
            continue
        if lo == p.num_short and p.chunks64 is not None and v.dtype == torch.bfloat16 and dkp <= 128 and dvp <= 128:
            nc = p.chunks64.shape[0]
            ws = torch.empty(nc * H * nv.lib().b2_delta_chunk_words(dkp, dvp), device=v.device, dtype=torch.int32)
            o = torch.empty((v.shape[0], H * dvp), device=v.device, dtype=torch.float32)
            nv.check(nv.lib().b2_delta_chunk(
                nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ptr(log_decay), nv.ptr(beta), nv.ptr(gate), nv.ptr(norm_w), nv.ptr(out),
                nv.ptr(state), nv.ptr(ws), nv.ptr(o), nv.ptr(p.chunks64), nv.ptr(p.first64), nv.ptr(p.starts), nv.ptr(p.slots),
                nc, lo, n, p.short_rows, p.rows - p.short_rows, H, G, dk, dkp, dv, dvp, nv.ctypes.c_longlong(gate.stride(0)),
                nv.ctypes.c_longlong(out.stride(0)), nv.ctypes.c_float(eps), nv.stream_ptr()), "delta_chunk")
            nv.count_launch(3)
            continue
        cu, st, sl = _sub(p, lo)
        nv.check(nv.lib().b2_delta_serial(
            nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ptr(log_decay), nv.ptr(beta), nv.ptr(gate), nv.ptr(norm_w), nv.ptr(out),
            nv.ptr(state), cu, st, sl, n, longest, H, G, dk, dkp, dv, dvp, nv.ctypes.c_longlong(gate.stride(0)),
            nv.ctypes.c_longlong(out.stride(0)), nv.ctypes.c_float(eps), int(v.dtype == torch.float32), nv.stream_ptr()),
            "delta_serial")
        nv.count_launch()


MEMORY_EPS = 1e-6     # added to the normaliser


def matrix_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: torch.Tensor, zi: torch.Tensor, zf: torch.Tensor,
                  bi: torch.Tensor, bf: torch.Tensor, out: torch.Tensor, S: torch.Tensor, n: torch.Tensor, m: torch.Tensor,
                  p: Portions, norm_w: torch.Tensor, dk: int, dv: int, cap: float, q_scale: float, out_scale: float,
                  eps: float) -> None:
    """Log gates ``i = cap tanh((zi + bi) / cap)``, ``f = logsigmoid(cap tanh((zf + bf) / cap))`` per head; with a running maximum
    ``m <- max(f + m, i)`` (from 0), ``S <- e^(f + m_old - m) S + e^(i - m) k v^T`` and ``n`` likewise with k alone,
    ``o = S^T q / (max(|n . q|, e^-m) + 1e-6)`` for ``q_scale q``; then ``out = rms(o) norm_w sigmoid(gate) out_scale``, the norm
    per head.  ``q, k [M, H*dkp]``, ``v, gate, out [M, H*dvp]`` are column slices (the first four of one matrix), ``zi, zf
    [M, H]`` fp32 column slices of one matrix, ``norm_w [H*dvp]``; ``S [slots, H, dkp, dvp]``, ``n [slots, H, dkp]``,
    ``m [slots, H]``."""
    H, dkp, dvp = S.shape[1:]
    if not q.is_cuda:
        M = q.shape[0]
        i = cap * torch.tanh((zi + bi.float()) / cap)
        f = torch.nn.functional.logsigmoid(cap * torch.tanh((zf + bf.float()) / cap))
        qf, kf = q.reshape(M, H, dkp).float() * q_scale, k.reshape(M, H, dkp).float()
        vf, gf = v.reshape(M, H, dvp).float(), gate.reshape(M, H, dvp).float()
        o = torch.zeros(M, H, dvp)
        for a, b, start, slot in _cpu_sequences(p):
            fresh = start == 0
            Ss, ns, ms = (torch.zeros_like(t[slot]) if fresh else t[slot].clone() for t in (S, n, m))
            for t in range(a, b):
                mt = torch.maximum(f[t] + ms, i[t])
                w, u = torch.exp(f[t] + ms - mt), torch.exp(i[t] - mt)
                Ss = w[:, None, None] * Ss + u[:, None, None] * kf[t, :, :, None] * vf[t, :, None, :]
                ns = w[:, None] * ns + u[:, None] * kf[t]
                ms = mt
                den = torch.maximum((ns * qf[t]).sum(-1).abs(), torch.exp(-ms)) + MEMORY_EPS
                o[t] = (Ss * qf[t, :, :, None]).sum(1) / den[:, None]
            S[slot], n[slot], m[slot] = Ss, ns, ms
        o = _head_rms(o, dv, eps) * norm_w.float().reshape(H, dvp) * torch.sigmoid(gf) * out_scale
        out.copy_(o.reshape(M, H * dvp).to(out.dtype))
        return
    assert q.stride(0) == k.stride(0) == v.stride(0) == gate.stride(0) and zi.stride(0) == zf.stride(0)
    assert zi.dtype == zf.dtype == torch.float32
    cf, cl = nv.ctypes.c_float, nv.ctypes.c_longlong
    for lo, cnt, longest in ((0, p.num_short, p.max_short), (p.num_short, p.nseq - p.num_short, p.max_long)):
        if cnt <= 0:
            continue
        if lo == p.num_short and p.chunks128 is not None and q.dtype == torch.bfloat16 and dkp <= 128 and dvp <= 128:
            nc = p.chunks128.shape[0]
            ws = torch.empty((nc, H, dkp, dvp), device=q.device, dtype=torch.float32)
            wn = torch.empty((nc, H, dkp), device=q.device, dtype=torch.float32)
            wg = torch.empty((nc, H, 3), device=q.device, dtype=torch.float32).view(-1)      # (sum of f, largest g), then the maxima
            nv.check(nv.lib().b2_memory_chunk(
                nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ptr(gate), nv.ptr(zi), nv.ptr(zf), cl(zi.stride(0)), nv.ptr(bi), nv.ptr(bf),
                nv.ptr(norm_w), nv.ptr(out), nv.ptr(ws), nv.ptr(wn), nv.ptr(wg), nv.ptr(wg[2 * nc * H:]), nv.ptr(S), nv.ptr(n), nv.ptr(m),
                nv.ptr(p.chunks128), nv.ptr(p.first128), nv.ptr(p.starts), nv.ptr(p.slots), nc, lo, cnt, H, dk, dkp, dv, dvp,
                cl(q.stride(0)), cl(out.stride(0)), cf(cap), cf(q_scale), cf(out_scale), cf(eps), nv.stream_ptr()), "memory_chunk")
            nv.count_launch(3)
            continue
        cu, st, sl = _sub(p, lo)
        nv.check(nv.lib().b2_memory_serial(
            nv.ptr(q), nv.ptr(k), nv.ptr(v), nv.ptr(gate), nv.ptr(zi), nv.ptr(zf), cl(zi.stride(0)), nv.ptr(bi), nv.ptr(bf),
            nv.ptr(norm_w), nv.ptr(out), nv.ptr(S), nv.ptr(n), nv.ptr(m), cu, st, sl, cnt, longest, H, dk, dkp, dv, dvp,
            cl(q.stride(0)), cl(out.stride(0)), cf(cap), cf(q_scale), cf(out_scale), cf(eps), int(q.dtype == torch.float32),
            nv.stream_ptr()), "memory_serial")
        nv.count_launch()
