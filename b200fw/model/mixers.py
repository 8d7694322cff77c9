"""Serving-side token mixers and feed-forward blocks for models whose layers differ from one another.

A block declares the column sections it wants from its layer's fused input projection (one GEMM per layer for everything
that reads the normed input) and how it turns them into an output.  Blocks marked ``joint`` write their pre-projection
activation into a slice of one concatenated buffer, so that the layer's output projections are a single GEMM accumulated
into the 32-bit residual stream.  Every constant of a mechanism is a constructor argument.

Head sizes and feature counts are stored padded to multiples of eight with zeros (:func:`b200fw.ops.portions.pad8`);
:class:`Slot` maps a tensor of the checkpoint onto its place inside the padded, fused storage.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops.portions import pad8


@dataclass
class Slot:
    """Where a checkpoint tensor lives: ``view`` (possibly a strided part of fused storage) holds ``shape`` reshaped."""
    view: torch.Tensor
    shape: Tuple[int, ...]

    def load(self, t: torch.Tensor) -> None:
        self.view.copy_(t.reshape(self.view.shape).to(self.view.dtype))

    def export(self) -> torch.Tensor:
        return self.view.detach().reshape(self.shape)


def _param(*shape, dtype, device) -> nn.Parameter:
    return nn.Parameter(torch.zeros(*shape, dtype=dtype, device=device), requires_grad=False)


class PackedRows(nn.Module):
    """Several ``[heads * d, in]`` projections of one input stacked into one weight, each head padded to ``pad8(d)`` rows."""

    def __init__(self, in_features: int, sections: List[Tuple[str, int, int]], dtype, device):
        super().__init__()
        self.in_features, self.sections, at = in_features, {}, 0
        for name, heads, d in sections:
            self.sections[name] = (at, heads, d)
            at += heads * pad8(d)
        self.weight = _param(at, pad8(in_features), dtype=dtype, device=device)

    def slot(self, name: str) -> Slot:
        at, heads, d = self.sections[name]
        rows = self.weight.data[at:at + heads * pad8(d)].view(heads, pad8(d), -1)
        return Slot(rows[:, :d, :self.in_features], (heads * d, self.in_features))

    def cols(self, y: torch.Tensor, first: str, last: Optional[str] = None) -> torch.Tensor:
        """Columns of section ``first`` (through ``last``) of this projection's output."""
        a, e = self.sections[first], self.sections[last or first]
        return y[:, a[0]:e[0] + e[1] * pad8(e[2])]

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return ops.linear(x, self.weight)


class PackedCols(nn.Module):
    """Several ``[out, heads * d]`` projections into one output side by side: their inputs are concatenated."""

    def __init__(self, out_features: int, sections: List[Tuple[str, int, int]], dtype, device):
        super().__init__()
        self.out_features, self.sections, at = out_features, {}, 0
        for name, heads, d in sections:
            self.sections[name] = (at, heads, d)
            at += heads * pad8(d)
        self.in_padded = at
        self.weight = _param(pad8(out_features), at, dtype=dtype, device=device)

    def slot(self, name: str) -> Slot:
        at, heads, d = self.sections[name]
        w = self.weight.data[:self.out_features, at:at + heads * pad8(d)].unflatten(1, (heads, pad8(d)))
        return Slot(w[:, :, :d], (self.out_features, heads * d))

    def cols(self, x: torch.Tensor, name: str) -> torch.Tensor:
        at, heads, d = self.sections[name]
        return x[:, at:at + heads * pad8(d)]

    def buffer(self, rows: int) -> torch.Tensor:
        return torch.empty((rows, self.in_padded), dtype=self.weight.dtype, device=self.weight.device)

    def forward(self, x: torch.Tensor, accumulate_into: Optional[torch.Tensor] = None) -> torch.Tensor:
        """fp32 result, or accumulated into the fp32 tensor given."""
        if accumulate_into is not None:
            return ops.gemm(x, self.weight, out=accumulate_into, accumulate=True)
        return ops.gemm(x, self.weight, out=torch.empty((x.shape[0], self.weight.shape[0]), dtype=torch.float32,
                                                        device=x.device))


class DenseGLU(nn.Module):
    """``W_down(silu(W_gate h) * (W_up h))``: declares its sections, the layer owns the fused projections."""
    joint = True

    def __init__(self, hidden: int, inner: int):
        super().__init__()
        self.in_sections = [("gate", 1, inner), ("up", 1, inner)]
        self.out_section = ("down", 1, inner)

    def tensors(self, prefix: str, inp: "Sections", out_slot: Slot) -> Dict[str, Slot]:
        return {prefix + "gate": inp.slot("gate"), prefix + "up": inp.slot("up"), prefix + "down": out_slot}

    def run(self, y: "Sections", out: torch.Tensor) -> None:
        ops.glu(y.cols("gate"), y.cols("up"), out)


class Sections:
    """A block's view of its layer's fused input projection: section names get the block's prefix."""

    def __init__(self, proj: PackedRows, prefix: str, y: Optional[torch.Tensor] = None):
        self.proj, self.prefix, self.y = proj, prefix, y

    def slot(self, name: str) -> Slot:
        return self.proj.slot(self.prefix + name)

    def cols(self, first: str, last: Optional[str] = None) -> torch.Tensor:
        return self.proj.cols(self.y, self.prefix + first, None if last is None else self.prefix + last)


class Retention(nn.Module):
    """Linear attention with a fixed decay per head, rotary positions on q and k, a per-head norm and a silu gate."""
    joint = True

    def __init__(self, hidden: int, heads: int, dim: int, vdim: int, decay: List[float], rot_base: float, rot_dims: int,
                 eps: float, dtype, device):
        super().__init__()
        if len(decay) != heads:
            raise ValueError(f"retention: {len(decay)} decays for {heads} heads")
        if rot_dims % 2 or not 0 <= rot_dims <= dim:
            raise ValueError(f"retention: rotary dims {rot_dims} must be even and at most the head size {dim}")
        self.heads, self.dim, self.vdim, self.eps = heads, dim, vdim, eps
        self.rot = (float(rot_base), int(rot_dims))
        self.in_sections = [("q", heads, dim), ("k", heads, dim), ("v", heads, vdim), ("g", heads, vdim)]
        self.out_section = ("o", heads, vdim)
        self.register_buffer("decay", torch.tensor(decay, dtype=torch.float32, device=device), persistent=False)

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return {"S": (self.heads, pad8(self.dim), pad8(self.vdim))}

    def tensors(self, prefix: str, inp: Sections, out_slot: Slot) -> Dict[str, Slot]:
        return {prefix + n: inp.slot(n) for n in "qkvg"} | {prefix + "o": out_slot}

    def run(self, y: Sections, out: torch.Tensor, p, state: Dict[str, torch.Tensor], rope) -> None:
        cos, sin = rope(*self.rot) if self.rot[1] else (None, None)
        ops.retention(y.cols("q"), y.cols("k"), y.cols("v"), y.cols("g"), out, state["S"], p, self.decay, self.dim, self.vdim,
                      cos, sin, self.dim ** -0.5, self.eps)


class BiasedChunkAttention(nn.Module):
    """Softmax attention inside fixed chunks of the sequence: per-head q / k norm, learned distance bias, a sink per head,
    an output gate per head.  Grouped query heads; no rotation."""

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, chunk: int, bias_rows: int,
                 bias_far: float, eps: float, dtype, device):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"attention: {heads} query heads do not divide over {kv_heads} key/value heads")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.chunk, self.eps = float(scale), int(chunk), eps
        self.in_sections = [("q", heads, dim), ("k", kv_heads, dim), ("v", kv_heads, vdim), ("g", 1, heads)]
        self.rel = _param(bias_rows, heads, dtype=dtype, device=device)
        self.sink = _param(heads, dtype=dtype, device=device)
        # distances past the last entry share its bucket: everything at `bias_far` or beyond is in the last one
        length = min(self.chunk, max(math.ceil(bias_far), bias_rows) + 1)
        self.register_buffer("bucket", ops.distance_buckets(bias_rows, bias_far, length, device), persistent=False)
        self.o = PackedCols(hidden, [("o", heads, vdim)], dtype, device)

    def kv_shape(self) -> Tuple[int, int, int]:
        return self.kv_heads, pad8(self.dim), pad8(self.vdim)

    def tensors(self, prefix: str, inp: Sections) -> Dict[str, Slot]:
        t = {prefix + n: inp.slot(n) for n in "qkvg"}
        t[prefix + "rel"] = Slot(self.rel.data, tuple(self.rel.shape))
        t[prefix + "sink"] = Slot(self.sink.data, tuple(self.sink.shape))
        t[prefix + "o"] = self.o.slot("o")
        return t

    def run(self, y: Sections, p, kv: Tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
        """fp32 ``[M, hidden]``: the output projection of the gated heads."""
        kc, vc = kv
        q = ops.qk_norm_store(y.cols("q"), y.cols("k"), y.cols("v"), kc, vc, p, self.heads, self.dim, True, self.eps)
        att = self.o.buffer(q.shape[0])
        ops.paged_attention(q, kc, vc, att, p, self.heads, self.scale, self.chunk, self.rel, self.bucket, self.sink,
                            y.cols("g")[:, :self.heads])
        return self.o(att)


class GatedDelta(nn.Module):
    """Gated delta rule with one learned decay per head and key channel; short convolutions on q, k and v; low-rank decay
    and output-gate projections (one block-diagonal GEMM for both second factors)."""

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, decay_rank: int, gate_rank: int,
                 eps: float, dtype, device):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"delta rule: {heads} heads do not divide over {kv_heads} key heads")
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps_n, self.eps = heads, kv_heads, dim, vdim, taps, eps
        self.ranks = (decay_rank, gate_rank)
        dkp, dvp = pad8(dim), pad8(vdim)
        self.in_sections = [("q", kv_heads, dim), ("k", kv_heads, dim), ("v", heads, vdim), ("b", 1, heads),
                            ("a1", 1, decay_rank), ("g1", 1, gate_rank)]
        ra, rg = pad8(decay_rank), pad8(gate_rank)
        self.taps = _param(2 * kv_heads * dkp + heads * dvp, taps, dtype=dtype, device=device)
        self.second = _param(heads * (dkp + dvp), ra + rg, dtype=dtype, device=device)   # [a2 0; 0 g2]
        self.A_log = _param(heads, dtype=dtype, device=device)
        self.dt_bias = _param(heads, dkp, dtype=dtype, device=device)
        self.norm = _param(dvp, dtype=dtype, device=device)
        self.o = PackedCols(hidden, [("o", heads, vdim)], dtype, device)

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return {"S": (self.heads, pad8(self.dim), pad8(self.vdim)), "conv": (self.taps.shape[0], self.taps_n - 1)}

    def tensors(self, prefix: str, inp: Sections) -> Dict[str, Slot]:
        H, G, dk, dv, K = self.heads, self.kv_heads, self.dim, self.vdim, self.taps_n
        dkp, dvp, (ra, rg) = pad8(dk), pad8(dv), self.ranks
        t = {prefix + n: inp.slot(n) for n in ("q", "k", "v", "b", "a1", "g1")}
        w, taps = G * dkp, self.taps.data
        for n, a, heads, d in (("q", 0, G, dk), ("k", w, G, dk), ("v", 2 * w, H, dv)):
            v = taps[a:a + heads * pad8(d)].view(heads, pad8(d), K)[:, :d]
            t[prefix + n + ".conv"] = Slot(v, (heads * d, K))
        a2 = self.second.data[:H * dkp].view(H, dkp, -1)[:, :dk, :ra]
        g2 = self.second.data[H * dkp:].view(H, dvp, -1)[:, :dv, pad8(ra):pad8(ra) + rg]
        t[prefix + "a2"], t[prefix + "g2"] = Slot(a2, (H * dk, ra)), Slot(g2, (H * dv, rg))
        t[prefix + "A_log"] = Slot(self.A_log.data, (H,))
        t[prefix + "dt_bias"] = Slot(self.dt_bias.data[:, :dk], (H * dk,))
        t[prefix + "norm"] = Slot(self.norm.data[:dv], (dv,))
        t[prefix + "o"] = self.o.slot("o")
        return t

    def run(self, y: Sections, p, state: Dict[str, torch.Tensor]) -> torch.Tensor:
        """fp32 ``[M, hidden]``: the output projection of the normed, gated heads."""
        H, dkp = self.heads, pad8(self.dim)
        low = y.cols("a1", "g1")
        z = ops.gemm(low, self.second, out=torch.empty((low.shape[0], self.second.shape[0]), dtype=torch.float32,
                                                       device=low.device))
        q, k, v, g, beta = ops.delta_inputs(y.cols("q", "v"), self.taps, y.cols("b")[:, :H], z[:, :H * dkp], self.A_log,
                                            self.dt_bias.view(-1), state["conv"], p, self.kv_heads, self.dim, self.vdim,
                                            self.dim ** -0.5)
        out = self.o.buffer(v.shape[0])
        ops.gated_delta(q, k, v, g, beta, z[:, H * dkp:], self.norm, out, state["S"], p, self.kv_heads, self.dim, self.vdim,
                        self.eps)
        return self.o(out)
