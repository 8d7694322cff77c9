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


@dataclass
class RowSplitSlot:
    """A checkpoint tensor whose leading rows live in several places: ``parts`` = (slot, rows) in order."""
    parts: List[Tuple[Slot, int]]
    shape: Tuple[int, ...]

    def load(self, t: torch.Tensor) -> None:
        for (slot, _), piece in zip(self.parts, t.split([n for _, n in self.parts])):
            slot.load(piece)

    def export(self) -> torch.Tensor:
        return torch.cat([slot.export() for slot, _ in self.parts])


@dataclass
class HalvesSlot:
    """Per-head channels (dimension 1 of ``view [heads, d, ...]``) of which ``rot``, from channel ``at`` on, are rotated in pairs of
    halves (the i-th of them with the one rot / 2 further) in the checkpoint and stored as neighbours (2 i, 2 i + 1): a score does not
    change when queries and keys are reordered alike, and the kernels rotate neighbours."""
    view: torch.Tensor
    rot: int
    shape: Tuple[int, ...]
    at: int = 0

    def _order(self) -> torch.Tensor:
        half, d, a = self.rot // 2, self.view.shape[1], self.at
        turned = a + torch.arange(self.rot).reshape(2, half).t().reshape(-1)
        return torch.cat([torch.arange(a), turned, torch.arange(a + self.rot, d)]).to(self.view.device)

    def load(self, t: torch.Tensor) -> None:
        self.view.copy_(t.to(self.view.device).reshape(self.view.shape)[:, self._order()].to(self.view.dtype))

    def export(self) -> torch.Tensor:
        out = torch.empty(self.view.shape, dtype=self.view.dtype, device=self.view.device)
        out[:, self._order()] = self.view.detach()
        return out.reshape(self.shape)


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

    def end(self, name: str) -> int:
        """Columns up to and with section ``name``."""
        at, heads, d = self.sections[name]
        return at + heads * pad8(d)

    def forward(self, x: torch.Tensor, act: Optional[str] = None, cols: Optional[int] = None) -> torch.Tensor:
        """``act`` on the first ``cols`` columns, in the product's epilogue (:func:`b200fw.ops.linear_act`)."""
        return ops.linear_act(x, self.weight, act, cols)

    def fp32(self, x: torch.Tensor) -> torch.Tensor:
        """The product with a 32-bit result."""
        return ops.linear_fp32(x, self.weight)


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


class SquaredReLU(nn.Module):
    """``W_down relu(W_up h)^2``, a pair of products of its own: for layers whose feed-forward reads what the mixer left."""

    def __init__(self, hidden: int, inner: int, dtype, device):
        super().__init__()
        self.up = PackedRows(hidden, [("up", 1, inner)], dtype, device)
        self.down = PackedCols(hidden, [("down", 1, inner)], dtype, device)

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        return {prefix + "up": self.up.slot("up"), prefix + "down": self.down.slot("down")}

    def run(self, h: torch.Tensor) -> torch.Tensor:
        """fp32 ``[M, hidden]``."""
        return self.down(self.up(h, "relu2"))


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


class Lightning(nn.Module):
    """Linear attention with a fixed decay per head over silu features of q, k and v; one norm over all heads together and a
    sigmoid gate.  No positions: the decay orders the tokens."""

    def __init__(self, hidden: int, heads: int, dim: int, vdim: int, decay: List[float], eps: float, dtype, device):
        super().__init__()
        if len(decay) != heads:
            raise ValueError(f"lightning: {len(decay)} decays for {heads} heads")
        self.heads, self.dim, self.vdim, self.eps = heads, dim, vdim, eps
        self.in_proj = PackedRows(hidden, [("q", heads, dim), ("k", heads, dim), ("v", heads, vdim), ("g", heads, vdim)], dtype,
                                  device)
        self.o = PackedCols(hidden, [("o", heads, vdim)], dtype, device)
        self.norm = _param(heads, pad8(vdim), dtype=dtype, device=device)
        self.register_buffer("decay", torch.tensor(decay, dtype=torch.float32, device=device), persistent=False)

    def kv_shape(self) -> None:
        return None

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return {"S": (self.heads, pad8(self.dim), pad8(self.vdim))}

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        t = {prefix + n: self.in_proj.slot(n) for n in "qkvg"}
        t[prefix + "o"] = self.o.slot("o")
        t[prefix + "norm"] = Slot(self.norm.data[:, :self.vdim], (self.heads * self.vdim,))
        return t

    def run(self, h: torch.Tensor, p, kv, state: Dict[str, torch.Tensor], rope) -> Tuple[torch.Tensor, Dict]:
        """fp32 ``[M, hidden]``, still to be divided by the heads' common root mean square: that factor of a row commutes with
        the projection, so the sum after it applies it (:func:`b200fw.ops.post_norm`)."""
        P = self.in_proj
        y = P(h, "silu", P.end("v"))
        out = self.o.buffer(y.shape[0])
        sumsq = torch.empty((y.shape[0], self.heads), dtype=torch.float32, device=y.device)
        ops.retention(P.cols(y, "q"), P.cols(y, "k"), P.cols(y, "v"), P.cols(y, "g"), out, state["S"], p, self.decay, self.dim,
                      self.vdim, None, None, 1.0, self.eps, self.norm.view(-1), sumsq)
        return self.o(out), {"sumsq": sumsq, "sumsq_n": self.heads * self.vdim}


class DifferentialAttention(nn.Module):
    """Two softmax attentions per head over one set of values, subtracted; sliding window, soft cap, biases, normed and rotated
    queries and keys (channel pairs), a norm per head without weight and a sigmoid gate per channel.  Grouped query heads."""

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, softcap: float, window: int,
                 rot_base: float, rot_dims: int, diff: float, eps: float, dtype, device):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"attention: {heads} query heads do not divide over {kv_heads} key/value heads")
        if rot_dims % 2 or not 0 <= rot_dims <= dim:
            raise ValueError(f"attention: rotary dims {rot_dims} must be even and at most the head size {dim}")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.softcap, self.window, self.diff, self.eps = float(scale), float(softcap), int(window), float(diff), eps
        self.rot = (float(rot_base), int(rot_dims))
        self.in_proj = PackedRows(hidden, [("q", 2 * heads, dim), ("k", 2 * kv_heads, dim), ("v", kv_heads, vdim), ("g", heads, vdim)],
                                  dtype, device)
        self.bias = _param(self.in_proj.end("v"), dtype=dtype, device=device)
        self.q_norm = _param(pad8(dim), dtype=dtype, device=device)
        self.k_norm = _param(pad8(dim), dtype=dtype, device=device)
        self.lam = _param(4, pad8(dim), dtype=dtype, device=device)
        self.o = PackedCols(hidden, [("o", heads, vdim)], dtype, device)
        self.o_bias = _param(pad8(hidden), dtype=dtype, device=device)
        self.hidden = hidden

    def kv_shape(self) -> Tuple[int, int, int]:
        return self.kv_heads, 2 * pad8(self.dim), pad8(self.vdim)

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return {}

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        t = {prefix + n: self.in_proj.slot(n) for n in "qkvg"}
        for n in "qkv":
            at, heads, d = self.in_proj.sections[n]
            t[prefix + n + ".b"] = Slot(self.bias.data[at:at + heads * pad8(d)].view(heads, pad8(d))[:, :d], (heads * d,))
        t[prefix + "q.norm"] = Slot(self.q_norm.data[:self.dim], (self.dim,))
        t[prefix + "k.norm"] = Slot(self.k_norm.data[:self.dim], (self.dim,))
        for i, n in enumerate(("lq1", "lk1", "lq2", "lk2")):
            t[prefix + n] = Slot(self.lam.data[i, :self.dim], (self.dim,))
        t[prefix + "o"] = self.o.slot("o")
        t[prefix + "o.b"] = Slot(self.o_bias.data[:self.hidden], (self.hidden,))
        return t

    def run(self, h: torch.Tensor, p, kv: Tuple[torch.Tensor, torch.Tensor], state, rope) -> Tuple[torch.Tensor, Dict]:
        """fp32 ``[M, hidden]`` without the output bias, which the sum after it adds."""
        kc, vc = kv
        kc = kc.view(kc.shape[0], kc.shape[1], 2 * self.kv_heads, pad8(self.dim))
        P = self.in_proj
        y = P(h)
        cos, sin = rope(*self.rot) if self.rot[1] else (None, None)
        q = ops.qk_norm_store(P.cols(y, "q"), P.cols(y, "k"), P.cols(y, "v"), kc, vc, p, 2 * self.heads, self.dim, True, self.eps,
                              self.q_norm, self.k_norm, self.bias, cos, sin)
        out = self.o.buffer(y.shape[0])
        ops.differential_attention(q, kc, vc, out, p, self.heads, self.scale, self.lam, self.diff, self.vdim, self.eps,
                                   P.cols(y, "g"), self.window, self.softcap)
        return self.o(out), {"bias": self.o_bias}


class LatentAttention(nn.Module):
    """Softmax attention whose keys and values are made from one cached latent per token, plus one rotated key part that all
    heads share.  ``w_key`` holds the key projection beside an identity for the rotated part.  Options: queries from a normed latent of
    their own (``q_rank``), a sliding ``window`` (0: none), a ``sink`` per head, a sigmoid ``gate`` per head on the output, rotated
    channels paired as ``halves`` in the checkpoint instead of as neighbours."""

    def __init__(self, hidden: int, heads: int, dim: int, rot_dim: int, vdim: int, rank: int, scale: float, rot_base: float,
                 eps: float, dtype, device, q_rank: Optional[int] = None, window: int = 0, sink: bool = True, gate: bool = False,
                 halves: bool = False):
        super().__init__()
        if rot_dim % 2 or rot_dim < 2:
            raise ValueError(f"latent attention: the rotated size {rot_dim} must be even and positive")
        self.heads, self.dim, self.rot_dim, self.vdim, self.rank, self.q_rank = heads, dim, rot_dim, vdim, rank, q_rank
        self.scale, self.eps, self.rot = float(scale), eps, (float(rot_base), int(rot_dim))
        self.window, self.halves = int(window), halves
        query = ("q", heads, dim + rot_dim) if q_rank is None else ("dq", 1, q_rank)
        self.in_proj = PackedRows(hidden, [query, ("c", 1, rank), ("kr", 1, rot_dim)] + ([("g", 1, heads)] if gate else []), dtype, device)
        self.q_up = None if q_rank is None else PackedRows(q_rank, [("uq", heads, dim + rot_dim)], dtype, device)
        self.q_norm = None if q_rank is None else _param(pad8(q_rank), dtype=dtype, device=device)
        self.c_norm = _param(pad8(rank), dtype=dtype, device=device)
        self.w_key = _param(heads, pad8(dim + rot_dim), pad8(rank) + pad8(rot_dim), dtype=dtype, device=device)
        i = torch.arange(rot_dim, device=device)
        self.w_key.data[:, dim + i, pad8(rank) + i] = 1.0
        self.w_value = _param(heads, pad8(vdim), pad8(rank), dtype=dtype, device=device)
        self.sink = _param(heads, dtype=dtype, device=device) if sink else None
        self.o = PackedCols(hidden, [("o", heads, vdim)], dtype, device)

    def kv_shape(self) -> Tuple[int, int, int]:
        return 1, pad8(self.rank) + pad8(self.rot_dim), 0

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return {}

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        H, hidden, P = self.heads, self.in_proj.in_features, self.in_proj

        def turned(s: Slot, at: int):
            return HalvesSlot(s.view, self.rot_dim, s.shape, at) if self.halves else s
        t = {prefix + "dkv": RowSplitSlot([(P.slot("c"), self.rank), (turned(P.slot("kr"), 0), self.rot_dim)], (self.rank + self.rot_dim, hidden)),
             prefix + "dkv.norm": Slot(self.c_norm.data[:self.rank], (self.rank,)),
             prefix + "uk": Slot(self.w_key.data[:, :self.dim, :self.rank], (H * self.dim, self.rank)),
             prefix + "uv": Slot(self.w_value.data[:, :self.vdim, :self.rank], (H * self.vdim, self.rank)), prefix + "o": self.o.slot("o")}
        if self.q_up is None:
            t[prefix + "q"] = turned(P.slot("q"), self.dim)
        else:
            t |= {prefix + "dq": P.slot("dq"), prefix + "dq.norm": Slot(self.q_norm.data[:self.q_rank], (self.q_rank,)),
                  prefix + "uq": turned(self.q_up.slot("uq"), self.dim)}
        if "g" in P.sections:
            t[prefix + "g"] = P.slot("g")
        if self.sink is not None:
            t[prefix + "sink"] = Slot(self.sink.data, (H,))
        return t

    def run(self, h: torch.Tensor, p, kv: Tuple[torch.Tensor, torch.Tensor], state, rope) -> Tuple[torch.Tensor, Dict]:
        """fp32 ``[M, hidden]``."""
        P, (cos, sin) = self.in_proj, rope(*self.rot)
        y = P(h)
        cq = P.cols(y, "dq") if self.q_up is not None else None
        q = P.cols(y, "q") if cq is None else None
        ops.latent_store(q, P.cols(y, "c"), P.cols(y, "kr"), kv[0], p, self.heads, self.dim, self.rank, self.rot_dim, self.c_norm, cos, sin,
                         self.eps, cq, self.q_norm, self.q_rank or 0)
        turn = None
        if cq is not None:
            q, turn = self.q_up(cq), (cos, sin, self.dim)
        gate = P.cols(y, "g")[:, :self.heads] if "g" in P.sections else None
        out = self.o.buffer(y.shape[0])
        ops.latent_attention(q, kv[0], out, p, self.w_key, self.w_value, self.scale, self.sink, self.window, gate, turn)
        return self.o(out), {}


class GatedFF(nn.Module):
    """``W_down(silu(W_gate h) * (W_up h))``, a pair of products of its own: for layers whose feed-forward reads what the mixer
    left and is normed before the sum."""

    def __init__(self, hidden: int, inner: int, dtype, device):
        super().__init__()
        self.up = PackedRows(hidden, [("gate", 1, inner), ("up", 1, inner)], dtype, device)
        self.down = PackedCols(hidden, [("down", 1, inner)], dtype, device)

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        return {prefix + "gate": self.up.slot("gate"), prefix + "up": self.up.slot("up"), prefix + "down": self.down.slot("down")}

    def run(self, h: torch.Tensor) -> torch.Tensor:
        """fp32 ``[M, hidden]``."""
        a = self.down.buffer(h.shape[0])
        ops.glu_linear(h, self.up.weight, a)
        return self.down(a)

    def add(self, x: torch.Tensor, h: torch.Tensor, norm: torch.Tensor, coef: float, n: int, eps: float) -> torch.Tensor:
        """``x += coef * norm(ff(h))``; the new ``x`` in the activation dtype."""
        return ops.norm_add(x, self.run(h), norm, coef, n, eps)


class ExpertFF(nn.Module):
    """Mixture of gated feed-forward experts with sigmoid or softmax scores, a learned correction of the choice, a choice limited to the
    best groups, and a shared expert behind a gate of its own.  Router logits and the shared gate are one 32-bit product.  A shared expert
    of the experts' size is stored as one more of them, which every token takes.  ``clamped = (alpha, limit)``: the experts' gated form
    (:func:`b200fw.ops.expert_glu`).  ``beside``: sections of other projections of the same input, made by the router's product."""

    def __init__(self, hidden: int, experts: int, inner: int, top: int, groups: int, keep: int, scale: float,
                 shared_inner: Optional[int], dtype, device, score: str = "sigmoid", corrected: bool = True,
                 clamped: Optional[Tuple[float, float]] = None, beside: List[Tuple[str, int, int]] = ()):
        super().__init__()
        self.score, self.clamped = score, clamped
        if groups < 1 or experts % groups or not 1 <= keep <= groups:
            raise ValueError(f"experts: {experts} do not form {groups} equal groups of which {keep} are kept")
        if not 1 <= top <= keep * (experts // groups):
            raise ValueError(f"experts: cannot choose {top} among {keep} groups of {experts // groups}")
        self.hidden, self.n, self.inner, self.top, self.groups, self.keep, self.scale = hidden, experts, inner, top, groups, keep, float(scale)
        self.joint = shared_inner == inner
        all_ = experts + int(self.joint)
        self.w_in = _param(all_, 2, pad8(inner), pad8(hidden), dtype=dtype, device=device)
        self.w_out = _param(all_, pad8(hidden), pad8(inner), dtype=dtype, device=device)
        self.correction = _param(experts, dtype=dtype, device=device) if corrected else None
        self.shared = GatedFF(hidden, shared_inner, dtype, device) if shared_inner is not None and not self.joint else None
        self.router = PackedRows(hidden, [("router", 1, experts)] + ([("sg", 1, 1)] if shared_inner is not None else []) + list(beside), dtype, device)
        self.shared_row = self.router.sections["sg"][0] if shared_inner is not None else -1

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        H, F = self.hidden, self.inner
        t: Dict[str, Slot] = {}
        for e in range(self.n + int(self.joint)):
            p = f"{prefix}e{e}." if e < self.n else prefix + "shared."
            t[p + "gate"], t[p + "up"] = (Slot(self.w_in.data[e, i, :F, :H], (F, H)) for i in range(2))
            t[p + "down"] = Slot(self.w_out.data[e, :H, :F], (H, F))
        t[prefix + "router"] = self.router.slot("router")
        if self.correction is not None:
            t[prefix + "correction"] = Slot(self.correction.data, (self.n,))
        if self.shared is not None:
            t |= self.shared.tensors(prefix + "shared.")
        if self.shared_row >= 0:
            t[prefix + "shared.sg"] = self.router.slot("sg")
        return t

    def add(self, x: torch.Tensor, h: torch.Tensor, norm: torch.Tensor, coef: float, n: int, eps: float) -> torch.Tensor:
        """``x += coef * norm(ff(h))``; the new ``x`` in the activation dtype."""
        r, gate = ops.router(h, self.router.weight, self.shared_row, self.correction, self.top, self.groups, self.keep, self.scale, self.joint)
        shared = None if self.shared is None else self.shared.run(h)
        return ops.moe_norm_add(x, self._experts(h, r), r, shared, gate, norm, coef, n, eps)

    def _experts(self, h: torch.Tensor, r: "ops.Routing") -> torch.Tensor:
        return ops.expert_down(ops.expert_glu(h, self.w_in, r, self.clamped), self.w_out, r)

    def run(self, h: torch.Tensor) -> Tuple[Tuple[torch.Tensor, "ops.Routing"], torch.Tensor]:
        """``(rows, routing)`` for the weighted sum of a token's experts, and the router's whole product (fp32), ``beside`` sections
        included.  Without a shared expert."""
        assert self.shared_row < 0
        z = self.router.fp32(h)
        r = ops.route(z, self.correction, self.top, self.groups, self.keep, self.scale, score=self.score, experts=self.n)
        return (self._experts(h, r), r), z


class LayerNorm(nn.Module):
    """Weight and bias of a layer norm over ``hidden`` channels, zero in the padding."""

    def __init__(self, hidden: int, dtype, device):
        super().__init__()
        self.hidden = hidden
        self.weight, self.bias = (_param(pad8(hidden), dtype=dtype, device=device) for _ in range(2))

    @property
    def pair(self) -> Tuple[torch.Tensor, torch.Tensor]:
        return self.weight, self.bias

    def tensors(self, name: str) -> Dict[str, Slot]:
        return {name: Slot(self.weight.data[:self.hidden], (self.hidden,)), name + ".b": Slot(self.bias.data[:self.hidden], (self.hidden,))}


class InputConv(nn.Module):
    """A short causal convolution of a sublayer's input per channel, added to it: ``h + conv(h)``."""

    def __init__(self, hidden: int, taps: int, dtype, device):
        super().__init__()
        if not 1 <= taps <= 17:
            raise ValueError(f"input convolution: {taps} taps (1 to 17)")
        self.hidden = hidden
        self.taps = _param(pad8(hidden), taps, dtype=dtype, device=device)

    def state_shape(self) -> Tuple[int, ...]:
        return (self.taps.shape[0], self.taps.shape[1] - 1)

    def slot(self) -> Slot:
        return Slot(self.taps.data[:self.hidden], (self.hidden, self.taps.shape[1]))

    def forward(self, h: torch.Tensor, state: torch.Tensor, p) -> torch.Tensor:
        return ops.causal_conv(h, None, self.taps, None, state, p, add_input=True)


class TokenInput(nn.Module):
    """A layer's own vector of the token, gated by the residual: ``x += coef * norm(W_proj (gelu(W_gate x) * e))``."""

    def __init__(self, hidden: int, dim: int, layer: int, dtype, device):
        super().__init__()
        self.hidden, self.first = hidden, layer * pad8(dim)
        self.gate = PackedRows(hidden, [("gate", 1, dim)], dtype, device)
        self.proj = PackedCols(hidden, [("proj", 1, dim)], dtype, device)
        self.norm = _param(pad8(hidden), dtype=dtype, device=device)

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        return {prefix + "gate": self.gate.slot("gate"), prefix + "proj": self.proj.slot("proj"),
                prefix + "norm": Slot(self.norm.data[:self.hidden], (self.hidden,))}

    def add(self, x: torch.Tensor, h: torch.Tensor, table: torch.Tensor, ids: torch.Tensor, vocab: int, coef: float, n: int,
            eps: float) -> torch.Tensor:
        g = ops.token_gate(h, self.gate.weight, table, ids, self.first, vocab)
        return ops.norm_add(x, self.proj(g), self.norm, coef, n, eps)


class CausalAttention(nn.Module):
    """Softmax attention over all keys up to the query: grouped query heads, optional biases, weighted norms of q and k per head,
    rotary positions on channel halves (optionally with stretched low frequencies), an optional sink per head; keys and values of
    its own, or those of another layer (``shared_kv``).  Sections of the layer's fused projections (``joint``)."""
    joint = True

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, rot_base: float, rot_dims: int,
                 stretch: Optional[Tuple[float, float, float, float]], bias: bool, sink: bool, shared_kv: bool, eps: float, dtype,
                 device):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"attention: {heads} query heads do not divide over {kv_heads} key/value heads")
        if rot_dims % 2 or not 0 <= rot_dims <= dim:
            raise ValueError(f"attention: rotary dims {rot_dims} must be even and at most the head size {dim}")
        self.heads, self.kv_heads, self.dim, self.vdim, self.scale, self.eps = heads, kv_heads, dim, vdim, float(scale), eps
        self.rot, self.shared_kv = (float(rot_base), int(rot_dims), stretch), shared_kv
        self.in_sections = [("q", heads, dim)] + ([] if shared_kv else [("k", kv_heads, dim), ("v", kv_heads, vdim)])
        self.out_section = ("o", heads, vdim)
        self.bias = _param(sum(n * pad8(d) for _, n, d in self.in_sections), dtype=dtype, device=device) if bias else None
        self.q_norm = _param(pad8(dim), dtype=dtype, device=device)
        self.k_norm = None if shared_kv else _param(pad8(dim), dtype=dtype, device=device)
        self.sink = _param(heads, dtype=dtype, device=device) if sink else None

    def kv_shape(self) -> Optional[Tuple[int, int, int]]:
        return None if self.shared_kv else (self.kv_heads, pad8(self.dim), pad8(self.vdim))

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return {}

    def tensors(self, prefix: str, inp: Sections, out_slot: Slot) -> Dict[str, Slot]:
        t, at, rot = {prefix + "o": out_slot}, 0, self.rot[1]

        for n, heads, d in self.in_sections:
            s = inp.slot(n)
            t[prefix + n] = s if n == "v" else HalvesSlot(s.view, rot, s.shape)
            if self.bias is not None:
                b = self.bias.data[at:at + heads * pad8(d)].view(heads, pad8(d))[:, :d]
                t[prefix + n + ".b"] = Slot(b, (heads * d,)) if n == "v" else HalvesSlot(b, rot, (heads * d,))
            at += heads * pad8(d)
        t[prefix + "q.norm"] = HalvesSlot(self.q_norm.data[None, :self.dim], rot, (self.dim,))
        if self.k_norm is not None:
            t[prefix + "k.norm"] = HalvesSlot(self.k_norm.data[None, :self.dim], rot, (self.dim,))
        if self.sink is not None:
            t[prefix + "sink"] = Slot(self.sink.data, (self.heads,))
        return t

    def run(self, h: torch.Tensor, y: Sections, out: torch.Tensor, p, kv: Tuple[torch.Tensor, torch.Tensor], state, rope,
            out_scale: float = 1.0) -> None:
        if out_scale != 1.0:
            raise ValueError("attention: its output takes no factor")
        k, v = (None, None) if self.shared_kv else (y.cols("k"), y.cols("v"))
        cos, sin = rope(*self.rot) if self.rot[1] else (None, None)
        q = ops.qk_norm_store(y.cols("q"), k, v, *kv, p, self.heads, self.dim, True, self.eps, self.q_norm, self.k_norm, self.bias,
                              cos, sin)
        ops.paged_attention(q, *kv, out, p, self.heads, self.scale, sink=self.sink)


class MatrixMemory(nn.Module):
    """Linear attention with exponential input and forget gates per head, a running maximum that keeps them in range and a
    normaliser; a norm per head with weights over all heads, and a sigmoid gate.  The gates' projections stay in 32-bit."""
    joint = True

    def __init__(self, hidden: int, heads: int, dim: int, vdim: int, cap: float, eps: float, dtype, device):
        super().__init__()
        self.heads, self.dim, self.vdim, self.cap, self.eps = heads, dim, vdim, float(cap), eps
        self.in_sections = [("q", heads, dim), ("k", heads, dim), ("v", heads, vdim), ("g", heads, vdim)]
        self.out_section = ("o", heads, vdim)
        self.gates = PackedRows(hidden, [("i", 1, heads), ("f", 1, heads)], dtype, device)
        self.bias = _param(2, heads, dtype=dtype, device=device)
        self.norm = _param(heads, pad8(vdim), dtype=dtype, device=device)

    def kv_shape(self) -> None:
        return None

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return {"S": (self.heads, pad8(self.dim), pad8(self.vdim)), "n": (self.heads, pad8(self.dim)), "m": (self.heads,)}

    def tensors(self, prefix: str, inp: Sections, out_slot: Slot) -> Dict[str, Slot]:
        t = {prefix + n: inp.slot(n) for n in "qkvg"} | {prefix + "o": out_slot}
        for i, n in enumerate("if"):
            t[prefix + n], t[prefix + n + ".b"] = self.gates.slot(n), Slot(self.bias.data[i], (self.heads,))
        t[prefix + "norm"] = Slot(self.norm.data[:, :self.vdim], (self.heads * self.vdim,))
        return t

    def run(self, h: torch.Tensor, y: Sections, out: torch.Tensor, p, kv, state: Dict[str, torch.Tensor], rope,
            out_scale: float = 1.0) -> None:
        z, H = self.gates.fp32(h), self.heads
        ops.matrix_memory(y.cols("q"), y.cols("k"), y.cols("v"), y.cols("g"), self.gates.cols(z, "i")[:, :H], self.gates.cols(z, "f")[:, :H],
                          self.bias[0], self.bias[1], out, state["S"], state["n"], state["m"], p, self.norm.view(-1), self.dim, self.vdim,
                          self.cap, self.dim ** -0.5, out_scale, self.eps)


class GatedRecurrence(nn.Module):
    """A gelu branch times a gated linear recurrence with one state per channel, behind a short convolution; the two gates are
    block-diagonal products of the convolution's output, in 32-bit."""
    joint = True

    def __init__(self, hidden: int, width: int, blocks: int, taps: int, dtype, device):
        super().__init__()
        if blocks < 1 or width % blocks:
            raise ValueError(f"recurrence: {width} channels do not form {blocks} equal blocks")
        if not 1 <= taps <= 17:
            raise ValueError(f"recurrence: {taps} convolution taps (1 to 17)")
        self.width, self.blocks, self.size, self.taps_n = width, blocks, width // blocks, taps
        B, n, np_ = blocks, self.size, pad8(self.size)
        self.in_sections = [("y", B, n), ("x", B, n)]
        self.out_section = ("o", B, n)

        def vec(*s):
            return _param(*s, dtype=dtype, device=device)
        self.y_bias, self.x_bias, self.conv_bias, self.lam = vec(B, np_), vec(B, np_), vec(B, np_), vec(B, np_)
        self.taps = vec(B, np_, taps)
        self.w_gates, self.gate_bias = vec(B, 2, np_, np_), vec(B, 2, np_)

    def kv_shape(self) -> None:
        return None

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        C = self.blocks * pad8(self.size)
        return {"S": (C,), "conv": (C, self.taps_n - 1)}

    def tensors(self, prefix: str, inp: Sections, out_slot: Slot) -> Dict[str, Slot]:
        B, n, C = self.blocks, self.size, self.width
        t = {prefix + "y": inp.slot("y"), prefix + "x": inp.slot("x"), prefix + "o": out_slot,
             prefix + "conv": Slot(self.taps.data[:, :n], (C, self.taps_n))}
        for name, v in (("y.b", self.y_bias), ("x.b", self.x_bias), ("conv.b", self.conv_bias), ("lam", self.lam)):
            t[prefix + name] = Slot(v.data[:, :n], (C,))
        for i, name in enumerate(("ra", "ri")):
            t[prefix + name] = Slot(self.w_gates.data[:, i, :n, :n], (B, n, n))
            t[prefix + name + ".b"] = Slot(self.gate_bias.data[:, i, :n], (B, n))
        return t

    def run(self, h: torch.Tensor, y: Sections, out: torch.Tensor, p, kv, state: Dict[str, torch.Tensor], rope,
            out_scale: float = 1.0) -> None:
        if out_scale != 1.0:
            raise ValueError("recurrence: its output takes no factor")
        ops.gated_recurrence(y.cols("y"), y.cols("x"), self.y_bias.view(-1), self.x_bias.view(-1), self.taps.view(out.shape[1], -1),
                             self.conv_bias.view(-1), self.w_gates, self.gate_bias, self.lam.view(-1), out, state["S"], state["conv"], p)
