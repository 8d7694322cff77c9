"""Ruburax: a decoder whose layers are causal attention (some over the keys and values of an earlier layer), attention beside a
matrix memory, or a gated linear recurrence; dense or expert feed-forwards; a vector of the token fed into every layer.  Each
sublayer reads the 32-bit residual directly and is normed on its way back into it.  Built from :mod:`b200fw.model.mixers`; the
cache, the step and the loop over layers belong to the inference runtime (:mod:`b200fw.infer.hybrid`)."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Iterator, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops.portions import pad8
from .mixers import (CausalAttention, ExpertFF, GatedFF, GatedRecurrence, MatrixMemory, PackedCols, PackedRows, Sections, Slot,
                     TokenInput)

_ATTENTION = {"heads", "kv_heads", "dim", "vdim", "scale", "rot"}
_FIELDS = {"attention": _ATTENTION, "parallel": {"left", "right", "left_scale", "right_scale"}, "rglru": {"width", "blocks", "conv"}}
_RIGHT = {"heads", "dim", "vdim", "gate_cap"}


def _need(where: str, have, fields) -> None:
    missing = set(fields) - set(have or {})
    if missing:
        raise ValueError(f"{where} is missing {sorted(missing)}")


@dataclass
class RuburaxConfig:
    """``config.json`` of the design."""
    vocab_size: int
    hidden_size: int
    layers: List[Dict[str, Any]]
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    side_dim: Optional[int] = None            # size of the token's vector of every layer
    rms_norm_eps: float = 1e-6
    init_std: float = 0.02
    # positions are computed, not looked up: nothing but the cache bounds the context
    max_position_embeddings: int = 1 << 30

    architecture = "Ruburax"

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            if l.get("type") not in _FIELDS:
                raise ValueError(f"layer {i}: unknown type {l.get('type')!r}")
            m, f = l.get("mixer"), l.get("mlp")
            _need(f"layer {i} ({l['type']}): the mixer", m, _FIELDS[l["type"]])
            if l["type"] == "parallel":
                _need(f"layer {i}: the left mixer", m["left"], _ATTENTION)
                _need(f"layer {i}: the right mixer", m["right"], _RIGHT)
            src = m.get("kv_from") if l["type"] == "attention" else None
            if src is not None:
                o = self.layers[src] if 0 <= src < i else {}
                if o.get("type") != "attention" or o["mixer"].get("kv_from") is not None:
                    raise ValueError(f"layer {i}: kv_from {src} is not an earlier attention layer with keys of its own")
                if any(o["mixer"][k] != m[k] for k in ("kv_heads", "dim", "vdim", "rot")):
                    raise ValueError(f"layer {i}: head counts, sizes or rotation differ from those of layer {src}")
            if f is not None:
                if f.get("kind") == "dense":
                    _need(f"layer {i}: the feed-forward", f, {"ff"})
                elif f.get("kind") == "moe":
                    _need(f"layer {i}: the feed-forward", f, {"expert", "router"})
                    _need(f"layer {i}: the router", f["router"], {"experts", "top", "scale"})
                else:
                    raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")

    @classmethod
    def from_dict(cls, d: Dict[str, Any], shapes: Optional[Dict[str, Tuple[int, ...]]] = None) -> "RuburaxConfig":
        missing = {"vocab", "width", "layers", "norm", "residual_mult", "logit_scale"} - set(d)
        if missing:
            raise ValueError(f"config.json is missing required fields: {sorted(missing)}")
        side = d.get("token_side")
        return cls(int(d["vocab"]), int(d["width"]), d["layers"], float(d["residual_mult"]), float(d["logit_scale"]),
                   None if side is None else int(side["dim"]), float(d["norm"]["eps"]))

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.rms_norm_eps},
             "residual_mult": self.residual_mult, "logit_scale": self.logit_scale, "layers": copy.deepcopy(self.layers)}
        return d if self.side_dim is None else d | {"token_side": {"dim": self.side_dim}}

    # ---- the summary numbers other parts of the framework show or size things by --------------------------------
    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def _attention(self) -> List[Dict[str, Any]]:
        return [l["mixer"]["left"] if l["type"] == "parallel" else l["mixer"] for l in self.layers if l["type"] != "rglru"]

    @property
    def num_heads(self) -> int:
        return max([a["heads"] for a in self._attention()] or [1])

    @property
    def num_kv_heads(self) -> int:
        return max([a["kv_heads"] for a in self._attention()] or [1])

    @property
    def head_dim(self) -> int:
        return max([a["dim"] for a in self._attention()] or [8])

    @property
    def intermediate_size(self) -> int:
        """Feed-forward channels a token passes through."""
        def size(f):
            if f["kind"] == "dense":
                return f["ff"]
            return f["expert"]["ff"] * f["router"]["top"] + (f["shared"]["ff"] if f.get("shared") is not None else 0)
        return max([size(l["mlp"]) for l in self.layers if l.get("mlp") is not None] or [0])

    def kv_bytes_per_token(self, element: int = 2) -> int:
        return sum(a["kv_heads"] * (pad8(a["dim"]) + pad8(a["vdim"])) for a in self._attention() if a.get("kv_from") is None) * element

    def num_params(self) -> int:
        with torch.device("meta"):
            return sum(torch.Size(s.shape).numel() for s in RuburaxModel(self, device="meta").checkpoint().values())

    def num_active_params(self) -> int:
        """Parameters one token is multiplied with: all but the experts that are not chosen (and the token tables' other rows)."""
        n = self.num_params() - self.vocab_size * (self.side_dim or 0) * self.num_layers
        for l in self.layers:
            f = l.get("mlp")
            if f is not None and f["kind"] == "moe":
                n -= (f["router"]["experts"] - f["router"]["top"]) * 3 * f["expert"]["ff"] * self.hidden_size
        return n


def _attention(m: Dict[str, Any], hidden: int, bias: bool, sink: bool, eps: float, dtype, device) -> CausalAttention:
    rot, s = m["rot"], m["rot"].get("scaling")
    stretch = None if s is None else tuple(float(s[k]) for k in ("factor", "low", "high", "original"))
    return CausalAttention(hidden, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], rot["base"], rot["dims"], stretch, bias, sink,
                           m.get("kv_from") is not None, eps, dtype, device)


def _feed_forward(f: Dict[str, Any], hidden: int, dtype, device) -> nn.Module:
    if f["kind"] == "dense":
        return GatedFF(hidden, f["ff"], dtype, device)
    r = f["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    shared = f["shared"]["ff"] if f.get("shared") is not None else None
    return ExpertFF(hidden, r["experts"], f["expert"]["ff"], r["top"], g["count"], g["keep"], r["scale"], shared, dtype, device)


class RuburaxLayer(nn.Module):
    """``x += c norm1(mixer(x))``, ``x += c norm2(ff(x))``, ``x += c norm(side(x, token))`` with one constant c (a layer may have no
    feed-forward).  Everything that reads ``x`` in a mixer is one GEMM, and so are the output projections of mixers that run side by
    side; their sum's norm, the residual and the 16-bit copy that the next sublayer reads are one kernel."""

    def __init__(self, cfg: RuburaxConfig, i: int, dtype=None, device=None):
        super().__init__()
        l, H, eps = cfg.layers[i], cfg.hidden_size, cfg.rms_norm_eps
        m = l["mixer"]
        self.kind, self.hidden, self.eps, self.mult, self.vocab = l["type"], H, eps, cfg.residual_mult, cfg.vocab_size
        self.kv_from = m.get("kv_from") if self.kind == "attention" else None
        self.y_scale = 1.0
        # (prefix, block, factor on its output before the joint projection; None: left out)
        if self.kind == "attention":
            blocks = [("", _attention(m, H, True, True, eps, dtype, device), 1.0)]
        elif self.kind == "rglru":
            blocks = [("", GatedRecurrence(H, m["width"], m["blocks"], m["conv"], dtype, device), 1.0)]
        else:
            r, a, b = m["right"], float(m["left_scale"]), float(m["right_scale"])
            # a L + b R = a (L + (b / a) R): the first factor goes to the norm of the sum, the second to the memory's output
            self.y_scale = a if a != 0.0 else b
            blocks = [("left.", _attention(m["left"], H, False, False, eps, dtype, device), 1.0 if a != 0.0 else None),
                      ("right.", MatrixMemory(H, r["heads"], r["dim"], r["vdim"], r["gate_cap"], eps, dtype, device), b / a if a != 0.0 else 1.0)]
        self.blocks = nn.ModuleList([b for _, b, _ in blocks])
        self.prefixes, self.factors = [p for p, _, _ in blocks], [f for _, _, f in blocks]
        self.in_proj = PackedRows(H, [(p + n, h, d) for p, b, _ in blocks for n, h, d in b.in_sections], dtype, device)
        self.out_proj = PackedCols(H, [(p + b.out_section[0],) + b.out_section[1:] for p, b, _ in blocks], dtype, device)

        def norm():
            return nn.Parameter(torch.zeros(pad8(H), dtype=dtype, device=device), requires_grad=False)
        self.norm1 = norm()
        self.ff = _feed_forward(l["mlp"], H, dtype, device) if l.get("mlp") is not None else None
        self.norm2 = norm() if self.ff is not None else None
        self.side = TokenInput(H, cfg.side_dim, i, dtype, device) if cfg.side_dim is not None else None
        self.side_table: Optional[torch.Tensor] = None      # the model's, for all layers

    def kv_shape(self) -> Optional[Tuple[int, int, int]]:
        return self.blocks[0].kv_shape()

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return self.blocks[-1].state_shapes()

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        def vec(p):
            return Slot(p.data[:self.hidden], (self.hidden,))
        t = {prefix + "norm1": vec(self.norm1)}
        for p, b in zip(self.prefixes, self.blocks):
            t |= b.tensors(f"{prefix}mix.{p}", Sections(self.in_proj, p), self.out_proj.slot(p + b.out_section[0]))
        if self.ff is not None:
            t[prefix + "norm2"] = vec(self.norm2)
            t |= self.ff.tensors(prefix + "mlp.")
        if self.side is not None:
            t |= self.side.tensors(prefix + "side.")
        return t

    def forward(self, x: torch.Tensor, h: torch.Tensor, p, kv, state, rope, next_norm: Optional[torch.Tensor]):
        """One layer over a step's rows.  ``x``: fp32 residual, updated in place; ``h``: the same in the activation dtype; returns
        the new ``h``.  ``p``: row layout; ``kv``, ``state``: this layer's pages and state slots; ``rope(base, dims, stretch)``: the
        step's rotary tables."""
        y, buf = self.in_proj(h), self.out_proj.buffer(x.shape[0])
        for prefix, block, factor in zip(self.prefixes, self.blocks, self.factors):
            out = self.out_proj.cols(buf, prefix + block.out_section[0])
            block.run(h, Sections(self.in_proj, prefix, y), out, p, kv, state, rope, 1.0 if factor is None else factor)
            if factor is None:
                out.zero_()
        h = ops.norm_add(x, self.out_proj(buf), self.norm1, self.mult, self.hidden, self.eps, self.y_scale)
        if self.ff is not None:
            h = self.ff.add(x, h, self.norm2, self.mult, self.hidden, self.eps)
        if self.side is not None:
            h = self.side.add(x, h, self.side_table, p.ids, self.vocab, self.mult, self.hidden, self.eps)
        return h


class RuburaxModel(nn.Module):
    """Weights and per-layer computation.  Inference only, one GPU (``tp_size`` 1)."""

    tp_size, tp_rank, tp_group = 1, 0, None
    layer_start, is_first_stage, is_last_stage, tied = 0, True, True, True

    def __init__(self, cfg: RuburaxConfig, dtype=None, device=None):
        super().__init__()
        dtype = dtype or torch.float32
        self.cfg, self.logit_scale = cfg, cfg.logit_scale
        W, L = pad8(cfg.hidden_size), len(cfg.layers)
        self.embed_tokens = nn.Parameter(torch.zeros(pad8(cfg.vocab_size), W, dtype=dtype, device=device), requires_grad=False)
        self.side_table = None
        if cfg.side_dim is not None:
            self.side_table = nn.Parameter(torch.zeros(cfg.vocab_size, L * pad8(cfg.side_dim), dtype=dtype, device=device), requires_grad=False)
        self.layers = nn.ModuleList([RuburaxLayer(cfg, i, dtype, device) for i in range(L)])
        for layer in self.layers:
            layer.__dict__["side_table"] = self.side_table        # a reference, not a parameter of the layer
        self.norm = nn.Parameter(torch.zeros(W, dtype=dtype, device=device), requires_grad=False)

    def checkpoint(self) -> Dict[str, Slot]:
        """Checkpoint name -> where the tensor lives."""
        c = self.cfg
        t = {"embed": Slot(self.embed_tokens.data[:c.vocab_size, :c.hidden_size], (c.vocab_size, c.hidden_size)),
             "final.norm": Slot(self.norm.data[:c.hidden_size], (c.hidden_size,))}
        if self.side_table is not None:
            L, d = len(c.layers), c.side_dim
            t["side.embed"] = Slot(self.side_table.data.view(c.vocab_size, L, pad8(d))[:, :, :d], (c.vocab_size, L * d))
        for i, layer in enumerate(self.layers):
            t |= layer.tensors(f"l{i}.")
        return t

    def named_checkpoint_tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        for name, slot in self.checkpoint().items():
            yield name, slot.export()

    @torch.no_grad()
    def init_weights(self, seed: int = 0, std: Optional[float] = None):
        """Deterministic random weights: projections N(0, std), norms 1, forget gates open, slow channels, other biases 0."""
        import zlib
        std = self.cfg.init_std if std is None else std
        dev = self.embed_tokens.device
        for name, slot in self.checkpoint().items():
            last = name.rsplit(".", 1)[-1]
            g = torch.Generator(device=dev).manual_seed((zlib.crc32(name.encode()) + 1000003 * seed) % (2 ** 62))
            r = torch.empty(slot.shape, dtype=torch.float32, device=dev)
            if last.startswith("norm"):
                r.fill_(1.0)
            elif name.endswith("right.f.b"):
                r.fill_(4.0)
            elif last in ("b", "sink", "correction"):
                r.zero_()
            elif last == "lam":
                r.uniform_(-8.0, -4.0, generator=g)
            elif last == "conv":
                r.uniform_(-0.5, 0.5, generator=g)
            else:
                r.normal_(0.0, std, generator=g)
            slot.load(r)

    # ---- what the runtime allocates for it --------------------------------------------------------------------
    def kv_layer_shapes(self) -> List[Optional[Tuple[int, int, int]]]:
        """Per layer ``(kv heads, key size, value size)`` of its pages, None for a layer without any."""
        return [l.kv_shape() for l in self.layers]

    def kv_sources(self) -> List[Optional[int]]:
        """Per layer the earlier layer whose pages it reads, None for its own."""
        return [l.kv_from for l in self.layers]

    def state_layer_shapes(self) -> List[Dict[str, Tuple[int, ...]]]:
        """Per layer the fp32 state tensors one sequence holds."""
        return [l.state_shapes() for l in self.layers]

    # ---- pieces the runner calls ------------------------------------------------------------------------------
    def embed(self, ids: torch.Tensor, p=None, state=None):
        """The residual stream's first rows (fp32) and the same in the activation dtype, which the first layer reads."""
        return ops.embedding_f32(ids, self.embed_tokens, self.cfg.vocab_size, h=True)

    def logits_from_hidden(self, h: torch.Tensor) -> torch.Tensor:
        out = torch.empty((h.shape[0], self.embed_tokens.shape[0]), dtype=torch.float32, device=h.device)
        return ops.gemm(h, self.embed_tokens, out=out)[:, :self.cfg.vocab_size]

    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor) -> torch.Tensor:
        """``[B, S]`` token ids -> ``[B, S, V]`` logits, recomputed from nothing (a cache that lives for the call)."""
        from ..infer.hybrid import whole_sequences
        return whole_sequences(self, input_ids)


def ruburax_preset(width: int, heads: int, depth: int, vocab: int, kv_heads: int, experts: int, top: int, expert_ff: int, groups: int,
                   keep: int, side: int, dim: int = 128, every: int = 4) -> RuburaxConfig:
    """A configuration at the scale of a real model: of every ``every`` layers two are attention, the second over the keys of the
    first, then one attention beside a matrix memory, the others gated recurrences; the first feed-forward dense, the others experts."""
    rot = {"base": 500000.0, "dims": dim, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    att = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5}
    layers: List[Dict[str, Any]] = []
    for i in range(depth):
        at = i % every
        if at < 2:
            l = {"type": "attention", "mixer": {**att, "rot": rot, **({"kv_from": i - 1} if at else {})}}
        elif at == 2:
            l = {"type": "parallel", "mixer": {
                "left": {**att, "rot": {"base": 10000.0, "dims": dim}}, "left_scale": 0.5, "right_scale": 0.5,
                "right": {"heads": heads, "dim": dim, "vdim": dim, "gate_cap": 15.0}}}
        else:
            l = {"type": "rglru", "mixer": {"width": width, "blocks": heads, "conv": 4}}
        l["mlp"] = {"kind": "dense", "ff": top * expert_ff + expert_ff} if i == 0 else {
            "kind": "moe", "expert": {"ff": expert_ff}, "shared": {"ff": expert_ff},
            "router": {"experts": experts, "top": top, "scale": 2.5, "groups": {"count": groups, "keep": keep}}}
        layers.append(l)
    return RuburaxConfig(vocab, width, layers, residual_mult=1.0, logit_scale=1.0, side_dim=side)


RUBURAX_PRESETS = {
    "ruburax-tiny": ruburax_preset(256, 2, 4, 1024, 1, 8, 2, 128, 4, 2, 32, dim=64),
    # the widths, head counts, depth and vocabulary of the framework's dense presets of the same size; as many feed-forward channels
    # per token as theirs, in five of the experts' size: four chosen and one shared
    "ruburax-0.6b": ruburax_preset(1024, 8, 28, 151936, 4, 32, 4, 640, 8, 4, 128),
    "ruburax-4b": ruburax_preset(2560, 16, 36, 151936, 4, 32, 4, 1920, 8, 4, 256),
}
