"""Sotazen: a decoder whose layers are differential attention, lightning (linear) attention or latent attention, each norm
after the sum: ``x <- norm(alpha x + sublayer(x))`` over a 32-bit residual stream that the sublayers read directly.  Built
from :mod:`b200fw.model.mixers`; the cache, the step and the loop over layers belong to the inference runtime
(:mod:`b200fw.infer.hybrid`)."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Iterator, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops.portions import pad8
from .mixers import DifferentialAttention, LatentAttention, Lightning, Slot, SquaredReLU

_FIELDS = {"lightning": {"heads", "dim", "vdim", "decay"},
           "attention": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap", "mask", "rot", "diff"},
           "latent_attention": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot"}}


@dataclass
class SotazenConfig:
    """``config.json`` of the design."""
    vocab_size: int
    hidden_size: int
    layers: List[Dict[str, Any]]
    embed_scale: float = 1.0
    alpha: float = 1.0
    rms_norm_eps: float = 1e-6
    init_std: float = 0.02
    # positions are computed, not looked up: nothing but the cache bounds the context
    max_position_embeddings: int = 1 << 30

    architecture = "Sotazen"

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            if l.get("type") not in _FIELDS:
                raise ValueError(f"layer {i}: unknown type {l.get('type')!r}")
            missing = _FIELDS[l["type"]] - set(l.get("mixer") or {})
            if missing:
                raise ValueError(f"layer {i} ({l['type']}): the mixer is missing {sorted(missing)}")
            if l.get("mlp") is not None and l["mlp"].get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {l['mlp'].get('kind')!r}")
            m = l["mixer"]
            if l["type"] == "latent_attention" and m["rot"]["dims"] != m["rot_dim"]:
                raise ValueError(f"layer {i}: rot.dims {m['rot']['dims']} is not the rotated size {m['rot_dim']}")

    @classmethod
    def from_dict(cls, d: Dict[str, Any], shapes: Optional[Dict[str, Tuple[int, ...]]] = None) -> "SotazenConfig":
        missing = {"vocab", "width", "layers", "norm", "embedding", "postln_alpha"} - set(d)
        if missing:
            raise ValueError(f"config.json is missing required fields: {sorted(missing)}")
        return cls(int(d["vocab"]), int(d["width"]), d["layers"], float(d["embedding"]["scale"]), float(d["postln_alpha"]),
                   float(d["norm"]["eps"]))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.rms_norm_eps}, "embedding": {"scale": self.embed_scale}, "postln_alpha": self.alpha,
                "layers": copy.deepcopy(self.layers)}

    # ---- the summary numbers other parts of the framework show or size things by --------------------------------
    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def _all(self, key: str, *types: str) -> List[int]:
        return [l["mixer"][key] for l in self.layers if not types or l["type"] in types]

    @property
    def num_heads(self) -> int:
        return max(self._all("heads") or [1])

    @property
    def num_kv_heads(self) -> int:
        return max(self._all("kv_heads", "attention") or [1])

    @property
    def head_dim(self) -> int:
        return max(self._all("dim", "attention", "latent_attention") or [8])

    @property
    def intermediate_size(self) -> int:
        return max([l["mlp"]["ff"] for l in self.layers if l.get("mlp") is not None] or [0])

    def kv_bytes_per_token(self, element: int = 2) -> int:
        n = 0
        for l in self.layers:
            m = l["mixer"]
            if l["type"] == "attention":
                n += m["kv_heads"] * (2 * pad8(m["dim"]) + pad8(m["vdim"]))
            elif l["type"] == "latent_attention":
                n += pad8(m["kv_rank"]) + pad8(m["rot_dim"])
        return n * element

    def num_params(self) -> int:
        with torch.device("meta"):
            return sum(torch.Size(s.shape).numel() for s in SotazenModel(self, device="meta").checkpoint().values())


def _mixer(l: Dict[str, Any], hidden: int, eps: float, dtype, device) -> nn.Module:
    m = l["mixer"]
    if l["type"] == "lightning":
        return Lightning(hidden, m["heads"], m["dim"], m["vdim"], m["decay"], eps, dtype, device)
    if l["type"] == "attention":
        return DifferentialAttention(hidden, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m["softcap"],
                                     m["mask"]["size"], m["rot"]["base"], m["rot"]["dims"], m["diff"], eps, dtype, device)
    return LatentAttention(hidden, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], m["rot"]["base"], eps,
                           dtype, device)


class SotazenLayer(nn.Module):
    """``x <- norm1(alpha x + mixer(x))``, then ``x <- norm2(alpha x + ff(x))`` (a layer may have no feed-forward).  Each sum, its
    norm and the 16-bit copy that the next sublayer reads are one kernel."""

    def __init__(self, cfg: SotazenConfig, i: int, dtype=None, device=None):
        super().__init__()
        l, H = cfg.layers[i], cfg.hidden_size
        self.kind, self.hidden, self.eps, self.alpha = l["type"], H, cfg.rms_norm_eps, cfg.alpha

        def norm():
            return nn.Parameter(torch.zeros(pad8(H), dtype=dtype, device=device), requires_grad=False)
        self.mix = _mixer(l, H, cfg.rms_norm_eps, dtype, device)
        self.norm1 = norm()
        self.ff = SquaredReLU(H, l["mlp"]["ff"], dtype, device) if l.get("mlp") is not None else None
        self.norm2 = norm() if self.ff is not None else None

    def kv_shape(self) -> Optional[Tuple[int, int, int]]:
        return self.mix.kv_shape()

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return self.mix.state_shapes()

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        t = {prefix + "norm1": Slot(self.norm1.data[:self.hidden], (self.hidden,))} | self.mix.tensors(prefix + "mix.")
        if self.ff is not None:
            t[prefix + "norm2"] = Slot(self.norm2.data[:self.hidden], (self.hidden,))
            t |= self.ff.tensors(prefix + "mlp.")
        return t

    def forward(self, x: torch.Tensor, h: torch.Tensor, p, kv, state, rope, next_norm: Optional[torch.Tensor]):
        """One layer over a step's rows.  ``x``: fp32 residual, updated in place; ``h``: the same in the activation dtype; returns
        the new ``h``.  ``p``: row layout; ``kv``, ``state``: this layer's pages and state slots; ``rope(base, dims)``: the
        step's rotary tables."""
        y, after = self.mix.run(h, p, kv, state, rope)
        h = ops.post_norm(x, y, self.norm1, self.alpha, self.hidden, self.eps, **after)
        if self.ff is not None:
            h = ops.post_norm(x, self.ff.run(h), self.norm2, self.alpha, self.hidden, self.eps)
        return h


class SotazenModel(nn.Module):
    """Weights and per-layer computation.  Inference only, one GPU (``tp_size`` 1)."""

    tp_size, tp_rank, tp_group = 1, 0, None
    layer_start, is_first_stage, is_last_stage, tied = 0, True, True, True

    def __init__(self, cfg: SotazenConfig, dtype=None, device=None):
        super().__init__()
        dtype = dtype or torch.float32
        self.cfg = cfg
        W = pad8(cfg.hidden_size)
        self.embed_tokens = nn.Parameter(torch.zeros(pad8(cfg.vocab_size), W, dtype=dtype, device=device), requires_grad=False)
        self.layers = nn.ModuleList([SotazenLayer(cfg, i, dtype, device) for i in range(len(cfg.layers))])
        self.norm = nn.Parameter(torch.zeros(W, dtype=dtype, device=device), requires_grad=False)

    def checkpoint(self) -> Dict[str, Slot]:
        """Checkpoint name -> where the tensor lives."""
        c = self.cfg
        t = {"embed": Slot(self.embed_tokens.data[:c.vocab_size, :c.hidden_size], (c.vocab_size, c.hidden_size)),
             "final.norm": Slot(self.norm.data[:c.hidden_size], (c.hidden_size,))}
        for i, layer in enumerate(self.layers):
            t |= layer.tensors(f"l{i}.")
        return t

    def named_checkpoint_tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        for name, slot in self.checkpoint().items():
            yield name, slot.export()

    @torch.no_grad()
    def init_weights(self, seed: int = 0, std: Optional[float] = None):
        """Deterministic random weights: projections N(0, std), norms 1, biases and sinks 0, the lambda vectors small."""
        import zlib
        std = self.cfg.init_std if std is None else std
        dev = self.embed_tokens.device
        for name, slot in self.checkpoint().items():
            last = name.rsplit(".", 1)[-1]
            g = torch.Generator(device=dev).manual_seed((zlib.crc32(name.encode()) + 1000003 * seed) % (2 ** 62))
            r = torch.empty(slot.shape, dtype=torch.float32, device=dev)
            if last.startswith("norm"):
                r.fill_(1.0)
            elif last in ("b", "sink"):
                r.zero_()
            else:
                r.normal_(0.0, 0.1 if last in ("lq1", "lk1", "lq2", "lk2") else std, generator=g)
            slot.load(r)

    # ---- what the runtime allocates for it --------------------------------------------------------------------
    def kv_layer_shapes(self) -> List[Optional[Tuple[int, int, int]]]:
        """Per layer ``(kv heads, key size, value size)`` of its pages, None for a layer without any."""
        return [l.kv_shape() for l in self.layers]

    def state_layer_shapes(self) -> List[Dict[str, Tuple[int, ...]]]:
        """Per layer the fp32 state tensors one sequence holds."""
        return [l.state_shapes() for l in self.layers]

    # ---- pieces the runner calls ------------------------------------------------------------------------------
    def embed(self, ids: torch.Tensor, p=None, state=None):
        """The residual stream's first rows (fp32) and the same in the activation dtype, which the first layer reads."""
        return ops.embedding_f32(ids, self.embed_tokens, self.cfg.vocab_size, self.cfg.embed_scale, h=True)

    def logits_from_hidden(self, h: torch.Tensor) -> torch.Tensor:
        out = torch.empty((h.shape[0], self.embed_tokens.shape[0]), dtype=torch.float32, device=h.device)
        return ops.gemm(h, self.embed_tokens, out=out)[:, :self.cfg.vocab_size]

    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor) -> torch.Tensor:
        """``[B, S]`` token ids -> ``[B, S, V]`` logits, recomputed from nothing (a cache that lives for the call)."""
        from ..infer.hybrid import whole_sequences
        return whole_sequences(self, input_ids)


def sotazen_preset(width: int, heads: int, depth: int, ff: int, vocab: int, kv_heads: int, window: int = 1024,
                   rank: int = 512, dim: int = 128, rot: int = 64, every: int = 4) -> SotazenConfig:
    """A configuration at the scale of a real model: of every ``every`` layers the last is latent attention, the one before it
    differential attention in a window, the others lightning."""
    layers: List[Dict[str, Any]] = []
    for i in range(depth):
        if i % every == every - 1:
            l = {"type": "latent_attention", "mixer": {
                "heads": heads, "dim": dim, "rot_dim": rot, "vdim": dim, "kv_rank": rank, "scale": (dim + rot) ** -0.5,
                "rot": {"base": 10000.0, "dims": rot}}}
        elif i % every == every - 2:
            l = {"type": "attention", "mixer": {
                "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "softcap": 30.0,
                "mask": {"size": window}, "rot": {"base": 10000.0, "dims": dim}, "diff": 0.4}}
        else:
            l = {"type": "lightning", "mixer": {
                "heads": heads, "dim": dim, "vdim": dim,
                "decay": [1.0 - 2.0 ** (-5.0 - 7.0 * h / max(1, heads - 1)) for h in range(heads)]}}
        layers.append({**l, "mlp": {"kind": "dense", "ff": ff}})
    return SotazenConfig(vocab, width, layers, embed_scale=width ** 0.5, alpha=(2.0 * depth) ** 0.25)


SOTAZEN_PRESETS = {
    "sotazen-tiny": sotazen_preset(256, 2, 4, 512, 1024, 1, window=64, rank=64, dim=64, rot=32),
    # the widths, depth and vocabulary of the framework's dense presets of the same size; the feed-forward, which has two matrices
    # instead of three, is wider
    "sotazen-0.6b": sotazen_preset(1024, 8, 28, 5120, 151936, 4),
    "sotazen-4b": sotazen_preset(2560, 16, 36, 15104, 151936, 4),
}
