"""Fetelorn: a decoder whose layers mix retention (fixed-decay linear attention) with layers that run chunked softmax
attention and a gated delta rule side by side, over a 32-bit residual stream; mixer and feed-forward of a layer read one
norm and are added together.  Built from :mod:`b200fw.model.mixers`; the cache, the step and the loop over layers belong to
the inference runtime (:mod:`b200fw.infer.hybrid`)."""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, Iterator, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops.portions import pad8
from .mixers import BiasedChunkAttention, DenseGLU, GatedDelta, PackedCols, PackedRows, Retention, Sections, Slot


@dataclass
class FetelornConfig:
    """``config.json`` of the design.  What only the tensors' shapes say (rows of the distance-bias tables, ranks of the two
    low-rank projections) is given per layer by ``ranks``: one dictionary per layer, filled in from the checkpoint."""
    vocab_size: int
    hidden_size: int
    layers: List[Dict[str, Any]]
    rms_norm_eps: float = 1e-6
    ranks: List[Dict[str, int]] = field(default_factory=list)
    init_std: float = 0.02
    # positions are computed, not looked up: nothing but the cache bounds the context
    max_position_embeddings: int = 1 << 30

    architecture = "Fetelorn"

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            if l.get("type") not in ("retention", "parallel"):
                raise ValueError(f"layer {i}: unknown type {l.get('type')!r}")
            if l.get("mlp") is not None and l["mlp"].get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {l['mlp'].get('kind')!r}")
        if not self.ranks:
            self.ranks = [{"bias_rows": 32, "decay_rank": 64, "gate_rank": 64} for _ in self.layers]

    @classmethod
    def from_dict(cls, d: Dict[str, Any], shapes: Optional[Dict[str, Tuple[int, ...]]] = None) -> "FetelornConfig":
        missing = {"vocab", "width", "layers", "norm"} - set(d)
        if missing:
            raise ValueError(f"config.json is missing required fields: {sorted(missing)}")
        ranks = []
        for i, l in enumerate(d["layers"] if shapes is not None else []):
            r = {}
            if l.get("type") == "parallel":
                p = f"l{i}.mix."
                try:
                    r = {"bias_rows": shapes[p + "left.rel"][0], "decay_rank": shapes[p + "right.a1"][0],
                         "gate_rank": shapes[p + "right.g1"][0]}
                except KeyError as e:
                    raise ValueError(f"checkpoint has no tensor {e.args[0]!r}") from None
            ranks.append(r)
        return cls(int(d["vocab"]), int(d["width"]), d["layers"], float(d["norm"]["eps"]), ranks)

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.rms_norm_eps}, "layers": copy.deepcopy(self.layers)}

    # ---- the summary numbers other parts of the framework show or size things by --------------------------------
    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def _attention(self) -> List[Dict[str, Any]]:
        return [l["mixer"]["left"] for l in self.layers if l["type"] == "parallel"]

    @property
    def num_heads(self) -> int:
        return max([a["heads"] for a in self._attention()] + [l["mixer"]["heads"] for l in self.layers if l["type"] == "retention"] or [1])

    @property
    def num_kv_heads(self) -> int:
        return max([a["kv_heads"] for a in self._attention()] or [1])

    @property
    def head_dim(self) -> int:
        return max([a["dim"] for a in self._attention()] or [8])

    @property
    def intermediate_size(self) -> int:
        return max([l["mlp"]["ff"] for l in self.layers if l.get("mlp") is not None] or [0])

    def kv_bytes_per_token(self, element: int = 2) -> int:
        return sum(a["kv_heads"] * (pad8(a["dim"]) + pad8(a["vdim"])) for a in self._attention()) * element

    def num_params(self) -> int:
        with torch.device("meta"):
            return sum(s.view.numel() for s in FetelornModel(self, device="meta").checkpoint().values())


class FetelornLayer(nn.Module):
    """``x += mixer(norm1(x)) + ff(norm1(x))``.  Everything that reads the normed input is one GEMM.  A retention mixer and the
    feed-forward also share the output GEMM, accumulated into the residual; a parallel mixer has two output projections of
    its own (each is normed before the sum) and only the feed-forward accumulates."""

    def __init__(self, cfg: FetelornConfig, i: int, dtype=None, device=None):
        super().__init__()
        l, r, H, eps = cfg.layers[i], cfg.ranks[i], cfg.hidden_size, cfg.rms_norm_eps
        m = l["mixer"]
        self.kind, self.hidden, self.eps = l["type"], H, eps
        self.norm1 = nn.Parameter(torch.zeros(pad8(H), dtype=dtype, device=device), requires_grad=False)
        self.ff = DenseGLU(H, l["mlp"]["ff"]) if l.get("mlp") is not None else None
        blocks: List[Tuple[str, nn.Module]] = []
        if self.kind == "retention":
            rot = m.get("rot") or {"base": 1.0, "dims": 0}
            self.retention = Retention(H, m["heads"], m["dim"], m["vdim"], m["decay"], rot["base"], rot["dims"], eps, dtype, device)
            blocks.append(("", self.retention))
        else:
            a, b = m["left"], m["right"]
            self.left = BiasedChunkAttention(H, a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], a["mask"]["size"],
                                             r["bias_rows"], a["bias_max"], eps, dtype, device)
            self.right = GatedDelta(H, b["heads"], b["kv_heads"], b["dim"], b["vdim"], b["conv"], r["decay_rank"],
                                    r["gate_rank"], eps, dtype, device)
            self.left_out = nn.Parameter(torch.zeros(pad8(H), dtype=dtype, device=device), requires_grad=False)
            self.right_out = nn.Parameter(torch.zeros(pad8(H), dtype=dtype, device=device), requires_grad=False)
            blocks += [("left.", self.left), ("right.", self.right)]
        if self.ff is not None:
            blocks.append(("ff.", self.ff))
        self.in_proj = PackedRows(H, [(p + n, h, d) for p, b in blocks for n, h, d in b.in_sections], dtype, device)
        joint = [(p + b.out_section[0],) + b.out_section[1:] for p, b in blocks if getattr(b, "joint", False)]
        self.out_proj = PackedCols(H, joint, dtype, device) if joint else None

    def kv_shape(self) -> Optional[Tuple[int, int, int]]:
        return self.left.kv_shape() if self.kind == "parallel" else None

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return (self.right if self.kind == "parallel" else self.retention).state_shapes()

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        H = self.hidden

        def vec(p):
            return Slot(p.data[:H], (H,))
        t = {prefix + "norm1": vec(self.norm1)}
        if self.kind == "retention":
            t |= self.retention.tensors(prefix + "mix.", Sections(self.in_proj, ""), self.out_proj.slot("o"))
        else:
            t |= self.left.tensors(prefix + "mix.left.", Sections(self.in_proj, "left."))
            t |= self.right.tensors(prefix + "mix.right.", Sections(self.in_proj, "right."))
            t[prefix + "mix.left.out"], t[prefix + "mix.right.out"] = vec(self.left_out), vec(self.right_out)
        if self.ff is not None:
            t |= self.ff.tensors(prefix + "mlp.", Sections(self.in_proj, "ff."), self.out_proj.slot("ff.down"))
        return t

    def forward(self, x: torch.Tensor, h: Optional[torch.Tensor], p, kv, state, rope, next_norm: Optional[torch.Tensor]):
        """One layer over a step's rows.  ``x``: fp32 residual, updated in place; ``h``: ``norm1(x)`` if the previous layer's
        last kernel already produced it.  ``p``: row layout (:class:`b200fw.ops.portions.Portions`); ``kv``, ``state``: this
        layer's pages and state slots; ``rope(base, dims)``: the step's rotary tables.  Returns the next layer's ``h`` or
        None."""
        if h is None:
            h = ops.rmsnorm_f32(x, self.norm1, self.hidden, self.eps)
        y = self.in_proj(h)
        buf = self.out_proj.buffer(x.shape[0]) if self.out_proj is not None else None
        if self.ff is not None:
            self.ff.run(Sections(self.in_proj, "ff.", y), self.out_proj.cols(buf, "ff.down"))
        if self.kind == "retention":
            self.retention.run(Sections(self.in_proj, "", y), self.out_proj.cols(buf, "o"), p, state, rope)
            self.out_proj(buf, accumulate_into=x)
            return None
        left = self.left.run(Sections(self.in_proj, "left.", y), p, kv)
        right = self.right.run(Sections(self.in_proj, "right.", y), p, state)
        if self.ff is not None:
            self.out_proj(buf, accumulate_into=x)
        return ops.merge_norm_add(x, left, right, self.left_out, self.right_out, 0.5, self.hidden, self.eps, next_norm)


class FetelornModel(nn.Module):
    """Weights and per-layer computation.  Inference only, one GPU (``tp_size`` 1)."""

    tp_size, tp_rank, tp_group = 1, 0, None
    layer_start, is_first_stage, is_last_stage, tied = 0, True, True, True

    def __init__(self, cfg: FetelornConfig, dtype=None, device=None):
        super().__init__()
        dtype = dtype or torch.float32
        self.cfg = cfg
        W = pad8(cfg.hidden_size)
        self.embed_tokens = nn.Parameter(torch.zeros(pad8(cfg.vocab_size), W, dtype=dtype, device=device), requires_grad=False)
        self.layers = nn.ModuleList([FetelornLayer(cfg, i, dtype, device) for i in range(len(cfg.layers))])
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
        """Deterministic random weights: projections N(0, std), norms 1, decays and biases in a usable range."""
        import zlib
        std = self.cfg.init_std if std is None else std
        for name, slot in self.checkpoint().items():
            last = name.rsplit(".", 1)[-1]
            g = torch.Generator(device=slot.view.device).manual_seed((zlib.crc32(name.encode()) + 1000003 * seed) % (2 ** 62))
            shape = slot.view.shape
            r = torch.empty(shape, dtype=torch.float32, device=slot.view.device)
            if last in ("norm1", "norm", "out"):
                r.fill_(1.0)
            elif last == "A_log":
                r.uniform_(0.0, 2.0, generator=g)
            elif last == "dt_bias":
                r.uniform_(-6.0, -2.0, generator=g)
            elif last == "conv":
                r.uniform_(-0.5, 0.5, generator=g)
            else:
                r.normal_(0.0, std, generator=g)
            slot.view.copy_(r.to(slot.view.dtype))

    # ---- what the runtime allocates for it --------------------------------------------------------------------
    def kv_layer_shapes(self) -> List[Optional[Tuple[int, int, int]]]:
        """Per layer ``(kv heads, key size, value size)`` of its pages, None for a layer without any."""
        return [l.kv_shape() for l in self.layers]

    def state_layer_shapes(self) -> List[Dict[str, Tuple[int, ...]]]:
        """Per layer the fp32 state tensors one sequence holds."""
        return [l.state_shapes() for l in self.layers]

    # ---- pieces the runner calls ------------------------------------------------------------------------------
    def embed(self, ids: torch.Tensor, p=None, state=None):
        """The residual stream's first rows (fp32), and what the first layer reads if that is not its own norm's business."""
        return ops.embedding_f32(ids, self.embed_tokens, self.cfg.vocab_size), None

    def logits_from_hidden(self, h: torch.Tensor) -> torch.Tensor:
        out = torch.empty((h.shape[0], self.embed_tokens.shape[0]), dtype=torch.float32, device=h.device)
        return ops.gemm(h, self.embed_tokens, out=out)[:, :self.cfg.vocab_size]

    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor) -> torch.Tensor:
        """``[B, S]`` token ids -> ``[B, S, V]`` logits, recomputed from nothing (a cache that lives for the call)."""
        from ..infer.hybrid import whole_sequences
        return whole_sequences(self, input_ids)


def hybrid_preset(width: int, heads: int, depth: int, ff: int, vocab: int, kv_heads: int, chunk: int = 1024,
                  every: int = 4) -> FetelornConfig:
    """A configuration at the scale of a real model: every ``every``-th layer parallel, the others retention; 128-wide heads."""
    layers: List[Dict[str, Any]] = []
    for i in range(depth):
        mlp = {"kind": "dense", "ff": ff}
        if i % every == every - 1:
            layers.append({"type": "parallel", "mlp": mlp, "mixer": {
                "left": {"heads": heads, "kv_heads": kv_heads, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                         "mask": {"size": chunk}, "bias_max": 512},
                "right": {"heads": heads, "kv_heads": heads, "dim": 128, "vdim": 128, "conv": 4}}})
        else:
            layers.append({"type": "retention", "mlp": mlp, "mixer": {
                "heads": heads, "dim": 128, "vdim": 128, "rot": {"base": 10000.0, "dims": 128},
                "decay": [1.0 - 2.0 ** (-5.0 - 7.0 * h / max(1, heads - 1)) for h in range(heads)]}})
    return FetelornConfig(vocab, width, layers)


FETELORN_PRESETS = {
    "fetelorn-tiny": hybrid_preset(256, 2, 4, 512, 1024, 1, chunk=64, every=2),
    # the widths, head counts, depth and vocabulary of the framework's dense presets of the same size
    "fetelorn-0.6b": hybrid_preset(1024, 8, 28, 3072, 151936, 4),
    "fetelorn-4b": hybrid_preset(2560, 16, 36, 9728, 151936, 4),
}
