"""Lufivik: a decoder whose layers are latent attention in a sliding window with an input convolution and a gate per head, and
clamped-gate experts behind a softmax router.  Each sublayer stands between two layer norms, ``x <- x + s norm_b(g sublayer(norm_a(x)))``
with a gate g made from the sublayer's input and a scale s per channel; a run of layers may be passed several times, each time with a
cache and state of its own; the embedding adds a vector of the pair of tokens.  Built from :mod:`b200fw.model.mixers`; the cache, the
step and the loop over layers belong to the inference runtime (:mod:`b200fw.infer.hybrid`)."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Iterator, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops.portions import pad8
from .mixers import ExpertFF, InputConv, LatentAttention, LayerNorm, PackedRows, Slot

GATE_SLOPE = 1.702          # of the experts' gate: g sigmoid(GATE_SLOPE g)
_MIXER = {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "mask", "rot"}


def _need(where: str, have, fields) -> None:
    missing = set(fields) - set(have or {})
    if missing:
        raise ValueError(f"{where} is missing {sorted(missing)}")


@dataclass
class LufivikConfig:
    """``config.json`` of the design."""
    vocab_size: int
    hidden_size: int
    layers: List[Dict[str, Any]]
    buckets: int = 1                          # of the table of token pairs, which has one more row
    mul_prev: int = 1
    mul_cur: int = 1
    taps: int = 1                             # of the input convolution
    loop: Optional[Dict[str, int]] = None     # {"start", "stop", "times"}: layers start .. stop - 1 run so many times in a row
    norm_eps: float = 1e-6
    init_std: float = 0.02
    # positions are computed, not looked up: nothing but the cache bounds the context
    max_position_embeddings: int = 1 << 30

    architecture = "Lufivik"

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            if l.get("type") != "latent_attention":
                raise ValueError(f"layer {i}: unknown type {l.get('type')!r}")
            m, f = l.get("mixer"), l.get("mlp")
            _need(f"layer {i}: the mixer", m, _MIXER)
            if m["rot"]["dims"] != m["rot_dim"]:
                raise ValueError(f"layer {i}: rot.dims {m['rot']['dims']} is not the rotated size {m['rot_dim']}")
            if m["mask"]["size"] < 1:
                raise ValueError(f"layer {i}: a window of {m['mask']['size']} tokens")
            if f is not None:
                if f.get("kind") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
                _need(f"layer {i}: the feed-forward", f, {"expert", "router"})
                _need(f"layer {i}: the experts", f["expert"], {"ff", "limit"})
                _need(f"layer {i}: the router", f["router"], {"experts", "top"})
        if self.loop is not None:
            _need("the loop", self.loop, {"start", "stop", "times"})
            if not 0 <= self.loop["start"] <= self.loop["stop"] <= len(self.layers) or self.loop["times"] < 1:
                raise ValueError(f"the loop {self.loop} does not fit {len(self.layers)} layers")
        if self.buckets < 1:
            raise ValueError("the table of token pairs needs a bucket")

    @classmethod
    def from_dict(cls, d: Dict[str, Any], shapes: Optional[Dict[str, Tuple[int, ...]]] = None) -> "LufivikConfig":
        _need("config.json", d, {"vocab", "width", "layers", "norm", "embedding", "canon"})
        _need("config.json: the embedding", d["embedding"], {"bigram"})
        b = d["embedding"]["bigram"]
        _need("config.json: the bigram embedding", b, {"buckets", "mul_prev", "mul_cur"})
        return cls(int(d["vocab"]), int(d["width"]), d["layers"], int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"]),
                   int(d["canon"]["taps"]), d.get("loop"), float(d["norm"]["eps"]))

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
             "canon": {"taps": self.taps}, "layers": copy.deepcopy(self.layers),
             "embedding": {"bigram": {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}}}
        return d if self.loop is None else d | {"loop": dict(self.loop)}

    def layer_runs(self) -> List[int]:
        """Which layer every run uses."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b = self.loop["start"], self.loop["stop"]
        return list(range(a)) + list(range(a, b)) * self.loop["times"] + list(range(b, n))

    # ---- the summary numbers other parts of the framework show or size things by --------------------------------
    @property
    def num_layers(self) -> int:
        """Layer runs: what has a cache of its own and costs time."""
        return len(self.layer_runs())

    @property
    def num_heads(self) -> int:
        return max([l["mixer"]["heads"] for l in self.layers] or [1])

    @property
    def num_kv_heads(self) -> int:
        return 1

    @property
    def head_dim(self) -> int:
        return max([l["mixer"]["dim"] for l in self.layers] or [8])

    @property
    def intermediate_size(self) -> int:
        """Feed-forward channels a token passes through."""
        return max([l["mlp"]["expert"]["ff"] * l["mlp"]["router"]["top"] for l in self.layers if l.get("mlp") is not None] or [0])

    def kv_bytes_per_token(self, element: int = 2) -> int:
        return sum(pad8(m["kv_rank"]) + pad8(m["rot_dim"]) for m in (self.layers[i]["mixer"] for i in self.layer_runs())) * element

    def num_params(self) -> int:
        with torch.device("meta"):
            return sum(torch.Size(s.shape).numel() for s in LufivikModel(self, device="meta").checkpoint().values())

    def num_active_params(self) -> int:
        """Parameters one token is multiplied with, once per run of their layer: no experts that are not chosen, no rows of the tables
        that are not looked up."""
        n = 2 * self.vocab_size * self.hidden_size          # head and, like elsewhere, the embedding
        with torch.device("meta"):
            layers = LufivikModel(self, device="meta").layers
            size = [sum(torch.Size(s.shape).numel() for s in l.tensors("").values()) for l in layers]
        for i in self.layer_runs():
            f = self.layers[i].get("mlp")
            n += size[i]
            if f is not None:
                n -= (f["router"]["experts"] - f["router"]["top"]) * 3 * f["expert"]["ff"] * self.hidden_size
        return n


class LufivikLayer(nn.Module):
    """One layer: the mixer reads ``norm1(x)`` through the input convolution, the experts read ``norm2(x)`` (a layer may have none).  What
    follows a sublayer's output projection (its gate, its norm, the scale per channel, the sum, and the norm that the next sublayer reads)
    is one kernel; for the experts it also makes the weighted sum of their rows."""

    def __init__(self, cfg: LufivikConfig, i: int, dtype=None, device=None):
        super().__init__()
        l, H = cfg.layers[i], cfg.hidden_size
        m, f = l["mixer"], l.get("mlp")
        self.kind, self.hidden, self.eps = l["type"], H, cfg.norm_eps

        def vec():
            return nn.Parameter(torch.zeros(pad8(H), dtype=dtype, device=device), requires_grad=False)
        self.norm1, self.norm1b = LayerNorm(H, dtype, device), LayerNorm(H, dtype, device)
        self.conv = InputConv(H, cfg.taps, dtype, device)
        self.mix = LatentAttention(H, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], m["rot"]["base"], self.eps, dtype,
                                   device, q_rank=m["q_rank"], window=m["mask"]["size"], sink=False, gate=True, halves=True)
        self.gate1, self.gate1_bias, self.scale1 = PackedRows(H, [("rg1", 1, H)], dtype, device), vec(), vec()
        self.ff = None
        if f is not None:
            r = f["router"]
            self.norm2, self.norm2b = LayerNorm(H, dtype, device), LayerNorm(H, dtype, device)
            self.ff = ExpertFF(H, r["experts"], f["expert"]["ff"], r["top"], 1, 1, 1.0, None, dtype, device, score="softmax", corrected=False,
                               clamped=(GATE_SLOPE, float(f["expert"]["limit"])), beside=[("rg2", 1, H)])
            self.gate2_bias, self.scale2 = vec(), vec()

    def kv_shape(self) -> Optional[Tuple[int, int, int]]:
        return self.mix.kv_shape()

    def state_shapes(self) -> Dict[str, Tuple[int, ...]]:
        return {**self.mix.state_shapes(), "canon": self.conv.state_shape()}

    def tensors(self, prefix: str) -> Dict[str, Slot]:
        def vec(p):
            return Slot(p.data[:self.hidden], (self.hidden,))
        t = {**self.norm1.tensors(prefix + "norm1"), **self.norm1b.tensors(prefix + "norm1b"), **self.mix.tensors(prefix + "mix."),
             prefix + "canon1": self.conv.slot(), prefix + "rg1": self.gate1.slot("rg1"), prefix + "rg1.b": vec(self.gate1_bias),
             prefix + "ls1": vec(self.scale1)}
        if self.ff is not None:
            t |= {**self.norm2.tensors(prefix + "norm2"), **self.norm2b.tensors(prefix + "norm2b"), **self.ff.tensors(prefix + "mlp."),
                  prefix + "rg2": self.ff.router.slot("rg2"), prefix + "rg2.b": vec(self.gate2_bias), prefix + "ls2": vec(self.scale2)}
        return t

    def forward(self, x: torch.Tensor, h: torch.Tensor, p, kv, state, rope, next_norm: Optional[LayerNorm]):
        """One run over a step's rows.  ``x``: fp32 residual, updated in place; ``h``: ``norm1(x)`` in the activation dtype; returns
        ``next_norm(x)``, which the next run reads (None after the last).  ``p``: row layout; ``kv``, ``state``: this run's pages and
        state slots; ``rope(base, dims)``: the step's rotary tables."""
        after = None if next_norm is None else next_norm.pair
        gate = self.gate1(h)
        y, _ = self.mix.run(self.conv(h, state["canon"], p), p, kv, state, rope)
        h = ops.branch_add(x, y, self.norm1b.pair, self.hidden, self.eps, gate, self.gate1_bias, self.scale1,
                           after if self.ff is None else self.norm2.pair)
        if self.ff is None:
            return h
        y, z = self.ff.run(h)
        return ops.branch_add(x, y, self.norm2b.pair, self.hidden, self.eps, self.ff.router.cols(z, "rg2"), self.gate2_bias, self.scale2, after)


class LufivikModel(nn.Module):
    """Weights and per-layer computation.  Inference only, one GPU (``tp_size`` 1)."""

    tp_size, tp_rank, tp_group = 1, 0, None
    layer_start, is_first_stage, is_last_stage, tied = 0, True, True, False

    def __init__(self, cfg: LufivikConfig, dtype=None, device=None):
        super().__init__()
        dtype = dtype or torch.float32
        self.cfg = cfg
        W = pad8(cfg.hidden_size)

        def table(rows):
            return nn.Parameter(torch.zeros(rows, W, dtype=dtype, device=device), requires_grad=False)
        self.embed_tokens, self.pairs, self.head = table(cfg.vocab_size), table(cfg.buckets + 1), table(pad8(cfg.vocab_size))
        self.embed_norm, self.norm = LayerNorm(cfg.hidden_size, dtype, device), LayerNorm(cfg.hidden_size, dtype, device)
        self.layers = nn.ModuleList([LufivikLayer(cfg, i, dtype, device) for i in range(len(cfg.layers))])

    def checkpoint(self) -> Dict[str, Slot]:
        """Checkpoint name -> where the tensor lives."""
        c = self.cfg

        def rows(p, n):
            return Slot(p.data[:n, :c.hidden_size], (n, c.hidden_size))
        t = {"embed": rows(self.embed_tokens, c.vocab_size), "bigram": rows(self.pairs, c.buckets + 1), "head": rows(self.head, c.vocab_size),
             **self.embed_norm.tensors("embed.norm"), **self.norm.tensors("final.norm")}
        for i, layer in enumerate(self.layers):
            t |= layer.tensors(f"l{i}.")
        return t

    def named_checkpoint_tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        for name, slot in self.checkpoint().items():
            yield name, slot.export()

    @torch.no_grad()
    def init_weights(self, seed: int = 0, std: Optional[float] = None):
        """Deterministic random weights: projections N(0, std), norms and scales 1, biases 0, small convolutions."""
        import zlib
        std = self.cfg.init_std if std is None else std
        dev = self.embed_tokens.device
        for name, slot in self.checkpoint().items():
            last = name.rsplit(".", 1)[-1]
            g = torch.Generator(device=dev).manual_seed((zlib.crc32(name.encode()) + 1000003 * seed) % (2 ** 62))
            r = torch.empty(slot.shape, dtype=torch.float32, device=dev)
            if last.startswith("norm") or last in ("ls1", "ls2"):
                r.fill_(1.0)
            elif last == "b":
                r.zero_()
            elif last == "canon1":
                r.uniform_(-0.3, 0.3, generator=g)
            else:
                r.normal_(0.0, std, generator=g)
            slot.load(r)

    # ---- what the runtime allocates for it --------------------------------------------------------------------
    def layer_runs(self) -> List[int]:
        """Which layer every run of the step uses."""
        return self.cfg.layer_runs()

    def kv_layer_shapes(self) -> List[Optional[Tuple[int, int, int]]]:
        """Per run ``(kv heads, key size, value size)`` of its pages."""
        return [self.layers[i].kv_shape() for i in self.layer_runs()]

    def state_layer_shapes(self) -> List[Dict[str, Tuple[int, ...]]]:
        """Per run the fp32 state tensors one sequence holds."""
        return [self.layers[i].state_shapes() for i in self.layer_runs()]

    def state_sequence_shapes(self) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        """What one sequence holds outside the layers: its last token."""
        return {"last": ((), torch.int32)}

    # ---- pieces the runner calls ------------------------------------------------------------------------------
    def embed(self, ids: torch.Tensor, p, state):
        """The residual stream's first rows (fp32) and their norm in the activation dtype, which the first run reads."""
        c, runs = self.cfg, self.layer_runs()
        first = self.layers[runs[0]].norm1 if runs else self.norm
        return ops.embedding_pairs(ids, self.embed_tokens, self.pairs, state["last"], p, c.vocab_size, c.mul_prev, c.mul_cur,
                                   self.embed_norm.pair, c.hidden_size, c.norm_eps, first.pair)

    def final_norm(self, x: torch.Tensor, rows: Optional[torch.Tensor]) -> torch.Tensor:
        return ops.layernorm_f32(x, self.norm.pair, self.cfg.hidden_size, self.cfg.norm_eps, rows)

    def logits_from_hidden(self, h: torch.Tensor) -> torch.Tensor:
        out = torch.empty((h.shape[0], self.head.shape[0]), dtype=torch.float32, device=h.device)
        return ops.gemm(h, self.head, out=out)[:, :self.cfg.vocab_size]

    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor) -> torch.Tensor:
        """``[B, S]`` token ids -> ``[B, S, V]`` logits, recomputed from nothing (a cache that lives for the call)."""
        from ..infer.hybrid import whole_sequences
        return whole_sequences(self, input_ids)


def lufivik_preset(width: int, heads: int, depth: int, vocab: int, q_rank: int, experts: int, top: int, expert_ff: int, loop: Tuple[int, int, int],
                   window: int = 1024, rank: int = 512, dim: int = 128, rot: int = 64, taps: int = 4) -> LufivikConfig:
    """A configuration at the scale of a real model: ``depth`` layers of which ``loop = (start, stop, times)`` says what runs again."""
    l = {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot, "vdim": dim, "q_rank": q_rank, "kv_rank": rank, "scale": (dim + rot) ** -0.5,
        "mask": {"size": window}, "rot": {"base": 10000.0, "dims": rot}},
        "mlp": {"kind": "moe", "expert": {"ff": expert_ff, "limit": 7.0}, "router": {"experts": experts, "top": top}}}
    return LufivikConfig(vocab, width, [copy.deepcopy(l) for _ in range(depth)], buckets=vocab, mul_prev=48271, mul_cur=16807, taps=taps,
                         loop=dict(zip(("start", "stop", "times"), loop)))


LUFIVIK_PRESETS = {
    "lufivik-tiny": lufivik_preset(256, 2, 3, 1024, 96, 8, 2, 128, (1, 2, 2), window=64, rank=64, dim=64, rot=32),
    # the widths, head counts, layer runs and vocabulary of the framework's other presets of the same size; as many feed-forward channels
    # per token as theirs, in four chosen experts
    "lufivik-0.6b": lufivik_preset(1024, 8, 20, 151936, 512, 32, 4, 768, (8, 12, 3)),
    "lufivik-4b": lufivik_preset(2560, 16, 24, 151936, 1024, 32, 4, 2432, (8, 14, 3)),
}
