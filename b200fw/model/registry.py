"""Model registry: which configuration, model class and checkpoint layout a ``config.json`` stands for, and which preset
names exist.  The inference engine, the command line and the trace runner choose the model here."""
from __future__ import annotations

import json
import os
import struct
from dataclasses import dataclass
from typing import Any, Callable, Dict, Iterable, Tuple

import torch

from . import hf_io
from .config import PRESETS as DENSE_PRESETS
from .config import ModelConfig
from .fetelorn import FETELORN_PRESETS, FetelornConfig, FetelornModel
from .lufivik import LUFIVIK_PRESETS, LufivikConfig, LufivikModel
from .qwen3 import ParallelTransformerModel
from .ruburax import RUBURAX_PRESETS, RuburaxConfig, RuburaxModel
from .sotazen import SOTAZEN_PRESETS, SotazenConfig, SotazenModel


@dataclass(frozen=True)
class Architecture:
    name: str
    config_type: type
    read_config: Callable[[str], Any]                       # folder -> configuration
    build: Callable[..., torch.nn.Module]                   # (config, dtype=, device=) -> model
    load: Callable[[torch.nn.Module, str], Tuple[int, int]]     # (model, folder) -> (loaded, missing)
    sources: Tuple[str, ...] = ()                           # csrc/ files its inference uses
    float32: bool = False                                   # its kernels also run in true 32-bit on a GPU


def safetensors_shapes(path: str) -> Dict[str, Tuple[int, ...]]:
    """Tensor name -> shape from the headers of a folder's ``*.safetensors`` files (the data is not read)."""
    shapes: Dict[str, Tuple[int, ...]] = {}
    for f in sorted(x for x in os.listdir(path) if x.endswith(".safetensors")):
        with open(os.path.join(path, f), "rb") as fh:
            (n,) = struct.unpack("<Q", fh.read(8))
            head = json.loads(fh.read(n))
        shapes.update({k: tuple(v["shape"]) for k, v in head.items() if k != "__metadata__"})
    return shapes


def _config_json(path: str) -> Dict[str, Any]:
    with open(os.path.join(path, "config.json")) as f:
        return json.load(f)


def load_slots(model, tensors: Iterable[Tuple[str, torch.Tensor]], strict: bool = True, where: str = "") -> Tuple[int, int]:
    """Copy named tensors into a model that maps its checkpoint with :class:`b200fw.model.mixers.Slot` (in place: captured
    graphs stay valid).  Shapes are checked for all of them before the first one is copied; ``strict`` wants exactly the
    model's tensors."""
    slots, copies, bad = model.checkpoint(), [], []
    for name, t in tensors:
        s = slots.get(name)
        if s is None:
            if strict:
                bad.append(f"{name}: not a tensor of this model")
            continue
        if tuple(t.shape) != s.shape:
            bad.append(f"{name}: checkpoint {tuple(t.shape)}, model {s.shape}")
        copies.append((name, s, t))
    missing = len(slots) - len({n for n, _, _ in copies})
    if strict and missing:
        bad += [f"{n}: missing" for n in slots if n not in {c[0] for c in copies}]
    if bad:
        raise ValueError(f"{where or 'weights'} do not fit this model ({len(bad)} tensors), nothing was loaded: "
                         + "; ".join(bad[:4]) + (" ..." if len(bad) > 4 else ""))
    with torch.no_grad():
        for _, s, t in copies:
            s.load(t)
    return len(copies), missing


def _load_slots_at(model, path: str, strict: bool = True) -> Tuple[int, int]:
    return load_slots(model, hf_io._load_all(path).items(), strict, path)


ARCHITECTURES: Dict[str, Architecture] = {
    "Qwen3ForCausalLM": Architecture("Qwen3ForCausalLM", ModelConfig, hf_io.read_hf_config,
                                     lambda mc, dtype=None, device=None: ParallelTransformerModel(mc, dtype=dtype, device=device),
                                     hf_io.load_from_hf_checkpoint,
                                     ("host", "gemm", "norm_rope", "attention_fwd", "paged", "sampling")),
    "Fetelorn": Architecture("Fetelorn", FetelornConfig,
                             lambda path: FetelornConfig.from_dict(_config_json(path), safetensors_shapes(path)),
                             FetelornModel, _load_slots_at,
                             ("host", "gemm", "residual", "linear_state", "retention_chunk", "delta_chunk", "attention_rows", "attention_fwd", "sampling"), float32=True),
    "Sotazen": Architecture("Sotazen", SotazenConfig, lambda path: SotazenConfig.from_dict(_config_json(path)), SotazenModel,
                            _load_slots_at, ("host", "gemm", "residual", "linear_state", "retention_chunk", "attention_rows",
                                             "attention_decode", "attention_latent", "attention_fwd", "sampling"), float32=True),
    "Ruburax": Architecture("Ruburax", RuburaxConfig, lambda path: RuburaxConfig.from_dict(_config_json(path)), RuburaxModel,
                            _load_slots_at, ("host", "gemm", "residual", "linear_state", "retention_chunk", "recurrence", "moe",
                                             "attention_rows", "attention_decode", "attention_latent", "attention_fwd", "sampling"),
                            float32=True),
    "Lufivik": Architecture("Lufivik", LufivikConfig, lambda path: LufivikConfig.from_dict(_config_json(path)), LufivikModel,
                            _load_slots_at, ("host", "gemm", "residual", "recurrence", "moe", "attention_decode", "attention_latent",
                                             "attention_fwd", "sampling"), float32=True),
}
PRESETS: Dict[str, Any] = {**DENSE_PRESETS, **FETELORN_PRESETS, **SOTAZEN_PRESETS, **RUBURAX_PRESETS, **LUFIVIK_PRESETS}


def architecture_at(path: str) -> Architecture:
    """The architecture a model folder holds: ``architecture`` of its config.json, else the dense decoder family (whose
    configuration check names what is missing)."""
    name = _config_json(path).get("architecture")
    if name is None:
        return ARCHITECTURES["Qwen3ForCausalLM"]
    if name not in ARCHITECTURES:
        raise ValueError(f"{path}: unknown architecture {name!r} (known: {sorted(ARCHITECTURES)})")
    return ARCHITECTURES[name]


def architecture_of(cfg) -> Architecture:
    """The architecture a configuration object belongs to."""
    for a in ARCHITECTURES.values():
        if isinstance(cfg, a.config_type):
            return a
    raise TypeError(f"no architecture is registered for {type(cfg).__name__}")


def read_config(path: str):
    return architecture_at(path).read_config(path)


def build_model(cfg, dtype=None, device=None):
    return architecture_of(cfg).build(cfg, dtype=dtype, device=device)


def load_checkpoint(model, path: str) -> Tuple[int, int]:
    return architecture_of(model.cfg).load(model, path)


def save_checkpoint(model, path: str) -> None:
    """Write a folder this registry reads back."""
    if not hasattr(model, "checkpoint"):
        hf_io.save_hf_checkpoint(model, path)
        return
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(model.cfg.to_dict(), f, indent=2)
    save_file({k: v.cpu().contiguous().clone() for k, v in model.named_checkpoint_tensors()},
              os.path.join(path, "model.safetensors"), metadata={"format": "pt"})
