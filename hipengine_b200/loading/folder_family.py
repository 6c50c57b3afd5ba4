"""What a family with checkpoint folders contributes, and the parts its readers share.

A family module provides ``config_from_json`` / ``config_to_json`` and ``tensor_shapes`` (every tensor of a checkpoint with
its shape, in file order); the registry names the module.
"""
from __future__ import annotations

from dataclasses import asdict
from importlib import import_module
from typing import Any, Callable, Dict, Mapping, Optional, Sequence, Tuple

import torch

from ..models.config import BandSpec, LoopSpec, ModelConfig, RotarySpec, YarnSpec
from ..quant.ggml import GGMLType
from .weights import ModelWeights, QTensor

Shapes = Mapping[str, Sequence[int]]


def family_module(cfg: ModelConfig):
    """The reader module of ``cfg``'s family."""
    from ..models.registry import plugin_for
    return import_module(plugin_for(cfg.arch).folder_reader)


def loop_from_json(c: Mapping[str, Any]) -> Optional[LoopSpec]:
    lp = c.get("loop")
    return LoopSpec(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None


def loop_to_json(loop: Optional[LoopSpec]) -> Optional[Dict[str, int]]:
    return {"start": loop.start, "stop": loop.stop, "times": loop.times} if loop else None


# keys of a rotation's scaling -> what it is
_SCALINGS = (BandSpec, ("factor", "low", "high", "original")), (YarnSpec, ("factor", "original", "fast", "slow"))


def rotary_from_json(r: Mapping[str, Any], halves: bool = False) -> RotarySpec:
    s, scaling = r.get("scaling"), None
    if s:
        found = [c(*(float(s[k]) for k in keys)) for c, keys in _SCALINGS if set(keys) <= set(s)]
        if not found:
            raise ValueError(f"unknown scaling of a rotation: {sorted(s)}")
        scaling = found[0]
    return RotarySpec(int(r["dims"]), float(r["base"]), scaling, halves)


def rotary_to_json(rot: RotarySpec) -> Dict[str, Any]:
    out: Dict[str, Any] = {"dims": rot.dims, "base": rot.base}
    if rot.scaling is not None:
        out["scaling"] = asdict(rot.scaling)
    return out


def check_tensors(cfg: ModelConfig, have: Shapes) -> None:
    """Every tensor the configuration needs is there, with its shape."""
    bad = [f"{n}: expected {list(s)}, found {list(have[n]) if n in have else 'nothing'}"
           for n, s in family_module(cfg).tensor_shapes(cfg).items() if n not in have or tuple(have[n]) != tuple(s)]
    if bad:
        raise KeyError(f"checkpoint does not match its configuration: {'; '.join(bad[:6])}"
                       + (f" and {len(bad) - 6} more" if len(bad) > 6 else ""))


def weights_from_tensors(cfg: ModelConfig, tensors: Mapping[str, torch.Tensor]) -> ModelWeights:
    """``ModelWeights`` over in-memory bfloat16 tensors under their checkpoint names."""
    check_tensors(cfg, {n: t.shape for n, t in tensors.items()})
    out = {}
    for n, t in tensors.items():
        b = t.to(torch.bfloat16).contiguous()
        rows = b.reshape(-1, b.shape[-1] if b.dim() else 1)
        out[n] = QTensor(n, GGMLType.BF16, tuple(b.shape), rows.view(torch.uint8))
    return ModelWeights(cfg, out, {"general.architecture": cfg.arch, "general.name": cfg.arch,
                                   "config": family_module(cfg).config_to_json(cfg)})


def build_random_folder(cfg: ModelConfig, seed: int = 0, device="cpu", std: float = 0.02,
                        adjust: Optional[Callable[[str, torch.Tensor], torch.Tensor]] = None) -> ModelWeights:
    """Random-init weights of a folder family; ``adjust`` maps (name, N(0, std) draw) to what is stored."""
    gen = torch.Generator(device=torch.device(device))
    gen.manual_seed(seed)
    tensors: Dict[str, torch.Tensor] = {}
    for n, shape in family_module(cfg).tensor_shapes(cfg).items():
        t = torch.randn(tuple(shape), generator=gen, device=device, dtype=torch.float32) * std
        tensors[n] = (adjust(n, t) if adjust is not None else t).to(torch.bfloat16)
    w = weights_from_tensors(cfg, tensors)
    w.metadata["general.name"] = f"random-init {cfg.arch} seed={seed}"
    return w
