"""Milutar checkpoints: config.json <-> ``ModelConfig``, tensor names and shapes, random-init weights.

Tensor names: ``embed``, ``head``, ``final.norm`` (a single number), ``loop.step`` [times, width]; per layer ``l<i>.norm1`` (a
single number), ``.ls1``, ``.shift`` and, with a feed-forward, ``.mlp.up/down`` and ``.ls2``; attention ``.mix.q`` (or
``.mix.dq``, ``.mix.dq.norm``, ``.mix.uq``), ``.mix.dkv``, ``.mix.dkv.norm``, ``.mix.uk``, ``.mix.uv``, ``.mix.o`` and
``.mix.sink`` where the softmax has one.  Linear weights are [out, in].
"""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch

from ..models.config import DenseMlpSpec, LatentAttentionSpec, LayerSpec, ModelConfig, milutar_config
from .folder_family import build_random_folder, loop_from_json, loop_to_json, rotary_from_json, rotary_to_json
from .weights import ModelWeights

# mixer name -> (queries go through a latent, the softmax has a sink)
MIXERS = {"latent_attention": (False, False), "latent_attention_2": (True, True)}


# ----------------------------------------------------------------------------- configuration
def _layer(i: int, l: Mapping[str, Any]) -> LayerSpec:
    if l["type"] not in MIXERS:
        raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
    q_latent, sink = MIXERS[l["type"]]
    m, mlp = l["mixer"], l.get("mlp")
    if mlp is not None and mlp["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    a = LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                            kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot=rotary_from_json(m["rot"]),
                            q_rank=int(m["q_rank"]) if q_latent else 0, window=int((m.get("mask") or {}).get("size", 0)),
                            sink=sink)
    return LayerSpec(a, DenseMlpSpec(int(mlp["ff"]), "relu2") if mlp is not None else None, parallel=True, token_shift=True)


def config_from_json(c: Mapping[str, Any]) -> ModelConfig:
    return milutar_config(int(c["width"]), int(c["vocab"]), tuple(_layer(i, l) for i, l in enumerate(c["layers"])),
                          loop_from_json(c), rms_eps=float(c["norm"]["eps"]), residual_mult=float(c["residual_mult"]))


def config_to_json(cfg: ModelConfig) -> Dict[str, Any]:
    layers: List[Dict[str, Any]] = []
    for l in cfg.layer_specs:
        a = l.mixer
        m: Dict[str, Any] = {"heads": a.heads, "dim": a.dim, "rot_dim": a.rot_dim, "vdim": a.vdim, "kv_rank": a.kv_rank,
                             "scale": a.scale, "rot": rotary_to_json(a.rot)}
        if a.q_rank:
            m["q_rank"] = a.q_rank
        if a.window:
            m["mask"] = {"size": a.window}
        layers.append({"type": next(n for n, f in MIXERS.items() if f == (a.q_rank > 0, a.sink)), "mixer": m,
                       "mlp": {"kind": "dense", "ff": l.mlp.ff} if l.mlp is not None else None})
    return {"architecture": "Milutar", "vocab": cfg.vocab, "width": cfg.hidden, "norm": {"eps": cfg.rms_eps},
            "residual_mult": cfg.residual_mult, "layers": layers, "loop": loop_to_json(cfg.loop)}


# ----------------------------------------------------------------------------- tensors
def tensor_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Every tensor of a checkpoint and its shape, in file order."""
    H = cfg.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, H)}
    if cfg.loop is not None:
        out["loop.step"] = (cfg.loop.times, H)
    for i, l in enumerate(cfg.layer_specs):
        a, p = l.mixer, f"l{i}."
        m = p + "mix."
        out[p + "norm1"] = ()
        q_rows = a.heads * (a.dim + a.rot_dim)
        if a.q_rank:
            out[m + "dq"], out[m + "dq.norm"], out[m + "uq"] = (a.q_rank, H), (a.q_rank,), (q_rows, a.q_rank)
        else:
            out[m + "q"] = (q_rows, H)
        out[m + "dkv"], out[m + "dkv.norm"] = (a.kv_rank + a.rot_dim, H), (a.kv_rank,)
        out[m + "uk"], out[m + "uv"] = (a.heads * a.dim, a.kv_rank), (a.heads * a.vdim, a.kv_rank)
        if a.sink:
            out[m + "sink"] = (a.heads,)
        out[m + "o"] = (H, a.heads * a.vdim)
        if l.mlp is not None:
            out[p + "mlp.up"], out[p + "mlp.down"] = (l.mlp.ff, H), (H, l.mlp.ff)
        out[p + "ls1"] = (H,)
        if l.mlp is not None:
            out[p + "ls2"] = (H,)
        out[p + "shift"] = (H,)
    out["final.norm"] = ()
    out["head"] = (cfg.vocab, H)
    return out


def build_random_milutar(cfg: ModelConfig, seed: int = 0, device="cpu", std: float = 0.02) -> ModelWeights:
    def adjust(name: str, t: torch.Tensor) -> torch.Tensor:
        if name.endswith(("norm1", "norm")):
            return 1.0 + t
        if name.endswith((".ls1", ".ls2")):
            return 0.5 + t
        return t + 0.3 if name.endswith(".shift") else t
    return build_random_folder(cfg, seed, device, std, adjust)
