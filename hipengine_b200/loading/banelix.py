"""Banelix checkpoints: config.json <-> ``ModelConfig``, tensor names and shapes, random-init weights.

Tensor names: ``embed``, ``head``, ``final.norm``; per layer ``l<i>.norm1`` and, with a feed-forward, ``.norm2`` and
``.mlp.gate/up/down``.  Attention layers have ``.mix.q``, ``.mix.k``, ``.mix.v`` with biases ``.b``, ``.mix.q.norm``,
``.mix.k.norm`` (no key and value tensors where they come from another layer) and ``.mix.o``.  Layers of two mixers have
``.mix.left.q/k/g/o`` (biases on q and k) and ``.mix.right.y/x`` with biases, ``.conv`` [channels, taps] with bias, ``.ra`` /
``.ri`` [blocks, n, n] with biases, ``.lam`` and ``.o``.  Linear weights are [out, in].
"""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Tuple

import torch

from ..models.config import (QK_NORM_ROWS, QK_NORM_UNIT, AttentionSpec, DenseMlpSpec, LayerSpec, ModelConfig, RecurrentSpec,
                             SideBySideSpec, banelix_config)
from .folder_family import build_random_folder, rotary_from_json, rotary_to_json
from .weights import ModelWeights

SINK_SCORE = 0.0           # of the unit in the softmax denominator of an attention layer


# ----------------------------------------------------------------------------- configuration
def _heads(m: Mapping[str, Any], **kw) -> AttentionSpec:
    return AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                         rot=rotary_from_json(m["rot"], halves=True), window=int((m.get("mask") or {}).get("size", 0)),
                         bias=True, **kw)


def _layer(i: int, l: Mapping[str, Any]) -> LayerSpec:
    m, mlp = l["mixer"], l.get("mlp")
    if mlp is not None and mlp["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    if l["type"] == "attention":
        src = m.get("kv_from")
        mixer: Any = _heads(m, sink_score=SINK_SCORE, qk_norm=QK_NORM_ROWS, kv_from=None if src is None else int(src))
    elif l["type"] == "parallel":
        r = m["right"]
        mixer = SideBySideSpec(_heads(m["left"], qk_norm=QK_NORM_UNIT, keys_as_values=True, head_gate=True),
                               RecurrentSpec(int(r["width"]), int(r["blocks"]), int(r["conv"])),
                               float(m["left_scale"]), float(m["right_scale"]))
    else:
        raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
    return LayerSpec(mixer, DenseMlpSpec(int(mlp["ff"])) if mlp is not None else None)


def config_from_json(c: Mapping[str, Any]) -> ModelConfig:
    return banelix_config(int(c["width"]), int(c["vocab"]), tuple(_layer(i, l) for i, l in enumerate(c["layers"])),
                          rms_eps=float(c["norm"]["eps"]), residual_mult=float(c["residual_mult"]),
                          embed_scale=float(c["embedding"]["scale"]))


def _heads_json(a: AttentionSpec) -> Dict[str, Any]:
    m: Dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                         "rot": rotary_to_json(a.rot)}
    if a.window:
        m["mask"] = {"size": a.window}
    if a.kv_from is not None:
        m["kv_from"] = a.kv_from
    return m


def config_to_json(cfg: ModelConfig) -> Dict[str, Any]:
    layers: List[Dict[str, Any]] = []
    for l in cfg.layer_specs:
        m = l.mixer
        if isinstance(m, SideBySideSpec):
            r = m.right
            body = {"left": _heads_json(m.left), "right": {"width": r.width, "blocks": r.blocks, "conv": r.taps},
                    "left_scale": m.left_scale, "right_scale": m.right_scale}
        else:
            body = _heads_json(m)
        layers.append({"type": "parallel" if isinstance(m, SideBySideSpec) else "attention", "mixer": body,
                       "mlp": {"kind": "dense", "ff": l.mlp.ff} if l.mlp is not None else None})
    return {"architecture": "Banelix", "vocab": cfg.vocab, "width": cfg.hidden, "embedding": {"scale": cfg.embed_scale},
            "norm": {"eps": cfg.rms_eps}, "residual_mult": cfg.residual_mult, "layers": layers}


# ----------------------------------------------------------------------------- tensors
def tensor_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Every tensor of a checkpoint and its shape, in file order."""
    H = cfg.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, H)}

    def biased(name: str, rows: int) -> None:
        out[name], out[name + ".b"] = (rows, H), (rows,)

    for i, l in enumerate(cfg.layer_specs):
        a, p = l.attention, f"l{i}."
        both = isinstance(l.mixer, SideBySideSpec)
        m = p + ("mix.left." if both else "mix.")
        out[p + "norm1"] = (H,)
        if l.mlp is not None:
            out[p + "norm2"] = (H,)
        biased(m + "q", a.heads * a.dim)
        if a.kv_from is None:
            biased(m + "k", a.kv_heads * a.dim)
            if not a.keys_as_values:
                biased(m + "v", a.kv_heads * a.vdim)
        if a.qk_norm == QK_NORM_ROWS:
            out[m + "q.norm"] = (a.heads * a.dim,)
            if a.kv_from is None:
                out[m + "k.norm"] = (a.kv_heads * a.dim,)
        if a.head_gate:
            out[m + "g"] = (a.heads, H)
        out[m + "o"] = (H, a.heads * a.vdim)
        if both:
            r, m = l.mixer.right, p + "mix.right."
            n = r.width // r.blocks
            biased(m + "y", r.width)
            biased(m + "x", r.width)
            out[m + "conv"], out[m + "conv.b"] = (r.width, r.taps), (r.width,)
            for g in ("ra", "ri"):
                out[m + g], out[m + g + ".b"] = (r.blocks, n, n), (r.blocks, n)
            out[m + "lam"] = (r.width,)
            out[m + "o"] = (H, r.width)
        if l.mlp is not None:
            for n in ("gate", "up"):
                out[p + "mlp." + n] = (l.mlp.ff, H)
            out[p + "mlp.down"] = (H, l.mlp.ff)
    out["final.norm"] = (H,)
    out["head"] = (cfg.vocab, H)
    return out


def build_random_banelix(cfg: ModelConfig, seed: int = 0, device="cpu", std: float = 0.02) -> ModelWeights:
    def adjust(name: str, t: torch.Tensor) -> torch.Tensor:
        if name.endswith(("norm1", "norm2", "norm")):
            return 1.0 + t
        if name.endswith(".conv"):
            return t / std / t.shape[-1]
        # a between 0.9 and 0.999 over the channels at r = 1: memories of ten to a thousand tokens
        return torch.log(torch.expm1(-torch.log(0.9 + 0.099 * torch.sigmoid(t / std)) / 8)) if name.endswith(".lam") else t
    return build_random_folder(cfg, seed, device, std, adjust)
