"""Mepatar checkpoints: config.json <-> ``ModelConfig``, tensor names and shapes, random-init weights.

Tensor names: ``embed``, ``head``, ``final.norm``; per layer ``l<i>.norm1``, ``.canon1`` [width, taps], ``.mix.*`` and, with a
feed-forward, ``.norm2`` and ``.mlp.*``.  Mixers: attention has ``.q``, ``.k``, ``.v``, ``.o`` with biases ``.b``, ``.q.norm`` and
``.k.norm`` [dim], ``.temp`` [heads]; retention ``.q``, ``.k``, ``.v``, ``.g``, ``.o``; the delta rule these five (the first
three with ``.conv`` [channels, taps]), the row maps ``.b`` and ``.a``, ``.A_log``, ``.dt_bias`` [heads] and ``.norm`` [vdim].
Feed-forwards: ``.gate``, ``.up``, ``.down``, or ``.router`` and those three per expert ``.e<j>``.  Linear weights are [out, in].
"""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Optional, Tuple, Union

import torch

from ..models.config import (DenseMlpSpec, LayerSpec, LinearAttentionSpec, ModelConfig, MoeMlpSpec, mepatar_attention,
                             mepatar_config, mepatar_experts, mepatar_layer)
from .folder_family import build_random_folder, rotary_from_json, rotary_to_json
from .weights import ModelWeights


# ----------------------------------------------------------------------------- configuration
def _mixer(kind: str, m: Mapping[str, Any]):
    heads, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    if kind == "attention":
        mask = m["mask"]
        if int(mask["size"]) < 1:
            raise ValueError(f"window of {mask['size']}")
        return mepatar_attention(heads, int(m["kv_heads"]), dim, vdim, float(m["scale"]), int(mask["size"]), int(mask["keep_first"]),
                                 rotary_from_json(m["rot"]))
    if kind == "retention":
        return LinearAttentionSpec(heads, heads, dim, vdim, tuple(float(x) for x in m["decay"]), rotary_from_json(m["rot"], halves=True))
    if kind == "delta":
        return LinearAttentionSpec(heads, int(m["kv_heads"]), dim, vdim, taps=int(m["conv"]))
    raise ValueError(f"unknown mixer {kind!r}")


def _mlp(m: Optional[Mapping[str, Any]]) -> Optional[Union[DenseMlpSpec, MoeMlpSpec]]:
    if m is None:
        return None
    if m["kind"] == "dense":
        return DenseMlpSpec(int(m["ff"]), "gelu_tanh")
    if m["kind"] == "moe":
        return mepatar_experts(int(m["router"]["experts"]), int(m["router"]["top"]), int(m["expert"]["ff"]), float(m["expert"]["limit"]))
    raise ValueError(f"unknown feed-forward kind {m['kind']!r}")


def config_from_json(c: Mapping[str, Any]) -> ModelConfig:
    layers: List[LayerSpec] = []
    for i, l in enumerate(c["layers"]):
        try:
            layers.append(mepatar_layer(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp")), int(c["canon"]["taps"])))
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    return mepatar_config(int(c["width"]), int(c["vocab"]), tuple(layers), rms_eps=float(c["norm"]["eps"]),
                          norm_groups=int(c["norm"]["groups"]), embed_scale=float(c["embedding"]["scale"]))


def config_to_json(cfg: ModelConfig) -> Dict[str, Any]:
    layers: List[Dict[str, Any]] = []
    for l in cfg.layer_specs:
        a, m = l.mixer, l.mlp
        body: Dict[str, Any] = {"heads": a.heads, "dim": a.dim, "vdim": a.vdim}
        if not isinstance(a, LinearAttentionSpec):
            kind = "attention"
            body.update(kv_heads=a.kv_heads, scale=a.scale, mask={"size": a.window, "keep_first": a.keep_first})
        elif a.delta:
            kind = "delta"
            body.update(kv_heads=a.kv_heads, conv=a.taps)
        else:
            kind = "retention"
            body["decay"] = list(a.decay)
        if a.rot is not None:
            body["rot"] = rotary_to_json(a.rot)
        mlp: Optional[Dict[str, Any]] = None
        if isinstance(m, MoeMlpSpec):
            mlp = {"kind": "moe", "router": {"experts": m.experts, "top": m.top}, "expert": {"ff": m.ff, "limit": m.limit}}
        elif m is not None:
            mlp = {"kind": "dense", "ff": m.ff}
        layers.append({"type": kind, "mixer": body, "mlp": mlp})
    return {"architecture": "Mepatar", "vocab": cfg.vocab, "width": cfg.hidden, "embedding": {"scale": cfg.embed_scale},
            "norm": {"eps": cfg.rms_eps, "groups": cfg.norm_groups}, "canon": {"taps": cfg.layer_specs[0].input_taps},
            "layers": layers}


# ----------------------------------------------------------------------------- tensors
def _mixer_shapes(a, H: int) -> Dict[str, Tuple[int, ...]]:
    out: Dict[str, Tuple[int, ...]] = {}
    rows = {"q": a.heads * a.dim, "k": a.kv_heads * a.dim, "v": a.kv_heads * a.vdim}
    if isinstance(a, LinearAttentionSpec):
        rows.update(q=a.kv_heads * a.dim, v=a.heads * a.vdim)
        for n, r in rows.items():
            out[n] = (r, H)
            if a.delta:
                out[n + ".conv"] = (r, a.taps)
        if a.delta:
            out.update({"b": (a.heads, H), "A_log": (a.heads,), "norm": (a.vdim,), "a": (a.heads, H), "dt_bias": (a.heads,)})
        out["g"], out["o"] = (a.heads * a.vdim, H), (H, a.heads * a.vdim)
        return out
    for n, r in rows.items():
        out[n], out[n + ".b"] = (r, H), (r,)
    out.update({"q.norm": (a.dim,), "k.norm": (a.dim,), "temp": (a.heads,), "o": (H, a.heads * a.vdim), "o.b": (H,)})
    return out


def tensor_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Every tensor of a checkpoint and its shape, in file order."""
    H = cfg.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, H)}
    for i, l in enumerate(cfg.layer_specs):
        p, m = f"l{i}.", l.mlp
        out[p + "norm1"] = (H,)
        if m is not None:
            out[p + "norm2"] = (H,)
        out.update({p + "mix." + n: s for n, s in _mixer_shapes(l.mixer, H).items()})
        if m is not None:
            moe = isinstance(m, MoeMlpSpec)
            for e in [f"e{j}." for j in range(m.experts)] if moe else [""]:
                for n in ("gate", "up"):
                    out[p + "mlp." + e + n] = (m.ff, H)
                out[p + "mlp." + e + "down"] = (H, m.ff)
            if moe:
                out[p + "mlp.router"] = (m.experts, H)
        out[p + "canon1"] = (H, l.input_taps)
    out["final.norm"] = (H,)
    out["head"] = (cfg.vocab, H)
    return out


def build_random_mepatar(cfg: ModelConfig, seed: int = 0, device="cpu", std: float = 0.02) -> ModelWeights:
    def adjust(name: str, t: torch.Tensor) -> torch.Tensor:
        if name.endswith(("norm1", "norm2", "norm", "temp")):
            return 1.0 + t
        if name.endswith((".conv", "canon1")):
            return t / std / t.shape[-1]
        # decays between 0.9 and 0.999 or so at a = 0: memories of ten to a thousand tokens
        return t / std if name.endswith("A_log") else t / std - 4.0 if name.endswith("dt_bias") else t
    return build_random_folder(cfg, seed, device, std, adjust)
