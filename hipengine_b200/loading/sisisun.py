"""Sisisun checkpoints: config.json <-> ``ModelConfig``, tensor names and shapes, random-init weights.

Tensor names: ``embed``, ``head``, ``final.norm``, ``loop.step`` [times, width]; per layer ``l<i>.norm1``, ``.mix.q/k/v/o``
with ``.mix.q.norm`` / ``.mix.k.norm``, ``.norm2`` and either ``.mlp.gate/up/down`` (dense) or ``.mlp.router``,
``.mlp.e<j>.gate/up/down`` and ``.mlp.shared.gate/up/down/sg`` (experts).  Linear weights are [out, in].
"""
from __future__ import annotations

from typing import Any, Dict, List, Mapping, Optional, Tuple

from ..models.config import AttentionSpec, DenseMlpSpec, LayerSpec, ModelConfig, MoeMlpSpec, sisisun_config
from .folder_family import build_random_folder, loop_from_json, loop_to_json
from .weights import ModelWeights


# ----------------------------------------------------------------------------- configuration
def _mlp_from_json(i: int, m: Optional[Mapping[str, Any]]):
    if m is None:
        return None
    kind = m["kind"]
    if kind == "dense":
        return DenseMlpSpec(int(m["ff"]), "clamped_glu", float(m["limit"]))
    if kind == "moe":
        r, shared = m["router"], m.get("shared")
        groups = r.get("groups") or {"count": 1, "keep": 1}
        return MoeMlpSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(m["expert"]["ff"]),
                          groups=int(groups["count"]), groups_kept=int(groups["keep"]),
                          scale=float(r.get("scale", 1.0)), shared_ff=int(shared["ff"]) if shared else 0)
    raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")


def config_from_json(c: Mapping[str, Any]) -> ModelConfig:
    layers: List[LayerSpec] = []
    for i, l in enumerate(c["layers"]):
        if l["type"] != "attention":
            raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
        m = l["mixer"]
        layers.append(LayerSpec(
            AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                          float(m.get("softcap") or 0.0)),
            _mlp_from_json(i, l.get("mlp"))))
    return sisisun_config(int(c["width"]), int(c["vocab"]), tuple(layers), loop_from_json(c), rms_eps=float(c["norm"]["eps"]))


def config_to_json(cfg: ModelConfig) -> Dict[str, Any]:
    layers = []
    for l in cfg.layer_specs:
        a, m = l.mixer, l.mlp
        mlp: Optional[Dict[str, Any]] = None
        if isinstance(m, DenseMlpSpec):
            mlp = {"kind": "dense", "ff": m.ff, "limit": m.limit}
        elif isinstance(m, MoeMlpSpec):
            mlp = {"kind": "moe", "expert": {"ff": m.ff}, "shared": {"ff": m.shared_ff} if m.shared_ff else None,
                   "router": {"experts": m.experts, "top": m.top, "scale": m.scale,
                              "groups": {"count": m.groups, "keep": m.groups_kept}}}
        layers.append({"type": "attention", "mlp": mlp,
                       "mixer": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim,
                                 "scale": a.scale, "softcap": a.softcap}})
    return {"architecture": "Sisisun", "vocab": cfg.vocab, "width": cfg.hidden, "norm": {"eps": cfg.rms_eps},
            "layers": layers, "loop": loop_to_json(cfg.loop)}


# ----------------------------------------------------------------------------- tensors
def tensor_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Every tensor of a checkpoint and its shape, in file order."""
    H = cfg.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, H)}
    if cfg.loop is not None:
        out["loop.step"] = (cfg.loop.times, H)

    def glu(p: str, ff: int) -> None:
        out[p + "gate"], out[p + "up"], out[p + "down"] = (ff, H), (ff, H), (H, ff)

    for i, l in enumerate(cfg.layer_specs):
        a, m, p = l.mixer, l.mlp, f"l{i}."
        out[p + "norm1"] = (H,)
        if m is not None:
            out[p + "norm2"] = (H,)
        out[p + "mix.q"] = (a.heads * a.dim, H)
        out[p + "mix.k"] = (a.kv_heads * a.dim, H)
        out[p + "mix.v"] = (a.kv_heads * a.vdim, H)
        out[p + "mix.q.norm"] = out[p + "mix.k.norm"] = (a.dim,)
        out[p + "mix.o"] = (H, a.heads * a.vdim)
        if isinstance(m, DenseMlpSpec):
            glu(p + "mlp.", m.ff)
        elif isinstance(m, MoeMlpSpec):
            for e in range(m.experts):
                glu(p + f"mlp.e{e}.", m.ff)
            out[p + "mlp.router"] = (m.experts, H)
            if m.shared_ff:
                glu(p + "mlp.shared.", m.shared_ff)
                out[p + "mlp.shared.sg"] = (1, H)
    out["final.norm"] = (H,)
    out["head"] = (cfg.vocab, H)
    return out


def build_random_sisisun(cfg: ModelConfig, seed: int = 0, device="cpu", std: float = 0.02) -> ModelWeights:
    return build_random_folder(cfg, seed, device, std, lambda n, t: 1.0 + t if n.endswith(("q.norm", "k.norm")) else t)
