"""Sisisun executor: listed attention layers without rotation, dense / expert feed-forwards, looped layer ranges.

The base (``listed.py``) holds the planes per layer run, the routes and the walk over runs; here are the weight packing and
the sublayers:
  * q | k | v and gate | up are stacked at load, experts are stacked per layer, norm weights are stored as 1 + w, head widths
    the attention kernels do not have are zero-padded;
  * up to 16 rows (decode steps, short portions) run on the streaming bf16 GEMV with the norm and the activation fused
    into it, more rows on the tcgen05 GEMM (split over K up to 128 rows); experts go through the selected-expert kernels
    or the grouped GEMM by the same rule;
  * ``dtype="float32"`` runs the same walk on fp32 CUDA-core kernels with fp32 activations and fp32 KV pages.
In both modes residual, norms, scores, softmax, router and positions are fp32.  Oracle: ``ref/sisisun.py``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from ..ops import kernels as K
from ..ops.kernels import DeviceWeight
from .config import DenseMlpSpec, MoeMlpSpec
from .executor import PAGE, BatchDesc
from .listed import ExpertWeights, ListedExecutor, pad2, up8


@dataclass
class _Layer:
    norm1: torch.Tensor                          # fp32 [Hp], 1 + w
    norm2: Optional[torch.Tensor]
    qkv: DeviceWeight                            # [q | k | v rows, Hp]
    q_norm: torch.Tensor                         # fp32 [dim]
    k_norm: torch.Tensor
    o: DeviceWeight                              # [Hp, heads * D]
    gate_up: Optional[DeviceWeight] = None       # dense: [gate | up rows, Hp]
    down: Optional[DeviceWeight] = None          # dense: [Hp, F]
    experts: Optional[ExpertWeights] = None


class SisisunExecutor(ListedExecutor):
    readds_embedding = True

    # ------------------------------------------------------------------ weights
    def _norm_weight(self, name: str) -> torch.Tensor:
        v = torch.zeros(self.hp, dtype=torch.float32, device=self.device)
        v[:self.cfg.hidden] = 1.0 + self._mat(name).float()
        self.f32[name] = v
        return v

    def _load_layers(self) -> None:
        cfg, dev, hp, mat, put, norm = self.cfg, self.device, self.hp, self._mat, self._put, self._norm_weight
        self.layers: List[_Layer] = []
        for i, spec in enumerate(cfg.layer_specs):
            a, m, p = spec.mixer, spec.mlp, f"l{i}."
            qkv = torch.cat([mat(p + "mix.q"), mat(p + "mix.k"), mat(p + "mix.v")], 0)
            for s in ("q.norm", "k.norm"):
                self.f32[p + "mix." + s] = mat(p + "mix." + s).float().contiguous()
            L = _Layer(norm(p + "norm1"), norm(p + "norm2") if m is not None else None,
                       put(p + "qkv", pad2(qkv, up8(qkv.shape[0]), hp)), self.f32[p + "mix.q.norm"],
                       self.f32[p + "mix.k.norm"], put(p + "o", self._out_mat(p + "mix.o", a.heads, a.vdim, a.width)))
            if isinstance(m, DenseMlpSpec):
                L.gate_up = put(p + "gate_up", self._gate_up(p + "mlp.", m.ff))
                L.down = put(p + "down", pad2(mat(p + "mlp.down"), hp, up8(m.ff)))
            elif isinstance(m, MoeMlpSpec):
                L.experts = self._load_experts(p, m)
            self.layers.append(L)
        i = torch.arange((cfg.hidden + 1) // 2, dtype=torch.float64)
        self.pos_freq = torch.pow(torch.tensor(10000.0, dtype=torch.float64), -2.0 * i / cfg.hidden).to(dev)

    # ------------------------------------------------------------------ layers
    def _attention(self, run: int, i: int, h: torch.Tensor, b: BatchDesc, route: str) -> None:
        cfg, sc, L = self.cfg, self.scratch, self.layers[i]
        a, T = cfg.layer_specs[i].mixer, b.T
        with self._stage("attn_qkv_gemm"):
            qkv = self._in_proj(h, L.norm1, L.qkv, "qkv", route)
        nq, nk = a.heads * a.dim, a.kv_heads * a.dim
        q_out = sc.get("q_out", (T, a.heads, a.width), self.act_dtype)
        K.qkv_post(qkv[:, :nq], qkv[:, nq:nq + nk], qkv[:, nq + nk:], L.q_norm, L.k_norm, q_out, None, self.kv[run],
                   self.block_table, b.slot, b.pos, a.heads, a.kv_heads, a.width, PAGE, False, 0, 1.0, cfg.rms_eps,
                   d_in=a.dim, dv_in=a.vdim)
        out = sc.get("attn_out", (T, a.heads * a.width), self.act_dtype)
        with self._stage("attn_core"):
            self._attend_run(run, a, q_out, b, out)
        with self._stage("out_gemm"):
            self._add_products(h, [(out, L.o, None)], route)

    # ------------------------------------------------------------------ whole model
    def _embed(self, b: BatchDesc, h: torch.Tensor, copy: Optional[torch.Tensor]) -> None:
        K.embed_sinusoid(self.embed_w, b.tokens, b.pos, self.pos_freq, h, copy)

    def _layer_run(self, run: int, i: int, h: torch.Tensor, b: BatchDesc, route: str, journal: Optional[dict]) -> None:
        self._attention(run, i, h, b, route)
        m = self.cfg.layer_specs[i].mlp
        if isinstance(m, DenseMlpSpec):
            L = self.layers[i]
            self._dense(L.norm2, L.gate_up, L.down, m, h, route)
        elif isinstance(m, MoeMlpSpec):
            L = self.layers[i]
            self._experts(L.experts, L.norm2, m, h, route)
