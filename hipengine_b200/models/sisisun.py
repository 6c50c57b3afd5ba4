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
from typing import List, Optional, Tuple

import torch

from ..ops import kernels as K
from ..ops.kernels import DeviceWeight
from .config import DenseMlpSpec, MoeMlpSpec
from .executor import PAGE, BatchDesc
from .listed import EXACT, FEW, MANY, ListedExecutor, pad2, up8


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
    router: Optional[DeviceWeight] = None        # [experts (+ shared gate), Hp], rows padded to eight
    e_gate_up: Optional[DeviceWeight] = None     # [experts * (gate | up), Hp]
    e_down: Optional[DeviceWeight] = None        # [experts * Hp, F]
    s_gate_up: Optional[DeviceWeight] = None
    s_down: Optional[DeviceWeight] = None


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
        gate_up = self._gate_up

        def glu(name: str, p: str, ff: int) -> Tuple[DeviceWeight, DeviceWeight]:
            return put(name + "gate_up", gate_up(p, ff)), put(name + "down", pad2(mat(p + "down"), hp, up8(ff)))

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
                L.gate_up, L.down = glu(p, p + "mlp.", m.ff)
            elif isinstance(m, MoeMlpSpec):
                fp = up8(m.ff)
                gu = torch.empty(m.experts * 2 * fp, hp, dtype=torch.bfloat16, device=dev)
                dn = torch.empty(m.experts * hp, fp, dtype=torch.bfloat16, device=dev)
                for e in range(m.experts):
                    gu[e * 2 * fp:(e + 1) * 2 * fp] = gate_up(p + f"mlp.e{e}.", m.ff)
                    dn[e * hp:(e + 1) * hp] = pad2(mat(p + f"mlp.e{e}.down"), hp, fp)
                L.e_gate_up, L.e_down = put(p + "experts.gate_up", gu), put(p + "experts.down", dn)
                rows = [mat(p + "mlp.router")]
                if m.shared_ff:
                    L.s_gate_up, L.s_down = glu(p + "shared.", p + "mlp.shared.", m.shared_ff)
                    rows.append(mat(p + "mlp.shared.sg"))
                r = torch.cat(rows, 0)
                L.router = put(p + "router", pad2(r, up8(r.shape[0]), hp))
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

    def _experts(self, L: _Layer, m: MoeMlpSpec, h: torch.Tensor, route: str) -> None:
        from ..ops import gemm as GM
        sc, cfg, T, E, k = self.scratch, self.cfg, h.shape[0], m.experts, m.top
        F = L.e_down.n_cols
        xn = None
        if route != FEW:
            with self._stage("norm"):
                xn = self._norm_rows(h, L.norm2)
        if route == MANY:
            logits = GM.gemm_bf16(xn, L.router.data, sc.get("moe_logits_f32", (T, L.router.n_rows), torch.float32))
        else:
            logits = self._in_proj(h, L.norm2, L.router, "moe_logits", route, xn=xn)
        ids = sc.get("moe_ids", (T, k), torch.int32)
        wts = sc.get("moe_wts", (T, k), torch.float32)
        K.moe_route_grouped(logits, k, ids, wts, E, m.groups, m.groups_kept, m.scale)
        sg = logits[:, E:E + 1] if m.shared_ff else None
        s_gu = L.s_gate_up.data if m.shared_ff else None
        s_dn = L.s_down.data if m.shared_ff else None
        if route != MANY:
            rows = sc.get("moe_act", (T * k, F), self.act_dtype)
            rows_s = sc.get("moe_act_sh", (T, L.s_down.n_cols), self.act_dtype) if m.shared_ff else None
            if route == EXACT:
                K.moe_exact(xn, ids, wts, L.e_gate_up.data, L.e_down.data, E, rows, h, sg, s_gu, s_dn, rows_s)
                return
            K.moe_gateup_float(h, L.norm2, cfg.rms_eps, cfg.hidden, ids, wts, L.e_gate_up.data, E, rows, sg, s_gu, rows_s)
            K.moe_down_float(rows, ids, L.e_down.data, E, h, rows_s, s_dn)
            return
        P = T * k
        bound = K.moe_sorted_rows_bound(P, E)
        pos = sc.get("moe_pos", (P,), torch.int32)
        tiles = sc.get("moe_tiles", (bound // 128,), torch.int32)
        K.moe_group(ids, E, pos, tiles, sc.get("moe_meta", (4,), torch.int32))
        xs = sc.get("moe_xs", (bound, self.hp), torch.bfloat16)
        K.moe_gather(xn, pos, k, xs)
        gu = sc.get("moe_gu", (bound, 2 * F), torch.bfloat16)
        GM.gemm_bf16_grouped(xs, L.e_gate_up.data, gu, E, tiles)
        act = sc.get("moe_act_g", (bound, F), torch.bfloat16)
        K.act_mul(gu, act, "silu")
        ys = sc.get("moe_ys", (bound, self.hp), torch.bfloat16)
        GM.gemm_bf16_grouped(act, L.e_down.data, ys, E, tiles)
        ysh = None
        if m.shared_ff:
            gus = self._proj(xn, L.s_gate_up, "moe_gus", "g")
            acts = sc.get("moe_acts", (T, L.s_down.n_cols), torch.bfloat16)
            K.act_mul(gus, acts, "silu")
            ysh = self._gemm(acts, L.s_down, sc.get("y_bf", (T, self.hp), torch.bfloat16), tag="d")
        K.moe_combine(h, ys, pos, wts, k, ysh, sg)

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
            self._experts(self.layers[i], m, h, route)
