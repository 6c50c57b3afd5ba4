"""Mepatar executor: mixer and feed-forward side by side under grouped norms, a convolution ahead of the mixer; the mixers are
attention over a window and the sequence's first tokens, retention, and the gated delta rule.

The base (``listed.py``) holds the planes and states per layer run, the routes, attention, feed-forwards and experts; here are
the weight packing and the layer.  A layer run:
  norm, convolution  one kernel gives both sublayers their rows (one norm pass, two gains) and advances the past rows;
  input              ONE product gives all rows of the mixer; for few rows the router's rows ride in the same launch;
  attention          head rows (bias, norm, rotation, page write) in one launch, then the split-K or flash kernel;
  linear attention   single tokens: one launch from rows to the gated output; prompt portions: chunks on tensor cores;
  output             mixer and dense feed-forward add into the residual together (one launch for few rows), experts on their own.
Both sublayers have read the residual by the time the first output is added to it.
``dtype="float32"`` runs the same walk on fp32 CUDA-core kernels with fp32 pages.  In both modes residual, norms, the input
convolution, angles, scores, softmax, router scores, decays, step sizes, unit norms and recurrent states are fp32.  Oracle:
``ref/mepatar.py``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from ..ops import kernels as K
from ..ops import linear as LN
from ..ops import mixers as MX
from ..ops.kernels import DeviceWeight
from .config import QK_NORM_HEAD, AttentionSpec, DenseMlpSpec, LinearAttentionSpec, MoeMlpSpec
from .executor import PAGE, BatchDesc
from .listed import FEW, ExpertWeights, ListedExecutor, pad2, up8


@dataclass
class _Layer:
    norm1: torch.Tensor                           # fp32 [hp]
    conv: torch.Tensor                            # fp32 [taps, hp], oldest first
    in_w: DeviceWeight                            # rows of every input projection, [n, hp]
    cols: Dict[str, Tuple[int, int]]              # q, k, v, g, b, a -> column range of the input rows
    o: DeviceWeight                               # [hp, heads * padded value width]
    o_bias: Optional[torch.Tensor] = None         # fp32 [hp]
    bias: Optional[torch.Tensor] = None           # attention: fp32 over the input rows
    gain: Optional[Dict[str, torch.Tensor]] = None      # attention: q [heads, dim] (times the factor of the scores), k [dim]
    freq: Optional[torch.Tensor] = None
    lin: Optional[LN.LinearParams] = None
    norm2: Optional[torch.Tensor] = None
    gate_up: Optional[DeviceWeight] = None
    down: Optional[DeviceWeight] = None
    experts: Optional[ExpertWeights] = None


class MepatarExecutor(ListedExecutor):
    # ------------------------------------------------------------------ weights
    def _norm_weight(self, name: str) -> torch.Tensor:
        return self._vec(name, self.hp)

    def _load_layers(self) -> None:
        cfg, hp, put, norm = self.cfg, self.hp, self._put, self._norm_weight
        self.layers: List[_Layer] = []
        for i, spec in enumerate(cfg.layer_specs):
            p, a, m = f"l{i}.", spec.mixer, spec.mlp
            linear = isinstance(a, LinearAttentionSpec)
            names = ["q", "k", "v"] + (["g"] if linear else []) + (["b", "a"] if linear and a.delta else [])
            mats = [self._mat(p + "mix." + n) for n in names]
            cols, at = {}, 0
            w = torch.zeros(sum(up8(t.shape[0]) for t in mats), hp, dtype=torch.bfloat16, device=self.device)
            for n, t in zip(names, mats):
                w[at:at + t.shape[0], :cfg.hidden] = t
                cols[n] = (at, at + up8(t.shape[0]))
                at = cols[n][1]
            conv = pad2(self._mat(p + "canon1").float().t().contiguous(), spec.input_taps, hp).contiguous()
            L = _Layer(norm(p + "norm1"), conv, put(p + "in", w), cols,
                       put(p + "o", self._out_mat(p + "mix.o", a.heads, a.vdim, a.vcols if linear else a.width)))
            if a.rot is not None:
                L.freq = torch.tensor(a.rot.table()[0], dtype=torch.float64, device=self.device)
            if linear:
                L.lin = self._load_linear(p + "mix.", a, L)
            else:
                self._load_attention(p + "mix.", a, L)
            if m is not None:
                L.norm2 = norm(p + "norm2")
            if isinstance(m, MoeMlpSpec):
                L.experts = self._load_experts(p, m)
            elif m is not None:
                L.gate_up = put(p + "gate_up", self._gate_up(p + "mlp.", m.ff))
                L.down = put(p + "down", pad2(self._mat(p + "mlp.down"), hp, up8(m.ff)))
            self.layers.append(L)

    def _load_attention(self, m: str, a: AttentionSpec, L: _Layer) -> None:
        L.bias = torch.zeros(L.in_w.n_rows, dtype=torch.float32, device=self.device)
        for n, (c0, _) in L.cols.items():
            b = self._mat(m + n + ".b").float()
            L.bias[c0:c0 + b.numel()] = b
        q, k, temp = (self._mat(m + n).float() for n in ("q.norm", "k.norm", "temp"))
        L.gain = {"q": (temp[:, None] * q[None]).contiguous(), "k": k.contiguous()}
        L.o_bias = self._vec(m + "o.b", self.hp)

    def _load_linear(self, m: str, a: LinearAttentionSpec, L: _Layer) -> LN.LinearParams:
        dev, c = self.device, L.cols
        p = LN.LinearParams(a, c["k"][0], c["v"][0], c["g"][0], L.freq)
        if not a.delta:
            p.g1 = (torch.tensor(a.decay, dtype=torch.float64) - 1.0).float().to(dev)
            p.powers = LN.decay_powers(a.decay).to(dev)
            return p
        p.conv = torch.zeros(a.taps, a.conv_cols, dtype=torch.float32, device=dev)
        for n in ("q", "k", "v"):
            w = self._mat(m + n + ".conv").float()
            p.conv[:, c[n][0]:c[n][0] + w.shape[0]] = w.t()
        p.rate, p.dt, p.gain = (self._mat(m + n).float().contiguous() for n in ("A_log", "dt_bias", "norm"))
        p.rate = torch.exp(p.rate)
        return p

    # ------------------------------------------------------------------ mixers
    def _input(self, L: _Layer, xs: torch.Tensor, xn: Optional[torch.Tensor], route: str):
        """(input rows [T, n], gate rows of the delta rule in fp32 or None, router products or None)."""
        T, w = xs.shape[0], L.in_w
        logits = None
        if route == FEW and L.experts is not None:
            rows = self.scratch.get("mix_in_f32", (T, w.n_rows), torch.float32)
            r = L.experts.router
            logits = self.scratch.get("moe_logits_f32", (T, r.n_rows), torch.float32)
            K.gemv_float(xs, [(w.data, None, rows, K.EPI_F32), (r.data, None, logits, K.EPI_F32, xn)])
        else:
            rows = self._in_proj(xs, None, w, "mix_in", route, xn=xs)
        if "b" not in L.cols:
            return rows, None, logits
        c0 = L.cols["b"][0]
        ab = rows[:, c0:]
        if rows.dtype != torch.float32:                    # what the decays are made of is not rounded
            from ..ops import gemm as GM
            ab = GM.gemm_bf16_splitk_det(xs, w.data[c0:], self.scratch.get("lin_ab", (T, w.n_rows - c0), torch.float32), self.scratch)
        return rows, ab, logits

    def _attention(self, run: int, i: int, rows: torch.Tensor, b: BatchDesc) -> torch.Tensor:
        sc, T, L = self.scratch, b.T, self.layers[i]
        a: AttentionSpec = self.cfg.layer_specs[i].mixer

        def heads(n: str, count: int, dim: int) -> MX.HeadRows:
            c = slice(*L.cols[n])
            return MX.HeadRows(rows[:, c], count, dim, L.bias[c], L.gain.get(n))

        q_out = sc.get("q_out", (T, a.heads, a.width), self.act_dtype)
        with self._stage("post"):
            MX.mixer_post(heads("q", a.heads, a.dim), heads("k", a.kv_heads, a.dim), heads("v", a.kv_heads, a.vdim), QK_NORM_HEAD,
                          a.rot, L.freq, 1.0, q_out, self.kv[run], PAGE, b, self.block_table, self.cfg.rms_eps)
        out = sc.get("mix_out", (T, a.heads * a.width), self.act_dtype)
        with self._stage("attn_core"):
            self._attend_run(run, a, q_out, b, out)
        return out

    def _linear(self, run: int, i: int, rows: torch.Tensor, ab: Optional[torch.Tensor], b: BatchDesc,
                journal: Optional[dict]) -> torch.Tensor:
        L = self.layers[i]
        a: LinearAttentionSpec = self.cfg.layer_specs[i].mixer
        out = self.scratch.get("mix_out", (b.T, a.heads * a.vcols), self.act_dtype)
        jS, jring = (None, None) if journal is None else (journal["gdn"][run], journal["conv"].get(run))
        with self._stage("linear_core"):
            LN.linear_attention(L.lin, rows, ab, up8(a.heads), self.gdn_state[run], self.conv_state.get(run), b, out,
                                self.cfg.rms_eps, self.scratch, jS, jring)
        return out

    # ------------------------------------------------------------------ whole model
    def _embed(self, b: BatchDesc, h: torch.Tensor, copy: Optional[torch.Tensor]) -> None:
        K.embed(self.embed_w, b.tokens, h, self.cfg.embed_scale)

    def _layer_run(self, run: int, i: int, h: torch.Tensor, b: BatchDesc, route: str, journal: Optional[dict]) -> None:
        sc, T, L, m = self.scratch, b.T, self.layers[i], self.cfg.layer_specs[i].mlp
        key = self.input_key(run)
        xs = sc.get("xn_mix", (T, self.hp), self.act_dtype)
        xn = None if m is None else sc.get("xn", (T, self.hp), self.act_dtype)
        with self._stage("norm"):
            LN.norm_conv(h, L.norm1, L.norm2, L.conv, self.conv_state.get(key), b, xs, xn, self.cfg.norm_groups, self.cfg.rms_eps,
                         self.cfg.hidden, journal=None if journal is None else journal["conv"].get(key))
        with self._stage("in_gemm"):
            rows, ab, logits = self._input(L, xs, xn, route)
        if L.lin is not None:
            mix = self._linear(run, i, rows, ab, b, journal)
        else:
            mix = self._attention(run, i, rows, b)
        parts = [(mix, L.o, None)]
        if isinstance(m, DenseMlpSpec):
            parts.append((self._dense_act(None, L.gate_up, L.down.n_cols, m, h, route, xn=xn), L.down, None))
        with self._stage("out_gemm"):
            self._add_products(h, parts, route, L.o_bias)
        if isinstance(m, MoeMlpSpec):
            with self._stage("experts"):
                self._experts(L.experts, None, m, h, route, xn=xn, logits=logits)
