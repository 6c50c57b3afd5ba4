"""Banelix executor: windowed attention layers, and layers of attention beside a gated linear recurrence.

The base (``listed.py``) holds the planes per layer run, the states, the routes, attention and feed-forward; here are the
weight packing and the two mixers.  A layer:
  input     ONE product gives query | key | value | head gate | output gate | recurrence rows (norm fused up to 16 rows);
  post      one launch: biases, norms, rotation, page write, and the recurrence's short convolution (``ops/mixers.py``);
  attention split-K kernel for single tokens and short portions, flash kernel for longer ones; sink, window and head gate
            inside them;
  recurrence one token per request: gate products and state step in one launch; otherwise the block-diagonal gate products
            (streaming product, or one grouped tcgen05 GEMM with a group per block) and a scan;
  output    both mixers' output products with their factors in one launch for few rows.
``dtype="float32"`` runs the same walk on fp32 CUDA-core kernels with fp32 pages.  In both modes residual, norms, angles,
scores, softmax, gates and recurrent state are fp32.  Oracle: ``ref/banelix.py``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from ..ops import kernels as K
from ..ops import mixers as MX
from ..ops.kernels import DeviceWeight
from .config import QK_NORM_ROWS, AttentionSpec, RecurrentSpec, SideBySideSpec, round_up
from .executor import PAGE, BatchDesc
from .listed import EXACT, FEW, ListedExecutor, pad2, up8


@dataclass
class _Attention:
    cols: Dict[str, Tuple[int, int]]              # q, k, v, g, y, x -> column range of the input rows
    bias: torch.Tensor                            # fp32 over the input rows
    gain: Dict[str, torch.Tensor]                 # norm over the whole projection: q, k
    freq: torch.Tensor                            # float64 [rot.dims / 2]
    amp: float
    o: DeviceWeight                               # [hp, heads * D]
    o_scale: torch.Tensor                         # fp32 [hp]
    sink: Optional[torch.Tensor]                  # fp32 [heads]


@dataclass
class _Recurrent:
    conv: torch.Tensor                            # fp32 [taps, C]
    conv_bias: torch.Tensor
    par: MX.Recurrence
    o: DeviceWeight                               # [hp, C]
    o_scale: torch.Tensor


@dataclass
class _Layer:
    norm1: torch.Tensor                           # fp32 [hp]
    in_w: DeviceWeight                            # rows of every input projection, [n, hp]
    att: _Attention
    rec: Optional[_Recurrent] = None
    norm2: Optional[torch.Tensor] = None
    gate_up: Optional[DeviceWeight] = None
    down: Optional[DeviceWeight] = None
    ff_scale: Optional[torch.Tensor] = None       # fp32 [hp]


class BanelixExecutor(ListedExecutor):
    # ------------------------------------------------------------------ weights
    def _norm_weight(self, name: str) -> torch.Tensor:
        return self._vec(name, self.hp)

    def _factor(self, value: float) -> torch.Tensor:
        return torch.full((self.hp,), value, dtype=torch.float32, device=self.device)

    @staticmethod
    def _pad_blocks(t: torch.Tensor, r: RecurrentSpec) -> torch.Tensor:
        """Channels along the first dimension -> every block zero-padded to ``block_cols``."""
        out = torch.zeros(r.blocks, r.block_cols, *t.shape[1:], dtype=t.dtype, device=t.device)
        out[:, :r.width // r.blocks] = t.reshape(r.blocks, -1, *t.shape[1:])
        return out.reshape(r.cols, *t.shape[1:])

    def _load_layers(self) -> None:
        cfg, hp, put, norm = self.cfg, self.hp, self._put, self._norm_weight
        self.layers: List[_Layer] = []
        for i, spec in enumerate(cfg.layer_specs):
            p, both = f"l{i}.", isinstance(spec.mixer, SideBySideSpec)
            a, m = spec.attention, p + ("mix.left." if both else "mix.")
            rows = ["q"] + ([] if a.kv_from is not None else ["k"] if a.keys_as_values else ["k", "v"])
            mats = [(n, self._mat(m + n), self._mat(m + n + ".b") if a.bias else None) for n in rows]
            if a.head_gate:
                mats.append(("g", self._mat(m + "g"), None))
            if both:
                r, mr = spec.mixer.right, p + "mix.right."
                mats += [(n, *(self._pad_blocks(self._mat(mr + n + s), r) for s in ("", ".b"))) for n in ("y", "x")]
            cols, at = {}, 0
            w = torch.zeros(sum(up8(t.shape[0]) for _, t, _ in mats), hp, dtype=torch.bfloat16, device=self.device)
            bias = torch.zeros(w.shape[0], dtype=torch.float32, device=self.device)
            for n, t, b in mats:
                w[at:at + t.shape[0], :cfg.hidden] = t
                if b is not None:
                    bias[at:at + t.shape[0]] = b.float()
                cols[n] = (at, at + up8(t.shape[0]))
                at = cols[n][1]
            freq, amp = a.rot.table()
            gain = {}
            if a.qk_norm == QK_NORM_ROWS:
                gain = {n: self._vec(m + n + ".norm", cols[n][1] - cols[n][0]) for n in rows if n != "v"}
            L = _Layer(norm(p + "norm1"), put(p + "in", w), _Attention(
                cols, bias, gain, torch.tensor(freq, dtype=torch.float64, device=self.device), amp,
                put(p + "o", self._out_mat(m + "o", a.heads, a.vdim, a.width)),
                self._factor(cfg.residual_mult * (spec.mixer.left_scale if both else 1.0)),
                None if a.sink_score is None else torch.full((a.heads,), a.sink_score, dtype=torch.float32, device=self.device)))
            if both:
                L.rec = self._load_recurrent(p, spec.mixer, L.att)
            if spec.mlp is not None:
                L.norm2 = norm(p + "norm2")
                L.gate_up = put(p + "gate_up", self._gate_up(p + "mlp.", spec.mlp.ff))
                L.down = put(p + "down", pad2(self._mat(p + "mlp.down"), hp, up8(spec.mlp.ff)))
                L.ff_scale = self._factor(cfg.residual_mult)
            self.layers.append(L)
        self._block_tiles: Dict[Tuple[int, int], torch.Tensor] = {}

    def _load_recurrent(self, p: str, mix: SideBySideSpec, att: _Attention) -> _Recurrent:
        r, m = mix.right, p + "mix.right."
        n, bc = r.width // r.blocks, r.block_cols
        vec = lambda name: self._pad_blocks(self._mat(m + name).float().reshape(r.width), r)
        gates = torch.zeros(r.blocks, 2, bc, bc, dtype=torch.bfloat16, device=self.device)
        gate_b = torch.zeros(r.blocks, 2, bc, dtype=torch.float32, device=self.device)
        for j, g in enumerate(("ra", "ri")):
            gates[:, j, :n, :n] = self._mat(m + g)
            gate_b[:, j, :n] = self._mat(m + g + ".b").float()
        gates = gates.reshape(r.blocks, 2 * bc, bc)
        self.dw[p + "gates"] = DeviceWeight(30, r.blocks * 2 * bc, bc, gates)
        decay = self._pad_blocks(-8.0 * torch.nn.functional.softplus(self._mat(m + "lam").float()), r)
        part = lambda name: att.bias[slice(*att.cols[name])].contiguous()
        return _Recurrent(self._pad_blocks(self._mat(m + "conv").float(), r).t().contiguous(), vec("conv.b"),
                          MX.Recurrence(gates, gate_b.reshape(r.blocks, 2 * bc), decay, part("y"), part("x"), r.taps),
                          self._put(p + "right.o", self._out_mat(m + "o", r.blocks, n, bc)),
                          self._factor(self.cfg.residual_mult * mix.right_scale))

    # ------------------------------------------------------------------ mixers
    def _conv_out(self, r: RecurrentSpec, T: int, route: str) -> torch.Tensor:
        """[T, blocks, block_cols] buffer of the convolution's output: token-major, or for the grouped product block-major with
        whole 128-row tiles per block."""
        if route in (FEW, EXACT):
            return self.scratch.get("rec_u", (T, r.blocks, r.block_cols), self.act_dtype)
        return self.scratch.get("rec_u", (r.blocks, round_up(T, 128), r.block_cols), self.act_dtype).transpose(0, 1)[:T]

    def _gate_products(self, R: _Recurrent, r: RecurrentSpec, u: torch.Tensor, route: str) -> torch.Tensor:
        """fp32 [T, blocks, 2 * block_cols]: every block of u times its two gate maps."""
        T, n = u.shape[0], 2 * r.block_cols
        if route in (FEW, EXACT):
            g = self.scratch.get("rec_gates", (T, r.blocks, n), torch.float32)
            (K.small_gemm_f32 if route == EXACT else K.gemv_float_batched)(u, R.par.gate_w, g)
            return g
        from ..ops import gemm as GM
        Tp = round_up(T, 128)
        tiles = self._block_tiles.get((r.blocks, Tp))
        if tiles is None:
            tiles = torch.arange(r.blocks, dtype=torch.int32, device=self.device).repeat_interleave(Tp // 128)
            self._block_tiles[(r.blocks, Tp)] = tiles
        g = self.scratch.get("rec_gates", (r.blocks, Tp, n), torch.float32)
        GM.gemm_bf16_grouped(self.scratch.get("rec_u", (r.blocks * Tp, r.block_cols), self.act_dtype),
                             R.par.gate_w.view(-1, r.block_cols), g.view(-1, n), r.blocks, tiles)
        return g.transpose(0, 1)[:T]

    def _recurrence(self, run: int, R: _Recurrent, r: RecurrentSpec, u: torch.Tensor, y: torch.Tensor, x: torch.Tensor,
                    b: BatchDesc, route: str, journal: Optional[dict]) -> torch.Tensor:
        out = self.scratch.get("rec_out", (b.T, r.cols), self.act_dtype)
        S, cs = self.gdn_state[run], self.conv_state.get(run)
        if route == FEW and b.n_seg == b.T and journal is None:
            MX.rglru_step(R.par, u, y, x, S, cs, b, out)
        else:
            g = self._gate_products(R, r, u, route)
            MX.rglru_scan(R.par, g, u, y, x, S, cs, b, out, journal=None if journal is None else journal["gdn"][run])
        return out

    def _mix(self, run: int, i: int, h: torch.Tensor, b: BatchDesc, route: str, journal: Optional[dict]) -> None:
        sc, L, T = self.scratch, self.layers[i], b.T
        mix, A, R = self.cfg.layer_specs[i].mixer, L.att, L.rec
        a: AttentionSpec = self.cfg.layer_specs[i].attention
        with self._stage("in_gemm"):
            rows = self._in_proj(h, L.norm1, L.in_w, "mix_in", route)
        part = {n: rows[:, c0:c1] for n, (c0, c1) in A.cols.items()}

        def heads(n: str, count: int, dim: int) -> Optional[MX.HeadRows]:
            if n not in part:
                return None
            return MX.HeadRows(part[n], count, dim, A.bias[slice(*A.cols[n])] if a.bias else None, A.gain.get(n))

        conv = None
        if R is not None:
            u = self._conv_out(mix.right, T, route)
            conv = MX.ConvRows(part["x"], R.par.x_bias, R.conv, R.conv_bias, u, self.conv_state.get(run),
                               None if journal is None else journal["conv"].get(run))
        q_out = sc.get("q_out", (T, a.heads, a.width), self.act_dtype)
        with self._stage("post"):
            MX.mixer_post(heads("q", a.heads, a.dim), heads("k", a.kv_heads, a.dim), heads("v", a.kv_heads, a.vdim), a.qk_norm,
                          a.rot, A.freq, A.amp, q_out, self.kv.get(run), PAGE, b, self.block_table, self.cfg.rms_eps, conv)
        outs = []
        if R is not None:
            with self._stage("recurrence"):
                outs = [(self._recurrence(run, R, mix.right, u, part["y"], part["x"], b, route, journal), R.o, R.o_scale)]
        attn = sc.get("attn_out", (T, a.heads * a.width), self.act_dtype)
        with self._stage("attn_core"):
            self._attend_run(run, a, q_out, b, attn, A.sink, part["g"] if a.head_gate else None)
        with self._stage("out_gemm"):
            self._add_products(h, [(attn, A.o, A.o_scale)] + outs, route)

    # ------------------------------------------------------------------ whole model
    def _embed(self, b: BatchDesc, h: torch.Tensor, copy: Optional[torch.Tensor]) -> None:
        K.embed(self.embed_w, b.tokens, h, self.cfg.embed_scale)

    def _layer_run(self, run: int, i: int, h: torch.Tensor, b: BatchDesc, route: str, journal: Optional[dict]) -> None:
        self._mix(run, i, h, b, route, journal)
        m, L = self.cfg.layer_specs[i].mlp, self.layers[i]
        if m is not None:
            self._dense(L.norm2, L.gate_up, L.down, m, h, route, L.ff_scale)
