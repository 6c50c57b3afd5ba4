"""Common base of the designs whose layers are listed one by one (``ModelConfig.layer_specs``), some of them run repeatedly.

On top of the hybrid executor (scratch, paged pool, block tables, decode and prefill graphs, journals) it holds what these
families share:
  * bfloat16 weights; widths that are no multiple of eight are zero-padded at load (norms average over the real width);
  * one cache plane per layer RUN: every pass of a looped range attends only to what the same pass wrote;
  * per-slot recurrent rows per layer run (token shift, the state of a recurrence and of its convolution), kept where the
    hybrid executor keeps its convolution windows and states, so admission, snapshots, the cold tier, graph warm-up and
    speculative commits treat them alike;
  * three kernel routes by row count: fp32, up to 16 rows (streaming GEMV), more (tcgen05 GEMM, split over K up to 128 rows);
  * grouped-query attention of packed segments, gated feed-forwards and scaled residual adds on these routes.
"""
from __future__ import annotations

from typing import Callable, Optional, Sequence, Tuple

import torch

from ..loading.weights import ModelWeights
from ..ops import kernels as K
from ..ops.kernels import DeviceWeight
from ..quant.ggml import GGMLType
from .config import AttentionSpec, DenseMlpSpec, SideBySideSpec
from .executor import PAGE, BatchDesc, HybridExecutor

# segments of up to this many rows attend through the split-K decode kernel, longer ones through the flash kernel
DECODE_SEG_ROWS = 8
EXACT, FEW, MANY = "exact", "few", "many"       # kernel routes of a forward


def up8(n: int) -> int:
    return -(-n // 8) * 8


def pad2(t: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    """``t`` in the upper left corner of a zero [rows, cols] matrix."""
    if t.shape == (rows, cols):
        return t
    out = torch.zeros(rows, cols, dtype=t.dtype, device=t.device)
    out[:t.shape[0], :t.shape[1]] = t
    return out


class ListedExecutor(HybridExecutor):
    keeps_hidden = False
    packs_mixed = True             # prompt portions and decode rows of one step run as one forward

    def __init__(self, weights: ModelWeights, dtype: str = "bfloat16", **kw):
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"compute dtype {dtype!r} (bfloat16 | float32)")
        self.exact = dtype == "float32"
        self.act_dtype = torch.float32 if self.exact else torch.bfloat16
        self.on_layer_run: Optional[Callable[[int, torch.Tensor], None]] = None    # (run, residual rows) observer
        super().__init__(weights, **kw)

    # ------------------------------------------------------------------ weights
    def _load(self, weights: ModelWeights) -> None:
        self.weights_in = weights
        self.hp = up8(self.cfg.hidden)
        self.runs = self.cfg.layer_runs()
        self._load_layers()
        self.embed_w = self._put("token_embd.weight", self._mat("embed"))
        self.head_w = self._put("output.weight", pad2(self._mat("head"), self.cfg.vocab, self.hp))
        self.f32["final.norm"] = self._norm_weight("final.norm")
        self.loop_step: Optional[torch.Tensor] = None
        if self.cfg.loop is not None:
            self.loop_step = pad2(self._mat("loop.step").float(), self.cfg.loop.times, self.hp).contiguous()
        del self.weights_in

    def _load_layers(self) -> None:
        raise NotImplementedError

    def _norm_weight(self, name: str) -> torch.Tensor:
        """fp32 gains [hp] of a norm over the residual width (zero in padded columns)."""
        raise NotImplementedError

    def _mat(self, name: str) -> torch.Tensor:
        t = self.weights_in[name]
        if t.ggml_type == GGMLType.BF16:
            return t.raw.to(self.device).reshape(-1).view(torch.bfloat16).reshape(t.shape)
        return t.dequant(self.device).to(torch.bfloat16)

    def _out_mat(self, name: str, heads: int, real: int, padded: int) -> torch.Tensor:
        """Output map [hp, heads * padded] of a matrix over heads (or blocks) of ``real`` columns."""
        out = torch.zeros(self.hp, heads, padded, dtype=torch.bfloat16, device=self.device)
        out[:self.cfg.hidden, :, :real] = self._mat(name).reshape(self.cfg.hidden, heads, real)
        return out.reshape(self.hp, -1)

    def _gate_up(self, p: str, ff: int) -> torch.Tensor:
        """[gate | up] rows of a gated feed-forward, each zero-padded to a multiple of eight."""
        return torch.cat([pad2(self._mat(p + n), up8(ff), self.hp) for n in ("gate", "up")], 0)

    def _put(self, name: str, t: torch.Tensor) -> DeviceWeight:
        w = self.dw[name] = DeviceWeight(int(GGMLType.BF16), t.shape[0], t.shape[1], t.contiguous())
        return w

    def _vec(self, name: str, width: int, factor: float = 1.0) -> torch.Tensor:
        """A vector as fp32, times ``factor``, zero-padded to ``width``."""
        t = self._mat(name).float().reshape(-1)
        v = torch.zeros(width, dtype=torch.float32, device=self.device)
        v[:t.numel()] = t * factor
        self.f32[name] = v
        return v

    # ------------------------------------------------------------------ state: one cache plane per layer run
    def _alloc_state(self) -> None:
        dev = self.device
        self.conv_state, self.gdn_state, self.kv = {}, {}, {}
        self.kv_run = {}                       # run -> run whose plane it attends to
        latest = {}                            # layer -> its latest run
        for run, (i, _) in enumerate(self.runs):
            spec = self.cfg.layer_specs[i]
            src = getattr(spec.attention, "kv_from", None)
            self.kv_run[run] = run if src is None else latest[src]
            latest[i] = run
            if src is None:
                self.kv[run] = torch.zeros(*self._plane_shape(spec.attention), dtype=self.act_dtype, device=dev)
            if spec.token_shift:
                self.conv_state[run] = torch.zeros(self.max_slots, self.hp, 1, dtype=torch.float32, device=dev)
            if isinstance(spec.mixer, SideBySideSpec):
                r = spec.mixer.right
                self.gdn_state[run] = torch.zeros(self.max_slots, r.cols, dtype=torch.float32, device=dev)
                if r.taps > 1:
                    self.conv_state[run] = torch.zeros(self.max_slots, r.taps - 1, r.cols, dtype=torch.float32, device=dev)
        self._alloc_tables()

    def _plane_shape(self, mixer):
        return self.n_pages, 2, mixer.kv_heads, PAGE, mixer.width

    # ------------------------------------------------------------------ dispatch
    def _resid_buffer(self, T: int) -> torch.Tensor:
        return self.scratch.get("h", (T, self.hp), torch.float32)

    def _norm_rows(self, h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        xn = self.scratch.get("xn", (h.shape[0], self.hp), self.act_dtype)
        return K.rmsnorm_rows(h, w, xn, self.cfg.rms_eps, n_mean=self.cfg.hidden)

    def _route(self, T: int) -> str:
        return EXACT if self.exact else FEW if T <= K.FLOAT_GEMV_MAX_ROWS else MANY

    # ------------------------------------------------------------------ projections
    def _in_proj(self, h: torch.Tensor, norm_w: torch.Tensor, w: DeviceWeight, name: str, route: str,
                 xn: Optional[torch.Tensor] = None) -> torch.Tensor:
        """norm(h) @ W^T (fp32, or bf16 rows for large batches); ``xn``: the normalised rows when they exist already."""
        T, cfg = h.shape[0], self.cfg
        if route == FEW:
            out = self.scratch.get(name + "_f32", (T, w.n_rows), torch.float32)
            K.gemv_float(h, [(w.data, None, out, K.EPI_F32)], norm_w=norm_w, eps=cfg.rms_eps, norm_n=cfg.hidden)
            return out
        if xn is None:
            with self._stage("norm"):
                xn = self._norm_rows(h, norm_w)
        if route == EXACT:
            return K.small_gemm_f32(xn, w.data, self.scratch.get(name + "_f32", (T, w.n_rows), torch.float32))
        return self._proj(xn, w, name, name)

    def _add_products(self, h: torch.Tensor, parts: Sequence[Tuple[torch.Tensor, DeviceWeight, Optional[torch.Tensor]]],
                      route: str) -> None:
        """h += sum of s * (x @ W^T) over one or two (x, W, s); ``s``: fp32 factor per column or None."""
        from ..ops import gemm as GM
        if route == FEW:
            K.gemv_sum(h, [(x, w.data, s) for x, w, s in parts])
            return
        for x, w, s in parts:
            if route == EXACT:
                K.small_gemm_f32(x, w.data, h, add=True, col_scale=s)
            elif h.shape[0] <= self.SPLITK_MAX_ROWS:
                GM.gemm_bf16_splitk_det(x, w.data, h, self.scratch, add=True, col_scale=s)
            else:
                GM.gemm_bf16(x, w.data, h, epi=GM.EPI_ADD, col_scale=s)

    # ------------------------------------------------------------------ attention
    def _attend_run(self, run: int, a: AttentionSpec, q: torch.Tensor, b: BatchDesc, out: torch.Tensor,
                    sink: Optional[torch.Tensor] = None, head_gate: Optional[torch.Tensor] = None) -> None:
        """Rows of a packed batch over the pages of run ``run``; ``sink`` fp32 [heads], ``head_gate`` [T, heads] logits."""
        D, kv = a.width, self.kv[self.kv_run[run]]
        if self.exact:
            K.attn_exact(q, kv, self.block_table, b.slot, b.ctx_len, out, a.heads, a.kv_heads, D, PAGE, a.scale,
                         a.softcap, a.window, sink, head_gate)
            return
        from ..ops import attention as A

        def decode(r0: int, r1: int, ctx: int) -> None:
            span = min(ctx, a.window) if a.window else ctx
            split_len, max_splits = K.attn_decode_split(span, r1 - r0, a.kv_heads)
            part = self.scratch.get("attn_part", (K.attn_decode_scratch_floats(r1 - r0, a.heads, max_splits, D),),
                                    torch.float32)
            K.attn_decode(q[r0:r1], None, kv, self.block_table, b.slot[r0:r1], b.ctx_len[r0:r1], part, out[r0:r1],
                          a.heads, a.kv_heads, D, PAGE, split_len, max_splits, a.scale, a.window, a.softcap, sink,
                          None if head_gate is None else head_gate[r0:r1])

        if b.segs_host is None:
            decode(0, b.T, b.max_ctx)
            return
        # neighbouring segments of the same kind share a launch: prompt portions the flash kernel, single tokens and
        # short portions the split-K kernel
        flash = A.flash_prefill_available(D)
        s, r0 = 0, 0
        while s < len(b.segs_host):
            long = flash and b.segs_host[s][2] > DECODE_SEG_ROWS
            e, r1, ctx = s, r0, 1
            while e < len(b.segs_host) and (flash and b.segs_host[e][2] > DECODE_SEG_ROWS) == long:
                _, p0, n = b.segs_host[e]
                ctx, r1, e = max(ctx, p0 + n), r1 + n, e + 1
            if long:
                A.flash_prefill_segs(q, None, kv, self.block_table, b.seg_start[s:], b.seg_slot[s:], b.pos,
                                     [n for _, _, n in b.segs_host[s:e]], out, a.heads, a.kv_heads, D, PAGE, a.scale,
                                     a.window, a.softcap, sink, head_gate)
            else:
                for c0 in range(r0, r1, 512):       # bounds the split-K scratch of long segments of very wide heads
                    decode(c0, min(r1, c0 + 512), ctx)
            s, r0 = e, r1

    # ------------------------------------------------------------------ feed-forward
    def _dense(self, norm_w: torch.Tensor, gate_up: DeviceWeight, down: DeviceWeight, m: DenseMlpSpec, h: torch.Tensor,
               route: str, scale: Optional[torch.Tensor] = None) -> None:
        """h += scale * (Wd act(Wg norm(h), Wu norm(h)))."""
        T, F = h.shape[0], down.n_cols
        act = self.scratch.get("ffn_act", (T, F), self.act_dtype)
        if route == FEW:
            gu = gate_up.data
            K.gemv_float(h, [(gu[:F], gu[F:], act, K.EPI_OF_ACT[m.act])], norm_w=norm_w, eps=self.cfg.rms_eps,
                         norm_n=self.cfg.hidden, limit=m.limit)
        else:
            with self._stage("ffn_gateup_gemm"):
                gu = self._in_proj(h, norm_w, gate_up, "ffn_gu", route)
            with self._stage("act_mul"):
                K.act_mul(gu, act, m.act, m.limit)
        with self._stage("ffn_down_gemm"):
            self._add_products(h, [(act, down, scale)], route)

    # ------------------------------------------------------------------ whole model
    def _embed(self, b: BatchDesc, h: torch.Tensor, copy: Optional[torch.Tensor]) -> None:
        raise NotImplementedError

    def _layer_run(self, run: int, i: int, h: torch.Tensor, b: BatchDesc, route: str, journal: Optional[dict]) -> None:
        raise NotImplementedError

    readds_embedding = False       # later passes of a loop start from x + the embedding output

    def forward(self, b: BatchDesc, journal: Optional[dict] = None, h_out: Optional[torch.Tensor] = None,
                defer_resid: bool = False) -> torch.Tensor:
        cfg, T = self.cfg, b.T
        route = self._route(T)
        direct = h_out is not None and h_out.shape[1] == self.hp and h_out.is_contiguous()
        h = h_out if direct else self._resid_buffer(T)
        lp = cfg.loop
        again = self.readds_embedding and lp is not None and lp.times > 1
        x0 = self.scratch.get("embed_out", (T, self.hp), torch.float32) if again else None
        self._embed(b, h, x0)
        for run, (i, t) in enumerate(self.runs):
            if t >= 0 and i == lp.start:
                K.resid_inject(h, x0 if t > 0 else None, self.loop_step[t])
            self._layer_run(run, i, h, b, route, journal)
            if self.on_layer_run is not None:
                self.on_layer_run(run, h[:, :cfg.hidden])
        if h_out is not None and not direct:
            h_out.copy_(h[:, :cfg.hidden])
            return h_out
        return h

    def logits(self, h_rows: torch.Tensor, out: Optional[torch.Tensor] = None,
               hidden_out: Optional[torch.Tensor] = None) -> torch.Tensor:
        cfg, R = self.cfg, h_rows.shape[0]
        if h_rows.shape[1] != self.hp:
            h_rows = pad2(h_rows, R, self.hp)
        norm_w = self.f32["final.norm"]
        if out is None:
            out = self.scratch.get("logits", (R, cfg.vocab), torch.float32)
        if hidden_out is not None:
            hid = self.scratch.get("hidden_rows", (R, self.hp), torch.float32)
            hidden_out.copy_(K.rmsnorm_rows(h_rows, norm_w, hid, cfg.rms_eps, n_mean=cfg.hidden)[:, :cfg.hidden])
        if self._route(R) == FEW:
            K.gemv_float(h_rows, [(self.head_w.data, None, out, K.EPI_F32)], norm_w=norm_w, eps=cfg.rms_eps,
                         norm_n=cfg.hidden)
            return out
        xn = self.scratch.get("xn_head", (R, self.hp), self.act_dtype)
        K.rmsnorm_rows(h_rows, norm_w, xn, cfg.rms_eps, n_mean=cfg.hidden)
        if self.exact:
            return K.small_gemm_f32(xn, self.head_w.data, out)
        from ..ops import gemm as GM
        return GM.gemm_bf16(xn, self.head_w.data, out)
