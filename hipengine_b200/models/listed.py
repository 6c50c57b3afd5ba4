"""Common base of the designs whose layers are listed one by one (``ModelConfig.layer_specs``), some of them run repeatedly.

On top of the hybrid executor (scratch, paged pool, block tables, decode and prefill graphs, journals) it holds what these
families share:
  * bfloat16 weights; widths that are no multiple of eight are zero-padded at load (norms average over the real width);
  * one cache plane per layer RUN: every pass of a looped range attends only to what the same pass wrote;
  * per-slot recurrent rows per layer run (token shift, the state of a recurrence and of its convolution), kept where the
    hybrid executor keeps its convolution windows and states, so admission, snapshots, the cold tier, graph warm-up and
    speculative commits treat them alike;
  * three kernel routes by row count: fp32, up to 16 rows (streaming GEMV), more (tcgen05 GEMM, split over K up to 128 rows);
  * grouped-query attention of packed segments, gated feed-forwards, routed experts and scaled residual adds on these routes.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Optional, Sequence, Tuple

import torch

from ..loading.weights import ModelWeights
from ..ops import kernels as K
from ..ops.kernels import DeviceWeight
from ..quant.ggml import GGMLType
from .config import AttentionSpec, DenseMlpSpec, LinearAttentionSpec, MoeMlpSpec, SideBySideSpec
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


@dataclass
class ExpertWeights:
    router: DeviceWeight                         # [experts (+ shared gate), hp], rows padded to eight
    gate_up: DeviceWeight                        # [experts * (gate | up), hp]
    down: DeviceWeight                           # [experts * hp, F]
    s_gate_up: Optional[DeviceWeight] = None     # shared expert
    s_down: Optional[DeviceWeight] = None


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

    def _load_experts(self, p: str, m: MoeMlpSpec) -> ExpertWeights:
        """Experts, router and shared expert of the layer whose tensors start with ``p``, stacked."""
        hp, fp, put = self.hp, up8(m.ff), self._put
        gu = torch.empty(m.experts * 2 * fp, hp, dtype=torch.bfloat16, device=self.device)
        dn = torch.empty(m.experts * hp, fp, dtype=torch.bfloat16, device=self.device)
        for e in range(m.experts):
            gu[e * 2 * fp:(e + 1) * 2 * fp] = self._gate_up(p + f"mlp.e{e}.", m.ff)
            dn[e * hp:(e + 1) * hp] = pad2(self._mat(p + f"mlp.e{e}.down"), hp, fp)
        rows, shared = [self._mat(p + "mlp.router")], (None, None)
        if m.shared_ff:
            rows.append(self._mat(p + "mlp.shared.sg"))
            shared = (put(p + "shared.gate_up", self._gate_up(p + "mlp.shared.", m.shared_ff)),
                      put(p + "shared.down", pad2(self._mat(p + "mlp.shared.down"), hp, up8(m.shared_ff))))
        r = torch.cat(rows, 0)
        return ExpertWeights(put(p + "router", pad2(r, up8(r.shape[0]), hp)), put(p + "experts.gate_up", gu),
                             put(p + "experts.down", dn), *shared)

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
            if src is None and spec.attention is not None:
                self.kv[run] = torch.zeros(*self._plane_shape(spec.attention), dtype=self.act_dtype, device=dev)
            if spec.token_shift:
                self.conv_state[run] = torch.zeros(self.max_slots, self.hp, 1, dtype=torch.float32, device=dev)
            if isinstance(spec.mixer, SideBySideSpec):
                r = spec.mixer.right
                self.gdn_state[run] = torch.zeros(self.max_slots, r.cols, dtype=torch.float32, device=dev)
                if r.taps > 1:
                    self.conv_state[run] = torch.zeros(self.max_slots, r.taps - 1, r.cols, dtype=torch.float32, device=dev)
            if isinstance(spec.mixer, LinearAttentionSpec):
                m = spec.mixer
                self.gdn_state[run] = torch.zeros(self.max_slots, m.heads, m.dim, m.vcols, dtype=torch.float32, device=dev)
                if m.delta and m.taps > 1:
                    self.conv_state[run] = torch.zeros(self.max_slots, m.taps, m.conv_cols, dtype=torch.float32, device=dev)
            if spec.input_taps > 1:
                self.conv_state[self.input_key(run)] = torch.zeros(self.max_slots, spec.input_taps - 1, self.hp,
                                                                   dtype=torch.float32, device=dev)
        self._alloc_tables()

    @staticmethod
    def input_key(run: int) -> str:
        """Key of the past of the convolution ahead of run ``run``'s mixer among the convolution states."""
        return f"{run}.in"

    def _plane_shape(self, mixer):
        return self.n_pages, 2, mixer.kv_heads, PAGE, mixer.width

    # ------------------------------------------------------------------ dispatch
    def _resid_buffer(self, T: int) -> torch.Tensor:
        return self.scratch.get("h", (T, self.hp), torch.float32)

    def _norm_rows(self, h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        return self._norm_into(h, w, self.scratch.get("xn", (h.shape[0], self.hp), self.act_dtype))

    def _norm_into(self, h: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        if self.cfg.norm_groups > 1:
            from ..ops import linear as LN
            return LN.grouped_norm(h, w, out, self.cfg.norm_groups, self.cfg.rms_eps, self.cfg.hidden)
        return K.rmsnorm_rows(h, w, out, self.cfg.rms_eps, n_mean=self.cfg.hidden)

    def _route(self, T: int) -> str:
        return EXACT if self.exact else FEW if T <= K.FLOAT_GEMV_MAX_ROWS else MANY

    # ------------------------------------------------------------------ projections
    def _in_proj(self, h: torch.Tensor, norm_w: torch.Tensor, w: DeviceWeight, name: str, route: str,
                 xn: Optional[torch.Tensor] = None) -> torch.Tensor:
        """norm(h) @ W^T (fp32, or bf16 rows for large batches); ``xn``: the normalised rows when they exist already."""
        T, cfg = h.shape[0], self.cfg
        if route == FEW:
            out = self.scratch.get(name + "_f32", (T, w.n_rows), torch.float32)
            norm = {} if xn is not None else dict(norm_w=norm_w, eps=cfg.rms_eps, norm_n=cfg.hidden)
            K.gemv_float(h if xn is None else xn, [(w.data, None, out, K.EPI_F32)], **norm)
            return out
        if xn is None:
            with self._stage("norm"):
                xn = self._norm_rows(h, norm_w)
        if route == EXACT:
            return K.small_gemm_f32(xn, w.data, self.scratch.get(name + "_f32", (T, w.n_rows), torch.float32))
        return self._proj(xn, w, name, name)

    def _add_products(self, h: torch.Tensor, parts: Sequence[Tuple[torch.Tensor, DeviceWeight, Optional[torch.Tensor]]],
                      route: str, bias: Optional[torch.Tensor] = None) -> None:
        """h += bias + sum of s * (x @ W^T) over one or two (x, W, s); ``s``: fp32 factor per column or None."""
        from ..ops import gemm as GM
        if route == FEW:
            K.gemv_sum(h, [(x, w.data, s) for x, w, s in parts], bias)
            return
        for x, w, s in parts:
            if route == EXACT:
                K.small_gemm_f32(x, w.data, h, add=True, col_scale=s, col_bias=bias)
            elif h.shape[0] <= self.SPLITK_MAX_ROWS:
                GM.gemm_bf16_splitk_det(x, w.data, h, self.scratch, add=True, col_scale=s, col_bias=bias)
            else:
                GM.gemm_bf16(x, w.data, h, epi=GM.EPI_ADD, col_scale=s, col_bias=bias)
            bias = None

    # ------------------------------------------------------------------ attention
    def _attend_run(self, run: int, a: AttentionSpec, q: torch.Tensor, b: BatchDesc, out: torch.Tensor,
                    sink: Optional[torch.Tensor] = None, head_gate: Optional[torch.Tensor] = None) -> None:
        """Rows of a packed batch over the pages of run ``run``; ``sink`` fp32 [heads], ``head_gate`` [T, heads] logits."""
        D, kv = a.width, self.kv[self.kv_run[run]]
        if self.exact:
            K.attn_exact(q, kv, self.block_table, b.slot, b.ctx_len, out, a.heads, a.kv_heads, D, PAGE, a.scale,
                         a.softcap, a.window, sink, head_gate, a.keep_first)
            return
        from ..ops import attention as A

        def decode(r0: int, r1: int, ctx: int) -> None:
            span = min(ctx, a.window + a.keep_first) if a.window else ctx
            split_len, max_splits = K.attn_decode_split(span, r1 - r0, a.kv_heads)
            part = self.scratch.get("attn_part", (K.attn_decode_scratch_floats(r1 - r0, a.heads, max_splits, D),),
                                    torch.float32)
            K.attn_decode(q[r0:r1], None, kv, self.block_table, b.slot[r0:r1], b.ctx_len[r0:r1], part, out[r0:r1],
                          a.heads, a.kv_heads, D, PAGE, split_len, max_splits, a.scale, a.window, a.softcap, sink,
                          None if head_gate is None else head_gate[r0:r1], a.keep_first)

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
                                     a.window, a.softcap, sink, head_gate, a.keep_first)
            else:
                for c0 in range(r0, r1, 512):       # bounds the split-K scratch of long segments of very wide heads
                    decode(c0, min(r1, c0 + 512), ctx)
            s, r0 = e, r1

    # ------------------------------------------------------------------ feed-forward
    def _dense(self, norm_w: torch.Tensor, gate_up: DeviceWeight, down: DeviceWeight, m: DenseMlpSpec, h: torch.Tensor,
               route: str, scale: Optional[torch.Tensor] = None) -> None:
        """h += scale * (Wd act(Wg norm(h), Wu norm(h)))."""
        act = self._dense_act(norm_w, gate_up, down.n_cols, m, h, route)
        with self._stage("ffn_down_gemm"):
            self._add_products(h, [(act, down, scale)], route)

    def _dense_act(self, norm_w: Optional[torch.Tensor], gate_up: DeviceWeight, F: int, m: DenseMlpSpec, h: torch.Tensor,
                   route: str, xn: Optional[torch.Tensor] = None) -> torch.Tensor:
        """act(Wg norm(h), Wu norm(h)) [T, F]; ``xn``: the normalised rows when they exist already."""
        act = self.scratch.get("ffn_act", (h.shape[0], F), self.act_dtype)
        if route == FEW:
            gu = gate_up.data
            norm = {} if xn is not None else dict(norm_w=norm_w, eps=self.cfg.rms_eps, norm_n=self.cfg.hidden)
            K.gemv_float(h if xn is None else xn, [(gu[:F], gu[F:], act, K.EPI_OF_ACT[m.act])], limit=m.limit, **norm)
        else:
            with self._stage("ffn_gateup_gemm"):
                gu = self._in_proj(h, norm_w, gate_up, "ffn_gu", route, xn=xn)
            with self._stage("act_mul"):
                K.act_mul(gu, act, m.act, m.limit)
        return act

    def _experts(self, W: ExpertWeights, norm_w: Optional[torch.Tensor], m: MoeMlpSpec, h: torch.Tensor, route: str,
                 xn: Optional[torch.Tensor] = None, logits: Optional[torch.Tensor] = None) -> None:
        """h += the routed experts (and the shared one) of norm(h); ``xn``: the normalised rows, ``logits``: the router's products
        (fp32), when they exist already."""
        from ..ops import gemm as GM
        sc, cfg, T, E, k = self.scratch, self.cfg, h.shape[0], m.experts, m.top
        F, fused = W.down.n_cols, xn is None and route == FEW
        if xn is None and not fused:
            with self._stage("norm"):
                xn = self._norm_rows(h, norm_w)
        if logits is None:
            if route == MANY:
                logits = GM.gemm_bf16(xn, W.router.data, sc.get("moe_logits_f32", (T, W.router.n_rows), torch.float32))
            else:
                logits = self._in_proj(h, norm_w, W.router, "moe_logits", route, xn=xn)
        ids = sc.get("moe_ids", (T, k), torch.int32)
        wts = sc.get("moe_wts", (T, k), torch.float32)
        if m.score == "softmax":
            K.moe_route(logits, k, ids, wts, n_experts=E, mode=2)
        else:
            K.moe_route_grouped(logits, k, ids, wts, E, m.groups, m.groups_kept, m.scale)
        sg = logits[:, E:E + 1] if m.shared_ff else None
        s_gu = W.s_gate_up.data if m.shared_ff else None
        s_dn = W.s_down.data if m.shared_ff else None
        if route != MANY:
            rows = sc.get("moe_act", (T * k, F), self.act_dtype)
            rows_s = sc.get("moe_act_sh", (T, W.s_down.n_cols), self.act_dtype) if m.shared_ff else None
            if route == EXACT:
                K.moe_exact(xn, ids, wts, W.gate_up.data, W.down.data, E, rows, h, sg, s_gu, s_dn, rows_s, m.act, m.limit)
                return
            K.moe_gateup_float(h if fused else xn, norm_w if fused else None, cfg.rms_eps, cfg.hidden, ids, wts, W.gate_up.data, E,
                               rows, sg, s_gu, rows_s, m.act, m.limit)
            K.moe_down_float(rows, ids, W.down.data, E, h, rows_s, s_dn)
            return
        P = T * k
        bound = K.moe_sorted_rows_bound(P, E)
        pos = sc.get("moe_pos", (P,), torch.int32)
        tiles = sc.get("moe_tiles", (bound // 128,), torch.int32)
        K.moe_group(ids, E, pos, tiles, sc.get("moe_meta", (4,), torch.int32))
        xs = sc.get("moe_xs", (bound, self.hp), torch.bfloat16)
        K.moe_gather(xn, pos, k, xs)
        gu = sc.get("moe_gu", (bound, 2 * F), torch.bfloat16)
        GM.gemm_bf16_grouped(xs, W.gate_up.data, gu, E, tiles)
        act = sc.get("moe_act_g", (bound, F), torch.bfloat16)
        K.act_mul(gu, act, m.act, m.limit)
        ys = sc.get("moe_ys", (bound, self.hp), torch.bfloat16)
        GM.gemm_bf16_grouped(act, W.down.data, ys, E, tiles)
        ysh = None
        if m.shared_ff:
            gus = self._proj(xn, W.s_gate_up, "moe_gus", "g")
            acts = sc.get("moe_acts", (T, W.s_down.n_cols), torch.bfloat16)
            K.act_mul(gus, acts, m.act, m.limit)
            ysh = self._gemm(acts, W.s_down, sc.get("y_bf", (T, self.hp), torch.bfloat16), tag="d")
        K.moe_combine(h, ys, pos, wts, k, ysh, sg)

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
            hidden_out.copy_(self._norm_into(h_rows, norm_w, hid)[:, :cfg.hidden])
        few = self._route(R) == FEW
        if few and cfg.norm_groups == 1:
            K.gemv_float(h_rows, [(self.head_w.data, None, out, K.EPI_F32)], norm_w=norm_w, eps=cfg.rms_eps,
                         norm_n=cfg.hidden)
            return out
        xn = self._norm_into(h_rows, norm_w, self.scratch.get("xn_head", (R, self.hp), self.act_dtype))
        if few:
            K.gemv_float(xn, [(self.head_w.data, None, out, K.EPI_F32)])
            return out
        if self.exact:
            return K.small_gemm_f32(xn, self.head_w.data, out)
        from ..ops import gemm as GM
        return GM.gemm_bf16(xn, self.head_w.data, out)
