"""Milutar executor: parallel layers over latent attention, token shift, layer scale, looped layer ranges.

The base (``listed.py``) holds the planes per layer run, the recurrent rows, the routes and the walk over runs.  A layer run:
  norm + shift   one kernel gives both sublayers their rows and advances the slot's previous row;
  projections    up to 16 rows: query / latent rows and the squared-ReLU feed-forward rows in ONE streaming launch (each
                 segment reads its own input); more rows: tcgen05 GEMMs with the activation in the epilogue;
  cache          latent norm, rotation and page write in one kernel; a page row is [latent | rotated key part];
  attention      single rows and short portions in latent space (the key map moved onto the query, the value map behind the
                 sum), long portions with keys and values expanded once per launch by GEMMs: the common head shapes on
                 tcgen05 with accumulators in tensor memory, the others on a register kernel;
  output         both output projections with their per-channel factors: one launch for few rows, two accumulating GEMMs
                 otherwise.
``dtype="float32"`` runs the same walk, in latent space throughout, on fp32 CUDA-core kernels and fp32 pages.  In both modes
residual, norms, angles, scores and softmax are fp32.  Oracle: ``ref/milutar.py``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Tuple

import torch

from ..ops import kernels as K
from ..ops import latent as LA
from ..ops.kernels import DeviceWeight
from .config import LatentAttentionSpec
from .executor import PAGE, BatchDesc
from .listed import DECODE_SEG_ROWS, EXACT, FEW, MANY, ListedExecutor, pad2, up8

EXPANDED_KV_BYTES = 1 << 30       # expanded keys and values of a launch: above this the heads are taken in groups
TC_MIN_ROWS = 65                  # longest portion from which the tensor-memory form (256-row tiles) is taken
LATENT_ROWS = 512                 # rows per latent-space launch (bounds its split-K scratch)


@dataclass
class _Layer:
    gain: torch.Tensor                     # fp32 [hp]: the norm's single number in every real column
    shift: torch.Tensor                    # fp32 [hp]
    dn: int                                # unrotated / value columns per head, padded to eight
    dv: int
    qd: int                                # query columns per head: dn + rotated, padded to eight
    in_w: DeviceWeight                     # [query (or query latent) rows | latent and rotated key rows, hp]
    n_q: int                               # rows of its first part
    kv_norm: torch.Tensor                  # fp32 [rank_cols]
    uk: DeviceWeight                       # [heads * dn, rank_cols]
    uv: DeviceWeight                       # [heads * dv, rank_cols]
    uk_t: torch.Tensor                     # [heads, rank_cols, dn]: the key map from the query's side
    freq: torch.Tensor                     # float64 [rot_dim / 2]
    amp: float
    o: DeviceWeight                        # [hp, heads * dv]
    s1: torch.Tensor                       # fp32 [hp]: layer scale times the residual factor
    q_norm: Optional[torch.Tensor] = None  # query latent: fp32 [q_rank padded]
    uq: Optional[DeviceWeight] = None      # [heads * qd, q_rank padded]
    sink: Optional[torch.Tensor] = None    # fp32 [heads]
    up: Optional[DeviceWeight] = None      # [ff padded, hp]
    down: Optional[DeviceWeight] = None    # [hp, ff padded]
    s2: Optional[torch.Tensor] = None


class MilutarExecutor(ListedExecutor):
    # ------------------------------------------------------------------ weights
    def _norm_weight(self, name: str) -> torch.Tensor:
        v = torch.zeros(self.hp, dtype=torch.float32, device=self.device)
        v[:self.cfg.hidden] = self._mat(name).float().reshape(())
        self.f32[name] = v
        return v

    @staticmethod
    def _pad_heads(w: torch.Tensor, heads: int, parts: Tuple[Tuple[int, int], ...], cols: int) -> torch.Tensor:
        """Rows of every head in ``parts`` of (real, padded) rows -> zero-padded rows and columns."""
        out = torch.zeros(heads, sum(p for _, p in parts), cols, dtype=w.dtype, device=w.device)
        src, dst = 0, 0
        w = w.reshape(heads, -1, w.shape[1])
        for real, padded in parts:
            out[:, dst:dst + real, :w.shape[2]] = w[:, src:src + real]
            src, dst = src + real, dst + padded
        return out

    def _load_layers(self) -> None:
        cfg, hp, mat, put = self.cfg, self.hp, self._mat, self._put
        self.layers: List[_Layer] = []
        for i, spec in enumerate(cfg.layer_specs):
            a, m, p = spec.mixer, spec.mlp, f"l{i}."
            dn, dv, rr = up8(a.dim), up8(a.vdim), up8(a.rot_dim)
            q_parts = ((a.dim, dn), (a.rot_dim, rr))
            qr = up8(a.q_rank) if a.q_rank else 0
            q = self._pad_heads(mat(p + ("mix.uq" if a.q_rank else "mix.q")), a.heads, q_parts, qr or hp)
            q = q.reshape(a.heads * (dn + rr), -1)
            first = pad2(mat(p + "mix.dq"), qr, hp) if a.q_rank else q
            down = pad2(mat(p + "mix.dkv"), up8(a.kv_rank + a.rot_dim), hp)
            uk = self._pad_heads(mat(p + "mix.uk"), a.heads, ((a.dim, dn),), a.rank_cols)
            uv = self._pad_heads(mat(p + "mix.uv"), a.heads, ((a.vdim, dv),), a.rank_cols)
            freq, amp = a.rot.table()
            uk_t = uk.transpose(1, 2).contiguous()
            self.dw[p + "uk_t"] = DeviceWeight(30, a.heads * a.rank_cols, dn, uk_t)
            L = _Layer(self._norm_weight(p + "norm1"), self._vec(p + "shift", hp), dn, dv, dn + rr,
                       put(p + "in", torch.cat([first, down], 0)), first.shape[0],
                       self._vec(p + "mix.dkv.norm", a.rank_cols),
                       put(p + "uk", uk.reshape(-1, a.rank_cols)), put(p + "uv", uv.reshape(-1, a.rank_cols)), uk_t,
                       torch.tensor(freq, dtype=torch.float64, device=self.device), amp,
                       put(p + "o", self._out_mat(p + "mix.o", a.heads, a.vdim, dv)),
                       self._vec(p + "ls1", hp, cfg.residual_mult))
            if a.q_rank:
                L.q_norm, L.uq = self._vec(p + "mix.dq.norm", qr), put(p + "uq", q)
            if a.sink:
                L.sink = self._vec(p + "mix.sink", a.heads)
            if m is not None:
                L.up = put(p + "up", pad2(mat(p + "mlp.up"), up8(m.ff), hp))
                L.down = put(p + "down", pad2(mat(p + "mlp.down"), hp, up8(m.ff)))
                L.s2 = self._vec(p + "ls2", hp, cfg.residual_mult)
            self.layers.append(L)

    def _plane_shape(self, mixer: LatentAttentionSpec):
        return self.n_pages, PAGE, mixer.row_cols

    # ------------------------------------------------------------------ projections
    def _in_projections(self, L: _Layer, a: LatentAttentionSpec, xn: torch.Tensor, xs: torch.Tensor, route: str):
        """(queries [T, heads * qd] fp32 or bf16, latent rows fp32, feed-forward rows or None)."""
        from ..ops import gemm as GM
        sc, T, w, eps = self.scratch, xn.shape[0], L.in_w, self.cfg.rms_eps
        act = None if L.up is None else sc.get("ffn_act", (T, L.up.n_rows), self.act_dtype)
        few_tiles = route == MANY and T <= self.SPLITK_MAX_ROWS
        if route == MANY and not few_tiles and L.uq is None:
            # long batches keep the queries in bf16 (rotated in place); the latents stay fp32 up to their norm
            q = GM.gemm_bf16(xs, w.data[:L.n_q], sc.get("lat_q_bf", (T, L.n_q), torch.bfloat16))
            down = GM.gemm_bf16(xs, w.data[L.n_q:], sc.get("lat_down_f32", (T, w.n_rows - L.n_q), torch.float32))
        else:
            rows = sc.get("lat_in_f32", (T, w.n_rows), torch.float32)
            if route == FEW:
                segs = [(w.data, None, rows, K.EPI_F32)]
                if act is not None:
                    segs.append((L.up.data, None, act, K.EPI_RELU2, xn))
                K.gemv_float(xs, segs)
            elif route == EXACT:
                K.small_gemm_f32(xs, w.data, rows)
            elif few_tiles:
                GM.gemm_bf16_splitk_det(xs, w.data, rows, sc)
            else:
                GM.gemm_bf16(xs, w.data, rows)
            q, down = rows[:, :L.n_q], rows[:, L.n_q:]
        if act is not None and route != FEW:
            if route == EXACT:
                K.small_gemm_f32(xn, L.up.data, act, mode=K.GEMM_RELU2)
            elif few_tiles:
                GM.gemm_bf16_splitk_det(xn, L.up.data, act, sc, relu2=True)
            else:
                GM.gemm_bf16(xn, L.up.data, act, epi=GM.EPI_RELU2)
        if L.uq is not None:
            n = L.uq.n_rows
            if route == FEW:
                qf = sc.get("lat_q_f32", (T, n), torch.float32)
                K.gemv_float(q, [(L.uq.data, None, qf, K.EPI_F32)], norm_w=L.q_norm, eps=eps, norm_n=a.q_rank)
            else:
                cq = sc.get("lat_cq", (T, L.n_q), self.act_dtype)
                K.rmsnorm_rows(q, L.q_norm, cq, eps, n_mean=a.q_rank)
                if route == EXACT:
                    qf = K.small_gemm_f32(cq, L.uq.data, sc.get("lat_q_f32", (T, n), torch.float32))
                elif few_tiles:
                    qf = GM.gemm_bf16_splitk_det(cq, L.uq.data, sc.get("lat_q_f32", (T, n), torch.float32), sc)
                else:
                    qf = GM.gemm_bf16(cq, L.uq.data, sc.get("lat_q_bf", (T, n), torch.bfloat16))
            q = qf
        return q, down, act

    # ------------------------------------------------------------------ attention
    def _segment_groups(self, L: _Layer, b: BatchDesc, route: str):
        """Neighbouring segments of a kind, as (expanded?, first segment, end segment, first row, end row, longest context)."""
        if route != MANY or b.segs_host is None or LA.prefill_tile_rows(L.qd, L.dv) == 0:
            return [(False, 0, b.n_seg, 0, b.T, b.max_ctx)]
        out, s, r = [], 0, 0
        segs = b.segs_host
        while s < len(segs):
            long = segs[s][2] > DECODE_SEG_ROWS
            e, r1, ctx = s, r, 1
            while e < len(segs) and (segs[e][2] > DECODE_SEG_ROWS) == long:
                ctx, r1, e = max(ctx, segs[e][1] + segs[e][2]), r1 + segs[e][2], e + 1
            out.append((long, s, e, r, r1, ctx))
            s, r = e, r1
        return out

    def _attend(self, run: int, a: LatentAttentionSpec, L: _Layer, q: torch.Tensor, down: torch.Tensor, b: BatchDesc,
                route: str) -> torch.Tensor:
        sc, T, H, kv = self.scratch, b.T, a.heads, self.kv[run]
        groups = self._segment_groups(L, b, route)
        out = sc.get("attn_out", (T, H * L.dv), self.act_dtype)
        q_lat = None
        if any(not g[0] for g in groups):
            q_lat = sc.get("lat_q_rows", (T, H, a.row_cols), self.act_dtype)
        q_out = None
        if any(g[0] for g in groups):
            q_out = q if q.dtype == torch.bfloat16 else sc.get("lat_q_bf", (T, H * L.qd), torch.bfloat16)
        LA.latent_post(down, q, L.kv_norm, L.freq, L.amp, kv, self.block_table, b.slot, b.pos, H, L.dn, a.rot_dim, a.kv_rank,
                       a.rank_cols, self.cfg.rms_eps, q_out=q_out, q_lat=q_lat)
        with self._stage("attn_core"):
            for long, s, e, r0, r1, ctx in groups:
                if long:
                    self._expanded(a, L, kv, q_out.view(T, H, L.qd), b, s, e, out)
                    continue
                for c0 in range(r0, r1, LATENT_ROWS):
                    self._latent_space(a, L, kv, q.unflatten(1, (H, L.qd)), q_lat, b, c0, min(r1, c0 + LATENT_ROWS), ctx, out)
        return out

    def _latent_space(self, a: LatentAttentionSpec, L: _Layer, kv: torch.Tensor, q: torch.Tensor, q_lat: torch.Tensor,
                      b: BatchDesc, r0: int, r1: int, ctx: int, out: torch.Tensor) -> None:
        """Rows r0..r1 against the cached latents themselves."""
        H, R, rank = a.heads, r1 - r0, a.rank_cols
        mul = (lambda x, w, o: K.small_gemm_f32(x, w, o)) if self.exact else K.gemv_float_batched
        ql, o_lat = q_lat[r0:r1], self.scratch.get("lat_o_rows", (R, H, rank), self.act_dtype)
        mul(q[r0:r1, :, :L.dn], L.uk_t, ql[:, :, :rank])
        args = (ql, kv, self.block_table, b.slot[r0:r1], b.ctx_len[r0:r1])
        if self.exact:
            LA.latent_exact(*args, o_lat, rank, a.scale, a.window, L.sink)
        else:
            plan = LA.decode_plan(min(ctx, a.window) if a.window else ctx, R, H, a.row_cols)
            part = self.scratch.get("attn_part", (plan.scratch_floats(R, H, rank),), torch.float32)
            LA.latent_decode(*args, part, o_lat, rank, a.scale, plan, a.window, L.sink)
        mul(o_lat, L.uv.data.view(H, L.dv, rank), out[r0:r1].view(R, H, L.dv))

    def _expanded(self, a: LatentAttentionSpec, L: _Layer, kv: torch.Tensor, q: torch.Tensor, b: BatchDesc, s: int, e: int,
                  out: torch.Tensor) -> None:
        """Segments s..e with full keys and values, expanded from the cache rows they can see."""
        from ..ops import gemm as GM
        segs, H = b.segs_host[s:e], a.heads
        keys, rows = LA.gathered_rows(segs, a.window), [n for _, _, n in segs]
        tc = LA.prefill_tc_ok(L.dn, L.qd, L.dv) and max(rows) >= TC_MIN_ROWS and a.scale > 0
        lat = self.scratch.get("lat_keys", (keys, a.row_cols), torch.bfloat16)
        LA.latent_gather(kv, self.block_table, b.seg_start[s:], b.seg_slot[s:], b.pos, e - s, a.window, lat)
        group = max(1, min(H, EXPANDED_KV_BYTES // (keys * (L.dn + L.dv) * 2)))
        c = lat[:, :a.rank_cols]
        for h0 in range(0, H, group):
            n = min(group, H - h0)
            uk, uv = L.uk.data[h0 * L.dn:(h0 + n) * L.dn], L.uv.data[h0 * L.dv:(h0 + n) * L.dv]
            kx = GM.gemm_bf16(c, uk, self.scratch.get("lat_kx", (keys, n * L.dn), torch.bfloat16))
            v = self.scratch.get("lat_v", (n * L.dv, keys) if tc else (keys, n * L.dv), torch.bfloat16)
            GM.gemm_bf16(*((uv, c) if tc else (c, uv)), v)
            LA.latent_prefill(q, kx, v, lat, b.seg_start[s:], b.pos, rows, out, H, h0, n, L.dn, L.dv, a.rank_cols, a.scale,
                              a.window, L.sink, transposed=tc)

    # ------------------------------------------------------------------ whole model
    def _embed(self, b: BatchDesc, h: torch.Tensor, copy: Optional[torch.Tensor]) -> None:
        K.embed(self.embed_w, b.tokens, h)

    def _layer_run(self, run: int, i: int, h: torch.Tensor, b: BatchDesc, route: str, journal: Optional[dict]) -> None:
        sc, T, L, a = self.scratch, b.T, self.layers[i], self.cfg.layer_specs[i].mixer
        xn, xs = (sc.get(n, (T, self.hp), self.act_dtype) for n in ("xn", "xn_shift"))
        with self._stage("norm"):
            K.norm_shift(h, L.gain, L.shift, self.conv_state[run], b.seg_start, b.seg_slot, b.tok_seg, xn, xs,
                         self.cfg.rms_eps, self.cfg.hidden, journal=None if journal is None else journal["conv"][run])
        with self._stage("in_gemm"):
            q, down, act = self._in_projections(L, a, xn, xs, route)
        attn = self._attend(run, a, L, q, down, b, route)
        with self._stage("out_gemm"):
            self._add_products(h, [(attn, L.o, L.s1)] + ([] if act is None else [(act, L.down, L.s2)]), route)
