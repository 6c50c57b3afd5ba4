"""Rows of ``families.py`` for Banelix: head rows with the convolution, the gated linear recurrence, attention with window, sink
and head gate, and the layer's products, beside the like kernels of the Sisisun decoder (same base, grouped-query attention)
and, for the recurrence, of the hybrid decoder's Gated-DeltaNet layers, at the layer sizes of an 8B-class model."""
from __future__ import annotations

from typing import Callable, Dict, List

import torch

from .families import _bf, _row, _variants, model_throughput
from .micro import time_launches

WIDTH, H, G, D, FF, C, BLOCKS, TAPS = 4096, 32, 8, 128, 14336, 4096, 16, 4
BC = C // BLOCKS


def _batch(T: int, decode: bool):
    from ..models.executor import make_batch
    return make_batch([(t, 4000, [0]) for t in range(T)] if decode else [(0, 0, [0] * T)], "cuda")


def _f32(*shape) -> torch.Tensor:
    return torch.randn(*shape, device="cuda")


def post_rows(T: int) -> List[Dict]:
    """The launch between input products and mixers, in both kinds of layer."""
    from ..models.config import BANELIX_8B
    from ..ops import kernels as K
    from ..ops import mixers as MX
    decode = T <= 16
    b, dt, es = _batch(T, decode), (torch.float32 if decode else torch.bfloat16), (4 if decode else 2)
    pages = max(T, 4000) // 16 + 2
    bt = (torch.arange(pages, dtype=torch.int32, device="cuda") + 1).repeat(max(T if decode else 1, 1), 1)
    out: List[Dict] = []
    q_out = torch.empty(T, H, D, device="cuda", dtype=torch.bfloat16)
    for both in (False, True):
        spec = BANELIX_8B.layer_specs[0 if both else 3].attention
        freq = torch.tensor(spec.rot.table()[0], dtype=torch.float64, device="cuda")
        nq, nk = H * D, G * D
        n_in = nq + nk + (2 * C if both else nk)
        # read: the rows that are used; write: queries, keys and values, the convolution's output
        nb = T * ((n_in - (C if both else 0)) * es + nq * 2 + 2 * nk * 2 + (C * (2 + 4 * (TAPS - 1) * decode) if both else 0))
        n = _variants(nb)
        rows = [torch.randn(T, n_in, device="cuda").to(dt) for _ in range(n)]
        kv = torch.empty(pages + 1, 2, G, 16, D, device="cuda", dtype=torch.bfloat16)
        bias, gain, conv = _f32(n_in), torch.ones(n_in, device="cuda"), None
        u = torch.empty((T, BLOCKS, BC) if decode else (BLOCKS, T, BC), device="cuda", dtype=torch.bfloat16)
        u = u if decode else u.transpose(0, 1)
        w, st = _f32(TAPS, C), torch.zeros(max(T, 1) if decode else 1, TAPS - 1, C, device="cuda")
        head = lambda r, c0, h: MX.HeadRows(r[:, c0:c0 + h * D], h, D, bias[c0:c0 + h * D], gain[c0:c0 + h * D])

        def new(i):
            r = rows[i]
            conv = MX.ConvRows(r[:, -C:], bias[-C:], w, bias[:C], u, st) if both else None
            MX.mixer_post(head(r, 0, H), head(r, nq, G), None if both else head(r, nq + nk, G), spec.qk_norm, spec.rot, freq, 1.0,
                          q_out, kv, 16, b, bt, 1e-6, conv)
        ms = time_launches(new, n)
        nw = torch.ones(D, device="cuda")
        like = lambda i: K.qkv_post(rows[i][:, :nq], rows[i][:, nq:nq + nk], rows[i][:, n_in - nk:], nw, nw, q_out, None, kv, bt,
                                    b.slot, b.pos, H, G, D, 16, False, 0, 1.0, 1e-6)
        lms = time_launches(like, n)
        lb = T * ((nq + 2 * nk) * es + nq * 2 + 2 * nk * 2)
        out.append(_row(f"head rows{' + convolution' if both else ''}, {T} tokens", "hbm", ms, nb, "qkv_post", lms, lb))
        del rows
    return out


def few_rows(R: int) -> List[Dict]:
    from ..ops import kernels as K
    from ..ops import mixers as MX
    out: List[Dict] = []
    x, nw, h = _f32(R, WIDTH), torch.ones(WIDTH, device="cuda"), torch.zeros(R, WIDTH, device="cuda")
    n_in = H * D + G * D + H + 2 * C
    nb = n_in * WIDTH * 2
    n = _variants(nb)
    ws, rows = [_bf(n_in, WIDTH) for _ in range(n)], torch.empty(R, n_in, device="cuda")
    n_like = (H + 2 * G) * D
    ms = time_launches(lambda i: K.gemv_float(x, [(ws[i], None, rows, K.EPI_F32)], norm_w=nw), n)
    lo = torch.empty(R, n_like, device="cuda")
    lms = time_launches(lambda i: K.gemv_float(x, [(ws[i][:n_like], None, lo, K.EPI_F32)], norm_w=nw), n)
    out.append(_row(f"input rows {R} x {n_in} x {WIDTH}", "hbm", ms, nb, f"gemv_float {n_like} rows", lms, n_like * WIDTH * 2))
    del ws
    nb = 2 * WIDTH * C * 2
    n = _variants(nb)
    wo, wr, s = [_bf(WIDTH, C) for _ in range(n)], [_bf(WIDTH, C) for _ in range(n)], torch.ones(WIDTH, device="cuda")
    o, o2 = (torch.randn(R, C, device="cuda").bfloat16() for _ in range(2))
    ms = time_launches(lambda i: K.gemv_sum(h, [(o, wo[i], s), (o2, wr[i], s)]), n)
    lms = time_launches(lambda i: K.gemv_sum(h, [(o, wo[i], None)]), n)
    out.append(_row(f"both output products {R} x {WIDTH} x {2 * C}", "hbm", ms, nb, "one output product", lms, nb // 2))
    del wo, wr
    nb = 2 * FF * WIDTH * 2
    n = _variants(nb)
    gu, act = [_bf(2 * FF, WIDTH) for _ in range(n)], torch.empty(R, FF, device="cuda", dtype=torch.bfloat16)
    run = lambda e: time_launches(lambda i: K.gemv_float(x, [(gu[i][:FF], gu[i][FF:], act, e)], norm_w=nw, limit=7.0), n)
    out.append(_row(f"gate/up SiLU {R} x {2 * FF} x {WIDTH}", "hbm", run(K.EPI_SILU_MUL), nb, "clamped GLU", run(K.EPI_CLAMPED_GLU), nb))
    del gu
    # one token of the recurrence beside one token of a Gated-DeltaNet layer (its two launches), every format its own bytes
    nb = 2 * C * BC * 2 + R * C * (2 + 4 * 2 + 2 + 4 * 2 + 4 * 2 * (TAPS - 1))
    n = _variants(nb)
    b, u = _batch(R, True), torch.randn(R, BLOCKS, BC, device="cuda").bfloat16()
    y, xr = rows[:, :C], rows[:, C:2 * C]
    ps = [MX.Recurrence(_bf(BLOCKS, 2 * BC, BC), _f32(BLOCKS, 2 * BC), -torch.rand(C, device="cuda"), _f32(C), _f32(C), TAPS)
          for _ in range(n)]
    S, cs = torch.zeros(R, C, device="cuda"), torch.zeros(R, TAPS - 1, C, device="cuda")
    ro = torch.empty(R, C, device="cuda", dtype=torch.bfloat16)
    ms = time_launches(lambda i: MX.rglru_step(ps[i], u, y, xr, S, cs, b, ro), n)
    Hv, Gk, Sd = 48, 16, 128
    cw = 2 * Gk * Sd + Hv * Sd
    lb = R * (Hv * Sd * Sd * 4 * 2 + cw * 4 * (2 * 3 + 2))
    ln = _variants(lb)
    xs, z = _f32(R, cw), _f32(R, Hv * Sd)
    ls, lc = [torch.zeros(R, Hv, Sd, Sd, device="cuda") for _ in range(ln)], torch.zeros(R, cw, 3, device="cuda")
    ab, one, q = _f32(R, Hv), torch.ones(Hv, device="cuda"), torch.empty(R, cw, device="cuda")
    dec, bet, og = torch.empty(R, Hv, device="cuda"), torch.empty(R, Hv, device="cuda"), torch.empty(R, Hv * Sd, device="cuda", dtype=torch.bfloat16)
    w4, nz = _f32(cw, 4), torch.ones(Sd, device="cuda")
    lms = time_launches(lambda i: K.gdn_decode(xs, w4, lc, ab, ab, -one, one, b.seg_slot, q, dec, bet, ls[i], z, nz, og, Gk, Hv, 1e-6), ln)
    out.append(_row(f"recurrence, one token of {R} requests, {C} channels", "hbm", ms, nb, "gdn_decode", lms, lb))
    return out


def recurrence_rows(T: int) -> List[Dict]:
    """Gate products and scan of a long portion."""
    from ..ops import gemm as GM
    from ..ops import kernels as K
    from ..ops import mixers as MX
    out: List[Dict] = []
    n = 3
    us, gw = [_bf(BLOCKS * T, BC) for _ in range(n)], _bf(BLOCKS, 2 * BC, BC)
    gates = [torch.randn(BLOCKS, T, 2 * BC, device="cuda") for _ in range(n)]
    tiles = torch.arange(BLOCKS, dtype=torch.int32, device="cuda").repeat_interleave(T // 128)
    ms = time_launches(lambda i: GM.gemm_bf16_grouped(us[i], gw.view(-1, BC), gates[i].view(-1, 2 * BC), BLOCKS, tiles), n)
    nb = T * C * (2 + 8) + 2 * C * BC * 2
    xl, wl = _bf(T, BC), _bf(2 * C, BC)
    lo = [torch.empty(T, 2 * C, device="cuda") for _ in range(n)]
    lms = time_launches(lambda i: GM.gemm_bf16(xl, wl, lo[i]), n)
    out.append(_row(f"gate products {T} x {BLOCKS} blocks x {2 * BC} x {BC}", "hbm", ms, nb, f"gemm_bf16 {T} x {2 * C} x {BC}, fp32 out", lms,
                    T * 2 * C * 4 + (T + 2 * C) * BC * 2))
    del lo
    rows = [_bf(T, 2 * C) for _ in range(n)]
    p = MX.Recurrence(gw, _f32(BLOCKS, 2 * BC), -torch.rand(C, device="cuda"), _f32(C), _f32(C), TAPS)
    S, cs, b = torch.zeros(1, C, device="cuda"), torch.zeros(1, TAPS - 1, C, device="cuda"), _batch(T, False)
    ro = torch.empty(T, C, device="cuda", dtype=torch.bfloat16)
    ms = time_launches(lambda i: MX.rglru_scan(p, gates[i].transpose(0, 1), us[i].view(BLOCKS, T, BC).transpose(0, 1),
                                               rows[i][:, :C], rows[i][:, C:], S, cs, b, ro), n)
    del gates, us, rows
    Hv, Gk, Sd = 48, 16, 128
    cw = 2 * Gk * Sd + Hv * Sd
    qs, o = [_f32(T, cw) for _ in range(n)], torch.empty(T, Hv, Sd, device="cuda")
    dec, bet = torch.rand(T, Hv, device="cuda"), torch.rand(T, Hv, device="cuda")
    st = torch.zeros(1, Hv, Sd, Sd, device="cuda")
    lms = time_launches(lambda i: K.gdn_scan_chunked(qs[i], dec, bet, st, b.seg_start, b.seg_slot, o, Gk, Hv), n)
    out.append(_row(f"recurrence scan {T} x {C}", "hbm", ms, T * C * (8 + 2 + 2 + 2), "gdn_scan_chunked", lms, T * (cw + Hv * Sd + 2 * Hv) * 4))
    return out


def products(M: int) -> List[Dict]:
    from ..models.executor import _Scratch
    from ..ops import gemm as GM
    few, sc = M <= 128, _Scratch(torch.device("cuda", torch.cuda.current_device()))
    out: List[Dict] = []
    s = torch.ones(WIDTH, device="cuda")
    for what, N, Kc, add in (("input rows", H * D + G * D + H + 2 * C, WIDTH, False), ("output, scaled add", WIDTH, C, True),
                             ("down, scaled add", WIDTH, FF, True)):
        n = _variants(N * Kc * 2)
        x, ws = _bf(M, Kc), [_bf(N, Kc) for _ in range(n)]
        h = torch.zeros(M, N, device="cuda")
        y = h if few else torch.empty(M, N, device="cuda", dtype=torch.bfloat16)
        if add:
            ms = time_launches((lambda i: GM.gemm_bf16_splitk_det(x, ws[i], h, sc, add=True, col_scale=s)) if few else
                               (lambda i: GM.gemm_bf16(x, ws[i], h, epi=GM.EPI_ADD, col_scale=s)), n)
            lms = time_launches((lambda i: GM.gemm_bf16_splitk_det(x, ws[i], h, sc, add=True)) if few else
                                (lambda i: GM.gemm_bf16(x, ws[i], h, epi=GM.EPI_ADD)), n)
            ln = N
        else:
            ln = (H + 2 * G) * D
            run = lambda k: time_launches((lambda i: GM.gemm_bf16_splitk_det(x, ws[i][:k], y[:, :k], sc)) if few else
                                          (lambda i: GM.gemm_bf16(x, ws[i][:k], y[:, :k])), n)
            ms, lms = run(N), run(ln)
        work = lambda k: k * Kc * 2 if few else 2.0 * M * k * Kc
        out.append(_row(f"{what} {M} x {N} x {Kc}", "hbm" if few else "bf16", ms, work(N), f"gemm_bf16 {ln} columns", lms, work(ln)))
        del ws
    GM.check_status()
    return out


def attention_prefill(T: int, window: int) -> Dict:
    from ..ops import attention as A
    pages, n = T // 16, 3
    q, out = _bf(T, H, D) * 20, torch.empty(T, H * D, device="cuda", dtype=torch.bfloat16)
    kv = [_bf(pages + 1, 2, G, 16, D) * 20 for _ in range(n)]
    bt = (torch.arange(pages, dtype=torch.int32, device="cuda") + 1)[None]
    b = _batch(T, False)
    sink, gate = torch.zeros(H, device="cuda"), _bf(T, H)
    kw = dict(window=window, sink=sink) if window else dict(head_gate=gate)
    run = lambda **k: time_launches(lambda i: A.flash_prefill_segs(q, None, kv[i], bt, b.seg_start, b.seg_slot, b.pos, [T], out, H, G, D,
                                                                   16, D ** -0.5, **k), n)
    full = 2.0 * T * T * H * D
    seen = 4.0 * H * D * sum(min(p + 1, window) for p in range(T)) if window else full
    return _row(f"flash prefill, {f'window {window} and sink' if window else 'head gate'}, T {T} heads {H}/{G} x {D}", "bf16",
                run(**kw), seen, "flash prefill, soft cap", run(softcap=50.0), full)


def attention_decode(ctx: int, R: int, window: int) -> Dict:
    from ..ops import kernels as K
    pages, span = ctx // 16, min(ctx, window or ctx)
    nb = R * span * 2 * G * D * 2
    n = _variants(nb)
    q, out = _bf(R, H, D) * 20, torch.empty(R, H * D, device="cuda", dtype=torch.bfloat16)
    kv = [_bf(R * pages + 1, 2, G, 16, D) * 20 for _ in range(n)]
    bt = (torch.arange(R * pages, dtype=torch.int32, device="cuda") + 1).view(R, pages)
    slot = torch.arange(R, dtype=torch.int32, device="cuda")
    kw = dict(window=window, sink=torch.zeros(H, device="cuda")) if window else dict(head_gate=_f32(R, H))

    def run(c: int, **k) -> float:
        cl = torch.full((R,), c, dtype=torch.int32, device="cuda")
        sl, ns = K.attn_decode_split(min(c, span), R, G)
        part = torch.empty(K.attn_decode_scratch_floats(R, H, ns, D), device="cuda")
        return time_launches(lambda i: K.attn_decode(q, None, kv[i], bt, slot, cl, part, out, H, G, D, 16, sl, ns, D ** -0.5, **k), n)
    ms, lms = run(ctx, **kw), run(span, softcap=50.0)
    K.check_status()
    return _row(f"decode attention, {f'window {window} and sink' if window else 'head gate'}, {R} x {ctx} heads {H}/{G} x {D}", "hbm", ms,
                nb, f"decode attention, soft cap, {R} x {span}", lms, nb)


def kernel_rows(emit: Callable[[Dict], None]) -> None:
    for T in (1, 8, 4096):
        for r in post_rows(T):
            emit(r)
    for R in (1, 8, 16):
        for r in few_rows(R):
            emit(r)
    for r in recurrence_rows(4096):
        emit(r)
    for M in (32, 4096):
        for r in products(M):
            emit(r)
    for T, w in ((4096, 0), (16384, 4096)):
        emit(attention_prefill(T, w))
    for ctx, R, w in ((4096, 1, 0), (32768, 1, 0), (4096, 16, 0), (32768, 1, 4096), (32768, 16, 4096)):
        emit(attention_decode(ctx, R, w))


def model_rows(emit: Callable[[Dict], None]) -> None:
    from ..models.config import BANELIX_8B, SISISUN_8B, banelix_config, sisisun_config
    m, d = BANELIX_8B, SISISUN_8B
    # eight layers each; two of Banelix's are windowed (the second on the keys and values of the first)
    new = banelix_config(m.hidden, 32768, m.layer_specs[:8], residual_mult=m.residual_mult, embed_scale=m.embed_scale)
    like = sisisun_config(d.hidden, 32768, d.layer_specs[:8])
    for cfg in (new, like):
        emit({"model": f"{cfg.hidden} wide, 8 layers", "family": cfg.arch, "weights": "bf16",
              **model_throughput(cfg, "bf16", rows=(1, 8, 16, 32))})
        torch.cuda.empty_cache()
