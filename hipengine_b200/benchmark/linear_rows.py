"""Rows of ``families.py`` for Mepatar: grouped norms with the input convolution, linear attention, attention over a window and the
first tokens, experts and the layer's products, beside the like kernels of the Sisisun decoder (same base, grouped-query attention,
experts), of Milutar (norm with a past row) and of the hybrid decoder (Gated-DeltaNet) at the layer sizes of an 8B-class model."""
from __future__ import annotations

from typing import Callable, Dict, List

import torch

from .families import _bf, _row, _variants, model_throughput
from .micro import time_launches

WIDTH, H, G, D, FF, TAPS, GROUPS = 4096, 32, 8, 128, 14336, 4, 8


def _batch(T: int, decode: bool):
    from ..models.executor import make_batch
    return make_batch([(t, 4000, [0]) for t in range(T)] if decode else [(0, 0, [0] * T)], "cuda")


def _f32(*shape) -> torch.Tensor:
    return torch.randn(*shape, device="cuda")


def norm_rows(T: int) -> Dict:
    from ..ops import kernels as K
    from ..ops import linear as LN
    decode = T <= 32
    n, b = _variants(T * WIDTH * 8), _batch(T, decode)
    x, w = [_f32(T, WIDTH) for _ in range(n)], torch.ones(WIDTH, device="cuda")
    cw, st, ls = _f32(TAPS, WIDTH), torch.zeros(T, TAPS - 1, WIDTH, device="cuda"), torch.zeros(T, WIDTH, device="cuda")
    a, p = (torch.empty(T, WIDTH, dtype=torch.bfloat16, device="cuda") for _ in range(2))
    ms = time_launches(lambda i: LN.norm_conv(x[i], w, w, cw, st, b, a, p, GROUPS, 1e-6, WIDTH), n)
    lms = time_launches(lambda i: K.norm_shift(x[i], w, w, ls, b.seg_start, b.seg_slot, b.tok_seg, a, p, 1e-6, WIDTH), n)
    return _row(f"norms + input convolution {T} x {WIDTH}", "hbm", ms, T * WIDTH * (8 + 8 * (TAPS - 1) * decode), "norm + token shift", lms,
                T * WIDTH * (16 if decode else 8))


def head_rows(T: int) -> Dict:
    from ..models.config import MEPATAR_8B
    from ..ops import kernels as K
    from ..ops import mixers as MX
    decode = T <= 32
    b, dt, es = _batch(T, decode), (torch.float32 if decode else torch.bfloat16), (4 if decode else 2)
    pages = max(T, 4000) // 16 + 2
    bt = (torch.arange(pages, dtype=torch.int32, device="cuda") + 1).repeat(max(T if decode else 1, 1), 1)
    spec = MEPATAR_8B.layer_specs[3].mixer
    freq, nq, nk = torch.tensor(spec.rot.table()[0], dtype=torch.float64, device="cuda"), H * D, G * D
    q_out, kv = torch.empty(T, H, D, device="cuda", dtype=torch.bfloat16), torch.empty(pages + 1, 2, G, 16, D, device="cuda", dtype=torch.bfloat16)
    nb = T * ((nq + 2 * nk) * es + nq * 2 + 2 * nk * 2)
    n = _variants(nb)
    rows, bias = [torch.randn(T, nq + 2 * nk, device="cuda").to(dt) for _ in range(n)], _f32(nq + 2 * nk)
    gq, gk, nw = _f32(H, D), _f32(D), torch.ones(D, device="cuda")
    head = lambda r, c0, h, g: MX.HeadRows(r[:, c0:c0 + h * D], h, D, bias[c0:c0 + h * D], g)
    ms = time_launches(lambda i: MX.mixer_post(head(rows[i], 0, H, gq), head(rows[i], nq, G, gk), head(rows[i], nq + nk, G, None), "head",
                                               spec.rot, freq, 1.0, q_out, kv, 16, b, bt, 1e-6), n)
    lms = time_launches(lambda i: K.qkv_post(rows[i][:, :nq], rows[i][:, nq:nq + nk], rows[i][:, nq + nk:], nw, nw, q_out, None, kv, bt,
                                             b.slot, b.pos, H, G, D, 16, False, 0, 1.0, 1e-6), n)
    return _row(f"head rows, {T} tokens", "hbm", ms, nb, "qkv_post", lms, nb)


def few_rows(R: int) -> List[Dict]:
    from ..ops import kernels as K
    out: List[Dict] = []
    xf, x, nw, h = _f32(R, WIDTH), torch.randn(R, WIDTH, device="cuda").bfloat16(), torch.ones(WIDTH, device="cuda"), torch.zeros(R, WIDTH, device="cuda")
    n_in, n_like = 2 * 16 * D + 2 * H * D + 2 * H, (H + 2 * G) * D       # the delta rule's rows
    nb = (n_in + 128) * WIDTH * 2
    n = _variants(nb)
    ws, rt = [_bf(n_in, WIDTH) for _ in range(n)], [_bf(128, WIDTH) for _ in range(n)]
    rows, lg = torch.empty(R, n_in, device="cuda"), torch.empty(R, 128, device="cuda")
    ms = time_launches(lambda i: K.gemv_float(x, [(ws[i], None, rows, K.EPI_F32), (rt[i], None, lg, K.EPI_F32, x)]), n)
    lo = torch.empty(R, n_like, device="cuda")
    lms = time_launches(lambda i: K.gemv_float(xf, [(ws[i][:n_like], None, lo, K.EPI_F32)], norm_w=nw), n)
    out.append(_row(f"input and router rows {R} x {n_in + 128} x {WIDTH}", "hbm", ms, nb, f"gemv_float {n_like} rows, norm fused", lms,
                    n_like * WIDTH * 2))
    del ws
    nb = 2 * FF * WIDTH * 2
    n = _variants(nb)
    gu, act = [_bf(2 * FF, WIDTH) for _ in range(n)], torch.empty(R, FF, device="cuda", dtype=torch.bfloat16)
    ms = time_launches(lambda i: K.gemv_float(x, [(gu[i][:FF], gu[i][FF:], act, K.EPI_GELU_MUL)]), n)
    lms = time_launches(lambda i: K.gemv_float(xf, [(gu[i][:FF], gu[i][FF:], act, K.EPI_CLAMPED_GLU)], norm_w=nw, limit=7.0), n)
    out.append(_row(f"gate/up GELU {R} x {2 * FF} x {WIDTH}", "hbm", ms, nb, "clamped GLU, norm fused", lms, nb))
    del gu
    nb = WIDTH * (H * D + FF) * 2
    n = _variants(nb)
    wo, wd, o, bias = [_bf(WIDTH, H * D) for _ in range(n)], [_bf(WIDTH, FF) for _ in range(n)], torch.randn(R, H * D, device="cuda").bfloat16(), _f32(WIDTH)
    ms = time_launches(lambda i: K.gemv_sum(h, [(o, wo[i], None), (act, wd[i], None)], bias), n)
    lms = time_launches(lambda i: K.gemv_sum(h, [(act, wd[i], None)]), n)
    out.append(_row(f"both output products + bias {R} x {WIDTH} x {H * D + FF}", "hbm", ms, nb, "one output product", lms, WIDTH * FF * 2))
    return out


def _linear_params(delta: bool, n_rows_extra: int = 0):
    from ..models.config import MEPATAR_8B
    from ..ops import linear as LN
    s = MEPATAR_8B.layer_specs[0 if delta else 1].mixer
    ck = s.kv_heads * s.dim
    p = LN.LinearParams(s, ck, 2 * ck, 2 * ck + s.heads * s.vdim)
    if delta:
        p.conv, p.rate, p.dt, p.gain = _f32(s.taps, s.conv_cols), torch.ones(s.heads, device="cuda"), _f32(s.heads), torch.ones(s.vdim, device="cuda")
    else:
        p.freq = torch.tensor(s.rot.table()[0], dtype=torch.float64, device="cuda")
        p.g1 = torch.tensor([d - 1 for d in s.decay], device="cuda")
        p.powers = LN.decay_powers(s.decay).cuda()
    return s, p, p.cz + s.heads * s.vdim


def step_rows(R: int) -> List[Dict]:
    """One token of R requests, beside the two launches of a Gated-DeltaNet layer with as many heads."""
    from ..models.executor import _Scratch
    from ..ops import kernels as K
    from ..ops import linear as LN
    out: List[Dict] = []
    sc, b = _Scratch("cuda"), _batch(R, True)
    Hv, Gk, Sd = 32, 16, 128
    cw = 2 * Gk * Sd + Hv * Sd
    lb = R * (Hv * Sd * Sd * 4 * 2 + cw * 4 * (2 * 3 + 2))
    ln = _variants(lb)
    xs, z = _f32(R, cw), _f32(R, Hv * Sd)
    ls, lc = [torch.zeros(R, Hv, Sd, Sd, device="cuda") for _ in range(ln)], torch.zeros(R, cw, 3, device="cuda")
    ab, one, q = _f32(R, Hv), torch.ones(Hv, device="cuda"), torch.empty(R, cw, device="cuda")
    dec, bet, og = torch.empty(R, Hv, device="cuda"), torch.empty(R, Hv, device="cuda"), torch.empty(R, Hv * Sd, device="cuda", dtype=torch.bfloat16)
    w4, nz = _f32(cw, 4), torch.ones(Sd, device="cuda")
    lms = time_launches(lambda i: K.gdn_decode(xs, w4, lc, ab, ab, -one, one, b.seg_slot, q, dec, bet, ls[i], z, nz, og, Gk, Hv, 1e-6), ln)
    for delta in (True, False):
        s, p, cols = _linear_params(delta)
        nb = R * (s.heads * s.dim * s.vcols * 8 + cols * 4 + s.heads * s.vcols * 2 + (s.conv_cols * s.taps * 4 if delta else 0))
        rows, abr = _f32(R, cols), _f32(R, 2 * s.heads)
        S = [torch.zeros(R, s.heads, s.dim, s.vcols, device="cuda") for _ in range(_variants(nb))]
        ring = torch.zeros(R, s.taps, s.conv_cols, device="cuda") if delta else None
        o = torch.empty(R, s.heads * s.vcols, device="cuda", dtype=torch.bfloat16)
        ms = time_launches(lambda i: LN.linear_attention(p, rows, abr, s.heads, S[i], ring, b, o, 1e-6, sc), len(S))
        out.append(_row(f"{'delta rule' if delta else 'retention'}, one token of {R} requests", "hbm", ms, nb, "gdn_decode", lms, lb))
    return out


def portion_rows(T: int) -> List[Dict]:
    """The three kernels of a long portion beside those of a Gated-DeltaNet layer; bytes: what enters and leaves the layer part."""
    from ..models.executor import _Scratch
    from ..ops import kernels as K
    from ..ops import linear as LN
    out: List[Dict] = []
    b, n = _batch(T, False), 3
    Hv, Gk, Sd = 32, 16, 128
    cw = 2 * Gk * Sd + Hv * Sd
    xs, conv = [_bf(T, cw) for _ in range(n)], torch.empty(T, cw, device="cuda")
    w4, cst, st = _f32(cw, 4), torch.zeros(1, cw, 3, device="cuda"), torch.zeros(1, Hv, Sd, Sd, device="cuda")
    dec, bet, a = torch.rand(T, Hv, device="cuda"), torch.rand(T, Hv, device="cuda"), _f32(T, Hv)
    one, o, z = torch.ones(Hv, device="cuda"), torch.empty(T, Hv, Sd, device="cuda"), _bf(T, Hv * Sd)
    og, nz = torch.empty(T, Hv * Sd, device="cuda", dtype=torch.bfloat16), torch.ones(Sd, device="cuda")

    def pre(i):
        K.conv1d(xs[i], w4, cst, b.seg_start, b.seg_slot, b.tok_seg, conv, cw)
        K.gdn_prepare(conv, a, a, -one, one, dec, bet, Gk, Hv, Sd)
    scan = lambda i: K.gdn_scan_chunked(conv, dec, bet, st, b.seg_start, b.seg_slot, o, Gk, Hv)
    norm = lambda i: K.gdn_gated_norm(o, z, nz, og, Hv, Sd, 1e-6)
    pre(0)
    like = {"prepare": (time_launches(pre, n), T * cw * 6), "scan": (time_launches(scan, n), T * (cw + Hv * Sd) * 4),
            "output": (time_launches(norm, n), T * Hv * Sd * 8)}
    names = {"prepare": "conv1d + gdn_prepare", "scan": "gdn_scan_chunked", "output": "gdn_gated_norm"}
    total = sum(t for t, _ in like.values())
    for delta in (True, False):
        s, p, cols = _linear_params(delta)
        rows, abr = [_bf(T, cols) for _ in range(n)], _f32(T, 2 * s.heads)
        S, ring = torch.zeros(1, s.heads, s.dim, s.vcols, device="cuda"), torch.zeros(1, s.taps, s.conv_cols, device="cuda") if delta else None
        res, sc = torch.empty(T, s.heads * s.vcols, device="cuda", dtype=torch.bfloat16), _Scratch("cuda")
        plans = [LN.plan(p, r, abr, s.heads, S, ring, b, res, 1e-6, sc) for r in rows]
        for a_, steps in plans:
            for st_ in steps:
                LN.launch(st_, a_)
        what, times = "delta rule" if delta else "retention", []
        planes, mats = T * s.kv_heads * s.dim * 8, T * s.heads * 64 * (4 if not delta else 8)
        nb = {"prepare": T * (s.conv_cols * 2 + s.heads * s.vcols * 2) + planes + mats,
              "scan": planes + mats + T * s.heads * s.vcols * 6, "output": T * s.heads * s.vcols * 8}
        for j, part in enumerate(("prepare", "scan", "output")):
            ms = time_launches(lambda i: LN.launch(plans[i][1][j], plans[i][0]), n)
            times.append(ms)
            out.append(_row(f"{what} {T} tokens, {part}", "hbm", ms, nb[part], names[part], *like[part]))
        out.append(_row(f"{what} {T} tokens, all three", "hbm", sum(times), T * (cols + s.heads * s.vcols) * 2, "the like kernels together",
                        total, T * (cw + 2 * Hv * Sd) * 2))
    return out


def expert_rows(T: int) -> List[Dict]:
    from ..ops import kernels as K
    E, k, W, F = 128, 8, 2048, 768
    h, x, nw = _f32(T, W), torch.randn(T, W, device="cuda").bfloat16(), torch.ones(W, device="cuda")
    n = max(4, min(16, E // (T * k)))
    ids = [torch.stack([torch.randperm(E, device="cuda")[:k] for _ in range(T)]).int() for _ in range(n)]
    touched = sum(len(set(i.flatten().tolist())) for i in ids) / n
    wts, gu = torch.full((T, k), 1.0 / k, device="cuda"), _bf(E * 2 * F, W)
    rows = torch.empty(T * k, F, device="cuda", dtype=torch.bfloat16)
    ms = time_launches(lambda i: K.moe_gateup_float(x, None, 1e-6, W, ids[i], wts, gu, E, rows, act="clamped_glu", limit=7.0), n)
    lms = time_launches(lambda i: K.moe_gateup_float(h, nw, 1e-6, W, ids[i], wts, gu, E, rows), n)
    nb = touched * 2 * F * W * 2
    return [_row(f"experts gate/up on prepared rows, {T} tokens top {k} of {E} x {F}", "hbm", ms, nb, "norm fused, SiLU", lms, nb)]


def router_rows(T: int) -> Dict:
    from ..ops import kernels as K
    E, k = 128, 8
    lg, ids, wts = _f32(T, E), torch.empty(T, k, dtype=torch.int32, device="cuda"), torch.empty(T, k, device="cuda")
    run = lambda m: time_launches(lambda i: K.moe_route(lg, k, ids, wts, mode=m), 4)
    nb = T * (E * 4 + k * 8)
    return _row(f"softmax router, scores as they are, {T} x {E}", "hbm", run(2), nb, "normalised", run(0), nb)


def products(M: int) -> List[Dict]:
    from ..models.executor import _Scratch
    from ..ops import gemm as GM
    few, sc = M <= 128, _Scratch(torch.device("cuda", torch.cuda.current_device()))
    out: List[Dict] = []
    bias = _f32(WIDTH)
    for what, N, Kc in (("retention input rows", 4 * H * D, WIDTH), ("output + bias", WIDTH, H * D), ("gate rows", 2 * H, WIDTH)):
        n = _variants(N * Kc * 2)
        x, ws = _bf(M, Kc), [_bf(N, Kc) for _ in range(n)]
        h = torch.zeros(M, N, device="cuda")
        work = lambda k: k * Kc * 2 if few else 2.0 * M * k * Kc
        if "bias" in what:
            ms = time_launches((lambda i: GM.gemm_bf16_splitk_det(x, ws[i], h, sc, add=True, col_bias=bias)) if few else
                               (lambda i: GM.gemm_bf16(x, ws[i], h, epi=GM.EPI_ADD, col_bias=bias)), n)
            lms, lk, like = time_launches((lambda i: GM.gemm_bf16_splitk_det(x, ws[i], h, sc, add=True)) if few else
                                          (lambda i: GM.gemm_bf16(x, ws[i], h, epi=GM.EPI_ADD)), n), N, "without bias"
        elif "gate" in what:
            if few:
                continue                                     # they ride in the input product
            ms = time_launches(lambda i: GM.gemm_bf16_splitk_det(x, ws[i], h, sc), n)
            r = _bf(128, Kc)
            lo = torch.empty(M, 128, device="cuda")
            lms, lk, like = time_launches(lambda i: GM.gemm_bf16(x, r, lo), n), 128, "router rows, 128 columns"
        else:
            y = h if few else torch.empty(M, N, device="cuda", dtype=torch.bfloat16)
            lk, like = (H + 2 * G) * D, "gemm_bf16 6144 columns"
            run = lambda k: time_launches((lambda i: GM.gemm_bf16_splitk_det(x, ws[i][:k], y[:, :k], sc)) if few else
                                          (lambda i: GM.gemm_bf16(x, ws[i][:k], y[:, :k])), n)
            ms, lms = run(N), run(lk)
        out.append(_row(f"{what} {M} x {N} x {Kc}", "hbm" if few else "bf16", ms, work(N), like, lms, work(lk)))
        del ws
    GM.check_status()
    return out


def attention_prefill(T: int, window: int, keep: int) -> Dict:
    from ..ops import attention as A
    pages, n = T // 16, 3
    q, out = _bf(T, H, D) * 20, torch.empty(T, H * D, device="cuda", dtype=torch.bfloat16)
    kv = [_bf(pages + 1, 2, G, 16, D) * 20 for _ in range(n)]
    bt = (torch.arange(pages, dtype=torch.int32, device="cuda") + 1)[None]
    b = _batch(T, False)
    run = lambda **k: time_launches(lambda i: A.flash_prefill_segs(q, None, kv[i], bt, b.seg_start, b.seg_slot, b.pos, [T], out, H, G, D,
                                                                   16, D ** -0.5, **k), n)
    seen = 4.0 * H * D * sum(min(p + 1, window + min(keep, max(0, p + 1 - window))) for p in range(T))
    return _row(f"flash prefill, window {window} and {keep} first tokens, T {T} heads {H}/{G} x {D}", "bf16", run(window=window, keep_first=keep),
                seen, "flash prefill, soft cap", run(softcap=50.0), 2.0 * T * T * H * D)


def attention_decode(ctx: int, R: int, window: int, keep: int) -> Dict:
    from ..ops import kernels as K
    pages, span = ctx // 16, min(ctx, window + keep)
    nb = R * span * 2 * G * D * 2
    n = _variants(nb)
    q, out = _bf(R, H, D) * 20, torch.empty(R, H * D, device="cuda", dtype=torch.bfloat16)
    kv = [_bf(R * pages + 1, 2, G, 16, D) * 20 for _ in range(n)]
    bt = (torch.arange(R * pages, dtype=torch.int32, device="cuda") + 1).view(R, pages)
    slot = torch.arange(R, dtype=torch.int32, device="cuda")

    def run(c: int, **k) -> float:
        cl = torch.full((R,), c, dtype=torch.int32, device="cuda")
        sl, ns = K.attn_decode_split(min(c, span), R, G)
        part = torch.empty(K.attn_decode_scratch_floats(R, H, ns, D), device="cuda")
        return time_launches(lambda i: K.attn_decode(q, None, kv[i], bt, slot, cl, part, out, H, G, D, 16, sl, ns, D ** -0.5, **k), n)
    ms, lms = run(ctx, window=window, keep_first=keep), run(span, softcap=50.0)
    K.check_status()
    return _row(f"decode attention, window {window} and {keep} first tokens, {R} x {ctx} heads {H}/{G} x {D}", "hbm", ms, nb,
                f"decode attention, soft cap, {R} x {span}", lms, nb)


def kernel_rows(emit: Callable[[Dict], None]) -> None:
    for T in (1, 8, 32, 4096):
        emit(norm_rows(T))
    for T in (1, 8, 4096):
        emit(head_rows(T))
    for R in (1, 8, 16):
        for r in few_rows(R):
            emit(r)
    for R in (1, 8, 32):
        for r in step_rows(R):
            emit(r)
    for r in portion_rows(4096):
        emit(r)
    for T in (1, 8):
        for r in expert_rows(T):
            emit(r)
    emit(router_rows(4096))
    for M in (32, 4096):
        for r in products(M):
            emit(r)
    for T, w, k in ((4096, 4096, 128), (16384, 4096, 128)):
        emit(attention_prefill(T, w, k))
    for ctx, R, w, k in ((4096, 1, 4096, 128), (32768, 1, 4096, 128), (32768, 16, 4096, 128)):
        emit(attention_decode(ctx, R, w, k))


def model_rows(emit: Callable[[Dict], None]) -> None:
    from ..models.config import MEPATAR_30B_MOE, MEPATAR_8B, SISISUN_30B_MOE, SISISUN_8B, mepatar_config, sisisun_config
    for what, m, d in (("dense", MEPATAR_8B, SISISUN_8B), ("experts", MEPATAR_30B_MOE, SISISUN_30B_MOE)):
        # eight layers each: three delta, three retention and two attention layers (dense), 4 / 2 / 2 (experts)
        new = mepatar_config(m.hidden, 32768, m.layer_specs[:8], norm_groups=m.norm_groups, embed_scale=m.embed_scale)
        like = sisisun_config(d.hidden, 32768, d.layer_specs[:8])
        for cfg in (new, like):
            emit({"model": f"{what}, {cfg.hidden} wide, 8 layers", "family": cfg.arch, "weights": "bf16",
                  **model_throughput(cfg, "bf16", rows=(1, 8, 16, 32))})
            torch.cuda.empty_cache()
