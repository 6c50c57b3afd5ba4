"""Rows of ``families.py`` for Milutar: latent attention, token shift and the parallel layer's products beside the like kernels
of the Sisisun decoder (grouped-query attention, plain norm, plain products) at the layer sizes of an 8B-class model."""
from __future__ import annotations

from typing import Callable, Dict, List

import torch

from .families import _bf, _row, _variants, model_throughput
from .micro import time_launches

H, RANK, RD, DIM, VDIM, QRANK, WIDTH, FF = 32, 512, 64, 128, 128, 1536, 4096, 20480
W = RANK + RD


def _pages(ctx: int, R: int, n: int, W_: int):
    pages = -(-ctx // 16)
    cache = [_bf(R * pages + 1, 16, W_) for _ in range(n)]
    return cache, (torch.arange(R * pages, dtype=torch.int32, device="cuda") + 1).view(R, pages)


def norm_rows(T: int) -> Dict:
    from ..ops import kernels as K
    n = _variants(T * WIDTH * 8)
    x, w = [torch.randn(T, WIDTH, device="cuda") for _ in range(n)], torch.ones(WIDTH, device="cuda")
    st = torch.zeros(T, WIDTH, device="cuda")
    decode = T <= 16
    start = torch.arange(T + 1, dtype=torch.int32, device="cuda") if decode else torch.tensor([0, T], dtype=torch.int32, device="cuda")
    slot = torch.arange(T, dtype=torch.int32, device="cuda")
    seg = slot if decode else torch.zeros_like(slot)
    h, hs = (torch.empty(T, WIDTH, dtype=torch.bfloat16, device="cuda") for _ in range(2))
    ms = time_launches(lambda i: K.norm_shift(x[i], w, w, st, start, slot, seg, h, hs, 1e-6, WIDTH), n)
    lms = time_launches(lambda i: K.rmsnorm_rows(x[i], w, h), n)
    return _row(f"norm + token shift {T} x {WIDTH}", "hbm", ms, T * WIDTH * (16 if decode else 8), "norm", lms, T * WIDTH * 6)


def few_rows(R: int) -> List[Dict]:
    from ..ops import kernels as K
    out: List[Dict] = []
    x, y = (torch.randn(R, WIDTH, device="cuda").bfloat16() for _ in range(2))
    xf, nw = torch.randn(R, WIDTH, device="cuda"), torch.ones(WIDTH, device="cuda")
    n_in = H * (DIM + RD) + W
    nb = (n_in + FF) * WIDTH * 2
    n = _variants(nb)
    wa, wb = [_bf(n_in, WIDTH) for _ in range(n)], [_bf(FF, WIDTH) for _ in range(n)]
    a, act = torch.empty(R, n_in, device="cuda"), torch.empty(R, FF, device="cuda", dtype=torch.bfloat16)
    ms = time_launches(lambda i: K.gemv_float(x, [(wa[i], None, a, K.EPI_F32), (wb[i], None, act, K.EPI_RELU2, y)]), n)
    lms = time_launches(lambda i: K.gemv_float(xf, [(wa[i], None, a, K.EPI_F32)], norm_w=nw), n)
    out.append(_row(f"query, latent and squared-ReLU rows {R} x {n_in + FF} x {WIDTH}", "hbm", ms, nb, "gemv_float, norm fused",
                    lms, n_in * WIDTH * 2))
    del wa, wb
    nb = WIDTH * (H * VDIM + FF) * 2
    n = _variants(nb)
    wo, wd, s = [_bf(WIDTH, H * VDIM) for _ in range(n)], [_bf(WIDTH, FF) for _ in range(n)], torch.ones(WIDTH, device="cuda")
    h, o = torch.zeros(R, WIDTH, device="cuda"), torch.randn(R, H * VDIM, device="cuda").bfloat16()
    ms = time_launches(lambda i: K.gemv_sum(h, [(o, wo[i], s), (act, wd[i], s)]), n)
    lms = time_launches(lambda i: K.gemv_float(act, [(wd[i], None, h, K.EPI_ADD_F32)]), n)
    out.append(_row(f"both output products {R} x {WIDTH} x {H * VDIM + FF}", "hbm", ms, nb, "gemv_float, residual add", lms,
                    WIDTH * FF * 2))
    del wo, wd
    nb = H * RANK * DIM * 2
    n = _variants(nb)
    uk, uv, like = ([_bf(*d) for _ in range(n)] for d in ((H, RANK, DIM), (H, VDIM, RANK), (512, 4096)))
    q, ql = torch.randn(R, H, DIM, device="cuda"), torch.empty(R, H, W, device="cuda", dtype=torch.bfloat16)
    ol, ao = torch.randn(R, H, RANK, device="cuda").bfloat16(), torch.empty(R, H, VDIM, device="cuda", dtype=torch.bfloat16)
    lo, xb = torch.empty(R, 512, device="cuda"), torch.randn(R, WIDTH, device="cuda").bfloat16()
    lms = time_launches(lambda i: K.gemv_float(xb, [(like[i], None, lo, K.EPI_F32)]), n)
    for what, f in (("key map onto the queries", lambda i: K.gemv_float_batched(q, uk[i], ql[:, :, :RANK])),
                    ("value map behind the sum", lambda i: K.gemv_float_batched(ol, uv[i], ao))):
        out.append(_row(f"{what} {R} x {H} heads x {RANK} x {DIM}", "hbm", time_launches(f, n), nb, "gemv_float 512 x 4096", lms, nb))
    return out


def products(M: int) -> List[Dict]:
    from ..models.executor import _Scratch
    from ..ops import gemm as G
    few, sc = M <= 128, _Scratch(torch.device("cuda", torch.cuda.current_device()))
    out: List[Dict] = []
    s = torch.ones(WIDTH, device="cuda")
    for what, N, Kc, add in (("up, squared ReLU", FF, WIDTH, False), ("down, scaled add", WIDTH, FF, True),
                             ("output, scaled add", WIDTH, H * VDIM, True)):
        n = _variants(N * Kc * 2)
        x, ws = _bf(M, Kc), [_bf(N, Kc) for _ in range(n)]
        acc, bf = torch.zeros(M, N, device="cuda"), torch.empty(M, N, device="cuda", dtype=torch.bfloat16)
        if few:
            new = (lambda i: G.gemm_bf16_splitk_det(x, ws[i], acc, sc, add=True, col_scale=s)) if add else \
                (lambda i: G.gemm_bf16_splitk_det(x, ws[i], bf, sc, relu2=True))
            like = lambda i: G.gemm_bf16_splitk_det(x, ws[i], acc, sc, add=add)
        else:
            new = (lambda i: G.gemm_bf16(x, ws[i], acc, epi=G.EPI_ADD, col_scale=s)) if add else \
                (lambda i: G.gemm_bf16(x, ws[i], bf, epi=G.EPI_RELU2))
            like = (lambda i: G.gemm_bf16(x, ws[i], acc, epi=G.EPI_ADD)) if add else (lambda i: G.gemm_bf16(x, ws[i], bf))
        work = N * Kc * 2 if few else 2.0 * M * N * Kc
        out.append(_row(f"{what} {M} x {N} x {Kc}", "hbm" if few else "bf16", time_launches(new, n), work, "gemm_bf16",
                        time_launches(like, n), work))
        G.check_status()
    return out


def cache_write(T: int) -> Dict:
    from ..ops import kernels as K
    from ..ops import latent as LA
    qd, n = DIM + RD, _variants(T * H * (DIM + RD) * 2)
    few = T <= 16
    q = [torch.randn(T, H * qd, device="cuda").to(torch.float32 if few else torch.bfloat16) for _ in range(n)]
    down, nw = torch.randn(T, W, device="cuda"), torch.ones(RANK, device="cuda")
    freq = torch.rand(RD // 2, dtype=torch.float64, device="cuda")
    (cache,), bt = _pages(T, 1, 1, W)
    slot, pos = torch.zeros(T, dtype=torch.int32, device="cuda"), torch.arange(T, dtype=torch.int32, device="cuda")
    lat = torch.empty(T, H, W, dtype=torch.bfloat16, device="cuda") if few else None
    ms = time_launches(lambda i: LA.latent_post(down, q[i], nw, freq, 1.0, cache, bt, slot, pos, H, DIM, RD, RANK, RANK, 1e-6,
                                                q_out=None if few else q[i], q_lat=lat), n)
    nb = T * (W * 4 + W * 2 + H * RD * (6 if few else 4))
    G, D = 8, 128
    qkv = [torch.randn(T, (H + 2 * G) * D, device="cuda").to(q[0].dtype) for _ in range(n)]
    kv = torch.zeros(bt.numel() + 1, 2, G, 16, D, dtype=torch.bfloat16, device="cuda")
    qo, qn = torch.empty(T, H, D, dtype=torch.bfloat16, device="cuda"), torch.ones(D, device="cuda")
    lms = time_launches(lambda i: K.qkv_post(qkv[i][:, :H * D], qkv[i][:, H * D:(H + G) * D], qkv[i][:, (H + G) * D:], qn, qn, qo,
                                             None, kv, bt, slot, pos, H, G, D, 16, False, 0, 1.0, 1e-6), n)
    e = q[0].element_size()
    return _row(f"latent norm, rotation, page write, {T} rows", "hbm", ms, nb, "qkv_post", lms, T * ((H + 2 * G) * D * (e + 2)))


def attention_prefill(T: int, window: int = 0) -> List[Dict]:
    from ..ops import attention as A
    from ..ops import gemm as GM
    from ..ops import latent as LA
    n = 3
    cache, bt = _pages(T, 1, n, W)
    q, out = _bf(T, H, DIM + RD) * 20, torch.empty(T, H * VDIM, device="cuda", dtype=torch.bfloat16)
    start, slot = torch.tensor([0, T], dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    pos, lat = torch.arange(T, dtype=torch.int32, device="cuda"), torch.empty(T, W, device="cuda", dtype=torch.bfloat16)
    ukv, kx, v = _bf(H * (DIM + VDIM), RANK), [_bf(T, H * DIM) for _ in range(n)], [_bf(H * VDIM, T) for _ in range(n)]
    sink = torch.zeros(H, device="cuda")
    lat.zero_()
    ms, reg = (time_launches(lambda i: LA.latent_prefill(q, kx[i], v[i] if tc else v[i].view(T, -1), lat, start, pos, [T], out, H, 0,
                                                         H, DIM, VDIM, RANK, (DIM + RD) ** -0.5, window, sink, transposed=tc), n)
               for tc in (True, False))
    G, D = 8, 128
    pages = -(-T // 16)
    kvl, q2 = [_bf(pages + 1, 2, G, 16, D) * 20 for _ in range(n)], _bf(T, H, D) * 20
    lms = time_launches(lambda i: A.flash_prefill(q2, None, kvl[i], bt, 0, 0, out, H, G, D, 16, D ** -0.5, window), n)
    seen = float(T) * T / 2 if not window else float(window) * (T - window / 2)
    rows = [_row(f"expanded attention{form}, T {T} heads {H} x {DIM + RD}/{VDIM}" + (f" window {window}" if window else ""),
                 "bf16", t, 2.0 * seen * H * (DIM + RD + VDIM), "flash prefill", lms, 2.0 * seen * H * 2 * D)
            for form, t in (("", ms), (" (register form)", reg))]
    if not window:
        fl = 2.0 * T * H * (DIM + VDIM) * RANK
        def expand(i):
            GM.gemm_bf16(lat[:, :RANK], ukv[:H * DIM], kx[i])
            GM.gemm_bf16(ukv[H * DIM:], lat[:, :RANK], v[i])
        gm = time_launches(expand, n)
        x, w2 = _bf(T, 4096), _bf(4096, 4096)
        y = torch.empty(T, 4096, device="cuda", dtype=torch.bfloat16)
        lm = time_launches(lambda i: GM.gemm_bf16(x, w2, y), n)
        rows.append(_row(f"expansion of {T} latents to {H} x {DIM + VDIM}", "bf16", gm, fl, "gemm_bf16 4096 x 4096", lm,
                         2.0 * T * 4096 * 4096))
        xs, wid = torch.empty(T, W, device="cuda", dtype=torch.bfloat16), torch.arange(T, dtype=torch.int32, device="cuda")
        from ..ops import kernels as K
        src = [_bf(T, W) for _ in range(8)]
        rows.append(_row(f"gather of {T} cache rows", "hbm",
                         time_launches(lambda i: LA.latent_gather(cache[i], bt, start, slot, pos, 1, 0, lat), n), T * W * 4,
                         "moe_gather", time_launches(lambda i: K.moe_gather(src[i], wid, 1, xs), 8), T * W * 4))
    GM.check_status()
    return rows


def attention_decode(ctx: int, R: int, heads: int = H) -> Dict:
    from ..ops import kernels as K
    from ..ops import latent as LA
    n = _variants(R * ctx * W * 2)
    cache, bt = _pages(ctx, R, n, W)
    q, out = _bf(R, heads, W) * 20, torch.empty(R, heads, RANK, device="cuda", dtype=torch.bfloat16)
    slot, cl = torch.arange(R, dtype=torch.int32, device="cuda"), torch.full((R,), ctx, dtype=torch.int32, device="cuda")
    plan = LA.decode_plan(ctx, R, heads, W)
    part = torch.empty(plan.scratch_floats(R, heads, RANK), device="cuda")
    ms = time_launches(lambda i: LA.latent_decode(q, cache[i], bt, slot, cl, part, out, RANK, 0.07, plan), n)
    del cache
    G, D = max(1, heads // 4), 128
    nl = _variants(R * ctx * 2 * G * D * 2)
    kv = [_bf(bt.numel() + 1, 2, G, 16, D) * 20 for _ in range(nl)]
    q2, o2 = _bf(R, heads, D) * 20, torch.empty(R, heads * D, device="cuda", dtype=torch.bfloat16)
    s2, n2 = K.attn_decode_split(ctx, R, G)
    p2 = torch.empty(K.attn_decode_scratch_floats(R, heads, n2, D), device="cuda")
    lms = time_launches(lambda i: K.attn_decode(q2, None, kv[i], bt, slot, cl, p2, o2, heads, G, D, 16, s2, n2, D ** -0.5), nl)
    K.check_status()
    return _row(f"latent-space attention {R} x {ctx} heads {heads} x {W}", "hbm", ms, R * ctx * W * 2,
                f"decode attention {heads}/{G} x {D}", lms, R * ctx * 2 * G * D * 2)


def kernel_rows(emit: Callable[[Dict], None]) -> None:
    for T in (1, 8, 4096):
        emit(norm_rows(T))
    for R in (1, 8, 16):
        for r in few_rows(R):
            emit(r)
    for M in (32, 4096):
        for r in products(M):
            emit(r)
    for T in (1, 8, 4096):
        emit(cache_write(T))
    for T, w in ((4096, 0), (16384, 4096)):
        for r in attention_prefill(T, w):
            emit(r)
    for ctx, R, heads in ((4096, 1, 32), (32768, 1, 32), (4096, 16, 32), (8192, 64, 32), (32768, 1, 16), (8192, 8, 128)):
        emit(attention_decode(ctx, R, heads))


def model_rows(emit: Callable[[Dict], None]) -> None:
    from ..models.config import MILUTAR_8B, SISISUN_8B, LoopSpec, milutar_config, sisisun_config
    m, d = MILUTAR_8B, SISISUN_8B
    # eight layer runs each (two with full attention): six layers of which two run twice
    new = milutar_config(m.hidden, 32768, m.layer_specs[:6], LoopSpec(2, 4, 2), residual_mult=m.residual_mult)
    like = sisisun_config(d.hidden, 32768, d.layer_specs[:6], LoopSpec(2, 4, 2))
    for cfg in (new, like):
        emit({"model": f"{cfg.hidden} wide, 8 layer runs", "family": cfg.arch, "weights": "bf16",
              **model_throughput(cfg, "bf16", rows=(1, 8, 16, 32))})
        torch.cuda.empty_cache()
