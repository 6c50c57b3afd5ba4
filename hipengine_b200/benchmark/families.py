"""A family beside its closest existing one at equal size: kernel by kernel against the roofline, then whole models.

    python bench.py --beside sisisun|milutar|banelix|mepatar    # what this module prints, as one JSON line per row
    python -m hipengine_b200.benchmark.families [family] [--kernels-only | --models-only]

Each kernel row gives the new design's kernel and the like kernel of the closest model (Sisisun beside the Qwen3-shaped
dense / MoE decoder on the hybrid executor, Milutar, Banelix and Mepatar beside Sisisun, ``latent_rows.py``,
``recurrent_rows.py`` and ``linear_rows.py``), their device times and the fraction of the measured peak that bounds them: HBM for the weight or KV
streams (every format counts its own bytes), the bf16 tensor peak for the large products.  Operands are rotated through more
than the L2 holds.  Weights are random.
"""
from __future__ import annotations

import argparse
import json
import sys
from typing import Callable, Dict, List, Optional

import torch

from ..utils.nvml_sampler import NvmlSampler, decode_reasons
from .micro import peaks, time_launches

L2_POOL = 300e6


def _variants(nbytes: float) -> int:
    return max(2, min(64, int(L2_POOL // max(nbytes, 1)) + 1))


def _bf(*shape) -> torch.Tensor:
    return (torch.randn(*shape, device="cuda") * 0.05).bfloat16()


def _quant(rows: int, cols: int, n: int, qtype: str):
    from ..ops import kernels as K
    from ..quant import ggml as Q
    t = {"q4_k": Q.GGMLType.Q4_K, "q8_0": Q.GGMLType.Q8_0}[qtype]
    raw = torch.cat([Q.quantize(torch.randn(min(4096, rows - r), cols, device="cuda") * 0.02, t).reshape(-1)
                     for r in range(0, rows, 4096)]).reshape(rows, -1)
    return [K.to_device_weight(raw.clone(), t, rows, cols) for _ in range(n)], rows * Q.row_bytes(t, cols)


def _row(what: str, bound: str, new_ms: float, new_work: float, like: str, like_ms: float, like_work: float) -> Dict:
    """``work``: bytes (bound 'hbm') or FLOPs (bound 'bf16')."""
    pk = peaks()
    peak = pk["hbm_gbs"] * 1e9 if bound == "hbm" else pk["bf16_tflops"] * 1e12
    f_new, f_like = new_work / (new_ms * 1e-3) / peak, like_work / (like_ms * 1e-3) / peak
    return {"kernel": what, "bound": f"{pk['src']} {bound}", "us": round(new_ms * 1e3, 2), "frac": round(f_new, 3),
            "like": like, "like_us": round(like_ms * 1e3, 2), "like_frac": round(f_like, 3),
            "distance_ratio": round(f_like / f_new, 2)}


# ----------------------------------------------------------------------------- projections
def gemv_rows(N: int, Kc: int, R: int, pair: bool, qtype: str = "q8_0") -> Dict:
    from ..ops import kernels as K
    x, nw = torch.randn(R, Kc, device="cuda"), torch.ones(Kc, device="cuda")
    rows = 2 * N if pair else N
    nb = rows * Kc * 2
    n = _variants(nb)
    ws = [_bf(rows, Kc) for _ in range(n)]
    out = torch.empty(R, N, device="cuda", dtype=torch.bfloat16 if pair else torch.float32)
    if pair:
        new = lambda i: K.gemv_float(x, [(ws[i][:N], ws[i][N:], out, K.EPI_CLAMPED_GLU)], norm_w=nw, limit=7.0)
    else:
        new = lambda i: K.gemv_float(x, [(ws[i], None, out, K.EPI_F32)], norm_w=nw)
    ms = time_launches(new, n)
    del ws
    a, qb = _quant(N, Kc, _variants(nb // 2), qtype)
    b = _quant(N, Kc, len(a), qtype)[0] if pair else None
    if pair:
        like = lambda i: K.gemv(x, [K.GemvSegment(a[i], out, K.EPI_SILU_MUL, b[i])], norm_w=nw)
    else:
        like = lambda i: K.gemv(x, [K.GemvSegment(a[i], out)], norm_w=nw)
    lms = time_launches(like, len(a))
    return _row(f"gemv_float{' gate/up' if pair else ''} {R} x {rows} x {Kc}", "hbm", ms, nb, f"gemv[{qtype}]", lms,
                qb * (2 if pair else 1))


def gemm(M: int, N: int, Kc: int, qtype: str = "q8_0") -> Dict:
    from ..models.executor import _Scratch
    from ..ops import gemm as G
    x, sc = _bf(M, Kc), _Scratch(torch.device("cuda", torch.cuda.current_device()))
    n = _variants(N * Kc * 2)
    ws = [_bf(N, Kc) for _ in range(n)]
    few = M <= 128
    out = torch.empty(M, N, device="cuda", dtype=torch.float32 if few else torch.bfloat16)
    ms = time_launches((lambda i: G.gemm_bf16_splitk_det(x, ws[i], out, sc)) if few else
                       (lambda i: G.gemm_bf16(x, ws[i], out)), n)
    del ws
    q, qb = _quant(N, Kc, _variants(N * Kc), qtype)
    lms = time_launches((lambda i: G.gemm_quant_splitk(x, q[i], out, sc)) if few else
                        (lambda i: G.gemm_quant(x, q[i], out, sc)), len(q))
    G.check_status()
    w = (N * Kc * 2, qb) if few else (2.0 * M * N * Kc,) * 2
    return _row(f"gemm_bf16 {M} x {N} x {Kc}", "hbm" if few else "bf16", ms, w[0], f"gemm_quant[{qtype}]", lms, w[1])


# ----------------------------------------------------------------------------- attention
def attention_prefill(T: int, H: int, G: int, D: int, cap: float = 50.0) -> Dict:
    from ..ops import attention as A
    pages = -(-T // 16)
    q, out = _bf(T, H, D) * 20, torch.empty(T, H * D, device="cuda", dtype=torch.bfloat16)
    n = 3
    kv = [_bf(pages + 1, 2, G, 16, D) * 20 for _ in range(n)]
    bt = (torch.arange(pages, dtype=torch.int32, device="cuda") + 1)[None]
    start = torch.tensor([0, T], dtype=torch.int32, device="cuda")
    slot = torch.zeros(1, dtype=torch.int32, device="cuda")
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    ms = time_launches(lambda i: A.flash_prefill_segs(q, None, kv[i], bt, start, slot, pos, [T], out, H, G, D, 16,
                                                      D ** -0.5, softcap=cap), n)
    lms = time_launches(lambda i: A.flash_prefill(q, None, kv[i], bt, 0, 0, out, H, G, D, 16, D ** -0.5), n)
    fl = 2.0 * T * T * H * D
    return _row(f"flash prefill, soft cap, T {T} heads {H}/{G} x {D}", "bf16", ms, fl, "flash prefill", lms, fl)


def attention_decode(ctx: int, R: int, H: int, G: int, D: int, cap: float = 50.0) -> Dict:
    from ..ops import kernels as K
    pages = -(-ctx // 16)
    nb = R * ctx * 2 * G * D * 2
    n = _variants(nb)
    q, out = _bf(R, H, D) * 20, torch.empty(R, H * D, device="cuda", dtype=torch.bfloat16)
    kv = [_bf(R * pages + 1, 2, G, 16, D) * 20 for _ in range(n)]
    bt = (torch.arange(R * pages, dtype=torch.int32, device="cuda") + 1).view(R, pages)
    slot = torch.arange(R, dtype=torch.int32, device="cuda")
    cl = torch.full((R,), ctx, dtype=torch.int32, device="cuda")
    sl, ns = K.attn_decode_split(ctx, R, G)
    part = torch.empty(K.attn_decode_scratch_floats(R, H, ns, D), device="cuda")
    run = lambda c: time_launches(lambda i: K.attn_decode(q, None, kv[i], bt, slot, cl, part, out, H, G, D, 16, sl, ns,
                                                          D ** -0.5, softcap=c), n)
    ms, lms = run(cap), run(0.0)
    K.check_status()
    return _row(f"decode attention, soft cap, {R} x {ctx} heads {H}/{G} x {D}", "hbm", ms, nb, "decode attention", lms, nb)


# ----------------------------------------------------------------------------- experts
def experts_few(T: int, E: int, k: int, H: int, F: int, qtype: str = "q8_0") -> List[Dict]:
    from ..ops import kernels as K
    h, nw = torch.randn(T, H, device="cuda"), torch.ones(H, device="cuda")
    # every launch routes to other experts; the experts of one launch are distinct, so each selected one is read once
    n = max(4, min(16, E // (T * k))) if T * k <= E else 4
    ids = [torch.stack([torch.randperm(E, device="cuda")[:k] for _ in range(T)]).int() if T > 1 else
           ((torch.arange(k, device="cuda") + i * k) % E)[None].int() for i in range(n)]
    touched = sum(len(set(i.flatten().tolist())) for i in ids) / n
    wts = torch.full((T, k), 1.0 / k, device="cuda")
    gu, dn = _bf(E * 2 * F, H), _bf(E * H, F)
    rows = torch.empty(T * k, F, device="cuda", dtype=torch.bfloat16)
    ms1 = time_launches(lambda i: K.moe_gateup_float(h, nw, 1e-6, H, ids[i], wts, gu, E, rows), n)
    ms2 = time_launches(lambda i: K.moe_down_float(rows, ids[i], dn, E, h), n)
    del gu, dn
    (qg,), qb = _quant(E * F, H, 1, qtype)
    (qu,), _ = _quant(E * F, H, 1, qtype)
    l1 = time_launches(lambda i: K.moe_gateup_sel(h, nw, 1e-6, ids[i], wts, qg, qu, F, rows), n)
    (qd,), qdb = _quant(E * H, F, 1, qtype)
    l2 = time_launches(lambda i: K.moe_down_sel(rows, ids[i], wts, qd, H, h), n)
    return [_row(f"experts gate/up, {T} tokens top {k} of {E} x {F}", "hbm", ms1, touched * 2 * F * H * 2,
                 f"moe_gateup_sel[{qtype}]", l1, touched * 2 * qb / E),
            _row(f"experts down, {T} tokens top {k} of {E} x {F}", "hbm", ms2, touched * F * H * 2,
                 f"moe_down_sel[{qtype}]", l2, touched * qdb / E)]


def experts_many(T: int, E: int, k: int, H: int, F: int, qtype: str = "q8_0") -> Dict:
    from ..ops import gemm as G
    from ..ops import kernels as K
    ids = torch.stack([torch.randperm(E, device="cuda")[:k] for _ in range(T)]).int()
    bound = K.moe_sorted_rows_bound(T * k, E)
    pos = torch.empty(T * k, dtype=torch.int32, device="cuda")
    tiles = torch.empty(bound // 128, dtype=torch.int32, device="cuda")
    K.moe_group(ids, E, pos, tiles, torch.empty(4, dtype=torch.int32, device="cuda"))
    xs, out = _bf(bound, H), torch.empty(bound, 2 * F, device="cuda", dtype=torch.bfloat16)
    gu = _bf(E * 2 * F, H)
    ms = time_launches(lambda i: G.gemm_bf16_grouped(xs, gu, out, E, tiles), 2)
    del gu
    (qg,), _ = _quant(E * F, H, 1, qtype)
    (qu,), _ = _quant(E * F, H, 1, qtype)

    def like(i):
        G.gemm_quant_grouped(xs, qg, out[:, :F], E, tiles)
        G.gemm_quant_grouped(xs, qu, out[:, F:], E, tiles)
    lms = time_launches(like, 2)
    G.check_status()
    fl = 2.0 * T * k * 2 * F * H
    return _row(f"grouped experts gate/up, {T} tokens top {k} of {E} x {F}", "bf16", ms, fl, f"grouped[{qtype}]", lms, fl)


def small_ops(T: int, E: int, k: int, H: int) -> List[Dict]:
    """Routing, embedding and the pass input against the like small kernels: bytes moved over HBM."""
    from ..ops import kernels as K
    lg = torch.randn(T, E, device="cuda")
    ids, wts = torch.empty(T, k, dtype=torch.int32, device="cuda"), torch.empty(T, k, device="cuda")
    nb = T * (E * 4 + k * 8)
    out = [_row(f"group-limited router {T} x {E}", "hbm",
                time_launches(lambda i: K.moe_route_grouped(lg, k, ids, wts, E, 8, 4, 2.5), 4), nb, "softmax router",
                time_launches(lambda i: K.moe_route(lg, k, ids, wts), 4), nb)]
    tab = K.DeviceWeight(30, 32768, H, _bf(32768, H))
    tok, pos = torch.randint(0, 32768, (T,), device="cuda"), torch.arange(T, dtype=torch.int32, device="cuda")
    freq = torch.rand((H + 1) // 2, dtype=torch.float64, device="cuda")
    h, x0 = torch.empty(T, H, device="cuda"), torch.empty(T, H, device="cuda")
    out.append(_row(f"embedding + positions {T} x {H}", "hbm",
                    time_launches(lambda i: K.embed_sinusoid(tab, tok, pos, freq, h, x0), 4), T * H * 10, "embedding",
                    time_launches(lambda i: K.embed(tab, tok, h), 4), T * H * 6))
    step = torch.randn(H, device="cuda")
    out.append(_row(f"pass input {T} x {H}", "hbm", time_launches(lambda i: K.resid_inject(h, x0, step), 4), T * H * 12,
                    "residual add", time_launches(lambda i: K.resid_add_f32(h, x0), 4), T * H * 12))
    return out


def kernel_rows(emit: Callable[[Dict], None]) -> None:
    for R in (1, 4, 8):
        for N, Kc, pair in ((6144, 4096, False), (14336, 4096, True), (4096, 14336, False)):
            emit(gemv_rows(N, Kc, R, pair))
    for M, N, Kc in ((4096, 6144, 4096), (4096, 28672, 4096), (4096, 4096, 14336), (32, 6144, 4096), (32, 4096, 14336)):
        emit(gemm(M, N, Kc))
    for T, H, G, D in ((4096, 32, 8, 128), (4096, 16, 2, 64), (2048, 16, 4, 256)):
        emit(attention_prefill(T, H, G, D))
    for ctx, R, H, G, D in ((4096, 1, 32, 8, 128), (32768, 1, 32, 8, 128), (4096, 16, 32, 4, 128), (8192, 4, 16, 2, 64)):
        emit(attention_decode(ctx, R, H, G, D))
    for T in (1, 8):
        for r in experts_few(T, 128, 8, 2048, 768):
            emit(r)
    emit(experts_many(4096, 128, 8, 2048, 768))
    for r in small_ops(4096, 128, 8, 4096):
        emit(r)


# ----------------------------------------------------------------------------- whole models
def _geometries():
    from ..models.config import (SISISUN_8B, SISISUN_30B_MOE, LoopSpec, ModelConfig, sisisun_config)
    d, m = SISISUN_8B, SISISUN_30B_MOE
    # eight layer runs each: six layers of which two run twice, beside eight plain layers
    dense = sisisun_config(d.hidden, 32768, d.layer_specs[:6], LoopSpec(2, 4, 2))
    moe = sisisun_config(m.hidden, 32768, m.layer_specs[:6], LoopSpec(2, 4, 2))
    base = dict(n_layers=8, vocab=32768, head_dim=128, rope_dim=128, qk_norm=True)
    a, b = d.layer_specs[0], m.layer_specs[0]
    like_dense = ModelConfig(arch="qwen3", hidden=d.hidden, n_heads=a.mixer.heads, n_kv_heads=a.mixer.kv_heads,
                             ffn=a.mlp.ff, **base)
    like_moe = ModelConfig(arch="qwen3moe", hidden=m.hidden, n_heads=b.mixer.heads, n_kv_heads=b.mixer.kv_heads, ffn=0,
                           n_experts=b.mlp.experts, n_experts_used=b.mlp.top, expert_ffn=b.mlp.ff,
                           shared_ffn=b.mlp.shared_ff, **base)
    return (("dense 4096 wide, 8 layer runs", dense, like_dense), ("128 experts 2048 wide, 8 layer runs", moe, like_moe))


def model_throughput(cfg, recipe: str, prompt: int = 4096, steps: int = 64, rows=(1, 8)) -> Dict:
    from ..loading.synth import build_random_model
    from ..models import make_executor
    from ..models.decode_graph import DecodeGraphRunner
    from ..models.executor import make_batch
    from ..ops import kernels as K
    w = build_random_model(cfg, seed=0, device="cuda", recipe=recipe)
    ex = make_executor(w, device="cuda", max_slots=max(rows), max_context=prompt + 1024)
    del w
    torch.cuda.empty_cache()
    out: Dict = {"weight_bytes": sum(d.data.numel() * d.data.element_size() for d in
                                     {id(v): v for v in ex.dw.values()}.values())}
    b = make_batch([(0, 0, torch.randint(0, cfg.vocab, (prompt,)).tolist())], ex.device)
    ev = lambda: torch.cuda.Event(enable_timing=True)

    def timed(fn, n):
        for _ in range(3):
            fn()
        e0, e1 = ev(), ev()
        torch.cuda.synchronize()
        e0.record()
        for _ in range(n):
            fn()
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1) / n
    ms = timed(lambda: ex.forward(b), 5)
    out["prefill_ms"], out["prefill_tok_s"] = round(ms, 3), round(prompt / ms * 1e3, 1)
    run = DecodeGraphRunner(ex, max_rows=max(rows))
    for R in rows:
        run.set_rows(list(range(R)), [1] * R, [prompt] * R)
        ms = timed(lambda: run.step(R, prompt + steps + 8), steps)
        out[f"decode_ms_{R}"], out[f"decode_tok_s_{R}"] = round(ms, 4), round(R / ms * 1e3, 1)
    K.check_status()
    return out


def model_rows(emit: Callable[[Dict], None]) -> None:
    for what, cfg, like in _geometries():
        emit({"model": what, "family": "sisisun", "weights": "bf16", **model_throughput(cfg, "bf16")})
        torch.cuda.empty_cache()
        for recipe in ("q8_0", "q4_k_m"):
            emit({"model": what, "family": like.arch, "weights": recipe, **model_throughput(like, recipe)})
            torch.cuda.empty_cache()


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="families")
    ap.add_argument("family", nargs="?", default="sisisun", choices=["sisisun", "milutar", "banelix", "mepatar"])
    ap.add_argument("--kernels-only", action="store_true")
    ap.add_argument("--models-only", action="store_true")
    a = ap.parse_args(argv)

    def emit(r: Dict) -> None:
        print(json.dumps(r), flush=True)
    if a.family == "milutar":
        from . import latent_rows as rows
    elif a.family == "banelix":
        from . import recurrent_rows as rows
    elif a.family == "mepatar":
        from . import linear_rows as rows
    else:
        rows = sys.modules[__name__]
    with NvmlSampler(device_index=torch.cuda.current_device(), interval_s=0.02) as clocks:
        def emit_clocked(r: Dict) -> None:
            """The row with the clocks and throttle reasons sampled since the last one."""
            seen, clocks.samples = clocks.samples, clocks.samples[-1:]      # a short row falls back on the last sample
            mhz = sorted(s.sm_mhz for s in seen if s.sm_mhz is not None)
            reasons = sorted({n for s in seen for n in decode_reasons(s.reasons)})
            emit({**r, "sm_mhz": mhz[len(mhz) // 2] if mhz else None, "clock_reasons": reasons})
        if not a.models_only:
            rows.kernel_rows(emit_clocked)
        if not a.kernels_only:
            rows.model_rows(emit_clocked)
    return 0


if __name__ == "__main__":
    sys.exit(main())
