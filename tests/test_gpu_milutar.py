"""Milutar on the GPU: every mechanism against the plain fp32 equations, then whole models through the executor, the paged
cache, mixed batches, the engine and the trace replay, in bfloat16 and float32."""
import json
import os
import subprocess
import sys
from dataclasses import replace

import pytest
import torch

from hipengine_b200.ref import milutar as R

from milutar_models import (HEADS, LOOPED, MODELS, ODD, ONES, TOL, WIDE, build, full, last_logits, logit_error, model,
                            needle, tokens, windowed, with_windows)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF, F32 = torch.bfloat16, torch.float32


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


def _close(got, want, rel):
    got, want = got.float().cpu(), want.float().cpu()
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-6))
    assert err <= rel, err


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


# ----------------------------------------------------------------------------- row kernels and products
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("real,width", [(5, 8), (132, 136), (1500, 1504), (4096, 4096)])
def test_norm_and_shift_rows(real, width, dtype):
    """Segments of one to five rows on slots with and without a past; the state takes the last row, the journal every one."""
    from hipengine_b200.ops import kernels as K
    g, lens, slots = _gen(real), [1, 5, 2, 1, 3], [2, 0, 5, 4, 1]
    T = sum(lens)
    x, w, s, st = torch.zeros(T, width), torch.zeros(width), torch.zeros(width), torch.zeros(6, width)
    x[:, :real] = torch.randn(T, real, generator=g) * 2
    w[:real], s[:real] = 0.8, torch.randn(real, generator=g)
    st[[0, 2, 4], :real] = torch.randn(3, real, generator=g)
    start = [sum(lens[:i]) for i in range(len(lens) + 1)]
    h = R.rms(x[:, :real], 1e-5) * 0.8
    want = torch.cat([R.token_shift(h[a:b], st[c, :real], s[:real]) for a, b, c in zip(start, start[1:], slots)])
    args = (x.cuda(), w.cuda(), s.cuda())
    desc = (_i32(start), _i32(slots), _i32([i for i, n in enumerate(lens) for _ in range(n)]))
    for journal in (None, torch.full((T, width), 7.0, device="cuda")):
        state = st.cuda()
        hn, hs = (torch.full((T, width), 7.0, dtype=dtype, device="cuda") for _ in range(2))
        K.norm_shift(*args, state, *desc, hn, hs, 1e-5, real, journal=journal)
        tol = 1e-5 if dtype == F32 else 0.01
        _close(hn[:, :real], h, tol)
        _close(hs[:, :real], want, tol)
        assert not hn[:, real:].any() and not hs[:, real:].any()
        if journal is not None:
            assert torch.equal(state.cpu(), st)
            _close(journal[:, :real], h, 1e-5)
            continue
        for c, b in zip(slots, start[1:]):
            _close(state[c, :real], h[b - 1], 1e-5)
        assert torch.equal(state[3].cpu(), st[3]) and not state[:, real:].any()


@pytest.mark.parametrize("rows", [1, 3, 8, 9, 16])
def test_streaming_products(rows):
    """Squared ReLU, segments with rows of their own, one matrix per head, and the sum of two products."""
    from hipengine_b200.ops import kernels as K
    g = _gen(rows)
    r = lambda *s: torch.randn(*s, generator=g)
    x, y, w, v = r(rows, 72), r(rows, 72), r(37, 72).to(BF), r(50, 72).to(BF)
    a, b = torch.zeros(rows, 37, device="cuda"), torch.zeros(rows, 50, dtype=BF, device="cuda")
    for dt in (F32, BF):
        K.gemv_float(x.to(dt).cuda(), [(w.cuda(), None, a, K.EPI_F32), (v.cuda(), None, b, K.EPI_RELU2, y.to(dt).cuda())])
        _close(a, x @ w.float().t(), 0.02)
        _close(b, R.squared_relu(y @ v.float().t()), 0.03)
    # batches: strided rows of a wider buffer, more rows than one launch takes
    R_, B = rows * 3, 5
    wide, wb = r(R_, B * 40 + 8), r(B, 21, 24).to(BF)
    for dt in (F32, BF):
        src = wide.to(dt).cuda()[:, :B * 40].unflatten(1, (B, 40))[:, :, :24]
        out = torch.full((R_, B, 32), 3.0, dtype=dt, device="cuda")
        K.gemv_float_batched(src, wb.cuda(), out[:, :, :21])
        _close(out[:, :, :21], torch.einsum("rbk,bnk->rbn", wide[:, :B * 40].reshape(R_, B, 40)[:, :, :24], wb.float()), 0.02)
        assert bool((out[:, :, 21:] == 3.0).all())
    # sums
    h, s1, s2 = r(rows, 37), r(37), r(37)
    for parts in ([(x, w, s1)], [(x, w, s1), (r(rows, 104), r(37, 104).to(BF), s2)], [(x, w, None), (y, w, s2)]):
        want = h + sum((s if s is not None else 1.0) * (p.to(BF).float() @ q.float().t()) for p, q, s in parts)
        got = h.cuda()
        K.gemv_sum(got, [(p.to(BF).cuda(), q.cuda(), None if s is None else s.cuda()) for p, q, s in parts])
        _close(got - h.cuda(), want - h, 1e-4)


@pytest.mark.parametrize("M,N,Kc", [(200, 264, 136), (130, 100, 72), (40, 136, 200), (17, 64, 1024)])
def test_gemm_epilogues(M, N, Kc):
    from hipengine_b200.models.executor import _Scratch
    from hipengine_b200.ops import gemm as G
    from hipengine_b200.ops import kernels as K
    g = _gen(M)
    x, w, s, h = (torch.randn(*d, generator=g) for d in ((M, Kc), (N, Kc), (N,), (M, N)))
    x, w = (x / Kc ** 0.5).to(BF), w.to(BF)
    y = x.float() @ w.float().t()
    xc, wc, sc = x.cuda(), w.cuda(), s.cuda()
    scr = _Scratch(torch.device("cuda", 0))
    for split in (False, True):
        act, hc = torch.empty(M, N, dtype=BF, device="cuda"), h.cuda()
        if split:
            G.gemm_bf16_splitk_det(xc, wc, act, scr, relu2=True)
            G.gemm_bf16_splitk_det(xc, wc, hc, scr, add=True, col_scale=sc)
        else:
            G.gemm_bf16(xc, wc, act, epi=G.EPI_RELU2)
            G.gemm_bf16(xc, wc, hc, epi=G.EPI_ADD, col_scale=sc)
        G.check_status()
        _close(act, R.squared_relu(y), 0.01)
        _close(hc - h.cuda(), s * y, 1e-4)
    hc, act = h.cuda(), torch.empty(M, N, device="cuda")
    K.small_gemm_f32(x.float().cuda(), wc, hc, add=True, col_scale=sc)
    K.small_gemm_f32(x.float().cuda(), wc, act, mode=K.GEMM_RELU2)
    _close(hc - h.cuda(), s * y, 1e-4)
    _close(act, R.squared_relu(y), 1e-4)
    xb, wb = torch.randn(M, 3, Kc + 4, generator=g), torch.randn(3, N, Kc, generator=g).to(BF)
    out = torch.zeros(M, 3, N, device="cuda")
    K.small_gemm_f32(xb.cuda()[:, :, :Kc], wb.cuda(), out)
    _close(out, torch.einsum("rbk,bnk->rbn", xb[:, :, :Kc], wb.float()), 1e-4)


def test_embedding_rows_are_padded():
    from hipengine_b200.ops import kernels as K
    w = torch.randn(50, 12, generator=_gen()).to(BF)
    out = torch.full((3, 16), 7.0, device="cuda")
    K.embed(K.DeviceWeight(30, 50, 12, w.cuda()), torch.tensor([49, 0, 7], device="cuda"), out)
    assert torch.equal(out[:, :12].cpu(), w[[49, 0, 7]].float()) and not out[:, 12:].any()


# ----------------------------------------------------------------------------- cache write
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("rank,rd,heads,dim", [(5, 2, 1, 3), (44, 12, 9, 20), (512, 64, 3, 128), (72, 24, 17, 40)])
def test_cache_rows_and_rotated_queries(rank, rd, heads, dim, dtype):
    """Positions up to 262143: latent norm, rotation with an amplitude, page addressing, all padding written as zeros."""
    from hipengine_b200.models.config import LatentAttentionSpec, RotarySpec, YarnSpec
    from hipengine_b200.ops import latent as LA
    up8 = lambda n: -(-n // 8) * 8
    a = LatentAttentionSpec(heads, dim, rd, 8, rank, 1.0, RotarySpec(rd, 5000.0, YarnSpec(4.0, 512.0, 20.0, 1.5)))
    g, pos = _gen(rank), [0, 1, 15, 16, 4097, 262143]
    T, dn, qd = len(pos), up8(dim), up8(dim) + up8(rd)
    down, q = torch.randn(T, up8(rank + rd), generator=g) * 3, torch.zeros(T, heads, qd)
    q[:, :, :dim] = torch.randn(T, heads, dim, generator=g)
    q[:, :, dn:dn + rd] = torch.randn(T, heads, rd, generator=g)
    nw = torch.zeros(a.rank_cols)
    nw[:rank] = 1 + torch.rand(rank, generator=g)
    freq, amp = a.rot.table()
    f, am = R.rotation_freqs(rd, 5000.0, {"factor": 4.0, "original": 512.0, "fast": 20.0, "slow": 1.5})
    pt = torch.tensor(pos)
    want_lat, want_rot = R.rms(down[:, :rank], 1e-4) * nw[:rank], R.rotate_pairs(down[:, rank:rank + rd], pt, f, am)
    want_q = q.clone()
    want_q[:, :, dn:dn + rd] = R.rotate_pairs(q[:, :, dn:dn + rd], pt, f, am)
    n_pages = 6
    cache = torch.full((n_pages, 16, a.row_cols), 7.0, dtype=dtype, device="cuda")
    bt = torch.zeros(T, 262144 // 16, dtype=torch.int32)
    for t, p in enumerate(pos):
        bt[t, p // 16] = t
    q_in = q.reshape(T, -1).cuda() if dtype == F32 else q.reshape(T, -1).to(BF).cuda()
    q_out, q_lat = torch.full_like(q_in, 7.0), torch.full((T, heads, a.row_cols), 7.0, dtype=dtype, device="cuda")
    common = (nw.cuda(), torch.tensor(freq, dtype=torch.float64, device="cuda"), amp, cache, bt.cuda(),
              torch.arange(T, dtype=torch.int32, device="cuda"), _i32(pos), heads, dn, rd, rank, a.rank_cols, 1e-4)
    LA.latent_post(down.cuda(), q_in, *common, q_out=q_out, q_lat=q_lat)
    tol = 2e-5 if dtype == F32 else 0.01
    for t, p in enumerate(pos):
        row = cache[t, p % 16].cpu().float()
        _close(row[:rank], want_lat[t], tol)
        _close(row[a.rank_cols:a.rank_cols + rd], want_rot[t], tol)
        assert not row[rank:a.rank_cols].any() and not row[a.rank_cols + rd:].any()
        assert bool((cache[t, (p + 1) % 16] == 7.0).all())              # no other row of the page
    _close(q_out.view(T, heads, qd), want_q, tol)
    _close(q_lat[:, :, a.rank_cols:a.rank_cols + rd], want_q[:, :, dn:dn + rd], tol)
    assert bool((q_lat[:, :, :a.rank_cols] == 7.0).all()) and not q_lat[:, :, a.rank_cols + rd:].any()
    LA.latent_post(down.cuda(), q_in, *common, q_out=q_in)                    # in place
    assert torch.equal(q_in, q_out)


# ----------------------------------------------------------------------------- attention
def _latent_cache(ctxs, rank, rd, seed=0, dtype=BF, big=None):
    """Latents and rotated parts of requests of ``ctxs`` tokens in shuffled pages: (cache, block table, lat, rot)."""
    g = _gen(seed)
    rc = -(-rank // 16) * 16
    W = -(-(rc + rd) // 32) * 32
    pages = [-(-c // 16) for c in ctxs]
    ids = (torch.randperm(sum(pages), generator=g) + 1).tolist()
    cache = torch.zeros(sum(pages) + 1, 16, W)
    cache[0] = float("nan")                                                   # the null page is never attended to
    bt = torch.zeros(len(ctxs), max(pages) + 3, dtype=torch.int32)
    lats, rots = [], []
    for s, c in enumerate(ctxs):
        lat, rot = torch.randn(c, rank, generator=g).to(dtype).float(), torch.randn(c, rd, generator=g).to(dtype).float()
        if big is not None and big[s] is not None:
            lat[big[s]] = (lat[big[s]] * 6).to(dtype).float()
        for i in range(pages[s]):
            bt[s, i] = ids.pop()
            n = min(16, c - 16 * i)
            cache[bt[s, i], :n, :rank], cache[bt[s, i], :n, rc:rc + rd] = lat[16 * i:16 * i + n], rot[16 * i:16 * i + n]
        lats.append(lat)
        rots.append(rot)
    return cache.to(dtype).cuda(), bt.cuda(), lats, rots, rc, W


@pytest.mark.parametrize("exact", [False, True])
@pytest.mark.parametrize("window,sink", [(0, False), (0, True), (1, False), (16, True), (65, False), (130, False)])
@pytest.mark.parametrize("heads,rank,rd", [(1, 8, 2), (6, 72, 24), (17, 136, 8), (40, 264, 32), (3, 520, 72), (16, 512, 64),
                                           (33, 512, 64), (2, 1008, 20)])
def test_latent_space_attention(heads, rank, rd, window, sink, exact):
    """Contexts around tile, page and window edges, spans of one tile and of several; one key of every request stands out,
    so a window or a span that is one key off shows."""
    from hipengine_b200.ops import kernels as K
    from hipengine_b200.ops import latent as LA
    ctxs = [1, 2, 16, 17, 63, 64, 65, 129, 300, 131]
    big = [None if not window or c <= window else c - window - (i % 2) for i, c in enumerate(ctxs)]   # just in, just out
    dtype = F32 if exact else BF
    cache, bt, lats, rots, rc, W = _latent_cache(ctxs, rank, rd, heads + rank, dtype, big)
    g, n = _gen(1), len(ctxs)
    q, sk = torch.randn(n, heads, rank + rd, generator=g).to(dtype).float(), torch.randn(heads, generator=g) + 1
    scale = 1.5 / (rank + rd) ** 0.5
    eye = torch.eye(rank).repeat(heads, 1)
    want = torch.stack([R.latent_attention(q[s:s + 1], lats[s], rots[s], eye, eye, torch.tensor([c - 1]), heads, scale,
                                           window, sk if sink else None)[0] for s, c in enumerate(ctxs)]).view(n, heads, rank)
    ql = torch.zeros(n, heads, W)
    ql[:, :, :rank], ql[:, :, rc:rc + rd] = q[:, :, :rank], q[:, :, rank:]
    ql, slot, ctx = ql.to(dtype).cuda(), torch.arange(n, dtype=torch.int32, device="cuda"), _i32(ctxs)
    skc = sk.cuda() if sink else None
    out = torch.full((n, heads, rc), 7.0, dtype=dtype, device="cuda")
    if exact:
        LA.latent_exact(ql, cache, bt, slot, ctx, out, rc, scale, window, skc)
        _close(out[:, :, :rank], want, 1e-4)
        assert not out[:, :, rank:].any()
        return
    for spans, cluster, tile in ((1, 1, 64), (1, 1, 32), (3, 3, 64), (8, 8, 32), (5, 1, 64), (6, 2, 32), (16, 8, 32)):
        plan = LA.DecodePlan(spans, cluster, tile)
        part = torch.full((max(1, plan.scratch_floats(n, heads, rc)),), float("nan"), device="cuda")
        out.fill_(7.0)
        LA.latent_decode(ql, cache, bt, slot, ctx, part, out, rc, scale, plan, window, skc)
        K.check_status()
        _close(out[:, :, :rank], want, 0.02)
        assert not out[:, :, rank:].any()


@pytest.mark.parametrize("window,sink", [(0, True), (0, False), (1, True), (33, False), (40, True), (1000, False)])
@pytest.mark.parametrize("heads,dim,rd,dv,rank", [(3, 20, 12, 28, 44), (2, 64, 40, 64, 72), (4, 64, 64, 96, 64),
                                                  (2, 128, 64, 128, 136), (2, 150, 50, 136, 80), (1, 8, 2, 8, 16),
                                                  (3, 60, 18, 122, 48), (2, 128, 8, 64, 512)])
def test_expanded_attention(heads, dim, rd, dv, rank, window, sink):
    """Portions of several requests (different slots, pages and starts) in one launch, heads in groups, against the plain
    equations; the keys just inside and just outside a window stand out."""
    from hipengine_b200.ops import gemm as G
    from hipengine_b200.ops import latent as LA
    up8 = lambda n: -(-n // 8) * 8
    segs = [(2, 0, 300), (0, 37, 9), (1, 128, 270)]                           # slot, first position, rows
    ctxs = [46, 398, 300]
    cache, bt, lats, rots, rc, W = _latent_cache(ctxs, rank, rd, rank + dim, BF, [20, 140, 60])
    g, T = _gen(2), sum(n for _, _, n in segs)
    dn, dvp, qd = up8(dim), up8(dv), up8(dim) + up8(rd)
    q = torch.randn(T, heads, dim + rd, generator=g).to(BF).float()
    wk, wv = (torch.randn(heads * d, rank, generator=g).to(BF).float() / rank ** 0.5 for d in (dim, dv))
    wk, wv, sk = wk.to(BF).float(), wv.to(BF).float(), torch.randn(heads, generator=g) + 1
    scale, want, row = 1.5 / (dim + rd) ** 0.5, [], 0
    for s, p0, n in segs:
        want.append(R.latent_attention(q[row:row + n], lats[s][:p0 + n], rots[s][:p0 + n], wk, wv, torch.arange(p0, p0 + n),
                                       heads, scale, window, sk if sink else None))
        row += n
    qp = torch.zeros(T, heads, qd)
    qp[:, :, :dim], qp[:, :, dn:dn + rd] = q[:, :, :dim], q[:, :, dim:]
    uk, uv = torch.zeros(heads, dn, rc), torch.zeros(heads, dvp, rc)
    uk[:, :dim, :rank], uv[:, :dv, :rank] = wk.view(heads, dim, rank), wv.view(heads, dv, rank)
    uk, uv = (x.view(-1, rc).to(BF).cuda() for x in (uk, uv))
    starts = [0]
    for _, _, n in segs:
        starts.append(starts[-1] + n)
    pos = _i32([p for _, p0, n in segs for p in range(p0, p0 + n)])
    start, slot = _i32(starts), _i32([s for s, _, _ in segs])
    qc, skc = qp.to(BF).cuda(), sk.cuda() if sink else None

    def run(first, group, tc, out):
        """Segments first.. with ``group`` heads a launch."""
        sub = segs[first:]
        keys = LA.gathered_rows(sub, window)
        lat = torch.full((keys, W), float("nan"), dtype=BF, device="cuda")
        LA.latent_gather(cache, bt, start[first:], slot[first:], pos, len(sub), window, lat)
        at = 0
        for s, p0, n in sub:
            a = max(0, p0 - window + 1) if window else 0
            _close(lat[at:at + p0 + n - a, :rank], lats[s][a:p0 + n], 0.0)
            at += -(-(p0 + n - a) // 8) * 8
            assert not lat[at - (-(p0 + n - a) % 8):at].any()
        assert at == keys
        for h0 in range(0, heads, group):
            n = min(group, heads - h0)
            kx, v = torch.empty(keys, n * dn, dtype=BF, device="cuda"), torch.empty(keys * n * dvp, dtype=BF, device="cuda")
            v = v.view(n * dvp, keys) if tc else v.view(keys, n * dvp)
            G.gemm_bf16(lat[:, :rc], uk[h0 * dn:(h0 + n) * dn], kx)
            G.gemm_bf16(*((uv[h0 * dvp:(h0 + n) * dvp], lat[:, :rc]) if tc else (lat[:, :rc], uv[h0 * dvp:(h0 + n) * dvp])), v)
            LA.latent_prefill(qc, kx, v, lat, start[first:], pos, [n for _, _, n in sub], out, heads, h0, n, dn, dvp, rc, scale,
                              window, skc, transposed=tc)
        G.check_status()

    full_want = torch.cat(want).view(T, heads, dv)
    for tc in (False, True):
        if tc and not LA.prefill_tc_ok(dn, qd, dvp):
            continue
        for group in sorted({heads, 1}):
            out = torch.full((T, heads * dvp), 7.0, dtype=BF, device="cuda")
            run(0, group, tc, out)
            _close(out.view(T, heads, dvp)[:, :, :dv], full_want, 0.03)
            assert not out.view(T, heads, dvp)[:, :, dv:].any()
        out = torch.full((T, heads * dvp), 7.0, dtype=BF, device="cuda")
        run(1, heads, tc, out)                                                # the later segments alone
        assert bool((out[:300] == 7.0).all())
        _close(out[300:].view(T - 300, heads, dvp)[:, :, :dv], full_want[300:], 0.03)


def test_growing_scores_in_the_tensor_memory_form():
    """Scores that rise key by key by far more than the tolerated growth, then fall: the accumulators are rescaled on the way
    and the last keys weigh nothing, in both tiles of a pair."""
    from hipengine_b200.ops import latent as LA
    T, H, dn, dv, rc, W = 300, 2, 64, 64, 16, 32
    g = _gen(3)
    k = torch.cat([torch.linspace(0, 40, 200), torch.linspace(40, -40, 100)])
    q, kx, v = torch.zeros(T, H, 72), torch.zeros(T, H, dn), torch.randn(T, H, dv, generator=g).to(BF).float()
    q[:, 0, 0], q[:, 1, 0], kx[:, :, 0] = 1.0, -1.0, k[:, None]
    kx, lat = kx.to(BF).float(), torch.zeros(T, W)
    want = torch.zeros(T, H, dv)
    for h in range(H):
        s = (q[:, h, :dn] @ kx[:, h].t()) * 3.0
        want[:, h] = R.softmax_with_sink(s, R.visible_keys(torch.arange(T), T)) @ v[:, h]
    out = torch.zeros(T, H * dv, dtype=BF, device="cuda")
    keys = LA.gathered_rows([(0, 0, T)], 0)
    pad = lambda x: torch.cat([x, torch.zeros(keys - T, *x.shape[1:])])
    c = lambda x: x.to(BF).cuda()
    LA.latent_prefill(c(q), c(pad(kx.reshape(T, -1))), c(pad(v.reshape(T, -1)).t().contiguous()), c(pad(lat)), _i32([0, T]),
                      torch.arange(T, dtype=torch.int32, device="cuda"), [T], out, H, 0, H, dn, dv, rc, 3.0, transposed=True)
    from hipengine_b200.ops import kernels as K
    K.check_status()
    _close(out.view(T, H, dv), want, 0.02)


# ----------------------------------------------------------------------------- whole models
DTYPES = ["float32", "bfloat16"]


def _executor(cfg_json, dtype, seed=0, max_slots=4, max_context=320, **kw):
    from hipengine_b200.models import make_executor
    w, ref, t = build(cfg_json, seed)
    return make_executor(w, dtype=dtype, device="cuda", max_slots=max_slots, max_context=max_context, **kw), ref, t


def _run(ex, segs):
    """Logits of every row; slots that start at position 0 start without a past."""
    from hipengine_b200.models.executor import make_batch
    from hipengine_b200.ops import kernels as K
    for slot, p0, _ in segs:
        if p0 == 0:
            ex.reset_slot(slot)
    h = ex.forward(make_batch(segs, ex.device))
    out = ex.logits(h).clone()
    K.check_status()
    return out.cpu()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_layers_one_by_one(name, dtype):
    ex, ref, _ = _executor(MODELS[name], dtype)
    for n in (37, 11):                                                        # both sides of the switch of kernels
        ids = tokens(n, MODELS[name]["vocab"], 2)
        got, want = [], []
        ex.on_layer_run = lambda run, h: got.append(h.clone().cpu())
        _run(ex, [(0, 0, ids)])
        ref.forward_raw(torch.tensor(ids), ref.new_state(), want)
        assert len(got) == len(want) == len(ex.cfg.layer_runs())
        for g, w in zip(got, want):
            _close(g, w, 5e-5 if dtype == "float32" else 0.04)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_prompts_portions_and_single_tokens_agree(name, dtype):
    """Whole prompt, portions of several sizes down to two tokens, and token by token: each against the oracle."""
    ex, ref, _ = _executor(MODELS[name], dtype)
    ids = tokens(150, MODELS[name]["vocab"], 5)
    want = ref.forward(torch.tensor(ids))[0]
    assert logit_error(_run(ex, [(0, 0, ids)]), want) < TOL[dtype]
    for slot, sizes in ((1, [2] * 75), (2, [31, 1, 2, 64, 3, 17, 16, 9, 7]), (3, [140] + [1] * 10)):
        parts, at = [], 0
        for n in sizes:
            parts.append(_run(ex, [(slot, at, ids[at:at + n])]))
            at += n
        assert at == 150 and logit_error(torch.cat(parts), want) < TOL[dtype], sizes
    parts = [_run(ex, [(0, p, [ids[p]])]) for p in range(50)]
    assert logit_error(torch.cat(parts), want[:50]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_few_and_many_rows_meet_at_every_batch_size(dtype):
    """Row counts on both sides of every switch of kernels (1, 8, 16, 17, 128, 129 rows)."""
    ex, ref, _ = _executor(ODD, dtype)
    ids = tokens(140, ODD["vocab"], 6)
    want = ref.forward(torch.tensor(ids))[0]
    for n in (1, 2, 8, 9, 16, 17, 33, 127, 128, 129, 140):
        assert logit_error(_run(ex, [(0, 0, ids[:n])]), want[:n]) < TOL[dtype], n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_unequal_requests_in_one_batch(name, dtype):
    """Portions of some requests beside single tokens of others, in any order, against each request alone."""
    ex, ref, _ = _executor(MODELS[name], dtype)
    seqs = [tokens(n, MODELS[name]["vocab"], n) for n in (90, 23, 61, 130)]
    want = [ref.forward(torch.tensor(s))[0] for s in seqs]
    at = [0] * 4
    plan = [[(3, 40), (0, 1)], [(0, 50), (1, 2), (3, 1)], [(2, 17), (3, 33), (1, 1), (0, 1)], [(0, 1), (3, 1), (1, 1)],
            [(1, 19), (2, 1), (0, 2), (3, 55)], [(2, 43), (0, 35)]]
    for step in plan:
        segs = [(r, at[r], seqs[r][at[r]:at[r] + n]) for r, n in step]
        got, row = _run(ex, segs), 0
        for r, n in step:
            assert logit_error(got[row:row + n], want[r][at[r]:at[r] + n]) < TOL[dtype], (step, r)
            row += n
            at[r] += n
    assert at == [90, 23, 61, 130]


@pytest.mark.parametrize("dtype", DTYPES)
def test_expanded_heads_in_groups(dtype, monkeypatch):
    """A small bound on the expanded keys and values: the heads of a long portion go through in several launches."""
    from hipengine_b200.models import milutar as M
    monkeypatch.setattr(M, "EXPANDED_KV_BYTES", 150 * 2 * 200)
    ex, ref, _ = _executor(HEADS, dtype)
    ids = tokens(150, HEADS["vocab"], 5)
    assert logit_error(_run(ex, [(0, 0, ids)]), ref.forward(torch.tensor(ids))[0]) < TOL[dtype]


def _ask(ex, slot, ids, cut):
    """Logits of the last token: the first ``cut`` tokens in one portion, the rest in another."""
    if cut:
        _run(ex, [(slot, 0, ids[:cut])])
    return _run(ex, [(slot, cut, ids[cut:])])[-1:]


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_at_every_border(dtype):
    """A key that decides the logits sits at the first tokens, at page borders and next to the asking token; it is asked
    for from a prompt, from a long and a short portion and from a decoded token."""
    from hipengine_b200.models import make_executor
    w, ref, _ = needle(LOOPED, strength=2.0)
    ex = make_executor(w, dtype=dtype, device="cuda", max_slots=4, max_context=320)
    base = [3 + t for t in tokens(131, LOOPED["vocab"] - 3, 8)]
    base[130] = 1
    plain = last_logits(ref, base)
    for p in (0, 1, 15, 16, 17, 63, 64, 111, 112, 128, 129):
        ids = list(base)
        ids[p] = 2
        want = last_logits(ref, ids)
        assert logit_error(plain, want) > 5 * TOL[dtype]
        for cut in (0, 97, 128, 130):
            assert logit_error(_ask(ex, 0, ids, cut), want) < TOL[dtype], (p, cut)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [1, 2, 16, 33])
def test_key_at_the_window_edge(size, dtype):
    """Keys just inside and just outside a window, in prompts, portions and decoding.  (A model of windows only; the oracle
    with windows one token longer or shorter gives other logits, so an edge that is one off shows.)"""
    from hipengine_b200.models import make_executor
    cfg = model(96, 160, [(windowed(4, 24, 8, 40, 32, 0.2, size), 64), (windowed(3, 16, 4, 16, 48, 0.25, size), 0)])
    w, ref, t = needle(cfg)
    ex = make_executor(w, dtype=dtype, device="cuda", max_slots=4, max_context=320)
    longer = R.MilutarRef(with_windows(cfg, 1), t)
    base = [3 + x for x in tokens(120, 157, 8)]
    for last in (47, 48, 63, 90, 119):
        for d in (size - 1, size):                                            # distance of the key from the asking token
            ids = base[:last + 1]
            ids[last] = 1
            if d:
                ids[last - d] = 2
            want = last_logits(ref, ids)
            if d == size:
                assert logit_error(last_logits(longer, ids), want) > 4 * TOL[dtype]
            for cut in (0, last - 20, last - 2, last):
                assert logit_error(_ask(ex, 1, ids, cut), want) < TOL[dtype], (last, d, cut)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_beside_one_and_many_keys(dtype):
    """The sink counts once, at the first token as after hundreds, in both forms of attention."""
    from hipengine_b200.models import make_executor
    cfg = model(64, 96, [(full(4, 16, 8, 16, 24, 0.05, 32), 0)], mult=1.0)
    w, ref, t = build(cfg, 3)
    t["l0.mix.sink"][:] = torch.tensor([7.0, 6.0, -2.0, 8.0])
    from hipengine_b200.loading.folder_family import weights_from_tensors
    w, ref = weights_from_tensors(w.config, t), R.MilutarRef(cfg, t)
    none = R.MilutarRef(cfg, {**t, "l0.mix.sink": torch.full((4,), -1e30)})
    ex = make_executor(w, dtype=dtype, device="cuda", max_slots=2, max_context=320)
    ids = tokens(300, 96, 1)
    want = ref.forward(torch.tensor(ids))[0]
    for p in (0, 20, 299):
        assert logit_error(none.forward(torch.tensor(ids))[0][p:p + 1], want[p:p + 1]) > 2 * TOL[dtype]
    assert logit_error(_run(ex, [(0, 0, ids[:299])]), want[:299]) < TOL[dtype]
    assert logit_error(_run(ex, [(0, 299, ids[299:])]), want[299:]) < TOL[dtype]
    assert logit_error(torch.cat([_run(ex, [(1, p, [ids[p]])]) for p in range(40)]), want[:40]) < TOL[dtype]


def test_scratch_contents_do_not_matter():
    from hipengine_b200.ops import kernels as K
    for dtype in DTYPES:
        for cfg in (ODD, WIDE):
            ex, _, _ = _executor(cfg, dtype)
            ex.scratch.canaries = True
            ids = tokens(150, cfg["vocab"], 1)
            work = [[(0, 0, ids)], [(1, 0, ids[:20])], [(1, 20, ids[:3]), (0, 150, ids[:1])], [(1, 23, ids[:30]), (0, 151, [3])]]
            first = [_run(ex, s) for s in work]
            for t in list(ex.scratch.bufs.values()) + list(ex.scratch.retired):
                t.view(torch.uint8).fill_(0xFF)
            for a, b in zip(first, [_run(ex, s) for s in work]):
                assert torch.equal(a, b) and bool(torch.isfinite(b).all())
            assert not ex.scratch.check_canaries()
            K.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [3, 17, 40])
def test_decode_graphs_of_many_rows(rows, dtype):
    """Captured decode steps of up to 40 requests of unequal lengths, each against itself alone; the captures do not move
    the state of the requests."""
    from hipengine_b200.models.decode_graph import DecodeGraphRunner
    from hipengine_b200.ops import kernels as K
    ex, ref, _ = _executor(ODD, dtype, max_slots=rows, max_context=96)
    seqs = [tokens(6 + (7 * r) % 31, ODD["vocab"], r) for r in range(rows)]
    for r, s in enumerate(seqs):
        _run(ex, [(r, 0, s[:-4])])
    run = DecodeGraphRunner(ex, max_rows=rows)
    for k in range(4):
        run.set_rows(list(range(rows)), [s[len(s) - 4 + k] for s in seqs], [len(s) - 4 + k for s in seqs])
        run.step(rows, 64, greedy=False)
        K.check_status()
        got = run.logits[:rows].cpu()
        for r in range(0, rows, 5):
            want = ref.forward(torch.tensor(seqs[r][:len(seqs[r]) - 3 + k]))[0][-1:]
            assert logit_error(got[r:r + 1], want) < TOL[dtype], (k, r)
    assert run.stats["captures"] == 1 and run.stats["hits"] == 3


# ----------------------------------------------------------------------------- engine
def _greedy(ref, prompt, n):
    """Oracle greedy continuation and, per step, the margin of the winner."""
    st, out, margin = ref.new_state(), [], []
    lg, st = ref.forward(torch.tensor(prompt), st)
    for _ in range(n):
        top = lg[-1].topk(2).values
        margin.append(float(top[0] - top[1]) / float(lg[-1].std()))
        out.append(int(lg[-1].argmax()))
        lg, st = ref.forward(torch.tensor(out[-1:]), st)
    return out, margin


def _check_greedy(ref, prompts, got, n):
    for p, g in zip(prompts, got):
        want, margin = _greedy(ref, p, n)
        cut = next((i for i, m in enumerate(margin) if m < 1e-4), n)
        assert g[:cut] == want[:cut]


@pytest.mark.parametrize("policy,prefix", [("protect_decode", "off"), ("mixed", "off"), ("mixed", "radix")])
def test_greedy_generation_through_the_engine(policy, prefix):
    """More requests than slots, a pool that forces pages to be used again, prompt chunks beside decode steps, with and
    without state snapshots inside the prompts: the ids of the float32 engine are the oracle's."""
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(ODD, 3)
    prompts = [tokens(n, ODD["vocab"], 100 + n) for n in (40, 3, 21, 70, 1, 33)]
    prompts.append(prompts[3][:48] + prompts[0][:9])                          # shares 48 tokens with an earlier one
    base = EngineConfig()
    eng = replace(base, scheduler=replace(base.scheduler, policy=policy, max_prefill_chunk_tokens=13),
                  kv=replace(base.kv, pool_pages=20, snapshot_interval_tokens=16))
    with LLM(w, engine_config=eng, dtype="float32", max_active_requests=3, max_sequence_length=256,
             prefix_cache=prefix) as llm:
        got = llm.generate_token_ids(prompts, SamplingParams(max_tokens=14, ignore_eos=True))
        snap = llm.live_loop_snapshot()["runner"]
    _check_greedy(ref, prompts, got, 14)
    assert ("mixed" in str(snap["launch_census"])) == (policy == "mixed")
    assert (snap["snapshots_taken"] > 0) == (prefix != "off")


def test_prefix_reuse_brings_the_state_along():
    """A cached prefix is only usable with the previous-row state of its last token: the continuation of a reused prefix
    is the oracle's, from the device cache and from the cold tier."""
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(LOOPED, 4)
    a = tokens(50, LOOPED["vocab"], 9)
    other = [tokens(60, LOOPED["vocab"], 20 + i) for i in range(4)]
    prompts = [a, a[:48] + tokens(5, LOOPED["vocab"], 2), a[:33] + tokens(3, LOOPED["vocab"], 3)]
    base = EngineConfig()
    eng = replace(base, kv=replace(base.kv, pool_pages=12, snapshot_interval_tokens=16, cold_tier_bytes=64 << 20,
                                   cold_restore_prefill_tok_s=1.0))
    with LLM(w, engine_config=eng, dtype="float32", max_active_requests=1, max_sequence_length=128,
             prefix_cache="radix") as llm:
        for batch in (prompts, other, prompts):
            for p in batch:
                _check_greedy(ref, [p], llm.generate_token_ids([p], SamplingParams(max_tokens=6, ignore_eos=True)), 6)
        snap = llm.live_loop_snapshot()["runner"]
    assert snap["prefix_hit_tokens"] >= 48 + 32 and snap.get("cold_restored_blocks", 0) > 0


def test_bf16_generation_follows_its_own_logits(tmp_path):
    """The served precision from a checkpoint folder: generated ids are the argmax of the logits of the sequence so far (long
    decode over many pages); a seeded sampled run repeats and its log-probabilities are those of the oracle's logits."""
    from hipengine_b200.llm import LLM, SamplingParams
    from hipengine_b200.loading.safetensors_dir import write_tensors
    _, ref, t = build(LOOPED, 4)
    (tmp_path / "config.json").write_text(json.dumps(LOOPED))
    write_tensors(tmp_path / "model.safetensors", t)
    prompt = tokens(50, LOOPED["vocab"], 9)
    sampled = SamplingParams(max_tokens=8, temperature=0.8, seed=5, logprobs=True, top_logprobs=3)
    with LLM(str(tmp_path), max_active_requests=2, max_sequence_length=512) as llm:
        a = llm.generate_token_ids([prompt], SamplingParams(max_tokens=180, ignore_eos=True))[0]
        s = [llm.generate_detailed([prompt], sampled)[0] for _ in range(2)]
    assert len(a) == 180 and s[0].token_ids == s[1].token_ids
    want = ref.forward(torch.tensor(prompt + a))[0]
    agree = total = 0
    for i, tok in enumerate(a):
        row = want[len(prompt) - 1 + i]
        top = row.topk(2).values
        if float(top[0] - top[1]) > 0.15 * float(row.std()):          # decided positions
            total += 1
            agree += int(row.argmax()) == tok
    assert total > 20 and agree == total
    rows = ref.forward(torch.tensor(prompt + list(s[0].token_ids)))[0][len(prompt) - 1:]
    for row, lp in zip(rows, s[0].logprobs):
        assert abs(float(torch.log_softmax(row / 0.8, -1)[lp.token_id]) - lp.logprob) < 0.15


@pytest.mark.parametrize("provider", ["prompt_lookup", "ngram"])
def test_speculation_keeps_greedy_output(provider):
    """Rejected drafts leave neither cache rows nor a previous-row state behind."""
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(LOOPED, 4)
    prompt = (tokens(12, LOOPED["vocab"], 9) * 3)[:30]
    with LLM(w, dtype="float32", max_active_requests=2, max_sequence_length=256, speculative_mtp_serving="on",
             speculative_provider=provider) as llm:
        got = llm.generate_token_ids([prompt, prompt[:17]], SamplingParams(max_tokens=40, ignore_eos=True))
    _check_greedy(ref, [prompt, prompt[:17]], got, 40)


# ----------------------------------------------------------------------------- trace replay
def _replay(cfg_json, dtype, max_tokens, seed=0):
    from hipengine_b200.generation.gpu_runner import GpuRunner
    from hipengine_b200.generation.trace_replay import TraceReplay, trace_engine_config
    w, ref, _ = build(cfg_json, seed)
    return TraceReplay(GpuRunner(w, trace_engine_config(max_tokens, dtype))), ref


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "ones"])
def test_replay_reuses_pages_and_slots(name, dtype):
    """Nine requests through four slots and a pool for 192 tokens, interleaved, some paused, with decode-only steps (the
    graph path) between mixed ones; every wanted row against the request alone."""
    cfg = MODELS[name]
    rep, ref = _replay(cfg, dtype, 192)
    lens = [40, 7, 64, 30, 18, 50, 33, 2, 61]
    seqs = {f"r{i}": tokens(n, cfg["vocab"], 50 + i) for i, n in enumerate(lens)}
    want = {r: ref.forward(torch.tensor(s))[0] for r, s in seqs.items()}
    waiting, live, used = list(seqs), {}, 0
    rng = torch.Generator().manual_seed(0)
    steps = decode_steps = 0
    pages = lambda n: -(-n // 64) * 64
    while waiting or live:
        steps += 1
        if waiting and len(live) < 4 and used + pages(len(seqs[waiting[0]])) <= 192:
            r = waiting.pop(0)
            used += pages(len(seqs[r]))
            live[r] = 0
        single = steps % 3 == 0 and all(p > 0 for p in live.values())
        entries, check, end = [], [], []
        for r in list(live):
            left = len(seqs[r]) - live[r]
            if live[r] > 0 and not single and int(torch.randint(0, 4, (1,), generator=rng)) == 0:
                continue                                                # sits this step out
            n = 1 if single else min(left, int(torch.randint(1, 24, (1,), generator=rng)))
            a = live[r]
            entries.append({"id": r, "tokens": seqs[r][a:a + n], "want": list(range(n))})
            check.append((r, a, n))
            live[r] += n
            if live[r] == len(seqs[r]):
                end.append(r)
        decode_steps += single
        got, row = rep.step(entries, end), 0
        for r, a, n in check:
            assert logit_error(got[row:row + n], want[r][a:a + n]) < TOL[dtype], (r, a, n)
            row += n
        for r in end:
            used -= pages(len(seqs[r]))
            live.pop(r)
    assert decode_steps > 3 and rep.runner.graphs.stats["captures"] > 0
    rep.runner.pool.assert_conserved()
    assert rep.runner.pool.n_free == 192 // 16 and len(rep.runner.free_slots) == 4


def test_decoding_across_a_graph_bucket():
    """A context that grows past 1024 tokens while decoding: another captured graph with more spans takes over."""
    rep, ref = _replay(LOOPED, "bfloat16", 1152)
    ids = tokens(1060, LOOPED["vocab"], 3)
    want = ref.forward(torch.tensor(ids))[0]
    rep.step([{"id": "a", "tokens": ids[:1010], "want": []}])
    for p in range(1010, 1060):
        got = rep.step([{"id": "a", "tokens": [ids[p]], "want": [0]}])
        assert logit_error(got, want[p:p + 1]) < TOL["bfloat16"], p
    assert rep.runner.graphs.stats["captures"] == 2


def test_trace_run_program(tmp_path):
    """The program end to end on a checkpoint folder: protocol, files, exit code."""
    import numpy as np
    from hipengine_b200.loading.safetensors_dir import write_tensors
    _, ref, t = build(HEADS)
    folder, out = tmp_path / "m", tmp_path / "o"
    folder.mkdir()
    out.mkdir()
    (folder / "config.json").write_text(json.dumps(HEADS))
    write_tensors(folder / "model.safetensors", t)
    a, b = tokens(20, HEADS["vocab"], 1), tokens(5, HEADS["vocab"], 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": [0, 17]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[18:19], "want": []}, {"id": "b", "tokens": b, "want": [4, 0]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[19:], "want": [0]}], "end": ["a"]}]
    for dtype in DTYPES:
        p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                           capture_output=True, text=True, timeout=300)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        la, lb = ref.forward(torch.tensor(a))[0], ref.forward(torch.tensor(b))[0]
        for step, want in ((0, la[[0, 17]]), (1, lb[[4, 0]]), (2, la[[19]])):
            got = np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(-1, HEADS["vocab"])
            assert logit_error(torch.from_numpy(got.copy()), want) < TOL[dtype]
