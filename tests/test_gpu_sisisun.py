"""Sisisun on the GPU: every mechanism against the plain fp32 equations, then whole models through the executor, the paged
cache, mixed batches, the engine and the trace replay, in bfloat16 and float32."""
import json
import os
import subprocess
import sys
from dataclasses import replace

import pytest
import torch

from hipengine_b200.ref import sisisun as R

from sisisun_models import (HEADS, LOOPED, MODELS, TOL, WIDE, attn, build, dense, logit_error, model, needle, tokens)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


def _close(got, want, rel):
    got, want = got.float().cpu(), want.float().cpu()
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-6))
    assert err <= rel, err


# ----------------------------------------------------------------------------- kernels
@pytest.mark.parametrize("rows", [1, 2, 7, 8, 9, 16])
@pytest.mark.parametrize("n,k,real", [(16, 8, 8), (40, 72, 65), (301, 320, 320), (1024, 2056, 2050)])
def test_streaming_gemv(rows, n, k, real):
    from hipengine_b200.ops import kernels as K
    g = _gen(rows * n + k)
    x = torch.zeros(rows, k)
    x[:, :real] = torch.randn(rows, real, generator=g) * 3
    nw = torch.zeros(k)
    nw[:real] = 1 + 0.3 * torch.randn(real, generator=g)
    w = (torch.randn(2 * n, k, generator=g) / k ** 0.5).to(torch.bfloat16)
    xc, wc, nc = x.cuda(), w.cuda(), nw.cuda()
    xn = R.rms_norm(x[:, :real], nw[:real], 1e-5)
    want = xn @ w[:, :real].float().t()
    out = torch.full((rows, 2 * n + 3), 7.0, device="cuda")
    other = torch.zeros(rows, n, dtype=torch.bfloat16, device="cuda")
    K.gemv_float(xc, [(wc, None, out[:, :2 * n], K.EPI_F32), (wc[n:], None, other, K.EPI_BF16)], norm_w=nc, eps=1e-5,
                 norm_n=real)
    _close(out[:, :2 * n], want, 0.02)
    assert bool((out[:, 2 * n:] == 7.0).all())
    _close(other, want[:, n:], 0.02)
    # residual add from bf16 rows, and the three gated activations
    xb = x.to(torch.bfloat16)
    acc = torch.ones(rows, n, device="cuda")
    K.gemv_float(xb.cuda(), [(wc[:n], None, acc, K.EPI_ADD_F32)])
    _close(acc, 1 + xb.float() @ w[:n].float().t(), 0.01)
    for act, f in (("silu", R.silu_glu), ("clamped_glu", lambda a, b: R.clamped_glu(a, b, 0.6)),
                   ("gelu_tanh", lambda a, b: torch.nn.functional.gelu(a, approximate="tanh") * b)):
        y = torch.zeros(rows, n, dtype=torch.bfloat16, device="cuda")
        K.gemv_float(xc, [(wc[:n], wc[n:], y, K.EPI_OF_ACT[act])], norm_w=nc, eps=1e-5, norm_n=real, limit=0.6)
        _close(y, f(want[:, :n], want[:, n:]), 0.02)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_clamped_activation_rows(dtype):
    from hipengine_b200.ops import kernels as K
    gu = (torch.randn(5, 48, generator=_gen()) * 4).to(dtype)
    want = R.clamped_glu(gu.float()[:, :24], gu.float()[:, 24:], 1.3)
    for out_dtype in ([torch.bfloat16] if dtype == torch.bfloat16 else [torch.bfloat16, torch.float32]):
        out = torch.empty(5, 24, dtype=out_dtype, device="cuda")
        K.act_mul(gu.cuda(), out, "clamped_glu", 1.3)
        _close(out, want, 1e-5 if out_dtype == torch.float32 else 0.01)


@pytest.mark.parametrize("experts,top,groups,keep,scale", [(12, 3, 4, 2, 1.6), (9, 2, 9, 5, 0.7), (8, 8, 1, 1, 1.0),
                                                           (16, 1, 4, 1, 2.5), (192, 8, 8, 3, 2.5), (640, 32, 40, 20, 3)])
def test_group_limited_router(experts, top, groups, keep, scale):
    from hipengine_b200.ops import kernels as K
    T = 67
    z = torch.randn(T, experts + 3, generator=_gen(experts)) * 2
    ids = torch.empty(T, top, dtype=torch.int32, device="cuda")
    wts = torch.empty(T, top, device="cuda")
    K.moe_route_grouped(z.cuda(), top, ids, wts, experts, groups, keep, scale)
    for t in range(T):
        want_ids, want_w = R.route(z[t, :experts], top, groups, keep, scale)
        assert ids[t].tolist() == want_ids
        assert torch.allclose(wts[t].cpu(), torch.tensor(want_w), rtol=1e-5, atol=1e-7)


def test_embedding_with_positions():
    from hipengine_b200.ops import kernels as K
    w = torch.randn(50, 45, generator=_gen()).to(torch.bfloat16)
    dw = K.DeviceWeight(30, 50, 45, w.cuda())
    pos = torch.tensor([0, 1, 2, 1000, 131071, 262143], dtype=torch.int32)
    ids = torch.tensor([3, 49, 0, 7, 7, 11])
    freq = torch.pow(torch.tensor(10000.0, dtype=torch.float64), -2.0 * torch.arange(23, dtype=torch.float64) / 45)
    out, copy = torch.full((6, 48), 9.0, device="cuda"), torch.zeros(6, 48, device="cuda")
    K.embed_sinusoid(dw, ids.cuda(), pos.cuda(), freq.cuda(), out, copy)
    want = w.float()[ids] + R.sinusoid(pos.long(), 45)
    assert float((out[:, :45].cpu() - want).abs().max()) < 2e-6 and bool((out[:, 45:] == 0).all())
    assert torch.equal(out, copy)


def test_pass_input():
    from hipengine_b200.ops import kernels as K
    g = _gen()
    h, x0, s = (torch.randn(3, 136, generator=g), torch.randn(3, 136, generator=g), torch.randn(136, generator=g))
    a = h.cuda()
    K.resid_inject(a, None, s.cuda())
    assert torch.equal(a.cpu(), h + s)
    K.resid_inject(a, x0.cuda(), s.cuda())
    assert torch.allclose(a.cpu(), h + s + x0 + s, atol=1e-6)


class _Pages:
    """KV pages of one slot, scattered over the pool, filled with given keys and values."""

    def __init__(self, k, v, D, dtype, n_slots=3, slot=1, spare=5):
        S, G, _ = k.shape
        n = -(-S // 16)
        perm = torch.randperm(n + spare, generator=_gen(S))[:n] + 1
        self.bt = torch.zeros(n_slots, n + 2, dtype=torch.int32)
        self.bt[slot, :n] = perm.int()
        kv = torch.randn(n + spare + 1, 2, G, 16, D, generator=_gen(3)).to(dtype)
        for p in range(S):
            for plane, t in ((0, k), (1, v)):
                kv[perm[p // 16], plane, :, p % 16, :] = 0
                kv[perm[p // 16], plane, :, p % 16, :t.shape[2]] = t[p].to(dtype)
        self.kv, self.bt, self.slot = kv.cuda(), self.bt.cuda(), slot


def _padq(q, D, dtype):
    out = torch.zeros(q.shape[0], q.shape[1], D, dtype=dtype)
    out[:, :, :q.shape[2]] = q.to(dtype)
    return out.cuda()


def _far_key(S, H, G, dim, vdim, needles, seed):
    """Random keys of unit size; the keys at ``needles`` line up with the queries so that their score stands out."""
    g = _gen(seed)
    q = torch.randn(1, H, dim, generator=g).repeat(S, 1, 1)
    k, v = torch.randn(S, G, dim, generator=g) * 0.5, torch.randn(S, G, vdim, generator=g)
    for p in needles:
        k[p] = 3 * q[0, ::H // G][:G]
    return q.to(torch.bfloat16).float(), k.to(torch.bfloat16).float(), v.to(torch.bfloat16).float()


ATTN = [(6, 2, 40, 24, 64), (5, 1, 64, 64, 64), (7, 1, 128, 72, 128), (24, 2, 128, 128, 128), (9, 1, 200, 136, 256),
        (4, 4, 300, 260, 512), (1, 1, 16, 16, 64), (8, 1, 64, 32, 64), (17, 1, 64, 64, 64)]


@pytest.mark.parametrize("H,G,dim,vdim,D", ATTN)
@pytest.mark.parametrize("cap", [0.0, 3.0, 60.0])
def test_decode_attention_soft_cap_and_groups(H, G, dim, vdim, D, cap):
    """One query row per context length around page borders and span borders, with far keys that stand out."""
    from hipengine_b200.ops import kernels as K
    S = 277
    q, k, v = _far_key(S, H, G, dim, vdim, (0, 15, 16, 100), H)
    pg = _Pages(k, v, D, torch.bfloat16)
    ctx = [1, 2, 15, 16, 17, 63, 64, 65, 101, 129, 256, 277]
    rows = torch.tensor([c - 1 for c in ctx])
    slot = torch.full((len(ctx),), pg.slot, dtype=torch.int32, device="cuda")
    out = torch.zeros(len(ctx), H * D, dtype=torch.bfloat16, device="cuda")
    scale = 0.35 / dim ** 0.5 * 4
    part = torch.zeros(K.attn_decode_scratch_floats(len(ctx), H, 5, D), device="cuda")
    K.attn_decode(_padq(q[rows], D, torch.bfloat16), None, pg.kv, pg.bt, slot,
                  torch.tensor(ctx, dtype=torch.int32, device="cuda"), part, out, H, G, D, 16, 64, 5, scale, softcap=cap)
    K.check_status()
    want = R.attention(q[rows], k, v, rows, scale, cap if cap > 0 else 1e6)
    got = out.view(len(ctx), H, D).cpu().float()
    _close(got[:, :, :vdim], want, 0.03)
    assert bool((got[:, :, vdim:] == 0).all())
    # the far key decides: without it the reference differs by far more than the tolerance
    k2 = k.clone()
    k2[0] = 0
    assert float((R.attention(q[rows], k2, v, rows, scale, cap if cap > 0 else 1e6) - want).abs().max()) > 0.2


@pytest.mark.parametrize("H,G,dim,vdim,D", [a for a in ATTN if a[4] <= 256])
@pytest.mark.parametrize("cap", [3.0, 60.0])
def test_prefill_attention_segments(H, G, dim, vdim, D, cap):
    """Three portions of two requests in one launch: from the start, from inside a page, and one short one."""
    from hipengine_b200.ops import attention as A
    S = 200
    q, k, v = _far_key(S, H, G, dim, vdim, (0, 31, 32, 64, 150), H + 1)
    pg = _Pages(k, v, D, torch.bfloat16)
    parts = [(0, 70), (83, 200), (13, 22)]
    pos = torch.tensor([p for a, b in parts for p in range(a, b)], dtype=torch.int32)
    start = torch.tensor([0, 70, 187, 196], dtype=torch.int32, device="cuda")
    slots = torch.full((3,), pg.slot, dtype=torch.int32, device="cuda")
    out = torch.zeros(len(pos), H * D, dtype=torch.bfloat16, device="cuda")
    scale = 1.2 / dim ** 0.5
    A.flash_prefill_segs(_padq(q[pos.long()], D, torch.bfloat16), None, pg.kv, pg.bt, start, slots, pos.cuda(),
                         [b - a for a, b in parts], out, H, G, D, 16, scale, softcap=cap)
    want = R.attention(q[pos.long()], k, v, pos.long(), scale, cap)
    _close(out.view(-1, H, D)[:, :, :vdim], want, 0.03)


@pytest.mark.parametrize("H,G,dim,vdim,D", ATTN)
def test_exact_attention(H, G, dim, vdim, D):
    from hipengine_b200.ops import kernels as K
    q, k, v = _far_key(70, H, G, dim, vdim, (0, 16), H + 2)
    pg = _Pages(k, v, D, torch.float32)
    rows = torch.tensor([0, 1, 2, 15, 16, 17, 47, 69])
    out = torch.zeros(len(rows), H * D, device="cuda")
    slot = torch.full((len(rows),), pg.slot, dtype=torch.int32, device="cuda")
    K.attn_exact(_padq(q[rows], D, torch.float32), pg.kv, pg.bt, slot, (rows + 1).int().cuda(), out, H, G, D, 16,
                 1.2 / dim ** 0.5, 5.0)
    _close(out.view(-1, H, D)[:, :, :vdim], R.attention(q[rows], k, v, rows, 1.2 / dim ** 0.5, 5.0), 2e-5)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_head_norm_and_cache_write_with_narrow_heads(dtype):
    from hipengine_b200.ops import kernels as K
    g = _gen(5)
    T, H, G, dim, vdim, D = 5, 3, 1, 40, 72, 128
    qkv = torch.randn(T, H * dim + G * (dim + vdim), generator=g)
    qn, kn = torch.rand(dim, generator=g) + 0.5, torch.rand(dim, generator=g) + 0.5
    kv = torch.full((4, 2, G, 16, D), 3.0, dtype=dtype, device="cuda")
    bt = torch.tensor([[0, 0], [2, 3]], dtype=torch.int32, device="cuda")
    pos = torch.tensor([14, 15, 16, 17, 31], dtype=torch.int32, device="cuda")
    q_out = torch.zeros(T, H, D, dtype=dtype, device="cuda")
    x = qkv.cuda()
    K.qkv_post(x[:, :H * dim], x[:, H * dim:(H + G) * dim], x[:, (H + G) * dim:], qn.cuda(), kn.cuda(), q_out, None, kv, bt,
               torch.ones(T, dtype=torch.int32, device="cuda"), pos, H, G, D, 16, False, 0, 1.0, 1e-5, d_in=dim, dv_in=vdim)
    tol = 0.01 if dtype == torch.bfloat16 else 1e-5
    _close(q_out[:, :, :dim], R.rms_norm(qkv[:, :H * dim].view(T, H, dim), qn, 1e-5), tol)
    assert bool((q_out[:, :, dim:] == 0).all())
    pages = [2, 2, 3, 3, 3]
    for t in range(T):
        row = kv[pages[t], :, 0, int(pos[t]) % 16].cpu().float()
        _close(row[0, :dim], R.rms_norm(qkv[t, H * dim:(H + G) * dim], kn, 1e-5), tol)
        _close(row[1, :vdim], qkv[t, (H + G) * dim:], tol)
        assert bool((row[0, dim:] == 0).all()) and bool((row[1, vdim:] == 0).all())


@pytest.mark.parametrize("exact", [False, True])
@pytest.mark.parametrize("shared", [True, False])
def test_selected_experts(exact, shared):
    from hipengine_b200.ops import kernels as K
    g = _gen(9)
    T, E, k, Kc, F, Fs, real = 5, 7, 3, 136, 40, 72, 131
    h = torch.zeros(T, Kc)
    h[:, :real] = torch.randn(T, real, generator=g)
    nw = torch.zeros(Kc)
    nw[:real] = 1 + 0.2 * torch.randn(real, generator=g)
    bf = lambda *s: (torch.randn(*s, generator=g) / s[-1] ** 0.5).to(torch.bfloat16)
    gu, dn, sgu, sdn = bf(E * 2 * F, Kc), bf(E * Kc, F), bf(2 * Fs, Kc), bf(Kc, Fs)
    ids = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)]).int()
    wts, sg = torch.rand(T, k, generator=g), torch.randn(T, 4, generator=g)
    xn = torch.zeros(T, Kc)
    xn[:, :real] = R.rms_norm(h[:, :real], nw[:real], 1e-5)
    want = h.clone()
    for t in range(T):
        for j in range(k):
            e = int(ids[t, j])
            y = gu.float().view(E, 2, F, Kc)[e] @ xn[t]
            want[t] += wts[t, j] * (dn.float().view(E, Kc, F)[e] @ R.silu_glu(y[0], y[1]))
        if shared:
            y = sgu.float().view(2, Fs, Kc) @ xn[t]
            want[t] += torch.sigmoid(sg[t, 2]) * (sdn.float() @ R.silu_glu(y[0], y[1]))
    dt = torch.float32 if exact else torch.bfloat16
    rows, rows_s = torch.zeros(T * k, F, dtype=dt, device="cuda"), torch.zeros(T, Fs, dtype=dt, device="cuda")
    hc, idc, wc, sgc = h.cuda(), ids.cuda(), wts.cuda(), sg.cuda()[:, 2:3]
    sh = (sgu.cuda(), sdn.cuda(), rows_s) if shared else (None, None, None)
    if exact:
        K.moe_exact(xn.cuda(), idc, wc, gu.cuda(), dn.cuda(), E, rows, hc, sgc if shared else None, *sh)
    else:
        K.moe_gateup_float(hc, nw.cuda(), 1e-5, real, idc, wc, gu.cuda(), E, rows, sgc if shared else None, sh[0], sh[2])
        K.moe_down_float(rows, idc, dn.cuda(), E, hc, sh[2], sh[1])
    _close(hc.cpu() - h, want - h, 1e-4 if exact else 0.02)


def test_bf16_weights_in_fp32_products():
    from hipengine_b200.ops import kernels as K
    g = _gen(1)
    x, w = torch.randn(70, 130, generator=g), torch.randn(67, 130, generator=g).to(torch.bfloat16)
    out = torch.ones(70, 67, device="cuda")
    K.small_gemm_f32(x.cuda(), w.cuda(), out, add=True)
    _close(out, 1 + x @ w.float().t(), 1e-5)


# ----------------------------------------------------------------------------- whole models
DTYPES = ["float32", "bfloat16"]


def _executor(cfg_json, dtype, seed=0, max_slots=4, max_context=320, **kw):
    from hipengine_b200.models import make_executor
    w, ref, t = build(cfg_json, seed, clear=dtype == "bfloat16")
    return make_executor(w, dtype=dtype, device="cuda", max_slots=max_slots, max_context=max_context, **kw), ref, t


def _run(ex, segs):
    from hipengine_b200.models.executor import make_batch
    from hipengine_b200.ops import kernels as K
    h = ex.forward(make_batch(segs, ex.device))
    out = ex.logits(h).clone()
    K.check_status()
    return out.cpu()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MODELS))
def test_layers_one_by_one(name, dtype):
    ex, ref, _ = _executor(MODELS[name], dtype)
    ids = tokens(37, MODELS[name]["vocab"], 2)
    got, want = [], []
    ex.on_layer_run = lambda run, h: got.append(h.clone().cpu())
    _run(ex, [(0, 0, ids)])
    ref.forward_raw(torch.tensor(ids), ref.new_state(), want)
    assert len(got) == len(want) == len(ex.cfg.layer_runs())
    for g, w in zip(got, want):
        _close(g, w, 2e-5 if dtype == "float32" else 0.05)


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
    ex, ref, _ = _executor(WIDE, dtype)
    ids = tokens(140, WIDE["vocab"], 6)
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
def test_far_key_at_every_border(dtype):
    """A key that decides the logits sits at the first tokens, at page borders and next to the asking token; it is asked
    for from a prompt, from a portion and from a decoded token."""
    from hipengine_b200.models import make_executor
    cfg = LOOPED
    w, ref, _ = needle(cfg)
    ex = make_executor(w, dtype=dtype, device="cuda", max_slots=4, max_context=320)
    base = [3 + t for t in tokens(131, cfg["vocab"] - 3, 8)]
    for p in (0, 1, 15, 16, 17, 63, 64, 111, 112, 128, 129):
        ids = list(base)
        ids[p], ids[130] = 2, 1
        want = ref.forward(torch.tensor(ids))[0][-1:]
        plain = ref.forward(torch.tensor(base[:130] + [1]))[0][-1:]
        assert logit_error(plain, want) > 5 * TOL[dtype]
        assert logit_error(_run(ex, [(0, 0, ids)])[-1:], want) < TOL[dtype], p
        _run(ex, [(1, 0, ids[:97])])
        assert logit_error(_run(ex, [(1, 97, ids[97:])])[-1:], want) < TOL[dtype], p
        _run(ex, [(2, 0, ids[:130])])
        assert logit_error(_run(ex, [(2, 130, ids[130:])]), want) < TOL[dtype], p


def test_scratch_contents_do_not_matter():
    from hipengine_b200.ops import kernels as K
    for dtype in DTYPES:
        ex, _, _ = _executor(WIDE, dtype)
        ex.scratch.canaries = True
        ids = tokens(150, WIDE["vocab"], 1)
        work = [[(0, 0, ids)], [(1, 0, ids[:20])], [(1, 20, ids[:3]), (0, 150, ids[:1])]]
        first = [_run(ex, s) for s in work]
        for t in list(ex.scratch.bufs.values()) + list(ex.scratch.retired):
            t.view(torch.uint8).fill_(0xFF)
        for a, b in zip(first, [_run(ex, s) for s in work]):
            assert torch.equal(a, b) and bool(torch.isfinite(b).all())
        assert not ex.scratch.check_canaries()
        K.check_status()


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


@pytest.mark.parametrize("policy", ["protect_decode", "mixed"])
def test_greedy_generation_through_the_engine(policy):
    """More requests than slots, a pool that forces pages to be used again, prompt chunks beside decode steps: the ids of
    the float32 engine are the oracle's."""
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(WIDE, 3)
    prompts = [tokens(n, WIDE["vocab"], 100 + n) for n in (40, 3, 21, 70, 1, 33)]
    base = EngineConfig()
    eng = replace(base, scheduler=replace(base.scheduler, policy=policy, max_prefill_chunk_tokens=13),
                  kv=replace(base.kv, pool_pages=20))
    with LLM(w, engine_config=eng, dtype="float32", max_active_requests=3, max_sequence_length=256,
             prefix_cache="off") as llm:
        got = llm.generate_token_ids(prompts, SamplingParams(max_tokens=14, ignore_eos=True))
        snap = llm.live_loop_snapshot()["runner"]
    for p, g in zip(prompts, got):
        want, margin = _greedy(ref, p, 14)
        cut = next((i for i, m in enumerate(margin) if m < 1e-4), 14)
        assert g[:cut] == want[:cut]
    assert snap["launch_census"]
    if policy == "mixed":
        assert "mixed" in str(snap["launch_census"])


def test_bf16_generation_follows_its_own_logits():
    """The served precision: sampled ids are the argmax of the logits of the sequence generated so far (long decode over
    many pages, prefix cache on, the second request reuses the first one's prompt pages)."""
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(LOOPED, 4, clear=True)
    prompt = tokens(50, LOOPED["vocab"], 9)
    with LLM(w, max_active_requests=2, max_sequence_length=512) as llm:
        a = llm.generate_token_ids([prompt], SamplingParams(max_tokens=180, ignore_eos=True))[0]
        b = llm.generate_token_ids([prompt], SamplingParams(max_tokens=180, ignore_eos=True))[0]
        hits = llm.live_loop_snapshot()["runner"]["prefix_hit_tokens"]
        s = llm.generate_detailed([prompt], SamplingParams(max_tokens=5, temperature=0.8, seed=1, logprobs=True,
                                                           top_logprobs=3))[0]
    assert len(a) == len(b) == 180 and hits == 48 and len(s.token_ids) == 5
    want = ref.forward(torch.tensor(prompt + a))[0]
    agree = total = 0
    for i, tok in enumerate(a):
        row = want[len(prompt) - 1 + i]
        top = row.topk(2).values
        if float(top[0] - top[1]) > 0.15 * float(row.std()):          # decided positions
            total += 1
            agree += int(row.argmax()) == tok
    assert total > 20 and agree == total


def test_prompt_lookup_speculation_keeps_greedy_output():
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(LOOPED, 4)
    prompt = (tokens(12, LOOPED["vocab"], 9) * 3)[:30]
    with LLM(w, dtype="float32", max_active_requests=2, max_sequence_length=256, speculative_mtp_serving="on",
             speculative_provider="prompt_lookup") as llm:
        got = llm.generate_token_ids([prompt], SamplingParams(max_tokens=40, ignore_eos=True))[0]
    want, margin = _greedy(ref, prompt, 40)
    cut = next((i for i, m in enumerate(margin) if m < 1e-4), 40)
    assert got[:cut] == want[:cut]


# ----------------------------------------------------------------------------- trace replay
def _replay(cfg_json, dtype, max_tokens, seed=0):
    from hipengine_b200.generation.gpu_runner import GpuRunner
    from hipengine_b200.generation.trace_replay import TraceReplay, trace_engine_config
    w, ref, _ = build(cfg_json, seed, clear=dtype == "bfloat16")
    return TraceReplay(GpuRunner(w, trace_engine_config(max_tokens, dtype))), ref


@pytest.mark.parametrize("dtype", DTYPES)
def test_replay_reuses_pages_and_slots(dtype):
    """Nine requests through four slots and a pool for 192 tokens, interleaved, some paused, with decode-only steps (the
    graph path) between mixed ones; every wanted row against the request alone."""
    rep, ref = _replay(WIDE, dtype, 192)
    lens = [40, 7, 64, 30, 18, 50, 33, 2, 61]
    seqs = {f"r{i}": tokens(n, WIDE["vocab"], 50 + i) for i, n in enumerate(lens)}
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


def test_replay_refuses_what_does_not_fit():
    from hipengine_b200.generation.trace_replay import TraceError
    rep, _ = _replay(LOOPED, "bfloat16", 64)
    for bad in ({"id": "a", "tokens": []}, {"id": "a", "tokens": [LOOPED["vocab"]]}, {"id": "a", "tokens": [-1]},
                {"id": "a", "tokens": [1], "want": [1]}):
        with pytest.raises(TraceError):
            rep.step([bad])
        if "a" in rep.live:
            rep.step([], ["a"])
    with pytest.raises(TraceError):
        rep.step([], ["never"])
    assert rep.step([{"id": "b", "tokens": [1, 2], "want": []}], ["b"]) is None


def test_trace_run_program(tmp_path):
    """The program end to end on a checkpoint folder: protocol, files, exit code."""
    import numpy as np
    from hipengine_b200.loading.safetensors_dir import write_tensors
    _, ref, t = build(HEADS, clear=True)
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
