"""Banelix on the GPU: every mechanism against the plain fp32 equations, then whole models through the executor, the paged
cache, mixed batches, the engine and the trace replay, in bfloat16 and float32."""
import json
import os
import subprocess
import sys
from dataclasses import replace

import pytest
import torch

from hipengine_b200.ref import banelix as R

from banelix_models import (HEADS, MODELS, ODD, TOL, WIDE, bands, both, build, last_logits, logit_error, model, needle,
                            rotation, tokens, windowed, with_windows, yarn)

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


def _up8(n):
    return -(-n // 8) * 8


# ----------------------------------------------------------------------------- head rows: bias, norm, rotation, pages
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("halves", [True, False])
@pytest.mark.parametrize("norm", ["none", "head", "rows", "unit"])
@pytest.mark.parametrize("T,H,G,dim,vdim,rd", [(6, 3, 1, 20, 28, 10), (2, 5, 5, 33, 33, 14), (150, 21, 3, 64, 48, 64),
                                               (9, 40, 4, 128, 128, 64), (150, 40, 8, 300, 264, 72), (1, 1, 1, 2, 2, 2)])
def test_head_rows(T, H, G, dim, vdim, rd, norm, halves, dtype):
    """Positions up to 262143, row buffers with other columns around, few and many tokens (parts of the heads per CTA or all of
    them), values of their own or the plain keys, or no keys at all; padding of heads is written as zeros."""
    from hipengine_b200.models.config import RotarySpec, YarnSpec, padded_head_width
    from hipengine_b200.models.executor import make_batch
    from hipengine_b200.ops import mixers as MX
    g, eps, D = _gen(H + dim), 1e-3, padded_head_width(max(dim, vdim))
    rot = RotarySpec(rd, 5000.0, YarnSpec(4.0, 512.0, 20.0, 1.5), halves)
    freq, amp = rot.table()
    pos = [0, 1, 15, 16, 4097, 262143] * 25
    pos = torch.tensor(pos[:T])
    widths = {"q": H * dim, "k": G * dim, "v": G * vdim}
    at, col, rows = 8, {}, []
    for n, w in widths.items():
        col[n] = (at, at + _up8(w))
        at = col[n][1] + 16
    x = torch.zeros(T, at)
    bias, gain = {}, {}
    for n, w in widths.items():
        x[:, col[n][0]:col[n][0] + w] = torch.randn(T, w, generator=g)
        bias[n], gain[n] = torch.zeros(_up8(w)), torch.zeros(_up8(w) if norm == "rows" else dim)
        bias[n][:w] = torch.randn(w, generator=g)
        gain[n][:w if norm == "rows" else dim] = 1 + torch.rand(w if norm == "rows" else dim, generator=g)
    x = x.to(dtype).float()
    real = {n: x[:, col[n][0]:col[n][0] + w] + bias[n][:w] for n, w in widths.items()}

    def turn(v):
        f = torch.tensor(freq, dtype=torch.float64)
        if halves:
            return R.rotate_halves(v, pos, f, amp)
        perm = torch.arange(rd).view(-1, 2).t().reshape(-1)              # neighbours -> halves and back
        out = v.clone()
        out[..., perm] = R.rotate_halves(v[..., perm], pos, f, amp)
        return out

    def want(n, heads):
        v = real[n]
        if norm == "rows":
            v = R.rms(v, eps) * gain[n][:v.shape[1]]
        v = v.reshape(T, heads, dim)
        if norm == "head":
            v = R.rms(v, eps) * gain[n]
        v = turn(v)
        return R.rms(v, eps) if norm == "unit" else v

    b = make_batch([(t, int(p), [0]) for t, p in enumerate(pos)], "cuda")
    bt = torch.zeros(T, 262144 // 16, dtype=torch.int32)
    for t, p in enumerate(pos):
        bt[t, p // 16] = t
    xc, bt = x.to(dtype).cuda(), bt.cuda()
    tol = 3e-5 if dtype == F32 else 0.01
    for keys in ("own values", "plain keys", "none"):
        if keys == "plain keys" and (norm == "rows" or dim < vdim):
            continue
        hr = lambda n, h, d: MX.HeadRows(xc[:, col[n][0]:col[n][1]], h, d, bias[n].cuda(), gain[n].cuda() if n != "v" else None)
        q_out = torch.full((T, H, D), 7.0, dtype=dtype, device="cuda")
        cache = torch.full((T, 2, G, 16, D), 7.0, dtype=dtype, device="cuda")
        MX.mixer_post(hr("q", H, dim), None if keys == "none" else hr("k", G, dim), hr("v", G, vdim) if keys == "own values" else None,
                      norm, rot, torch.tensor(freq, dtype=torch.float64, device="cuda"), amp, q_out,
                      None if keys == "none" else cache, 16, b, bt, eps)
        _close(q_out[:, :, :dim], want("q", H), tol)
        assert not q_out[:, :, dim:].any()
        if keys == "none":
            assert bool((cache == 7.0).all())
            continue
        got = torch.stack([cache[t, :, :, p % 16] for t, p in enumerate(pos)]).cpu()
        _close(got[:, 0, :, :dim], want("k", G), tol)
        v, w = ("v", vdim) if keys == "own values" else ("k", dim)
        _close(got[:, 1, :, :w], real[v].reshape(T, G, w), tol)
        assert not got[:, 0, :, dim:].any() and not got[:, 1, :, w:].any()
        for t, p in enumerate(pos):
            assert bool((cache[t, :, :, (p + 1) % 16] == 7.0).all())         # no other row of the page


# ----------------------------------------------------------------------------- convolution and recurrence
def _segments(lens, slots):
    from hipengine_b200.models.executor import make_batch
    return make_batch([(s, 5, [0] * n) for n, s in zip(lens, slots)], "cuda")


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("blocks,block,taps", [(1, 8, 1), (4, 15, 3), (3, 40, 2), (5, 256, 4), (2, 700, 6)])
def test_convolution(blocks, block, taps, dtype):
    """Segments shorter and longer than the convolution on slots with and without a past; the journal has the state after
    every token, the state itself stays; a block-major and a token-major result."""
    from hipengine_b200.ops import mixers as MX
    g, bc, lens, slots = _gen(block), _up8(block), [1, 5, 2, 1, 9], [2, 0, 5, 4, 1]
    T, C, b = sum(lens), blocks * bc, _segments(lens, slots)
    x, bias, w, cb = (torch.randn(*s, generator=g) for s in ((T, C), (C,), (taps, C), (C,)))
    st = torch.randn(6, taps - 1, C, generator=g)
    st[[1, 5]] = 0
    x = x.to(dtype).float()
    want, hist, row = [], [], 0
    for n, s in zip(lens, slots):
        xs = x[row:row + n] + bias
        want.append(R.causal_conv(xs, st[s], w.t(), cb))
        full = torch.cat([st[s], xs])
        hist += [full[t + 1:t + taps] for t in range(n)]
        row += n
    want = torch.cat(want).view(T, blocks, bc)
    q = MX.HeadRows(torch.zeros(T, 8, dtype=dtype, device="cuda"), 1, 8)
    rows = torch.full((T, C + 24), 3.0, dtype=dtype, device="cuda")
    rows[:, 16:16 + C] = x.cuda()
    for major in (0, 1):
        for journal in (None, torch.full((T, taps - 1, C), 7.0, device="cuda") if taps > 1 else None):
            u = torch.full((T, blocks, bc) if major == 0 else (blocks, T + 3, bc), 7.0, dtype=dtype, device="cuda")
            uv = u if major == 0 else u.transpose(0, 1)[:T]
            state = st.cuda() if taps > 1 else None
            MX.mixer_post(q, None, None, "none", None, torch.zeros(1, dtype=torch.float64, device="cuda"), 1.0,
                          torch.empty(T, 1, 64, dtype=dtype, device="cuda"), None, 16, b, torch.zeros(6, 4, dtype=torch.int32, device="cuda"),
                          1e-5, MX.ConvRows(rows[:, 16:16 + C], bias.cuda(), w.cuda(), cb.cuda(), uv, state, journal))
            _close(uv, want, 2e-6 if dtype == F32 else 0.005)
            assert state is None or torch.equal(state.cpu(), st)
            if journal is not None:
                _close(journal, torch.stack(hist), 1e-6)
            assert major == 0 or bool((u[:, T:] == 7.0).all())


def _lru(blocks, block, taps, dtype, seed):
    """Parameters, and the oracle's view of them without the padding."""
    from hipengine_b200.ops import mixers as MX
    g, bc = _gen(seed), _up8(block)
    ra, ri = (torch.randn(blocks, block, block, generator=g).to(BF) / block ** 0.5 for _ in range(2))
    rb, ib = (torch.randn(blocks, block, generator=g) - 0.5 for _ in range(2))
    lam, yb, xb = torch.randn(blocks * block, generator=g) * 2 - 4, torch.randn(blocks * bc, generator=g), torch.randn(blocks * bc, generator=g)
    w, gb = torch.zeros(blocks, 2, bc, bc, dtype=BF), torch.zeros(blocks, 2, bc)
    w[:, 0, :block, :block], w[:, 1, :block, :block], gb[:, 0, :block], gb[:, 1, :block] = ra, ri, rb, ib
    decay = torch.zeros(blocks, bc)
    decay[:, :block] = -8 * torch.nn.functional.softplus(lam).view(blocks, block)
    p = MX.Recurrence(w.view(blocks, 2 * bc, bc).cuda(), gb.view(blocks, 2 * bc).cuda(), decay.view(-1).cuda(), yb.cuda(), xb.cuda(), taps)
    return p, (ra.float(), ri.float(), rb, ib, lam, yb.view(blocks, bc)[:, :block].reshape(-1))


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("blocks,block,taps,lens", [
    (4, 15, 3, [1, 1, 1]), (3, 40, 4, [1] * 13), (1, 8, 1, [1]), (16, 64, 2, [1] * 16), (2, 328, 4, [1] * 5),
    (4, 15, 3, [1, 7, 2, 40, 1]), (3, 40, 4, [8, 9, 255, 256, 257, 2]), (1, 8, 1, [700, 3]), (2, 320, 4, [513, 1, 16]),
    (5, 256, 2, [1] * 40)])
def test_recurrence(blocks, block, taps, lens, dtype):
    """One-token steps and scans (segments around the tile's group, warp and tile edges, memories up to thousands of tokens),
    gates from every product: outputs, states, convolution states; with a journal the states stay."""
    from hipengine_b200.ops import kernels as K
    from hipengine_b200.ops import mixers as MX
    n_seg, T, bc, C = len(lens), sum(lens), _up8(block), blocks * _up8(block)
    slots = [(3 * s + 1) % (n_seg + 3) for s in range(n_seg)] if (n_seg + 3) % 3 else list(range(n_seg))
    p, (ra, ri, rb, ib, lam, yb) = _lru(blocks, block, taps, dtype, T)
    g, b = _gen(T), _segments(lens, slots)
    tight = lambda x: x.reshape(*x.shape[:-1], blocks, bc)[..., :block].reshape(*x.shape[:-1], blocks * block)
    u = torch.zeros(T, blocks, bc)
    u[:, :, :block] = torch.randn(T, blocks, block, generator=g)
    y, x = torch.randn(T, C, generator=g).to(dtype).float(), torch.randn(T, C, generator=g).to(dtype).float()
    u, S, cs = u.to(dtype).float(), torch.randn(n_seg + 3, C, generator=g), torch.randn(n_seg + 3, taps - 1, C, generator=g)
    uf, want, states, row = tight(u.view(T, C)), [], [], 0
    r, i = torch.sigmoid(R.block_product(uf, ra, rb)), torch.sigmoid(R.block_product(uf, ri, ib))
    for n, s in zip(lens, slots):
        o, _ = R.gated_recurrence(uf[row:row + n], r[row:row + n], i[row:row + n], lam, tight(S)[s])
        want.append(o)
        row += n
    history = torch.cat(want)
    want = history * R.gelu_tanh(tight(y) + yb)
    gates = torch.einsum("tbk,bnk->tbn", u.cuda(), p.gate_w.float())
    rows = torch.full((T, 2 * C + 16), 3.0, dtype=dtype, device="cuda")
    rows[:, :C], rows[:, C + 8:2 * C + 8] = y.cuda(), x.cuda()
    yr, xr = rows[:, :C], rows[:, C + 8:2 * C + 8]
    tol = 5e-5 if dtype == F32 else 0.006
    runs = [(m, j) for m in ("token-major", "block-major") for j in (False, True)]
    if dtype == BF and max(lens) == 1 and n_seg <= 16:
        runs += [("step", False)]
    for how, with_journal in runs:
        Sc, cc = S.cuda(), cs.cuda() if taps > 1 else None
        out = torch.full((T, C + 8), 7.0, dtype=dtype, device="cuda")
        journal = torch.full((T, C), 7.0, device="cuda") if with_journal else None
        uc, gc = u.to(dtype).cuda(), gates
        if how == "block-major":
            uc, gc = uc.transpose(0, 1).contiguous().transpose(0, 1), gc.transpose(0, 1).contiguous().transpose(0, 1)
        if how == "step":
            MX.rglru_step(p, uc, yr, xr, Sc, cc, b, out[:, :C])
        else:
            MX.rglru_scan(p, gc, uc, yr, xr, Sc, cc, b, out[:, :C], journal=journal)
        K.check_status()
        _close(tight(out[:, :C].cpu().float()), want, tol)
        assert bool((out[:, C:] == 7.0).all())
        if with_journal:
            assert torch.equal(Sc.cpu(), S) and (cc is None or torch.equal(cc.cpu(), cs))
            _close(tight(journal.cpu()), history, 5e-5)
            continue
        row, xb = 0, p.x_bias.cpu()
        for n, s in zip(lens, slots):
            _close(tight(Sc[s].cpu()), history[row + n - 1], 5e-5)
            if taps > 1:
                _close(cc[s], torch.cat([cs[s], x[row:row + n] + xb])[n:], 1e-6)
            row += n
        for s in set(range(n_seg + 3)) - set(slots):
            assert torch.equal(Sc[s].cpu(), S[s]) and (taps == 1 or torch.equal(cc[s].cpu(), cs[s]))


def test_long_memories_keep_their_accuracy():
    """Channels that forget one part in ten thousand per token, driven by a constant for 3000 tokens: the sum neither drifts
    nor is its drive biased."""
    from hipengine_b200.ops import mixers as MX
    T, C = 3000, 16
    lam = torch.linspace(-9.0, -4.0, C)
    decay = -8 * torch.nn.functional.softplus(lam)
    p = MX.Recurrence(torch.zeros(1, 2 * C, C, dtype=BF, device="cuda"), torch.zeros(1, 2 * C, device="cuda"), decay.cuda(),
                      torch.full((C,), 3.0, device="cuda"), torch.zeros(C, device="cuda"), 1)
    b = _segments([T], [0])
    u, rows, S = torch.ones(T, 1, C, device="cuda"), torch.zeros(T, C, device="cuda"), torch.zeros(1, C, device="cuda")
    out = torch.empty(T, C, device="cuda")
    MX.rglru_scan(p, torch.zeros(T, 1, 2 * C, device="cuda"), u, rows, rows, S, None, b, out)
    half, d = torch.full((T, C), 0.5).double(), lam.double()
    want, _ = R.gated_recurrence(torch.ones(T, C).double(), half, half, d, torch.zeros(C).double())
    _close(S[0], want[-1], 6e-5)                       # one decay rounded to fp32 is this far off after 3000 tokens
    _close(out, want * R.gelu_tanh(torch.tensor(3.0).double()), 6e-5)


# ----------------------------------------------------------------------------- attention: window, sink, gate per head
def _cache(ctxs, G, D, dtype, seed):
    """Keys and values of requests of ``ctxs`` tokens in shuffled pages: (cache, block table, keys, values)."""
    g, pages = _gen(seed), [-(-c // 16) for c in ctxs]
    ids = (torch.randperm(sum(pages), generator=g) + 1).tolist()
    cache = torch.zeros(sum(pages) + 1, 2, G, 16, D)
    cache[0] = float("nan")                                                   # the null page is never attended to
    bt, ks, vs = torch.zeros(len(ctxs), max(pages) + 3, dtype=torch.int32), [], []
    for s, c in enumerate(ctxs):
        k, v = (torch.randn(c, G, D, generator=g).to(dtype).float() for _ in range(2))
        for i in range(pages[s]):
            bt[s, i] = ids.pop()
            n = min(16, c - 16 * i)
            cache[bt[s, i], 0, :, :n], cache[bt[s, i], 1, :, :n] = k[16 * i:16 * i + n].transpose(0, 1), v[16 * i:16 * i + n].transpose(0, 1)
        ks.append(k)
        vs.append(v)
    return cache.to(dtype).cuda(), bt.cuda(), ks, vs


@pytest.mark.parametrize("window", [0, 1, 16, 65, 130])
@pytest.mark.parametrize("H,G,D", [(1, 1, 64), (6, 2, 64), (15, 3, 128), (40, 4, 128), (4, 4, 256), (14, 2, 64), (3, 1, 512)])
def test_attention_with_window_sink_and_gate(H, G, D, window):
    """Single tokens (spans of one tile and of several), portions of several requests in one launch, and the fp32 form; keys
    just inside and just outside the window stand out; sinks above and below every score."""
    from hipengine_b200.ops import attention as A
    from hipengine_b200.ops import kernels as K
    ctxs = [1, 2, 16, 17, 64, 65, 129, 300, 131, 67]
    g, n, scale = _gen(H), len(ctxs), 1.5 / D ** 0.5
    sink = torch.linspace(-3, 6, H) if H > 1 else torch.tensor([0.0])
    segs = [(7, 100, 200), (2, 3, 13), (6, 0, 129)]

    def plain(q, k, v, pos, gate, with_sink):
        seen, out = R.visible_keys(pos, k.shape[0], window), []
        for h in range(H):
            s = torch.where(seen, q[:, h] @ k[:, h // (H // G)].t() * scale, torch.tensor(float("-inf")))
            if with_sink:
                s = torch.cat([s, sink[h].expand(s.shape[0], 1)], 1)
            o = torch.softmax(s, -1)[:, :k.shape[0]] @ v[:, h // (H // G)]
            out.append(o * torch.sigmoid(gate[:, h:h + 1]) if gate is not None else o)
        return torch.stack(out, 1)

    for dtype in (BF, F32):
        cache, bt, ks, vs = _cache(ctxs, G, D, dtype, H + D)
        q = torch.randn(n, H, D, generator=g).to(dtype).float()
        for s, c in enumerate(ctxs):                                          # one key stands out: just inside or just outside
            j = c - 1 - (window - 1 + s % 2) if window else 0
            if 0 <= j < c:
                ks[s][j] = (q[s, ::H // G] * 3).to(dtype).float()
                cache[bt[s, j // 16], 0, :, j % 16] = ks[s][j].to(dtype).cuda()
        wide = torch.randn(n, H + 9, generator=g).to(dtype)
        gate = wide[:, 5:5 + H]
        qs = torch.randn(sum(m for _, _, m in segs), H, D, generator=g).to(dtype).float()
        gs = torch.randn(qs.shape[0], H + 3, generator=g).to(dtype)
        for use_sink, use_gate in ((False, False), (True, True), (True, False), (False, True)):
            want = torch.cat([plain(q[s:s + 1], ks[s], vs[s], torch.tensor([c - 1]), gate[s:s + 1].float() if use_gate else None,
                                    use_sink) for s, c in enumerate(ctxs)])
            out = torch.full((n, H * D), 7.0, dtype=dtype, device="cuda")
            kw = dict(sink=sink.cuda() if use_sink else None, head_gate=wide.cuda()[:, 5:5 + H] if use_gate else None)
            rows = (cache, bt, torch.arange(n, dtype=torch.int32, device="cuda"), _i32(ctxs))
            if dtype == F32:
                K.attn_exact(q.cuda(), *rows, out, H, G, D, 16, scale, 0.0, window, **kw)
                _close(out.view(n, H, D), want, 1e-4)
                continue
            for span in (64, 128, 320):
                splits = -(-(min(300, window) if window else 300) // span)
                part = torch.full((K.attn_decode_scratch_floats(n, H, splits, D),), float("nan"), device="cuda")
                K.attn_decode(q.to(BF).cuda(), None, *rows, part, out, H, G, D, 16, span, splits, scale, window, **kw)
                K.check_status()
                _close(out.view(n, H, D), want, 0.02)
            if not A.flash_prefill_available(D):
                continue
            start = [0]
            for _, _, m in segs:
                start.append(start[-1] + m)
            want = torch.cat([plain(qs[a:a + m], ks[s][:p0 + m], vs[s][:p0 + m], torch.arange(p0, p0 + m),
                                    gs[a:a + m, 2:2 + H].float() if use_gate else None, use_sink)
                              for (s, p0, m), a in zip(segs, start)])
            out = torch.full((qs.shape[0], H * D), 7.0, dtype=BF, device="cuda")
            kw["head_gate"] = gs.cuda()[:, 2:2 + H] if use_gate else None
            pos = _i32([p for _, p0, m in segs for p in range(p0, p0 + m)])
            for first in (0, 1):                                              # all segments; the later ones alone
                A.flash_prefill_segs(qs.to(BF).cuda(), None, cache, bt, _i32(start)[first:], _i32([s for s, _, _ in segs])[first:],
                                     pos, [m for _, _, m in segs[first:]], out, H, G, D, 16, scale, window, **kw)
                _close(out[start[first]:].view(-1, H, D), want[start[first]:], 0.03)


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
        assert len(got) == len(want) == len(ex.cfg.layer_specs)
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
    cfg = model(96, 160, [(both(4, 2, 24, 0.5, rotation(8, 500.0), 32, 2, 3, 1.0, 0.3), 64), (both(6, 3, 40, 0.4, rotation(
        16, 900.0, bands(4.0, 1.0, 4.0, 64.0)), 48, 3, 4, 0.8, 0.5), 0)])
    w, ref, _ = needle(cfg, strength=2.0)
    ex = make_executor(w, dtype=dtype, device="cuda", max_slots=4, max_context=320)
    base = [3 + t for t in tokens(131, 157, 8)]
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
    """Keys just inside and just outside a window, in prompts, portions and decoding, also where the keys are another layer's.
    (A model of windows only; the oracle with windows one token longer gives other logits, so an edge that is off shows.)"""
    from hipengine_b200.models import make_executor
    r = rotation(8, 500.0, yarn(2.0, 64.0, 4.0, 1.0))
    cfg = model(96, 160, [(windowed(4, 2, 24, 16, 0.3, size, r), 64), (windowed(4, 2, 24, 16, 0.25, size, r, kv_from=0), 0)])
    w, ref, t = needle(cfg, 2.0)
    ex = make_executor(w, dtype=dtype, device="cuda", max_slots=4, max_context=320)
    longer = R.BanelixRef(with_windows(cfg, 1), t)
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
def test_extra_unit_beside_one_and_many_keys(dtype, monkeypatch):
    """The unit in the denominator counts once, at the first token as behind a full window, in both forms of attention."""
    from hipengine_b200.models import make_executor
    cfg = model(64, 96, [(windowed(4, 2, 24, 24, 0.02, 40, rotation(8, 50.0)), 0)], mult=1.5, embed=0.5)
    w, ref, _ = build(cfg, 3)
    ids = tokens(300, 96, 1)
    want = ref.forward(torch.tensor(ids))[0]
    with monkeypatch.context() as m:
        real = R.weights_over
        m.setattr(R, "weights_over", lambda s, seen, extra: real(s, seen, False))
        none = ref.forward(torch.tensor(ids))[0]
    assert logit_error(none[:3], want[:3]) > 4 * TOL[dtype]
    ex = make_executor(w, dtype=dtype, device="cuda", max_slots=2, max_context=320)
    assert logit_error(_run(ex, [(0, 0, ids[:299])]), want[:299]) < TOL[dtype]
    assert logit_error(_run(ex, [(0, 299, ids[299:])]), want[299:]) < TOL[dtype]
    assert logit_error(torch.cat([_run(ex, [(1, p, [ids[p]])]) for p in range(40)]), want[:40]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_slot_used_again_starts_without_a_past(dtype):
    """Recurrent and convolution states of the last request in a slot do not reach the next one; state in other slots stays."""
    ex, ref, _ = _executor(ODD, dtype)
    a, b = tokens(40, ODD["vocab"], 1), tokens(30, ODD["vocab"], 2)
    _run(ex, [(0, 0, a), (1, 0, b[:20])])
    assert logit_error(_run(ex, [(0, 0, b)]), ref.forward(torch.tensor(b))[0]) < TOL[dtype]
    assert logit_error(_run(ex, [(1, 20, b[20:])]), ref.forward(torch.tensor(b))[0][20:]) < TOL[dtype]


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
    """A cached prefix is only usable with the recurrent state at its last token: the continuation of a reused prefix
    is the oracle's, from the device cache and from the cold tier."""
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(HEADS, 4)
    a = tokens(50, HEADS["vocab"], 9)
    other = [tokens(60, HEADS["vocab"], 20 + i) for i in range(4)]
    prompts = [a, a[:48] + tokens(5, HEADS["vocab"], 2), a[:33] + tokens(3, HEADS["vocab"], 3)]
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
    _, ref, t = build(HEADS, 4)
    (tmp_path / "config.json").write_text(json.dumps(HEADS))
    write_tensors(tmp_path / "model.safetensors", t)
    prompt = tokens(50, HEADS["vocab"], 9)
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
    """Rejected drafts leave neither cache rows nor recurrent states behind."""
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(HEADS, 4)
    prompt = (tokens(12, HEADS["vocab"], 9) * 3)[:30]
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
    rep, ref = _replay(HEADS, "bfloat16", 1152)
    ids = tokens(1060, HEADS["vocab"], 3)
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
