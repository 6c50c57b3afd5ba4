"""Mepatar on the GPU: every mechanism against the plain fp32 equations, then whole models through the executor, the paged
cache, mixed batches, the engine and the trace replay, in bfloat16 and float32."""
import json
import os
import subprocess
import sys
from dataclasses import replace

import pytest
import torch

from hipengine_b200.ref import mepatar as R

from mepatar_models import (EXACT_MODELS, HEADS, MODELS, ODD, TOL, WIDE, attention, build, delta, dense, last_logits, logit_error, model, moe,
                            needle, retention, tokens, with_masks)

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


def _segments(lens, slots, starts=None):
    from hipengine_b200.models.executor import make_batch
    starts = starts or [0] * len(lens)
    return make_batch([(s, p, [0] * n) for n, s, p in zip(lens, slots, starts)], "cuda")


# ----------------------------------------------------------------------------- grouped norms and the input convolution
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("width,groups,taps", [(132, 6, 4), (248, 4, 2), (160, 1, 7), (64, 64, 1), (96, 3, 3), (4096, 8, 4), (66, 11, 16)])
def test_norm_and_input_convolution(width, groups, taps, dtype):
    """Segments shorter and longer than the convolution and than a tile, on slots with and without a past; groups of one and of
    odd numbers of channels; padded columns; the journal has the past rows after every token while the state stays."""
    from hipengine_b200.ops import linear as LN
    g, hp, eps = _gen(width), _up8(width), 1e-4
    for lens in ([1, 1, 1], [1, 5, 2, 1, 40], [600, 3, 1, 33], [2]):
        n_seg, T = len(lens), sum(lens)
        slots = [(3 * s + 1) % (n_seg + 3) for s in range(n_seg)] if (n_seg + 3) % 3 else list(range(n_seg))
        b, past = _segments(lens, slots), taps - 1
        x = torch.zeros(T, hp)
        x[:, :width] = torch.randn(T, width, generator=g) * torch.logspace(-2, 2, width)
        w1, w2, cw, st = (torch.zeros(*s) for s in ((hp,), (hp,), (taps, hp), (n_seg + 3, past, hp)))
        for t in (w1, w2, cw, st):
            t[..., :width] = torch.randn(*t.shape[:-1], width, generator=g)
        st[slots[0]] = 0
        n1, n2 = (R.grouped_norm(x[:, :width], w[:width], groups, eps) for w in (w1, w2))
        want, states, hist, row = [], {}, [], 0
        for n, s in zip(lens, slots):
            y, states[s] = R.causal_conv(n1[row:row + n], st[s][:, :width], cw[:, :width].t())
            full = torch.cat([st[s][:, :width], n1[row:row + n]])
            hist += [full[t + 1:t + 1 + past] for t in range(n)]
            want.append(n1[row:row + n] + y)
            row += n
        want, tol = torch.cat(want), 3e-6 if dtype == F32 else 0.005
        for journal in ([None, torch.full((T, past, hp), 7.0, device="cuda")] if past else [None]):
            for plain in (True, False):
                a = torch.full((T, hp), 7.0, dtype=dtype, device="cuda")
                p = torch.full((T, hp), 7.0, dtype=dtype, device="cuda") if plain else None
                sc = st.cuda() if past else None
                LN.norm_conv(x.cuda(), w1.cuda(), w2.cuda() if plain else None, cw.cuda(), sc, b, a, p, groups, eps, width, journal=journal)
                step = width // groups if width > groups else width              # groups differ in size
                for i in range(0, width, step):
                    c = slice(i, i + step)
                    _close(a[:, c], want[:, c], tol)
                    if plain:
                        _close(p[:, c], n2[:, c], tol)
                assert not a[:, width:].any() and (p is None or not p[:, width:].any())
                if past == 0:
                    continue
                if journal is not None:
                    _close(journal[..., :width], torch.stack(hist), 3e-6)
                    assert torch.equal(sc.cpu(), st) and not journal[..., width:].any()
                    continue
                for s in range(n_seg + 3):
                    if s in states:
                        _close(sc[s][:, :width], states[s], 3e-6)
                        assert not sc[s][:, width:].any()
                    else:
                        assert torch.equal(sc[s].cpu(), st[s])
        out = torch.full((T, hp), 7.0, dtype=dtype, device="cuda")
        _close(LN.grouped_norm(x.cuda(), w1.cuda(), out, groups, eps, width)[:, :width], n1, tol)
        assert not out[:, width:].any()


# ----------------------------------------------------------------------------- linear attention
def _linear_case(spec, T, seed, dtype, ends):
    """Projected rows, parameters, and what the oracle makes of whole sequences."""
    from hipengine_b200.ops import linear as LN
    g, H, G, d, dv = _gen(seed), spec.heads, spec.kv_heads, spec.dim, spec.vdim
    widths = {"q": G * d, "k": G * d, "v": H * dv, "g": H * dv}
    col, at = {}, 0
    for n, w in widths.items():
        col[n] = (at, at + w)
        at += _up8(w)
    rows = torch.zeros(T, at + 8)
    for n, (a, z) in col.items():
        rows[:, a:z] = torch.randn(T, z - a, generator=g)
    rows = rows.to(dtype).float()
    p = LN.LinearParams(spec, col["k"][0], col["v"][0], col["g"][0])
    q, k, v, z = (rows[:, slice(*col[n])] for n in "qkvg")
    pos = torch.arange(T)
    extra = {}
    if spec.delta:
        conv = {n: torch.randn(widths[n], spec.taps, generator=g) * 0.7 for n in "qkv"}
        p.conv = torch.zeros(spec.taps, spec.conv_cols)
        for n in "qkv":
            p.conv[:, col[n][0]:col[n][1]] = conv[n].t()
        a_log, dt = torch.randn(H, generator=g) * 0.5 - 0.5, torch.randn(H, generator=g) - 2.5
        ab = torch.randn(T, 2 * _up8(H), generator=g)
        p.rate, p.dt, p.gain = torch.exp(a_log), dt, 1 + 0.3 * torch.randn(dv, generator=g)
        past = torch.zeros(spec.taps - 1, 1)
        qc, kc, vc = (R.silu(R.causal_conv(x, past.expand(-1, x.shape[1]), conv[n])[0]) for x, n in ((q, "q"), (k, "k"), (v, "v")))
        spread = lambda x: R.unit(x.reshape(T, G, d)).repeat_interleave(H // G, 1)
        beta = torch.sigmoid(ab[:, :H])
        decay = torch.exp(-p.rate * torch.nn.functional.softplus(ab[:, _up8(H):_up8(H) + H] + dt))
        args = (spread(qc) * d ** -0.5, spread(kc), vc.reshape(T, H, dv), decay, beta)
        run = lambda a, b, S: R.delta_rule(*(x[a:b] for x in args), S)
        extra["ab"] = ab
    else:
        turn = lambda x: R.rotate_halves(x.reshape(T, H, d), pos, spec.rot.dims, spec.rot.base)
        args = (turn(q), turn(k) * d ** -0.5, v.reshape(T, H, dv))
        dec = torch.tensor(spec.decay, dtype=torch.float32)
        run = lambda a, b, S: R.retention(*(x[a:b] for x in args), dec, S)
        p.freq = torch.tensor(spec.rot.table()[0], dtype=torch.float64)
        p.g1 = (torch.tensor(spec.decay, dtype=torch.float64) - 1).float()
        p.powers = LN.decay_powers(spec.decay)
    S, outs, states = torch.zeros(H, d, dv), [], {}
    cuts = sorted(set(ends) | {T})
    a = 0
    for b in cuts:
        o, S = run(a, b, S)
        outs.append(o)
        states[b] = S.clone()
        a = b
    o = R.rms(torch.cat(outs), 1e-3)
    if spec.delta:
        o = o * p.gain
    want = o * R.silu(z.reshape(T, H, dv))
    for n in ("freq", "g1", "powers", "rate", "dt", "conv", "gain"):
        if getattr(p, n) is not None:
            setattr(p, n, getattr(p, n).cuda())
    return p, rows, extra.get("ab"), want, states


def _specs():
    from hipengine_b200.models.config import LinearAttentionSpec as L, RotarySpec
    rot = lambda d, b=5000.0: RotarySpec(d, b, halves=True)
    dec = lambda h: tuple(1 - 0.5 / (2 ** (i % 9)) for i in range(h))
    return {
        "delta-20": L(6, 3, 20, 28, taps=3), "delta-128": L(4, 2, 128, 128, taps=4), "delta-64": L(2, 2, 64, 64, taps=2),
        "delta-1": L(1, 1, 1, 1, taps=1), "delta-wide": L(3, 1, 136, 264, taps=6), "delta-100": L(8, 1, 100, 40, taps=5),
        "delta-512": L(2, 1, 512, 512, taps=3), "delta-40": L(2, 1, 40, 200, taps=4), "delta-16": L(4, 4, 16, 36, taps=9),
        "ret-33": L(3, 3, 33, 18, dec(3), rot(14)), "ret-128": L(4, 4, 128, 128, dec(4), rot(128)),
        "ret-64": L(9, 9, 64, 64, dec(9), rot(64, 1e6)), "ret-2": L(1, 1, 2, 1, (1.0,), rot(2)),
        "ret-wide": L(2, 2, 300, 72, dec(2), rot(200)), "ret-100": L(5, 5, 100, 200, dec(5), rot(32)),
    }


CUTS = {"steps": [1] * 40, "mixed": [5, 1, 1, 30, 2, 64, 1, 7], "chunks": [64, 65, 63, 128, 1, 20], "long": [200, 141], "short": [3, 2, 15]}


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("cut", list(CUTS))
@pytest.mark.parametrize("name", ["delta-20", "delta-128", "delta-64", "delta-1", "delta-wide", "delta-100", "delta-512", "delta-40",
                                  "delta-16", "ret-33", "ret-128", "ret-64", "ret-2", "ret-wide", "ret-100"])
def test_linear_attention(name, cut, dtype):
    """Two sequences, cut differently, in the same batches as a third one that waits between; every form (one-token steps, serial
    scans, chunks) from the states the others left; outputs, states, the convolution's past, states of other slots."""
    from hipengine_b200.models.executor import _Scratch
    from hipengine_b200.ops import kernels as K
    from hipengine_b200.ops import linear as LN
    s = _specs()[name]
    sizes = CUTS[cut]
    T = sum(sizes)
    ends, at = [], 0
    for n in sizes:
        at += n
        ends.append(at)
    cases = [_linear_case(s, T, 10 + i, dtype, ends) for i in range(2)]
    sc, C = _Scratch("cuda", canaries=True), s.conv_cols
    slots, p0 = [2, 0], cases[0][0]
    S = torch.zeros(4, s.heads, s.dim, s.vcols, device="cuda")
    S[1], S[3] = 5.0, 6.0
    ring = torch.zeros(4, s.taps, C, device="cuda") if s.delta and s.taps > 1 else None
    if ring is not None:
        ring[1] = 8.0
    # the parameters are those of the first case; the second sequence's rows go with them too
    rows2 = cases[1][1]
    want2, states2 = _linear_again(s, p0, rows2, cases[1][2], ends)
    want, states = [cases[0][3], want2], [cases[0][4], states2]
    got = [[], []]
    tol = 2e-5 if dtype == F32 else 0.012
    prev = 0
    for j, e in enumerate(ends):
        order = (0, 1) if j % 2 == 0 else (1, 0)
        lens = [e - prev] * 2
        rows = torch.cat([cases[i][1][prev:e] for i in order]).to(dtype).cuda()
        ab = torch.cat([cases[i][2][prev:e] for i in order]).cuda() if s.delta else None
        b = _segments(lens, [slots[i] for i in order], [prev, prev])
        out = torch.full((2 * (e - prev), s.heads * s.vcols), 7.0, dtype=dtype, device="cuda")
        LN.linear_attention(p0, rows, ab, _up8(s.heads), S, ring, b, out, 1e-3, sc)
        K.check_status()
        for k, i in enumerate(order):
            got[i].append(out[k * (e - prev):(k + 1) * (e - prev)].cpu())
            st = S[slots[i]].cpu()
            # chunks take the convolution's values in bfloat16 and everything else as pairs of bfloat16
            _close(st[..., :s.vdim], states[i][e], 2e-5 if dtype == F32 or s.dim > 128 else 6e-3 if s.delta else 5e-5)
            assert not st[..., s.vdim:].any()
        prev = e
    for i in range(2):
        o = torch.cat(got[i]).view(T, s.heads, s.vcols)
        _close(o[..., :s.vdim], want[i], tol)
        assert not o[..., s.vdim:].any()
        if ring is not None:
            for q in range(max(0, T - s.taps + 1), T):
                assert torch.equal(ring[slots[i], q % s.taps].cpu(), cases[i][1][q, :C])
    assert bool((S[1] == 5.0).all()) and bool((S[3] == 6.0).all()) and not sc.check_canaries()
    assert ring is None or (bool((ring[1] == 8.0).all()) and not ring[3].any())


def _linear_again(s, p, rows, ab, ends):
    """The oracle on other rows with the parameters of ``p``."""
    H, G, d, dv, T = s.heads, s.kv_heads, s.dim, s.vdim, rows.shape[0]
    q, k, v, z = rows[:, :G * d], rows[:, p.ck:p.ck + G * d], rows[:, p.cv:p.cv + H * dv], rows[:, p.cz:p.cz + H * dv]
    if s.delta:
        w = p.conv.cpu()
        conv = lambda x, c: R.silu(R.causal_conv(x, torch.zeros(s.taps - 1, x.shape[1]), w[:, c:c + x.shape[1]].t())[0])
        spread = lambda x: R.unit(x.reshape(T, G, d)).repeat_interleave(H // G, 1)
        decay = torch.exp(-p.rate.cpu() * torch.nn.functional.softplus(ab[:, _up8(H):_up8(H) + H] + p.dt.cpu()))
        args = (spread(conv(q, 0)) * d ** -0.5, spread(conv(k, p.ck)), conv(v, p.cv).reshape(T, H, dv), decay, torch.sigmoid(ab[:, :H]))
        run = lambda a, b, S: R.delta_rule(*(x[a:b] for x in args), S)
    else:
        turn = lambda x: R.rotate_halves(x.reshape(T, H, d), torch.arange(T), s.rot.dims, s.rot.base)
        args = (turn(q), turn(k) * d ** -0.5, v.reshape(T, H, dv))
        run = lambda a, b, S: R.retention(*(x[a:b] for x in args), torch.tensor(s.decay, dtype=torch.float32), S)
    S, outs, states, a = torch.zeros(H, d, dv), [], {}, 0
    for b in sorted(set(ends) | {T}):
        o, S = run(a, b, S)
        outs.append(o)
        states[b] = S.clone()
        a = b
    o = R.rms(torch.cat(outs), 1e-3)
    return (o * p.gain.cpu() if s.delta else o) * R.silu(z.reshape(T, H, dv)), states


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", ["delta-20", "delta-100", "ret-33", "delta-1"])
def test_journals_hold_the_state_after_every_token(name, dtype):
    """Verify chains: the states stay, and putting a journalled state in place continues the sequence."""
    from hipengine_b200.models.executor import _Scratch
    from hipengine_b200.ops import linear as LN
    s, T = _specs()[name], 30
    p, rows, ab, want, states = _linear_case(s, T, 3, dtype, list(range(1, T + 1)))
    sc, rows = _Scratch("cuda"), rows.to(dtype).cuda()
    ab = ab.cuda() if s.delta else None
    S = torch.zeros(2, s.heads, s.dim, s.vcols, device="cuda")
    ring = torch.zeros(2, s.taps, s.conv_cols, device="cuda") if s.delta and s.taps > 1 else None
    part = lambda a, z: (rows[a:z], None if ab is None else ab[a:z], _up8(s.heads))
    out = lambda n: torch.empty(n, s.heads * s.vcols, dtype=dtype, device="cuda")
    LN.linear_attention(p, *part(0, 20), S, ring, _segments([20], [1]), out(20), 1e-3, sc)
    keep = (S.clone(), None if ring is None else ring.clone())
    jS = torch.full((6, *S.shape[1:]), 7.0, device="cuda")
    jr = torch.full((6, *ring.shape[1:]), 7.0, device="cuda") if ring is not None else None
    o = out(6)
    LN.linear_attention(p, *part(20, 26), S, ring, _segments([6], [1], [20]), o, 1e-3, sc, jS, jr)
    assert torch.equal(S, keep[0]) and (ring is None or torch.equal(ring, keep[1]))
    _close(o.view(6, s.heads, -1)[..., :s.vdim], want[20:26], 2e-5 if dtype == F32 else 0.012)
    for j in range(6):
        _close(jS[j][..., :s.vdim], states[21 + j], 2e-5 if dtype == F32 else 6e-3)
        assert not jS[j][..., s.vdim:].any()
    for accepted in (1, 4, 6):
        S[1] = jS[accepted - 1]
        if ring is not None:
            ring[1] = jr[accepted - 1]
        a = 20 + accepted
        o = out(T - a)
        LN.linear_attention(p, *part(a, T), S, ring, _segments([T - a], [1], [a]), o, 1e-3, sc)
        _close(o.view(T - a, s.heads, -1)[..., :s.vdim], want[a:], 2e-5 if dtype == F32 else 0.012)


@pytest.mark.parametrize("form", ["chunks", "serial", "steps"])
def test_long_memories_keep_their_accuracy(form):
    """Heads that forget one part in fifty thousand per token, driven by a constant for 3000 tokens, neither drift nor lose
    what came first; the delta rule unlearns a key it is shown again."""
    from hipengine_b200.models.config import LinearAttentionSpec, RotarySpec
    from hipengine_b200.models.executor import _Scratch
    from hipengine_b200.ops import linear as LN
    T, dec = 3000, (1 - 2e-5, 1 - 1e-3, 1 - 2.0 ** -10)
    s = LinearAttentionSpec(3, 3, 16, 8, dec, RotarySpec(2, 10.0, halves=True))
    dtype = BF if form == "chunks" else F32
    p = LN.LinearParams(s, 48, 96, 120, torch.zeros(1, dtype=torch.float64).cuda(), (torch.tensor(dec, dtype=torch.float64) - 1).float().cuda(),
                        LN.decay_powers(dec).cuda())
    rows = torch.ones(T, 144, dtype=dtype, device="cuda")
    S, sc = torch.zeros(1, 3, 16, 8, device="cuda"), _Scratch("cuda")
    if form == "steps":
        for t in range(0, 600):
            LN.linear_attention(p, rows[:1], None, 8, S, None, _segments([1], [0], [t]), torch.empty(1, 24, device="cuda"), 1e-3, sc)
        n = 600
    else:
        n = T
        LN.linear_attention(p, rows, None, 8, S, None, _segments([T], [0]), torch.empty(T, 24, dtype=dtype, device="cuda"), 1e-3, sc)
    d = torch.tensor(dec, dtype=torch.float64)
    want = 0.25 * (1 - d ** n) / (1 - d)
    _close(S[0, :, 3, 4], want, 3e-5)


# ----------------------------------------------------------------------------- attention: window and kept first tokens
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


@pytest.mark.parametrize("window,keep", [(1, 0), (1, 1), (16, 5), (40, 16), (65, 33), (64, 300), (130, 64), (0, 9)])
@pytest.mark.parametrize("H,G,D", [(1, 1, 64), (6, 2, 64), (15, 3, 128), (40, 4, 128), (4, 4, 256), (14, 2, 64), (3, 1, 512)])
def test_attention_over_a_window_and_the_first_tokens(H, G, D, window, keep):
    """Single tokens, portions of several requests in one launch, and the fp32 form, with contexts that end inside, at and behind
    the kept tokens and the window; one key stands out, just inside or just outside the window or the kept tokens."""
    from hipengine_b200.ops import attention as A
    from hipengine_b200.ops import kernels as K
    ctxs = [1, 2, 16, 17, 64, 65, 129, 300, 131, 67, 290, 299]
    g, n, scale = _gen(H), len(ctxs), 1.5 / D ** 0.5
    segs = [(7, 100, 200), (2, 3, 13), (6, 0, 129), (10, 280, 10)]
    sc = torch.full((H,), scale)

    def plain(q, k, v, pos):
        return R.attention(q, k, v, pos, sc, window or k.shape[0] + 1, keep)

    for dtype in (BF, F32):
        cache, bt, ks, vs = _cache(ctxs, G, D, dtype, H + D)
        q = torch.randn(n, H, D, generator=g).to(dtype).float()
        for s, c in enumerate(ctxs):
            j = (c - window, c - window - 1, keep - 1, keep)[s % 4] if window else s
            if 0 <= j < c:
                ks[s][j] = (q[s, ::H // G] * 3).to(dtype).float()
                cache[bt[s, j // 16], 0, :, j % 16] = ks[s][j].to(dtype).cuda()
        want = torch.cat([plain(q[s:s + 1], ks[s], vs[s], torch.tensor([c - 1])) for s, c in enumerate(ctxs)])
        out = torch.full((n, H * D), 7.0, dtype=dtype, device="cuda")
        rows = (cache, bt, torch.arange(n, dtype=torch.int32, device="cuda"), _i32(ctxs))
        if dtype == F32:
            K.attn_exact(q.cuda(), *rows, out, H, G, D, 16, scale, 0.0, window, keep_first=keep)
            _close(out.view(n, H, D), want, 1e-4)
            continue
        for span in (64, 128, 320):
            splits = -(-(min(300, window + keep) if window else 300) // span)
            part = torch.full((K.attn_decode_scratch_floats(n, H, splits, D),), float("nan"), device="cuda")
            K.attn_decode(q.to(BF).cuda(), None, *rows, part, out, H, G, D, 16, span, splits, scale, window, keep_first=keep)
            K.check_status()
            _close(out.view(n, H, D), want, 0.02)
        if not A.flash_prefill_available(D):
            continue
        start = [0]
        for _, _, m in segs:
            start.append(start[-1] + m)
        qs = torch.randn(start[-1], H, D, generator=g).to(BF).float()
        for (s, p0, m), a in zip(segs, start):                              # rows that ask for the edge keys
            for r in range(0, m, 3):
                p = p0 + r
                j = (p - window + 1, p - window, keep - 1, keep)[r % 4] if window else r
                if 0 <= j <= p:
                    qs[a + r] = (ks[s][j].repeat_interleave(H // G, 0) * 2).to(BF).float()
        want = torch.cat([plain(qs[a:a + m], ks[s][:p0 + m], vs[s][:p0 + m], torch.arange(p0, p0 + m))
                          for (s, p0, m), a in zip(segs, start)])
        out = torch.full((qs.shape[0], H * D), 7.0, dtype=BF, device="cuda")
        pos = _i32([p for _, p0, m in segs for p in range(p0, p0 + m)])
        for first in (0, 1):
            A.flash_prefill_segs(qs.to(BF).cuda(), None, cache, bt, _i32(start)[first:], _i32([s for s, _, _ in segs])[first:],
                                 pos, [m for _, _, m in segs[first:]], out, H, G, D, 16, scale, window, keep_first=keep)
            _close(out[start[first]:].view(-1, H, D), want[start[first]:], 0.03)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("T,H,G,dim,vdim,rd", [(6, 3, 1, 20, 28, 10), (150, 21, 3, 64, 48, 64), (9, 40, 4, 128, 128, 64), (1, 1, 1, 2, 2, 2)])
def test_head_rows_with_gains_per_head(T, H, G, dim, vdim, rd, dtype):
    """Biases, norm, rotation of neighbours; query gains of their own for every head carry the factor of the scores."""
    from hipengine_b200.models.config import RotarySpec, padded_head_width
    from hipengine_b200.models.executor import make_batch
    from hipengine_b200.ops import mixers as MX
    g, eps, D = _gen(H + dim), 1e-3, padded_head_width(max(dim, vdim))
    rot = RotarySpec(rd, 5000.0)
    pos = torch.tensor(([0, 1, 15, 16, 4097, 70001] * 25)[:T])
    x = {n: torch.randn(T, w, generator=g).to(dtype).float() for n, w in (("q", H * dim), ("k", G * dim), ("v", G * vdim))}
    bias = {n: torch.randn(t.shape[1], generator=g) for n, t in x.items()}
    gain, temp = {n: 1 + torch.rand(dim, generator=g) for n in "qk"}, torch.randn(H, generator=g)
    head = lambda n, h: R.rotate_neighbours(R.rms((x[n] + bias[n]).reshape(T, h, dim), eps) * gain[n], pos, rd, 5000.0)
    pad = lambda t: torch.nn.functional.pad(t, (0, _up8(t.shape[-1]) - t.shape[-1]))
    rows = lambda n, h, d, gn: MX.HeadRows(pad(x[n]).to(dtype).cuda(), h, d, pad(bias[n]).cuda(), None if gn is None else gn.cuda())
    b = make_batch([(t, int(p), [0]) for t, p in enumerate(pos)], "cuda")
    bt = torch.zeros(T, 70016 // 16, dtype=torch.int32)
    for t, p in enumerate(pos):
        bt[t, p // 16] = t
    q_out = torch.full((T, H, D), 7.0, dtype=dtype, device="cuda")
    cache = torch.full((T, 2, G, 16, D), 7.0, dtype=dtype, device="cuda")
    MX.mixer_post(rows("q", H, dim, temp[:, None] * gain["q"]), rows("k", G, dim, gain["k"]), rows("v", G, vdim, None), "head", rot,
                  torch.tensor(rot.table()[0], dtype=torch.float64, device="cuda"), 1.0, q_out, cache, 16, b, bt.cuda(), eps)
    tol = 3e-5 if dtype == F32 else 0.01
    _close(q_out[:, :, :dim], head("q", H) * temp[:, None], tol)
    got = torch.stack([cache[t, :, :, p % 16] for t, p in enumerate(pos)])
    _close(got[:, 0, :, :dim], head("k", G), tol)
    _close(got[:, 1, :, :vdim], (x["v"] + bias["v"]).reshape(T, G, vdim), tol)
    assert not q_out[:, :, dim:].any() and not got[:, 0, :, dim:].any() and not got[:, 1, :, vdim:].any()


# ----------------------------------------------------------------------------- experts, output biases
@pytest.mark.parametrize("E,k", [(1, 1), (5, 2), (8, 8), (40, 6), (200, 32), (512, 3)])
def test_softmax_routing_keeps_the_scores(E, k):
    from hipengine_b200.ops import kernels as K
    T = 37
    lg = torch.randn(T, _up8(E) + 8, generator=_gen(E)) * 3
    ids, w = torch.zeros(T, k, dtype=torch.int32, device="cuda"), torch.zeros(T, k, device="cuda")
    K.moe_route(lg.cuda(), k, ids, w, n_experts=E, mode=2)
    wi, ww = R.routing(lg[:, :E], k)
    assert torch.equal(ids.cpu().long(), wi)
    assert torch.allclose(w.cpu(), ww, rtol=2e-6, atol=1e-9)


@pytest.mark.parametrize("mode", ["few fp32 rows", "few bf16 rows", "float32"])
def test_clamped_experts_of_prepared_rows(mode):
    """Experts on rows that are normalised already, with a limit that binds on both branches."""
    from hipengine_b200.ops import kernels as K
    g, T, E, k, H, F, limit = _gen(1), 13, 6, 3, 72, 40, 0.7
    x = torch.randn(T, H, generator=g).to(BF).float()
    gu, dn = (torch.randn(E, 2 * F, H, generator=g) / 6).to(BF), (torch.randn(E, H, F, generator=g) / 5).to(BF)
    ids = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)])
    w = torch.rand(T, k, generator=g)
    h = torch.randn(T, H, generator=g)
    want = h.clone()
    for t in range(T):
        for j in range(k):
            e = int(ids[t, j])
            want[t] += w[t, j] * R.clamped_expert(x[t:t + 1], gu[e, :F].float(), gu[e, F:].float(), dn[e].float(), limit)[0]
    hc, ic, wc = h.cuda(), ids.int().cuda(), w.cuda()
    guc, dnc = gu.reshape(-1, H).cuda(), dn.reshape(-1, F).cuda()
    if mode == "float32":
        K.moe_exact(x.cuda(), ic, wc, guc, dnc, E, torch.empty(T * k, F, device="cuda"), hc, act="clamped_glu", limit=limit)
    else:
        rows = torch.empty(T * k, F, dtype=BF, device="cuda")
        K.moe_gateup_float(x.to(BF if "bf16" in mode else F32).cuda(), None, 1e-5, H, ic, wc, guc, E, rows, act="clamped_glu", limit=limit)
        K.moe_down_float(rows, ic, dnc, E, hc)
    _close(hc - h.cuda(), want - h, 1e-5 if mode == "float32" else 0.01)


@pytest.mark.parametrize("T", [1, 9, 16, 100, 128, 300])
def test_output_bias_is_added_once(T):
    from hipengine_b200.models.executor import _Scratch
    from hipengine_b200.ops import gemm as GM
    from hipengine_b200.ops import kernels as K
    g, N, K1 = _gen(T), 264, 136
    x, w, h, bias = torch.randn(T, K1, generator=g).to(BF), (torch.randn(N, K1, generator=g) / 12).to(BF), torch.randn(T, N, generator=g), torch.randn(N, generator=g)
    prod, xc, wc, bc = x.float() @ w.float().t(), x.cuda(), w.cuda(), bias.cuda()
    runs = {"exact": lambda o: K.small_gemm_f32(xc.float(), wc, o, add=True, col_bias=bc),
            "gemm": lambda o: GM.gemm_bf16(xc, wc, o, epi=GM.EPI_ADD, col_bias=bc)}
    if T <= 128:
        runs["split"] = lambda o: GM.gemm_bf16_splitk_det(xc, wc, o, _Scratch("cuda"), add=True, col_bias=bc)
    if T <= 16:
        runs["few"] = lambda o: K.gemv_sum(o, [(xc, wc, None)], bc)
        runs["two"] = lambda o: K.gemv_sum(o, [(xc, wc, None), (xc, wc, None)], bc)
    for name, run in runs.items():
        o = h.cuda()
        run(o)
        _close(o, h + bias + prod * (2 if name == "two" else 1), 1e-4)
    K.check_status()


# ----------------------------------------------------------------------------- whole models
DTYPES = ["float32", "bfloat16"]


def _executor(cfg_json, dtype, seed=0, max_slots=4, max_context=320, clear=True, **kw):
    from hipengine_b200.models import make_executor
    w, ref, t = build(cfg_json, seed, clear)
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


def _tol(name, dtype):
    return 3e-3 if name == "single" else TOL[dtype]


NAMES = [(n, "float32") for n in EXACT_MODELS] + [(n, "bfloat16") for n in MODELS]


@pytest.mark.parametrize("name,dtype", NAMES)
def test_layers_one_by_one(name, dtype):
    ex, ref, _ = _executor(EXACT_MODELS[name], dtype)
    for n in (37, 11):                                                        # both sides of the switch of kernels
        ids = tokens(n, EXACT_MODELS[name]["vocab"], 2)
        got, want = [], []
        ex.on_layer_run = lambda run, h: got.append(h.clone().cpu())
        _run(ex, [(0, 0, ids)])
        ref.forward_raw(torch.tensor(ids), ref.new_state(), want)
        assert len(got) == len(want) == len(ex.cfg.layer_specs)
        for g, w in zip(got, want):
            _close(g, w, 2e-3 if name == "single" else 5e-5 if dtype == "float32" else 0.04)


@pytest.mark.parametrize("name", ["odd", "heads", "wide"])
def test_undecided_routers_in_float32(name):
    """Random routers, whose choices bfloat16 would turn now and then."""
    ex, ref, _ = _executor(MODELS[name], "float32", seed=2, clear=False)
    ids = tokens(120, MODELS[name]["vocab"], 2)
    assert logit_error(_run(ex, [(0, 0, ids)]), ref.forward(torch.tensor(ids))[0]) < TOL["float32"]


@pytest.mark.parametrize("name,dtype", NAMES)
def test_prompts_portions_and_single_tokens_agree(name, dtype):
    """Whole prompt, portions of several sizes down to two tokens, and token by token: each against the oracle."""
    ex, ref, _ = _executor(EXACT_MODELS[name], dtype)
    ids = tokens(150, EXACT_MODELS[name]["vocab"], 5)
    want = ref.forward(torch.tensor(ids))[0]
    assert logit_error(_run(ex, [(0, 0, ids)]), want) < _tol(name, dtype)
    for slot, sizes in ((1, [2] * 75), (2, [31, 1, 2, 64, 3, 17, 16, 9, 7]), (3, [140] + [1] * 10)):
        parts, at = [], 0
        for n in sizes:
            parts.append(_run(ex, [(slot, at, ids[at:at + n])]))
            at += n
        assert at == 150 and logit_error(torch.cat(parts), want) < _tol(name, dtype), sizes
    parts = [_run(ex, [(0, p, [ids[p]])]) for p in range(50)]
    assert logit_error(torch.cat(parts), want[:50]) < _tol(name, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_few_and_many_rows_meet_at_every_batch_size(dtype):
    """Row counts on both sides of every switch of kernels (1, 8, 16, 17, 64, 128, 129 rows)."""
    ex, ref, _ = _executor(ODD, dtype)
    ids = tokens(140, ODD["vocab"], 6)
    want = ref.forward(torch.tensor(ids))[0]
    for n in (1, 2, 8, 9, 15, 16, 17, 33, 63, 64, 65, 127, 128, 129, 140):
        assert logit_error(_run(ex, [(0, 0, ids[:n])]), want[:n]) < TOL[dtype], n


@pytest.mark.parametrize("name,dtype", NAMES)
def test_unequal_requests_in_one_batch(name, dtype):
    """Portions of some requests beside single tokens of others, in any order, against each request alone."""
    ex, ref, _ = _executor(EXACT_MODELS[name], dtype)
    seqs = [tokens(n, EXACT_MODELS[name]["vocab"], n) for n in (90, 23, 61, 130)]
    want = [ref.forward(torch.tensor(s))[0] for s in seqs]
    at = [0] * 4
    plan = [[(3, 40), (0, 1)], [(0, 50), (1, 2), (3, 1)], [(2, 17), (3, 33), (1, 1), (0, 1)], [(0, 1), (3, 1), (1, 1)],
            [(1, 19), (2, 1), (0, 2), (3, 55)], [(2, 43), (0, 35)]]
    for step in plan:
        segs = [(r, at[r], seqs[r][at[r]:at[r] + n]) for r, n in step]
        got, row = _run(ex, segs), 0
        for r, n in step:
            assert logit_error(got[row:row + n], want[r][at[r]:at[r] + n]) < _tol(name, dtype), (step, r)
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
    cfg = model(96, 160, [(attention(4, 2, 24, 24, 1.5, 400, 0, 8, 500.0), dense(64)), (attention(6, 3, 40, 32, 1.0, 30, 200, 16, 900.0), None)])
    w, ref, _ = needle(cfg, strength=2.0)
    ex = make_executor(w, dtype=dtype, device="cuda", max_slots=4, max_context=320)
    base = [3 + t for t in tokens(131, 157, 8)]
    base[130] = 1
    plain = last_logits(ref, base)
    for p in (0, 1, 15, 16, 17, 63, 64, 111, 112, 128, 129):
        ids = list(base)
        ids[p] = 2
        want = last_logits(ref, ids)
        assert logit_error(plain, want) > 4 * TOL[dtype]
        for cut in (0, 97, 128, 130):
            assert logit_error(_ask(ex, 0, ids, cut), want) < TOL[dtype], (p, cut)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep", [(1, 0), (1, 1), (2, 16), (16, 5), (33, 20), (40, 0)])
def test_key_at_the_edges_of_the_mask(size, keep, dtype):
    """Keys just inside and just outside the window, and the last kept and the next token, in prompts, portions and decoding.
    (The oracle with masks one token longer gives other logits, so an edge that is off shows.)"""
    from hipengine_b200.models import make_executor
    cfg = model(96, 160, [(attention(4, 2, 24, 16, 1.0, size, keep, 8, 500.0), dense(64)), (attention(4, 2, 24, 24, 0.9, size, keep, 8, 500.0), None)])
    w, ref, t = needle(cfg, 2.0)
    ex = make_executor(w, dtype=dtype, device="cuda", max_slots=4, max_context=320)
    base = [3 + x for x in tokens(120, 157, 8)]
    for last in (47, 48, 63, 90, 119):
        for place in ("window in", "window out", "first in", "first out"):
            at = {"window in": last - size + 1, "window out": last - size, "first in": keep - 1, "first out": keep}[place]
            if not 0 <= at <= last:
                continue
            ids = base[:last + 1]
            ids[last] = 1
            if at < last:
                ids[at] = 2
            want = last_logits(ref, ids)
            if place.endswith("out") and at < last - size + 1 and at >= keep:
                longer = with_masks(cfg, size=1) if place == "window out" else with_masks(cfg, keep=1)
                assert logit_error(last_logits(R.MepatarRef(longer, t), ids), want) > 4 * TOL[dtype]
            for cut in (0, last - 20, last - 2, last):
                assert logit_error(_ask(ex, 1, ids, cut), want) < TOL[dtype], (last, place, cut)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["delta", "retention"])
def test_long_decoding_carries_the_state(kind, dtype):
    """One token at a time for several hundred tokens after a prompt, states of long memory."""
    mix = delta(4, 2, 24, 32, 4) if kind == "delta" else retention(3, 40, 24, (0.999, 0.99, 0.9995), 20, 5000.0)
    cfg = model(96, 160, [(mix, dense(64)), (mix, None)], groups=3)
    ex, ref, _ = _executor(cfg, dtype, max_context=512)
    ids = tokens(400, 160, 1)
    want = ref.forward(torch.tensor(ids))[0]
    assert logit_error(_run(ex, [(1, 0, ids[:70])]), want[:70]) < TOL[dtype]
    got = torch.cat([_run(ex, [(1, p, [ids[p]])]) for p in range(70, 400)])
    assert logit_error(got, want[70:]) < TOL[dtype]


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
        for cfg in (ODD, WIDE, HEADS):
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
    """A cached prefix is only usable with the states at its last token: the continuation of a reused prefix is the oracle's,
    from the device cache and from the cold tier."""
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(ODD, 4)
    a = tokens(50, ODD["vocab"], 9)
    other = [tokens(60, ODD["vocab"], 20 + i) for i in range(4)]
    prompts = [a, a[:48] + tokens(5, ODD["vocab"], 2), a[:33] + tokens(3, ODD["vocab"], 3)]
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


def test_a_model_without_a_cache_generates():
    """No attention layer at all: pages are accounted for and hold nothing."""
    from hipengine_b200.llm import LLM, SamplingParams
    cfg = model(96, 160, [(delta(4, 2, 24, 32, 3), dense(64)), (retention(3, 40, 24, (0.99, 0.9, 0.999), 20, 5000.0), moe(4, 2, 24, 1.0))], groups=3)
    w, ref, _ = build(cfg, 1)
    assert w.config.kv_bytes_per_token() == 0
    prompts = [tokens(n, 160, n) for n in (20, 1, 33)]
    with LLM(w, dtype="float32", max_active_requests=2, max_sequence_length=128) as llm:
        got = llm.generate_token_ids(prompts, SamplingParams(max_tokens=10, ignore_eos=True))
    _check_greedy(ref, prompts, got, 10)


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
    """Rejected drafts leave neither cache rows nor states behind."""
    from hipengine_b200.llm import LLM, SamplingParams
    w, ref, _ = build(ODD, 4)
    prompt = (tokens(12, ODD["vocab"], 9) * 3)[:30]
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


@pytest.mark.parametrize("name,dtype", [("odd", "float32"), ("ones", "float32"), ("odd", "bfloat16"), ("heads", "bfloat16")])
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
