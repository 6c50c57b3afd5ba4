"""Plain fp32 reference of the Milutar decoder, one function per mechanism, token order preserved.

Written from the layer equations and kept apart from the product path: it takes the decoded ``config.json`` (a dict) and
the checkpoint tensors under their own names; no configuration reader, weight packing or kernel launcher is involved.
Used as the oracle of the tests and by the ``cpu_reference`` backend.

    x_p    = E[token_p]
    layer  : h = g x / rms(x);  x += m (a * mixer(shift(h)) + b * ff(h))       a, b: per-channel vectors, m: a constant
    shift  : h_p + s * (h_{p-1} - h_p), with h_{-1} = 0
    mixer  : attention whose keys and values are two linear maps of one short latent row per position, plus a rotated
             key part that all heads share; full causal with a learned sink, or a sliding window
    loop   : a range of layers runs several times with the same weights; pass t starts from x + step_t
    logits = head norm(x)
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def token_shift(h: torch.Tensor, before: torch.Tensor, amount: torch.Tensor) -> torch.Tensor:
    """Move every row of h [T, W] towards the row before it; ``before`` [W] precedes the first one."""
    prev = torch.cat([before[None], h[:-1]], 0)
    return h + (prev - h) * amount


def rotation_freqs(dims: int, base: float, scaling: Optional[Mapping[str, Any]] = None) -> Tuple[torch.Tensor, float]:
    """(angular frequency per pair [dims / 2], amplitude of sine and cosine)."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=torch.float64), 1.0
    factor, orig = float(scaling["factor"]), float(scaling["original"])

    def pair_of(turns: float) -> float:
        """Index of the pair that makes ``turns`` turns over the original context."""
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x: torch.Tensor, pos: torch.Tensor, freqs: torch.Tensor, amp: float) -> torch.Tensor:
    """Rotate neighbouring pairs (x_{2i}, x_{2i+1}) of the last dimension by pos * freqs[i]; x [T, ..., 2 * pairs]."""
    a = pos.double()[:, None] * freqs[None]
    a = a.reshape(a.shape[0], *([1] * (x.dim() - 2)), a.shape[1])
    c, s = (torch.cos(a) * amp).float(), (torch.sin(a) * amp).float()
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


def visible_keys(pos: torch.Tensor, n_keys: int, window: int = 0) -> torch.Tensor:
    """[T, n_keys] bool: key j is seen from position i iff 0 <= i - j (< window when there is one)."""
    d = pos[:, None] - torch.arange(n_keys)[None, :]
    return (d >= 0) & (d < window) if window > 0 else d >= 0


def softmax_with_sink(s: torch.Tensor, seen: torch.Tensor, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Weights over the seen keys; ``sink`` (a scalar) adds one more term to the denominator only."""
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    if sink is None:
        return torch.softmax(s, -1)
    return torch.softmax(torch.cat([s, sink.expand(s.shape[0], 1)], 1), -1)[:, :-1]


def latent_attention(q: torch.Tensor, lat: torch.Tensor, rot: torch.Tensor, w_key: torch.Tensor, w_val: torch.Tensor,
                     pos: torch.Tensor, heads: int, scale: float, window: int = 0,
                     sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [T, heads, dim + rot_dim] (rotated part last, already rotated); lat [S, rank] and rot [S, rot_dim] of positions
    0..S-1; w_key [heads * dim, rank], w_val [heads * vdim, rank].  Returns [T, heads * vdim]."""
    T, S, rd = q.shape[0], lat.shape[0], rot.shape[1]
    dim = q.shape[2] - rd
    keys = (lat @ w_key.t()).reshape(S, heads, dim)
    vals = (lat @ w_val.t()).reshape(S, heads, -1)
    seen = visible_keys(pos, S, window)
    out = []
    for h in range(heads):
        s = (q[:, h, :dim] @ keys[:, h].t() + q[:, h, dim:] @ rot.t()) * scale
        out.append(softmax_with_sink(s, seen, None if sink is None else sink[h]) @ vals[:, h])
    return torch.cat(out, 1)


def squared_relu(x: torch.Tensor) -> torch.Tensor:
    return torch.relu(x) ** 2


class MilutarState:
    """What one request carries, per layer run: latents, rotated key parts and the last normalised row."""

    def __init__(self):
        self.pos = 0
        self.lat: Dict[int, torch.Tensor] = {}
        self.rot: Dict[int, torch.Tensor] = {}
        self.last: Dict[int, torch.Tensor] = {}

    def clone(self) -> "MilutarState":
        c = MilutarState()
        c.pos = self.pos
        c.lat, c.rot, c.last = ({i: t.clone() for i, t in d.items()} for d in (self.lat, self.rot, self.last))
        return c


class MilutarRef:
    def __init__(self, config: Mapping[str, Any], tensors: Mapping[str, torch.Tensor]):
        self.c = config
        self.t = {n: v.detach().to("cpu", torch.float32) for n, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])
        self.mult = float(config["residual_mult"])

    def new_state(self) -> MilutarState:
        return MilutarState()

    def schedule(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass) per layer run; pass is None outside the loop."""
        n, loop = len(self.c["layers"]), self.c.get("loop")
        order: List[Tuple[int, Optional[int]]] = []
        for i in range(n):
            if loop and i == loop["start"]:
                order += [(j, t) for t in range(loop["times"]) for j in range(loop["start"], loop["stop"])]
            elif not loop or not loop["start"] < i < loop["stop"]:
                order.append((i, None))
        return order

    def scalar_norm(self, x: torch.Tensor, name: str) -> torch.Tensor:
        return rms(x, self.eps) * self.t[name].reshape(())

    def mixer(self, i: int, run: int, h: torch.Tensor, st: MilutarState, pos: torch.Tensor) -> torch.Tensor:
        L, p = self.c["layers"][i], f"l{i}.mix."
        m, t = L["mixer"], self.t
        H, rank = m["heads"], m["kv_rank"]
        if L["type"] == "latent_attention_2":
            q = (rms(h @ t[p + "dq"].t(), self.eps) * t[p + "dq.norm"]) @ t[p + "uq"].t()
            sink: Optional[torch.Tensor] = t[p + "sink"]
        else:
            q, sink = h @ t[p + "q"].t(), None
        q = q.reshape(h.shape[0], H, -1)
        down = h @ t[p + "dkv"].t()
        lat = rms(down[:, :rank], self.eps) * t[p + "dkv.norm"]
        f, amp = rotation_freqs(m["rot"]["dims"], float(m["rot"]["base"]), m["rot"].get("scaling"))
        rot = rotate_pairs(down[:, rank:], pos, f, amp)
        d = m["dim"]
        q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], pos, f, amp)], -1)
        for store, new in ((st.lat, lat), (st.rot, rot)):
            store[run] = torch.cat([store[run], new], 0) if run in store else new
        window = int((m.get("mask") or {}).get("size", 0))
        o = latent_attention(q, st.lat[run], st.rot[run], t[p + "uk"], t[p + "uv"], pos, H, float(m["scale"]), window, sink)
        return o @ t[p + "o"].t()

    def ff(self, i: int, h: torch.Tensor) -> torch.Tensor:
        p = f"l{i}.mlp."
        return squared_relu(h @ self.t[p + "up"].t()) @ self.t[p + "down"].t()

    def forward_raw(self, tokens: torch.Tensor, st: MilutarState, trace: Optional[list] = None) -> torch.Tensor:
        """Residual rows [T, width] after the last layer for ``tokens`` at positions st.pos ..; ``trace`` collects the
        residual after every layer run."""
        T = tokens.shape[0]
        pos = torch.arange(st.pos, st.pos + T)
        x = self.t["embed"][tokens.long()]
        loop = self.c.get("loop")
        for run, (i, t) in enumerate(self.schedule()):
            p = f"l{i}."
            if t is not None and i == loop["start"]:
                x = x + self.t["loop.step"][t]
            h = self.scalar_norm(x, p + "norm1")
            before = st.last.get(run, torch.zeros(x.shape[1]))
            st.last[run] = h[-1]
            add = self.t[p + "ls1"] * self.mixer(i, run, token_shift(h, before, self.t[p + "shift"]), st, pos)
            if self.c["layers"][i]["mlp"] is not None:
                add = add + self.t[p + "ls2"] * self.ff(i, h)
            x = x + self.mult * add
            if trace is not None:
                trace.append(x.clone())
        st.pos += T
        return x

    def forward_hidden(self, tokens: torch.Tensor, st: MilutarState) -> torch.Tensor:
        return self.scalar_norm(self.forward_raw(tokens, st), "final.norm")

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return hidden @ self.t["head"].t()

    def forward(self, tokens: torch.Tensor, st: Optional[MilutarState] = None) -> Tuple[torch.Tensor, MilutarState]:
        st = st or self.new_state()
        return self.logits(self.forward_hidden(tokens, st)), st
