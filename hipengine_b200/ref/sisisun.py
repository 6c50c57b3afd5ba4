"""Plain fp32 reference of the Sisisun decoder, one function per mechanism, token order preserved.

Written from the layer equations and kept apart from the product path on purpose: it takes the decoded ``config.json``
(a dict) and the checkpoint tensors under their own names, so neither the configuration reader, nor the weight packing,
nor any kernel launcher is involved.  Used as the oracle of the tests and by the ``cpu_reference`` backend.

    x_p    = E[token_p] + s_p                        s_p: interleaved sin / cos of p * 10000^(-2i/width)
    layer  : x += attention(norm1(x)); x += ff(norm2(x))         norm(x) = x / rms(x) * (1 + w)
    loop   : a range of layers runs several times with the same weights; pass t starts from x + [t > 0] x_p + step_t
    logits = head norm(x)
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) * w over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sinusoid(pos: torch.Tensor, width: int) -> torch.Tensor:
    """[T, width]: entry 2i = sin(p * 10000^(-2i/width)), entry 2i + 1 = cos of the same angle."""
    out = torch.zeros(pos.numel(), width, dtype=torch.float64)
    for c in range(width):
        i = c // 2
        ang = pos.double() * (10000.0 ** (-2.0 * i / width))
        out[:, c] = torch.sin(ang) if c % 2 == 0 else torch.cos(ang)
    return out.to(torch.float32)


def softcap_score(s: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(s / cap)


def attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, pos: torch.Tensor, scale: float,
              cap: float) -> torch.Tensor:
    """q [T, H, D] at positions ``pos``; k [S, G, D], v [S, G, Dv] for positions 0..S-1 -> [T, H, Dv]."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    out = torch.zeros(T, H, v.shape[2], dtype=torch.float32)
    visible = torch.arange(S)[None, :] <= pos[:, None]
    for h in range(H):
        g = h // (H // G)
        s = softcap_score((q[:, h] @ k[:, g].t()) * scale, cap)
        p = torch.softmax(torch.where(visible, s, torch.full_like(s, -math.inf)), -1)
        out[:, h] = p @ v[:, g]
    return out


def clamped_glu(g: torch.Tensor, u: torch.Tensor, limit: float) -> torch.Tensor:
    g = torch.minimum(g, torch.full_like(g, limit))
    u = u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def silu_glu(g: torch.Tensor, u: torch.Tensor) -> torch.Tensor:
    return g * torch.sigmoid(g) * u


def route(z: torch.Tensor, top: int, n_groups: int, keep: int, scale: float) -> Tuple[List[int], List[float]]:
    """One token's router logits -> (expert ids, weights): sigmoid scores; groups of neighbouring experts ranked by the
    sum of their two largest scores, the best ``keep`` stay; the ``top`` best experts of those, weights normalised."""
    s = torch.sigmoid(z).tolist()
    size = len(s) // n_groups
    rank = sorted(range(n_groups), key=lambda a: -sum(sorted(s[a * size:(a + 1) * size])[-2:]))
    open_experts = [e for a in rank[:keep] for e in range(a * size, (a + 1) * size)]
    ids = sorted(open_experts, key=lambda e: (-s[e], e))[:top]
    tot = sum(s[e] for e in ids) + 1e-20
    return ids, [s[e] / tot * scale for e in ids]


class SisisunState:
    """Keys and values of one request, per layer run."""

    def __init__(self):
        self.pos = 0
        self.k: Dict[int, torch.Tensor] = {}
        self.v: Dict[int, torch.Tensor] = {}

    def clone(self) -> "SisisunState":
        c = SisisunState()
        c.pos = self.pos
        c.k = {i: t.clone() for i, t in self.k.items()}
        c.v = {i: t.clone() for i, t in self.v.items()}
        return c


class SisisunRef:
    def __init__(self, config: Mapping[str, Any], tensors: Mapping[str, torch.Tensor]):
        self.c = config
        self.t = {n: v.detach().to("cpu", torch.float32) for n, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])

    def new_state(self) -> SisisunState:
        return SisisunState()

    def schedule(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass) per layer run; pass is None outside the loop."""
        n, loop = len(self.c["layers"]), self.c.get("loop")
        if not loop:
            return [(i, None) for i in range(n)]
        a, b = loop["start"], loop["stop"]
        out: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(a)]
        for t in range(loop["times"]):
            out += [(i, t) for i in range(a, b)]
        return out + [(i, None) for i in range(b, n)]

    def norm(self, x: torch.Tensor, name: str) -> torch.Tensor:
        return rms_norm(x, 1.0 + self.t[name], self.eps)

    def mixer(self, i: int, run: int, x: torch.Tensor, st: SisisunState, pos: torch.Tensor) -> torch.Tensor:
        m, p = self.c["layers"][i]["mixer"], f"l{i}.mix."
        T = x.shape[0]
        q = (x @ self.t[p + "q"].t()).reshape(T, m["heads"], m["dim"])
        k = (x @ self.t[p + "k"].t()).reshape(T, m["kv_heads"], m["dim"])
        v = (x @ self.t[p + "v"].t()).reshape(T, m["kv_heads"], m["vdim"])
        q = rms_norm(q, self.t[p + "q.norm"], self.eps)
        k = rms_norm(k, self.t[p + "k.norm"], self.eps)
        st.k[run] = k if run not in st.k else torch.cat([st.k[run], k], 0)
        st.v[run] = v if run not in st.v else torch.cat([st.v[run], v], 0)
        o = attention(q, st.k[run], st.v[run], pos, float(m["scale"]), float(m["softcap"]))
        return o.reshape(T, -1) @ self.t[p + "o"].t()

    def ff(self, i: int, x: torch.Tensor) -> torch.Tensor:
        m, p = self.c["layers"][i]["mlp"], f"l{i}.mlp."
        lin = lambda n: x @ self.t[p + n].t()
        if m["kind"] == "dense":
            return clamped_glu(lin("gate"), lin("up"), float(m["limit"])) @ self.t[p + "down"].t()
        r = m["router"]
        z = lin("router")
        out = torch.zeros_like(x)
        for t in range(x.shape[0]):
            ids, wts = route(z[t], r["top"], r["groups"]["count"], r["groups"]["keep"], float(r["scale"]))
            for e, w in zip(ids, wts):
                e_ = f"{p}e{e}."
                a = silu_glu(self.t[e_ + "gate"] @ x[t], self.t[e_ + "up"] @ x[t])
                out[t] += w * (self.t[e_ + "down"] @ a)
        if m.get("shared"):
            a = silu_glu(lin("shared.gate"), lin("shared.up"))
            out = out + torch.sigmoid(lin("shared.sg")) * (a @ self.t[p + "shared.down"].t())
        return out

    def forward_raw(self, tokens: torch.Tensor, st: SisisunState, trace: Optional[list] = None) -> torch.Tensor:
        """Residual rows [T, width] after the last layer for ``tokens`` at positions st.pos ..; ``trace`` collects the
        residual after every layer run."""
        T = tokens.shape[0]
        pos = torch.arange(st.pos, st.pos + T)
        x0 = self.t["embed"][tokens.long()] + sinusoid(pos, self.c["width"])
        x = x0.clone()
        first = (self.c.get("loop") or {}).get("start")
        for run, (i, t) in enumerate(self.schedule()):
            if t is not None and i == first:
                if t > 0:
                    x = x + x0
                x = x + self.t["loop.step"][t]
            x = x + self.mixer(i, run, self.norm(x, f"l{i}.norm1"), st, pos)
            if self.c["layers"][i]["mlp"] is not None:
                x = x + self.ff(i, self.norm(x, f"l{i}.norm2"))
            if trace is not None:
                trace.append(x.clone())
        st.pos += T
        return x

    def forward_hidden(self, tokens: torch.Tensor, st: SisisunState) -> torch.Tensor:
        return self.norm(self.forward_raw(tokens, st), "final.norm")

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return hidden @ self.t["head"].t()

    def forward(self, tokens: torch.Tensor, st: Optional[SisisunState] = None) -> Tuple[torch.Tensor, SisisunState]:
        st = st or self.new_state()
        return self.logits(self.forward_hidden(tokens, st)), st
