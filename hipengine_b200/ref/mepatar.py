"""Plain fp32 reference of the Mepatar decoder, one function per mechanism, token order preserved.

Written from the layer equations and kept apart from the product path: it takes the decoded ``config.json`` (a dict) and
the checkpoint tensors under their own names; no configuration reader, weight packing or kernel launcher is involved.
Used as the oracle of the tests and by the ``cpu_reference`` backend.

    x_p   = c E[token_p]
    layer : x += mix(a) + ff(norm2(x)),  a = n + conv(n),  n = norm1(x)       norms over groups of channels
    mix   : softmax attention (a window, and the first tokens of the sequence), retention (linear attention with a decay per
            head), or the gated delta rule
    ff    : W_d (gelu(W_g h) * (W_u h)); a weighted sum of a few of many clamped experts; or none
    logits = head norm(x)
"""
from __future__ import annotations

import math
from typing import Any, Dict, Mapping, Optional, Tuple

import torch


# ----------------------------------------------------------------------------- norms
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def grouped_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Every one of ``groups`` equal runs of channels over its own root mean square, times a gain per channel."""
    return rms(x.reshape(*x.shape[:-1], groups, -1), eps).reshape(x.shape) * w


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)


# ----------------------------------------------------------------------------- convolutions
def causal_conv(x: torch.Tensor, before: torch.Tensor, w: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """Per channel: x [T, C] behind ``before`` [taps - 1, C]; w [C, taps], newest tap last.  (result, inputs to keep)"""
    taps, T = w.shape[1], x.shape[0]
    full = torch.cat([before, x], 0)
    return sum(full[j:j + T] * w[:, j] for j in range(taps)), full[T:]


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


# ----------------------------------------------------------------------------- positions
def angles(pos: torch.Tensor, dims: int, base: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """(cosine, sine) [T, 1, dims / 2] of position * base^(-2 i / dims)."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = pos.double()[:, None, None] * f
    return torch.cos(a).float(), torch.sin(a).float()


def rotate_halves(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """Dimension i turns with i + dims / 2; x [T, heads, d], dimensions from ``dims`` on stay."""
    c, s = angles(pos, dims, base)
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def rotate_neighbours(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """Dimension 2i turns with 2i + 1."""
    c, s = angles(pos, dims, base)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., dims:]], -1)


# ----------------------------------------------------------------------------- mixers
def visible_keys(pos: torch.Tensor, n_keys: int, window: int, first: int) -> torch.Tensor:
    """[T, n_keys] bool: of the keys up to position i, the last ``window`` ones and the sequence's ``first`` ones."""
    j = torch.arange(n_keys)[None, :]
    d = pos[:, None] - j
    return (d >= 0) & ((d < window) | (j < first))


def attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, pos: torch.Tensor, scale: torch.Tensor, window: int,
              first: int) -> torch.Tensor:
    """q [T, H, d], k [S, G, d], v [S, G, dv] of positions 0..S-1, scale [H]; query head h reads key head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    seen = visible_keys(pos, k.shape[0], window, first)
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].t() * scale[h]).masked_fill(~seen, -math.inf)
        out.append(torch.softmax(s, -1) @ v[:, g])
    return torch.stack(out, 1)


def retention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor,
              S: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """S_t = decay S_{t-1} + k_t v_t^T, o_t = S_t^T q_t; q, k [T, H, d], v [T, H, dv], decay [H], S [H, d, dv]."""
    out = []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor,
               S: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  q, k [T, H, d], v [T, H, dv], g and beta [T, H]."""
    out = []
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


# ----------------------------------------------------------------------------- feed-forward
def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_ff(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return (gelu_tanh(h @ gate.t()) * (h @ up.t())) @ down.t()


def clamped_expert(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ gate.t(), max=limit)
    u = torch.clamp(h @ up.t(), -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.t()


def routing(logits: torch.Tensor, top: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """(expert ids, weights) [T, top]: the largest softmax scores as they are."""
    w, ids = torch.topk(torch.softmax(logits, -1), top, -1)
    return ids, w


# ----------------------------------------------------------------------------- model
class MepatarState:
    """What one request carries per layer: keys and values, recurrent states, the last inputs of the convolutions."""

    def __init__(self):
        self.pos = 0
        self.k: Dict[int, torch.Tensor] = {}
        self.v: Dict[int, torch.Tensor] = {}
        self.S: Dict[int, torch.Tensor] = {}
        self.conv: Dict[Any, torch.Tensor] = {}

    def clone(self) -> "MepatarState":
        c = MepatarState()
        c.pos = self.pos
        c.k, c.v, c.S, c.conv = ({i: t.clone() for i, t in d.items()} for d in (self.k, self.v, self.S, self.conv))
        return c


class MepatarRef:
    def __init__(self, config: Mapping[str, Any], tensors: Mapping[str, torch.Tensor]):
        self.c = config
        self.t = {n: v.detach().to("cpu", torch.float32) for n, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])

    def new_state(self) -> MepatarState:
        return MepatarState()

    def norm(self, x: torch.Tensor, name: str) -> torch.Tensor:
        return grouped_norm(x, self.t[name], int(self.c["norm"]["groups"]), self.eps)

    def conv(self, x: torch.Tensor, name: str, key: Any, st: MepatarState) -> torch.Tensor:
        w = self.t[name]
        y, st.conv[key] = causal_conv(x, st.conv.get(key, torch.zeros(w.shape[1] - 1, x.shape[1])), w)
        return y

    def project(self, h: torch.Tensor, name: str, heads: int) -> torch.Tensor:
        y = h @ self.t[name].t()
        if name + ".b" in self.t:
            y = y + self.t[name + ".b"]
        return y.reshape(h.shape[0], heads, -1)

    def attention_mixer(self, i: int, h: torch.Tensor, st: MepatarState, pos: torch.Tensor) -> torch.Tensor:
        m, p, t = self.c["layers"][i]["mixer"], f"l{i}.mix.", self.t
        turn = lambda x, n: rotate_neighbours(rms(x, self.eps) * t[p + n + ".norm"], pos, int(m["rot"]["dims"]),
                                              float(m["rot"]["base"]))
        q = turn(self.project(h, p + "q", m["heads"]), "q")
        k, v = turn(self.project(h, p + "k", m["kv_heads"]), "k"), self.project(h, p + "v", m["kv_heads"])
        for store, new in ((st.k, k), (st.v, v)):
            store[i] = torch.cat([store[i], new], 0) if i in store else new
        o = attention(q, st.k[i], st.v[i], pos, float(m["scale"]) * t[p + "temp"], int(m["mask"]["size"]),
                      int(m["mask"]["keep_first"]))
        return o.flatten(1) @ t[p + "o"].t() + t[p + "o.b"]

    def retention_mixer(self, i: int, h: torch.Tensor, st: MepatarState, pos: torch.Tensor) -> torch.Tensor:
        m, p, t = self.c["layers"][i]["mixer"], f"l{i}.mix.", self.t
        H = int(m["heads"])
        turn = lambda x: rotate_halves(x, pos, int(m["rot"]["dims"]), float(m["rot"]["base"]))
        q, k, v = (self.project(h, p + n, H) for n in "qkv")
        S = st.S.get(i, torch.zeros(H, int(m["dim"]), int(m["vdim"])))
        o, st.S[i] = retention(turn(q), turn(k) * float(m["dim"]) ** -0.5, v, torch.tensor(m["decay"], dtype=torch.float32), S)
        return (rms(o, self.eps).flatten(1) * silu(h @ t[p + "g"].t())) @ t[p + "o"].t()

    def delta_mixer(self, i: int, h: torch.Tensor, st: MepatarState, pos: torch.Tensor) -> torch.Tensor:
        m, p, t = self.c["layers"][i]["mixer"], f"l{i}.mix.", self.t
        H, G, d, dv = (int(m[n]) for n in ("heads", "kv_heads", "dim", "vdim"))
        q, k, v = (silu(self.conv(h @ t[p + n].t(), p + n + ".conv", (i, n), st)) for n in "qkv")
        spread = lambda x: unit(x.reshape(-1, G, d)).repeat_interleave(H // G, 1)
        beta = torch.sigmoid(h @ t[p + "b"].t())
        g = torch.exp(-torch.exp(t[p + "A_log"]) * torch.nn.functional.softplus(h @ t[p + "a"].t() + t[p + "dt_bias"]))
        S = st.S.get(i, torch.zeros(H, d, dv))
        o, st.S[i] = delta_rule(spread(q) * d ** -0.5, spread(k), v.reshape(-1, H, dv), g, beta, S)
        return ((rms(o, self.eps) * t[p + "norm"]).flatten(1) * silu(h @ t[p + "g"].t())) @ t[p + "o"].t()

    def experts(self, i: int, h: torch.Tensor) -> torch.Tensor:
        m, p, t = self.c["layers"][i]["mlp"], f"l{i}.mlp.", self.t
        ids, w = routing(h @ t[p + "router"].t(), int(m["router"]["top"]))
        y = torch.zeros_like(h)
        for e in range(int(m["router"]["experts"])):
            rows, place = (ids == e).nonzero(as_tuple=True)
            if rows.numel():
                out = clamped_expert(h[rows], *(t[p + f"e{e}.{n}"] for n in ("gate", "up", "down")), float(m["expert"]["limit"]))
                y[rows] += w[rows, place][:, None] * out
        return y

    def layer(self, i: int, x: torch.Tensor, st: MepatarState, pos: torch.Tensor) -> torch.Tensor:
        L, p = self.c["layers"][i], f"l{i}."
        n = self.norm(x, p + "norm1")
        a = n + self.conv(n, p + "canon1", (i, "in"), st)
        y = {"attention": self.attention_mixer, "retention": self.retention_mixer, "delta": self.delta_mixer}[L["type"]](
            i, a, st, pos)
        if L["mlp"] is not None:
            h = self.norm(x, p + "norm2")
            if L["mlp"]["kind"] == "moe":
                y = y + self.experts(i, h)
            else:
                y = y + gated_ff(h, *(self.t[p + "mlp." + n] for n in ("gate", "up", "down")))
        return x + y

    def forward_raw(self, tokens: torch.Tensor, st: MepatarState, trace: Optional[list] = None) -> torch.Tensor:
        """Residual rows [T, width] after the last layer for ``tokens`` at positions st.pos ..; ``trace`` collects the
        residual after every layer."""
        T = tokens.shape[0]
        pos = torch.arange(st.pos, st.pos + T)
        x = self.t["embed"][tokens.long()] * float(self.c["embedding"]["scale"])
        for i in range(len(self.c["layers"])):
            x = self.layer(i, x, st, pos)
            if trace is not None:
                trace.append(x.clone())
        st.pos += T
        return x

    def forward_hidden(self, tokens: torch.Tensor, st: MepatarState) -> torch.Tensor:
        return self.norm(self.forward_raw(tokens, st), "final.norm")

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return hidden @ self.t["head"].t()

    def forward(self, tokens: torch.Tensor, st: Optional[MepatarState] = None) -> Tuple[torch.Tensor, MepatarState]:
        st = st or self.new_state()
        return self.logits(self.forward_hidden(tokens, st)), st
