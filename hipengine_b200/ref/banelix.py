"""Plain fp32 reference of the Banelix decoder, one function per mechanism, token order preserved.

Written from the layer equations and kept apart from the product path: it takes the decoded ``config.json`` (a dict) and
the checkpoint tensors under their own names; no configuration reader, weight packing or kernel launcher is involved.
Used as the oracle of the tests and by the ``cpu_reference`` backend.

    x_p   = c E[token_p]
    layer : x += m mix(norm1(x));  x += m ff(norm2(x))          m: one constant, norms with a gain per channel
    mix   : windowed softmax attention with one more unit in the denominator, keys possibly those of an earlier layer; or
            l A(h) + r R(h): attention over unit keys whose values are the plain keys, beside a gated linear recurrence
    ff    : W_d (silu(W_g h) * (W_u h))
    logits = head norm(x)
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


# ----------------------------------------------------------------------------- positions
def plain_freqs(dims: int, base: float) -> List[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_freqs(freqs: List[float], s: Mapping[str, Any]) -> List[float]:
    """Waves that fit ``high`` times into the original context keep their frequency, those that do not fit ``low`` times
    are ``factor`` times slower, those between are mixed."""
    factor, low, high, n = (float(s[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for f in freqs:
        wave = 2.0 * math.pi / f
        if wave < n / high:
            out.append(f)
        elif wave > n / low:
            out.append(f / factor)
        else:
            t = (n / wave - low) / (high - low)
            out.append(t * f + (1.0 - t) * f / factor)
    return out


def ramped_freqs(freqs: List[float], dims: int, base: float, s: Mapping[str, Any]) -> Tuple[List[float], float]:
    """Slow pairs are ``factor`` times slower, fast ones kept, a linear ramp over the pair's index between; and the
    amplitude of sine and cosine."""
    factor, n = float(s["factor"]), float(s["original"])

    def index_of(turns: float) -> float:
        return dims * math.log(n / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index_of(float(s["fast"]))), 0)
    hi = min(math.ceil(index_of(float(s["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotation(rot: Mapping[str, Any]) -> Tuple[torch.Tensor, float]:
    """(angular frequency per pair, amplitude) of a layer's rotation."""
    dims, base, s = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    f, amp = plain_freqs(dims, base), 1.0
    if s and "high" in s:
        f = banded_freqs(f, s)
    elif s:
        f, amp = ramped_freqs(f, dims, base, s)
    return torch.tensor(f, dtype=torch.float64), amp


def rotate_halves(x: torch.Tensor, pos: torch.Tensor, freqs: torch.Tensor, amp: float = 1.0) -> torch.Tensor:
    """Rotate the pairs (x_i, x_{i + n}) of the first 2n dimensions by pos * freqs[i], n = len(freqs); x [T, heads, d]."""
    n = freqs.numel()
    a = pos.double()[:, None, None] * freqs[None, None]
    c, s = (torch.cos(a) * amp).float(), (torch.sin(a) * amp).float()
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


# ----------------------------------------------------------------------------- attention
def visible_keys(pos: torch.Tensor, n_keys: int, window: int = 0) -> torch.Tensor:
    """[T, n_keys] bool: key j is seen from position i iff 0 <= i - j (< window when there is one)."""
    d = pos[:, None] - torch.arange(n_keys)[None, :]
    return (d >= 0) & (d < window) if window > 0 else d >= 0


def weights_over(s: torch.Tensor, seen: torch.Tensor, extra: bool) -> torch.Tensor:
    """Softmax over the seen keys; with ``extra`` the denominator has one unit more."""
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    if not extra:
        return torch.softmax(s, -1)
    top = s.max(-1, keepdim=True).values.clamp_min(0.0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, pos: torch.Tensor, scale: float, window: int = 0,
              extra: bool = False) -> torch.Tensor:
    """q [T, H, d], k [S, G, d], v [S, G, dv] of positions 0..S-1; query head h reads key head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    seen = visible_keys(pos, k.shape[0], window)
    return torch.stack([weights_over(q[:, h] @ k[:, h // (H // G)].t() * scale, seen, extra) @ v[:, h // (H // G)]
                        for h in range(H)], 1)


# ----------------------------------------------------------------------------- recurrence
def causal_conv(x: torch.Tensor, before: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """Per channel: x [T, C], ``before`` [taps - 1, C] the inputs ahead of x, w [C, taps] with the newest tap last."""
    taps, T = w.shape[1], x.shape[0]
    full = torch.cat([before, x], 0)
    return sum(full[j:j + T] * w[:, j] for j in range(taps)) + b


def block_product(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """x [T, C] cut into blocks, each times its own square matrix: w [blocks, n, n] (out, in), b [blocks, n]."""
    n = w.shape[1]
    return torch.cat([x[:, i * n:(i + 1) * n] @ w[i].t() + b[i] for i in range(w.shape[0])], 1)


def gated_recurrence(u: torch.Tensor, r: torch.Tensor, i: torch.Tensor, lam: torch.Tensor,
                     S: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """S_t = a_t S_{t-1} + sqrt(1 - a_t^2) i_t u_t with log a_t = -8 r_t softplus(lam); returns (every S_t, the last)."""
    log_a = -8.0 * r * torch.nn.functional.softplus(lam)
    a, out = torch.exp(log_a), []
    drive = torch.sqrt(1.0 - a * a) * i * u
    for t in range(u.shape[0]):
        S = a[t] * S + drive[t]
        out.append(S)
    return torch.stack(out), S


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_ff(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    g = h @ gate.t()
    return (g * torch.sigmoid(g) * (h @ up.t())) @ down.t()


# ----------------------------------------------------------------------------- model
class BanelixState:
    """What one request carries per layer: keys and values, the recurrent state, the convolution's last inputs."""

    def __init__(self):
        self.pos = 0
        self.k: Dict[int, torch.Tensor] = {}
        self.v: Dict[int, torch.Tensor] = {}
        self.S: Dict[int, torch.Tensor] = {}
        self.conv: Dict[int, torch.Tensor] = {}

    def clone(self) -> "BanelixState":
        c = BanelixState()
        c.pos = self.pos
        c.k, c.v, c.S, c.conv = ({i: t.clone() for i, t in d.items()} for d in (self.k, self.v, self.S, self.conv))
        return c


class BanelixRef:
    def __init__(self, config: Mapping[str, Any], tensors: Mapping[str, torch.Tensor]):
        self.c = config
        self.t = {n: v.detach().to("cpu", torch.float32) for n, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])
        self.mult = float(config["residual_mult"])

    def new_state(self) -> BanelixState:
        return BanelixState()

    def norm(self, x: torch.Tensor, name: str) -> torch.Tensor:
        return rms(x, self.eps) * self.t[name]

    def biased(self, h: torch.Tensor, name: str) -> torch.Tensor:
        return h @ self.t[name].t() + self.t[name + ".b"]

    def extend(self, i: int, st: BanelixState, k: torch.Tensor, v: torch.Tensor) -> None:
        for store, new in ((st.k, k), (st.v, v)):
            store[i] = torch.cat([store[i], new], 0) if i in store else new

    def windowed_attention(self, i: int, h: torch.Tensor, st: BanelixState, pos: torch.Tensor) -> torch.Tensor:
        m, p, T = self.c["layers"][i]["mixer"], f"l{i}.mix.", h.shape[0]
        f, amp = rotation(m["rot"])
        turn = lambda x, heads: rotate_halves(x.reshape(T, heads, m["dim"]), pos, f, amp)
        q = turn(self.norm(self.biased(h, p + "q"), p + "q.norm"), m["heads"])
        src = m.get("kv_from")
        if src is None:
            src = i
            k = turn(self.norm(self.biased(h, p + "k"), p + "k.norm"), m["kv_heads"])
            self.extend(i, st, k, self.biased(h, p + "v").reshape(T, m["kv_heads"], m["vdim"]))
        o = attention(q, st.k[src], st.v[src], pos, float(m["scale"]), int(m["mask"]["size"]), extra=True)
        return o.reshape(T, -1) @ self.t[p + "o"].t()

    def unit_key_attention(self, i: int, h: torch.Tensor, st: BanelixState, pos: torch.Tensor) -> torch.Tensor:
        m, p, T = self.c["layers"][i]["mixer"]["left"], f"l{i}.mix.left.", h.shape[0]
        f, amp = rotation(m["rot"])
        q = self.biased(h, p + "q").reshape(T, m["heads"], m["dim"])
        k = self.biased(h, p + "k").reshape(T, m["kv_heads"], m["dim"])
        unit = lambda x: rms(rotate_halves(x, pos, f, amp), self.eps)
        self.extend(i, st, unit(k), k)
        o = attention(unit(q), st.k[i], st.v[i], pos, float(m["scale"]))
        o = o * torch.sigmoid(h @ self.t[p + "g"].t())[:, :, None]
        return o.reshape(T, -1) @ self.t[p + "o"].t()

    def recurrent_block(self, i: int, h: torch.Tensor, st: BanelixState) -> torch.Tensor:
        p, t = f"l{i}.mix.right.", self.t
        y, x = gelu_tanh(self.biased(h, p + "y")), self.biased(h, p + "x")
        taps = t[p + "conv"].shape[1]
        before = st.conv.get(i, torch.zeros(taps - 1, x.shape[1]))
        u = causal_conv(x, before, t[p + "conv"], t[p + "conv.b"])
        st.conv[i] = torch.cat([before, x], 0)[x.shape[0]:]
        r = torch.sigmoid(block_product(u, t[p + "ra"], t[p + "ra.b"]))
        g = torch.sigmoid(block_product(u, t[p + "ri"], t[p + "ri.b"]))
        S, st.S[i] = gated_recurrence(u, r, g, t[p + "lam"], st.S.get(i, torch.zeros(u.shape[1])))
        return (S * y) @ t[p + "o"].t()

    def mixer(self, i: int, h: torch.Tensor, st: BanelixState, pos: torch.Tensor) -> torch.Tensor:
        L = self.c["layers"][i]
        if L["type"] == "attention":
            return self.windowed_attention(i, h, st, pos)
        m = L["mixer"]
        return (float(m["left_scale"]) * self.unit_key_attention(i, h, st, pos)
                + float(m["right_scale"]) * self.recurrent_block(i, h, st))

    def forward_raw(self, tokens: torch.Tensor, st: BanelixState, trace: Optional[list] = None) -> torch.Tensor:
        """Residual rows [T, width] after the last layer for ``tokens`` at positions st.pos ..; ``trace`` collects the
        residual after every layer."""
        T = tokens.shape[0]
        pos = torch.arange(st.pos, st.pos + T)
        x = self.t["embed"][tokens.long()] * float(self.c["embedding"]["scale"])
        for i, L in enumerate(self.c["layers"]):
            p = f"l{i}."
            x = x + self.mult * self.mixer(i, self.norm(x, p + "norm1"), st, pos)
            if L["mlp"] is not None:
                w = (self.t[p + "mlp." + n] for n in ("gate", "up", "down"))
                x = x + self.mult * gated_ff(self.norm(x, p + "norm2"), *w)
            if trace is not None:
                trace.append(x.clone())
        st.pos += T
        return x

    def forward_hidden(self, tokens: torch.Tensor, st: BanelixState) -> torch.Tensor:
        return self.norm(self.forward_raw(tokens, st), "final.norm")

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return hidden @ self.t["head"].t()

    def forward(self, tokens: torch.Tensor, st: Optional[BanelixState] = None) -> Tuple[torch.Tensor, BanelixState]:
        st = st or self.new_state()
        return self.logits(self.forward_hidden(tokens, st)), st
