"""Small Sisisun models with random weights for the tests: (config dict, tensors under their checkpoint names)."""
import json

import torch

from hipengine_b200.loading.folder_family import weights_from_tensors
from hipengine_b200.loading.sisisun import config_from_json, tensor_shapes
from hipengine_b200.ref.sisisun import SisisunRef, route


def attn(heads, kv_heads, dim, vdim, scale, softcap):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, count, keep, scale, shared=None):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None,
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


def model(width, vocab, layers, loop=None, eps=1e-5):
    return {"architecture": "Sisisun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "loop": loop,
            "layers": [{"type": "attention", "mixer": a, "mlp": m} for a, m in layers]}


# unequal widths and groups everywhere: heads of different shapes per layer, a width that is no multiple of eight, a layer
# without a feed-forward, a loop in the middle, single-expert groups
WIDE = model(132, 301, [
    (attn(6, 2, 40, 24, 0.21, 9.0), dense(100, 0.8)),
    (attn(5, 1, 16, 72, 0.4, 30.0), moe(12, 3, 36, 4, 2, 1.6, shared=20)),
    (attn(4, 4, 64, 64, 0.1, 4.0), None),
    (attn(7, 1, 24, 16, 0.3, 50.0), moe(9, 2, 24, 9, 5, 0.7)),
    (attn(24, 2, 32, 32, 0.2, 12.0), dense(64, 2.5)),
], loop={"start": 1, "stop": 4, "times": 2}, eps=1e-5)
# wide heads, no loop, every group open
HEADS = model(256, 512, [
    (attn(2, 1, 128, 128, 0.09, 20.0), moe(8, 4, 64, 1, 1, 1.0, shared=64)),
    (attn(3, 3, 200, 136, 0.07, 15.0), dense(192, 7.0)),
])
# the loop covers the whole stack
LOOPED = model(96, 160, [
    (attn(4, 2, 24, 40, 0.25, 25.0), dense(128, 1.2)),
    (attn(4, 2, 24, 40, 0.25, 25.0), moe(10, 2, 16, 2, 1, 3.0, shared=12)),
], loop={"start": 0, "stop": 2, "times": 4})
MODELS = {"wide": WIDE, "heads": HEADS, "looped": LOOPED}


_LEVELS = {}


def _clear_levels(cfg_json, g):
    """Per token one level per expert channel such that every router of the model chooses the same experts whatever the
    position vector adds (at most one per channel) and however the row is scaled: no choice is a close call."""
    key = (json.dumps(cfg_json), g.initial_seed())
    if key in _LEVELS:
        return _LEVELS[key]
    routers = [l["mlp"]["router"] for l in cfg_json["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"]
    E = max([r["experts"] for r in routers], default=0)
    rows = []
    while len(rows) < cfg_json["vocab"]:
        lv = torch.randn(E, generator=g) * 9
        stable = True
        for r in routers:
            n = r["experts"]
            pick = lambda z: set(route(z[:n], r["top"], r["groups"]["count"], r["groups"]["keep"], 1.0)[0])
            near = [(lv + 1.5 * torch.randn(E, generator=g).sign()) * f for f in (0.08, 0.2, 0.4) for _ in range(8)]
            stable = stable and all(pick(z) == pick(lv * 0.2) for z in near)
        if stable:
            rows.append(lv)
    _LEVELS[key] = torch.stack(rows)
    return _LEVELS[key]


def build(cfg_json, seed=0, clear=False):
    """(ModelWeights, oracle, tensors) with weights scaled so that every branch contributes visibly.  ``clear``: the first
    channels hold per-token expert levels that no layer writes and only the routers read, so that bf16 rounding cannot
    turn a routing decision (random routers decide some rows by less than that)."""
    cfg = config_from_json(cfg_json)
    g = torch.Generator().manual_seed(seed)
    t = {}
    for n, shape in tensor_shapes(cfg).items():
        x = torch.randn(*shape, generator=g)
        if n.endswith(("q.norm", "k.norm")):
            x = 1.0 + 0.2 * x
        elif n.endswith(("norm1", "norm2", "final.norm")):
            x = 0.2 * x
        elif n == "loop.step":
            x = 0.5 * x
        elif n not in ("embed",):
            x = x * 1.5 / shape[-1] ** 0.5
        t[n] = x.to(torch.bfloat16)
    if clear:
        lv = _clear_levels(cfg_json, g)
        E = lv.shape[1]
        t["embed"] *= 3
        t["embed"][:, :E] = lv.to(torch.bfloat16)
        for n, x in t.items():
            if n.endswith(".router"):
                x.zero_()
                x.fill_diagonal_(1.5)
            elif n.endswith(("norm1", "norm2")):
                x[:E] = 0
            elif n == "loop.step":
                x[:, :E] = 0
            elif n.endswith((".o", ".down")):
                x[:E] = 0
            elif n.endswith((".q", ".k", ".v", ".gate", ".up", ".sg")):
                x[:, :E] = 0
    w = weights_from_tensors(cfg, t)
    return w, SisisunRef(cfg_json, t), t


def logit_error(got, want):
    """Largest row error: rms of the difference (its mean taken off) over the rms spread of the wanted logits."""
    d = got.float().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    spread = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float((d.pow(2).mean(-1).sqrt() / spread).max())


TOL = {"bfloat16": 0.04, "float32": 1e-4}


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def needle(cfg_json, scale_up=1.0):
    """A model in which token 1 asks for token 2 and nothing else: the query of token 1 lines up with the key of token
    2 in every layer, so one score stands out among any number of keys and the value of token 2 decides the logits."""
    w, _, t = build(cfg_json, seed=7)
    W = cfg_json["width"]
    t["embed"][:] = (t["embed"].float() * 0.5).to(torch.bfloat16)
    ask, answer = torch.zeros(W), torch.zeros(W)
    ask[0], answer[1] = 40.0, 40.0
    t["embed"][1] += ask.to(torch.bfloat16)
    t["embed"][2] += answer.to(torch.bfloat16)
    for i, l in enumerate(cfg_json["layers"]):
        m = l["mixer"]
        q, k = t[f"l{i}.mix.q"], t[f"l{i}.mix.k"]
        pattern = torch.where(torch.arange(m["dim"]) % 2 == 0, 1.0, -1.0) * scale_up
        q[:, 0] = pattern.repeat(m["heads"]).to(torch.bfloat16)
        k[:, 1] = pattern.repeat(m["kv_heads"]).to(torch.bfloat16)
    cfg = config_from_json(cfg_json)
    return weights_from_tensors(cfg, t), SisisunRef(cfg_json, t), t
