"""Small Mepatar models with random weights for the tests: (config dict, tensors under their checkpoint names)."""
import copy

import torch

from hipengine_b200.loading.folder_family import weights_from_tensors
from hipengine_b200.loading.mepatar import config_from_json, tensor_shapes
from hipengine_b200.ref.mepatar import MepatarRef
from sisisun_models import logit_error, tokens  # noqa: F401  (used by the Mepatar tests)

TOL = {"bfloat16": 0.04, "float32": 1e-4}


def attention(heads, kv_heads, dim, vdim, scale, size, keep, dims, base):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                         "mask": {"size": size, "keep_first": keep}, "rot": {"dims": dims, "base": base}}


def retention(heads, dim, vdim, decay, dims, base):
    return "retention", {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"dims": dims, "base": base}}


def delta(heads, kv_heads, dim, vdim, conv):
    return "delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def model(width, vocab, layers, groups=2, taps=3, eps=3e-5, embed=3.0):
    return {"architecture": "Mepatar", "width": width, "vocab": vocab, "embedding": {"scale": embed},
            "norm": {"eps": eps, "groups": groups}, "canon": {"taps": taps},
            "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


# unequal widths everywhere (a width, heads and groups that are no multiples of eight or four, odd heads), every kind of mixer
# and feed-forward, layers without a feed-forward
ODD = model(132, 301, [
    (delta(6, 3, 20, 28, 3), dense(100)),
    (attention(6, 3, 20, 28, 0.5, 21, 5, 10, 300.0), moe(5, 2, 36, 1.2)),
    (retention(3, 33, 18, (0.9, 0.97, 0.999), 14, 700.0), None),
    (retention(5, 12, 30, (0.995, 0.8, 0.99, 0.96, 1.0), 12, 90.0), moe(7, 3, 20, 0.8)),
    (delta(2, 2, 44, 10, 5), None),
], groups=6, taps=4, eps=1e-4, embed=1.4)
# many heads per group (more than one chunk of the decode kernel), heads as wide as the chunked kernels take them
HEADS = model(248, 520, [
    (attention(40, 4, 24, 24, 0.6, 33, 20, 16, 4000.0), dense(192)),
    (delta(12, 4, 100, 72, 2), moe(16, 4, 64, 2.0)),
    (retention(4, 128, 128, (0.99, 0.95, 0.999, 0.9), 64, 15000.0), dense(256)),
    (attention(21, 3, 64, 48, 0.4, 70, 1, 64, 15000.0), None),
    (delta(4, 1, 128, 40, 4), dense(128)),
], groups=4, taps=2)
# wide heads (every size class of the kernels, heads too wide for the chunked ones), long convolutions
WIDE = model(160, 200, [
    (attention(2, 1, 150, 136, 0.2, 60, 40, 150, 9000.0), dense(96)),
    (delta(3, 1, 136, 264, 6), moe(3, 3, 40, 1.0)),
    (retention(2, 300, 72, (0.98, 0.999), 200, 20000.0), None),
    (attention(4, 2, 264, 20, 0.1, 9, 64, 72, 2000.0), moe(40, 8, 24, 3.0)),
], groups=1, taps=7)
# sizes of one: one head, one pair, windows of one and two tokens, no or one first token, no convolutions, one expert, no decay
ONES = model(64, 96, [
    (attention(1, 1, 2, 3, 1.0, 1, 1, 2, 100.0), dense(16)),
    (delta(6, 6, 16, 24, 1), moe(1, 1, 8, 1.0)),
    (retention(8, 16, 24, (1.0,) * 8, 2, 50.0), dense(8)),
    (attention(2, 2, 16, 16, 0.5, 2, 0, 16, 50.0), moe(2, 1, 24, 1.5)),
    (delta(8, 4, 8, 16, 1), None),
], groups=8, taps=1)
# single heads of linear attention down to one column.  Their norm makes any rounding large (a single column keeps only its
# sign): for float32 alone
SINGLE = model(48, 80, [
    (delta(1, 1, 1, 1, 1), dense(8)), (retention(1, 2, 1, (1.0,), 2, 50.0), moe(2, 2, 8, 1.0)), (delta(1, 1, 3, 2, 2), None),
    (attention(1, 1, 2, 1, 1.0, 3, 1, 2, 10.0), None)], groups=48, taps=2, embed=1.0)
MODELS = {"odd": ODD, "heads": HEADS, "wide": WIDE, "ones": ONES}
EXACT_MODELS = {**MODELS, "single": SINGLE}


def random_tensors(cfg_json, seed=0):
    """Weights scaled so that every branch contributes visibly; routers decide clearly (a choice turned by rounding would move
    a row by far more than rounding does)."""
    g = torch.Generator().manual_seed(seed)
    t = {}
    for n, shape in tensor_shapes(config_from_json(cfg_json)).items():
        x = torch.randn(shape, generator=g)
        if n.endswith(("norm1", "norm2", ".norm")):
            x = 1.0 + 0.4 * x
        elif n.endswith(".temp"):
            x = 1.2 + 0.5 * x
        elif n.endswith(".b") and len(shape) == 1:
            x = 0.4 * x
        elif n.endswith(".A_log"):
            x = 0.5 * x - 0.5
        elif n.endswith(".dt_bias"):
            x = x - 2.5
        elif n.endswith((".conv", "canon1")):
            x = 0.6 * x
        elif n.endswith((".mix.a", ".mix.b")):
            x = x * 1.0 / shape[-1] ** 0.5
        elif n != "embed":
            x = x * 1.3 / shape[-1] ** 0.5
        t[n] = x.to(torch.bfloat16)
    return t


def decided(cfg_json, t):
    """The same tensors with routers that read the first channels of the token's own embedding only, where every token has a
    clear order of the experts: which are chosen does not depend on rounding."""
    t = dict(t)
    vocab, width = t["embed"].shape
    most = max([l["mlp"]["router"]["experts"] for l in cfg_json["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"], default=0)
    if not most:
        return t
    g = torch.Generator().manual_seed(5)
    order = torch.stack([torch.randperm(most, generator=g) for _ in range(vocab)]).float()
    embed = t["embed"].float()
    embed[:, :most] = (order - (most - 1) / 2) * (4.0 / most)
    t["embed"] = embed.to(torch.bfloat16)
    for n, x in t.items():
        if n.endswith(".router"):
            r = torch.zeros_like(x)
            r[:, :most] = torch.eye(most)[:x.shape[0]] * 0.2 * most
            t[n] = r
        elif n.endswith((".mix.o", ".down", ".o.b")):          # nothing is added to these channels
            y = x.clone()
            y[:most] = 0
            t[n] = y
        elif n.endswith(("norm1", "norm2", "final.norm")):
            y = x.clone()
            y[:most] = 1
            t[n] = y
    return t


def build(cfg_json, seed=0, clear=True):
    """(ModelWeights, oracle, tensors)."""
    t = random_tensors(cfg_json, seed)
    if clear:
        t = decided(cfg_json, t)
    return weights_from_tensors(config_from_json(cfg_json), t), MepatarRef(cfg_json, t), t


def needle(cfg_json, strength=1.0, seed=7):
    """A model of attention layers in which token 1 asks for token 2 and nothing else: the query of token 1 lines up with the key
    of token 2 in the dimensions that are not rotated, in every layer, so one score stands out among any number of keys."""
    t = random_tensors(cfg_json, seed)
    t["embed"][:] = (t["embed"].float() * 0.5).to(torch.bfloat16)
    t["embed"][:, :2] = 0
    t["embed"][1, 0] = t["embed"][2, 1] = 12.0
    t["head"][:, :2] = 0
    for i, l in enumerate(cfg_json["layers"]):
        m, p = l["mixer"], f"l{i}.mix."
        t[f"l{i}.canon1"][:2] = 0                              # neighbours do not ask
        t[p + "temp"] = t[p + "temp"].abs()
        for n in ("q.norm", "k.norm"):
            t[p + n] = torch.ones_like(t[p + n])
        pattern = torch.where(torch.arange(m["dim"]) % 2 == 0, 1.0, -1.0) * strength
        pattern[:m["rot"]["dims"]] = 0
        t[p + "q"][:, 0] = pattern.repeat(m["heads"]).to(torch.bfloat16)
        t[p + "k"][:, 1] = pattern.repeat(m["kv_heads"]).to(torch.bfloat16)
    return weights_from_tensors(config_from_json(cfg_json), t), MepatarRef(cfg_json, t), t


def with_masks(cfg_json, size=0, keep=0):
    """The same configuration with every window ``size`` and every run of kept first tokens ``keep`` tokens longer."""
    c = copy.deepcopy(cfg_json)
    for l in c["layers"]:
        if "mask" in l["mixer"]:
            l["mixer"]["mask"]["size"] += size
            l["mixer"]["mask"]["keep_first"] = max(0, l["mixer"]["mask"]["keep_first"] + keep)
    return c


def last_logits(ref, ids):
    return ref.forward(torch.tensor(ids))[0][-1:]
