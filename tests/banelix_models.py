"""Small Banelix models with random weights for the tests: (config dict, tensors under their checkpoint names)."""
import copy

import torch

from hipengine_b200.loading.banelix import config_from_json, tensor_shapes
from hipengine_b200.loading.folder_family import weights_from_tensors
from hipengine_b200.ref.banelix import BanelixRef
from sisisun_models import logit_error, tokens  # noqa: F401  (used by the Banelix tests)

TOL = {"bfloat16": 0.04, "float32": 1e-4}


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def bands(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def rotation(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = scaling
    return r


def windowed(heads, kv_heads, dim, vdim, scale, size, rot, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot, "mask": {"size": size}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def both(heads, kv_heads, dim, scale, rot, width, blocks, conv, left=0.9, right=0.8):
    return "parallel", {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "rot": rot},
                        "right": {"width": width, "blocks": blocks, "conv": conv}, "left_scale": left, "right_scale": right}


def model(width, vocab, layers, eps=3e-5, mult=0.8, embed=3.0):
    return {"architecture": "Banelix", "width": width, "vocab": vocab, "embedding": {"scale": embed}, "norm": {"eps": eps},
            "residual_mult": mult,
            "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None} for (t, m), ff in layers]}


_ODD_ROT = rotation(10, 300.0, yarn(6.0, 256.0, 16.0, 1.0))
# unequal widths everywhere (a width, heads and blocks that are no multiples of eight, odd heads), layers without a
# feed-forward, a layer on the keys and values of an earlier one with another window and scale, two convolution lengths
ODD = model(132, 301, [
    (windowed(6, 3, 20, 28, 0.5, 21, _ODD_ROT), 100),
    (both(4, 2, 33, 0.35, rotation(14, 700.0, bands(5.0, 1.0, 4.0, 120.0)), 60, 4, 3, 1.8, 0.6), 64),
    (both(3, 1, 18, 0.5, rotation(6, 90.0, bands(3.0, 1.0, 2.5, 64.0)), 44, 2, 4, 0.6, 2.0), 0),
    (windowed(6, 3, 20, 28, 0.4, 7, _ODD_ROT, kv_from=0), 72),
], eps=1e-4, mult=0.75, embed=1.4)
# many heads per group (more than one chunk of the decode kernel), the source of the keys in the middle of the stack
_HEADS_ROT = rotation(64, 15000.0, yarn(2.0, 128.0, 4.0, 0.5))
HEADS = model(248, 520, [
    (both(40, 4, 24, 0.2, rotation(24, 4000.0, bands(8.0, 0.5, 6.0, 300.0)), 192, 6, 2), 192),
    (windowed(21, 3, 64, 48, 0.15, 33, _HEADS_ROT), 256),
    (windowed(21, 3, 64, 48, 0.2, 70, _HEADS_ROT, kv_from=1), 0),
    (both(16, 16, 100, 0.1, rotation(20, 900.0), 96, 1, 3, 1.1, 0.6), 128),
])
# wide heads (every size class of the kernels) and a long convolution
WIDE = model(160, 200, [
    (windowed(2, 1, 150, 136, 0.08, 60, rotation(150, 9000.0, yarn(5.0, 300.0, 10.0, 1.0))), 96),
    (both(4, 2, 264, 0.03, rotation(72, 20000.0, bands(4.0, 1.0, 4.0, 512.0)), 136, 1, 6), 80),
    (both(2, 2, 96, 0.06, rotation(96, 2000.0, bands(2.0, 1.0, 2.0, 100.0)), 288, 3, 4), 0),
])
# sizes of one: one head, one pair, windows of one and two tokens, blocks of one channel, no convolution, factors of one
ONES = model(64, 96, [
    (both(1, 1, 7, 1.0, rotation(2, 100.0, bands(1.0, 1.0, 4.0, 32.0)), 16, 16, 1, 1.0, 1.0), 16),
    (windowed(1, 1, 8, 3, 0.5, 1, rotation(2, 100.0, yarn(1.0, 32.0, 2.0, 1.0))), 8),
    (windowed(2, 2, 16, 16, 0.3, 2, rotation(16, 50.0)), 24),
    (both(3, 3, 8, 0.5, rotation(4, 10.0), 8, 1, 2, 1.0, 1.0), 8),
], mult=1.0, embed=1.0)
MODELS = {"odd": ODD, "heads": HEADS, "wide": WIDE, "ones": ONES}


def random_tensors(cfg_json, seed=0):
    """Weights scaled so that every branch contributes visibly."""
    g = torch.Generator().manual_seed(seed)
    t = {}
    for n, shape in tensor_shapes(config_from_json(cfg_json)).items():
        x = torch.randn(shape, generator=g)
        if n.endswith(("norm1", "norm2", ".norm")):
            x = 1.0 + 0.4 * x
        elif n.endswith((".ra.b", ".ri.b")):
            x = x - 0.5
        elif n.endswith(".b"):
            x = 0.4 * x
        elif n.endswith(".lam"):
            x = x - 3.0
        elif n.endswith(".conv"):
            x = 0.6 * x
        elif n.endswith(("left.g", "left.q", "left.k")):
            x = x * 2.5 / shape[-1] ** 0.5
        elif n != "embed":
            x = x * 1.3 / shape[-1] ** 0.5
        t[n] = x.to(torch.bfloat16)
    return t


def build(cfg_json, seed=0):
    """(ModelWeights, oracle, tensors)."""
    t = random_tensors(cfg_json, seed)
    return weights_from_tensors(config_from_json(cfg_json), t), BanelixRef(cfg_json, t), t


def needle(cfg_json, strength=1.0, seed=7):
    """A model in which token 1 asks for token 2 and nothing else: the query of token 1 lines up with the key of token 2 in
    the dimensions that are not rotated, in every layer, so one score stands out among any number of keys."""
    t = random_tensors(cfg_json, seed)
    t["embed"][:] = (t["embed"].float() * 0.5).to(torch.bfloat16)
    t["embed"][:, :2] = 0
    t["embed"][1, 0] = t["embed"][2, 1] = 12.0
    t["head"][:, :2] = 0
    for i, l in enumerate(cfg_json["layers"]):
        two = l["type"] == "parallel"
        m, p = (l["mixer"]["left"], f"l{i}.mix.left.") if two else (l["mixer"], f"l{i}.mix.")
        pattern = torch.where(torch.arange(m["dim"]) % 2 == 0, 1.0, -1.0) * strength
        pattern[:m["rot"]["dims"]] = 0
        t[p + "q"][:, 0] = pattern.repeat(m["heads"]).to(torch.bfloat16)
        if m.get("kv_from") is None:
            t[p + "k"][:, 1] = pattern.repeat(m["kv_heads"]).to(torch.bfloat16)
        if two:                                            # the recurrence does not see which token asks or is asked for
            for n in ("x", "y"):
                t[f"l{i}.mix.right.{n}"][:, :2] = 0
    return weights_from_tensors(config_from_json(cfg_json), t), BanelixRef(cfg_json, t), t


def with_windows(cfg_json, delta):
    """The same configuration with every window ``delta`` tokens longer."""
    c = copy.deepcopy(cfg_json)
    for l in c["layers"]:
        if "mask" in l["mixer"]:
            l["mixer"]["mask"]["size"] += delta
    return c


def last_logits(ref, ids):
    return ref.forward(torch.tensor(ids))[0][-1:]
