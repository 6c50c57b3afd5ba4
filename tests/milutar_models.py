"""Small Milutar models with random weights for the tests: (config dict, tensors under their checkpoint names)."""
import copy

import torch

from hipengine_b200.loading.folder_family import weights_from_tensors
from hipengine_b200.loading.milutar import config_from_json, tensor_shapes
from hipengine_b200.ref.milutar import MilutarRef
from sisisun_models import logit_error, tokens  # noqa: F401  (used by the Milutar tests)

TOL = {"bfloat16": 0.04, "float32": 1e-4}


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def windowed(heads, dim, rot, vdim, rank, scale, size, base=10000.0, scaling=None):
    r = {"dims": rot, "base": base}
    if scaling:
        r["scaling"] = scaling
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
                                "rot": r, "mask": {"size": size}}


def full(heads, dim, rot, vdim, rank, scale, q_rank, base=10000.0):
    return "latent_attention_2", {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
                                  "q_rank": q_rank, "rot": {"dims": rot, "base": base}}


def model(width, vocab, layers, loop=None, eps=3e-5, mult=0.8):
    return {"architecture": "Milutar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None,
            "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None} for (t, m), ff in layers]}


# unequal widths everywhere (a width and heads that are no multiple of eight, an odd unrotated part), a layer without a
# feed-forward, two windows, a loop in the middle
ODD = model(132, 301, [
    (windowed(5, 20, 12, 28, 44, 0.5, 21, 300.0, yarn(6.0, 256.0, 16.0, 1.0)), 100),
    (full(3, 33, 6, 17, 30, 0.5, 26, 700.0), 64),
    (windowed(2, 16, 4, 40, 24, 0.6, 7, 100.0, yarn(3.0, 64.0, 8.0, 2.0)), 0),
    (full(4, 8, 10, 12, 50, 0.6, 40, 400.0), 72),
], loop=(1, 3, 2), eps=1e-4, mult=0.55)
# many heads (more than one chunk of the decode kernel), no loop
HEADS = model(248, 520, [
    (full(40, 24, 20, 16, 136, 0.15, 96), 192),
    (windowed(17, 64, 32, 48, 72, 0.11, 33, 15000.0, yarn(2.0, 128.0, 4.0, 0.5)), 256),
])
# wide latents and heads: every size class of the kernels, one layer whose heads the prefill kernel does not take
WIDE = model(160, 200, [
    (windowed(2, 150, 50, 136, 260, 0.07, 60, 9000.0, yarn(5.0, 300.0, 10.0, 1.0)), 96),
    (full(3, 200, 72, 264, 520, 0.06, 144), 80),
    (full(2, 96, 32, 100, 512, 0.08, 64), 0),
])
# the loop covers the whole stack
LOOPED = model(96, 160, [
    (windowed(4, 24, 8, 40, 32, 0.2, 48, 2000.0, yarn(4.0, 128.0, 8.0, 1.0)), 128),
    (full(4, 24, 8, 40, 32, 0.2, 64), 112),
], loop=(0, 2, 4), mult=0.75)
# sizes of one: one head, one pair, windows of one and two tokens, one pass, no residual factor, a scaling that scales by one
ONES = model(64, 96, [
    (windowed(1, 8, 2, 8, 8, 0.4, 1, 100.0, yarn(1.0, 32.0, 2.0, 1.0)), 16),
    (full(1, 5, 2, 3, 16, 0.5, 16), 8),
    (windowed(2, 16, 16, 16, 16, 0.2, 2), 24),
], loop=(2, 3, 1), mult=1.0)
MODELS = {"odd": ODD, "heads": HEADS, "wide": WIDE, "looped": LOOPED, "ones": ONES}


def random_tensors(cfg_json, seed=0):
    """Weights scaled so that every branch contributes visibly."""
    g = torch.Generator().manual_seed(seed)
    t = {}
    for n, shape in tensor_shapes(config_from_json(cfg_json)).items():
        x = torch.randn(shape, generator=g)
        if n.endswith(("norm1", "final.norm")):
            x = 0.7 + 0.2 * x.abs()
        elif n.endswith(("dq.norm", "dkv.norm")):
            x = 1.0 + 0.4 * x
        elif n.endswith((".ls1", ".ls2")):
            x = 0.6 + 0.2 * x
        elif n.endswith(".shift"):
            x = 0.4 + 0.2 * x
        elif n.endswith(".sink"):
            x = 1.0 + x
        elif n == "loop.step":
            x = 0.5 * x
        elif n != "embed":
            x = x * 1.3 / shape[-1] ** 0.5
        t[n] = x.to(torch.bfloat16)
    return t


def build(cfg_json, seed=0):
    """(ModelWeights, oracle, tensors)."""
    t = random_tensors(cfg_json, seed)
    return weights_from_tensors(config_from_json(cfg_json), t), MilutarRef(cfg_json, t), t


def needle(cfg_json, strength=1.0, seed=7):
    """A model in which token 1 asks for token 2 and nothing else: the query of token 1 lines up with the key of token 2 in
    every layer, so one score stands out among any number of keys and the value of token 2 decides the logits."""
    t = random_tensors(cfg_json, seed)
    W = cfg_json["width"]
    t["embed"][:] = (t["embed"].float() * 0.5).to(torch.bfloat16)
    t["embed"][:, :2] = 0
    t["embed"][1, 0] = t["embed"][2, 1] = 12.0
    t["head"][:, :2] = 0
    if "loop.step" in t:
        t["loop.step"][:, :2] = 0
    for i, l in enumerate(cfg_json["layers"]):
        m, p = l["mixer"], f"l{i}."
        t[p + "shift"][:2] = 0
        pattern = torch.where(torch.arange(m["dim"]) % 2 == 0, 1.0, -1.0) * strength
        t[p + "mix.dkv"][0, 1] = 2.0 * W ** 0.5
        t[p + "mix.uk"][:, 0] = pattern.repeat(m["heads"]).to(torch.bfloat16)
        q = torch.zeros(m["heads"], m["dim"] + m["rot_dim"])
        q[:, :m["dim"]] = pattern
        if l["type"] == "latent_attention_2":
            t[p + "mix.dq"][0, 0] = 2.0 * W ** 0.5
            t[p + "mix.uq"][:, 0] = q.reshape(-1).to(torch.bfloat16)
        else:
            t[p + "mix.q"][:, 0] = q.reshape(-1).to(torch.bfloat16)
    return weights_from_tensors(config_from_json(cfg_json), t), MilutarRef(cfg_json, t), t


def with_windows(cfg_json, delta):
    """The same configuration with every window ``delta`` tokens longer."""
    c = copy.deepcopy(cfg_json)
    for l in c["layers"]:
        if "mask" in l["mixer"]:
            l["mixer"]["mask"]["size"] += delta
    return c


def last_logits(ref, ids):
    return ref.forward(torch.tensor(ids))[0][-1:]
