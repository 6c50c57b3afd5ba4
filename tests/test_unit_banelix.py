"""Banelix on the host: configuration and checkpoint folders, the oracle's own consistency, the reference backend."""
import copy
import json
import math
from dataclasses import replace

import pytest
import torch

from hipengine_b200.llm import LLM, SamplingParams
from hipengine_b200.loading import safetensors_dir as S
from hipengine_b200.loading.banelix import config_from_json, config_to_json, tensor_shapes
from hipengine_b200.loading.model_loader import describe_model_source, load_model
from hipengine_b200.models.config import NAMED_CONFIGS, TINY_BANELIX, BandSpec, RotarySpec, YarnSpec
from hipengine_b200.models.registry import folder_plugin, load_object, plugin_for, supported_architectures
from hipengine_b200.ref import banelix as R

from banelix_models import (HEADS, MODELS, ODD, TOL, bands, both, build, last_logits, logit_error, model, needle,
                            random_tensors, rotation, tokens, windowed, with_windows, yarn)


def _write(path, cfg_json, t):
    (path / "config.json").write_text(json.dumps(cfg_json))
    S.write_tensors(path / "model.safetensors", t)


# ----------------------------------------------------------------------------- configuration, checkpoint folders
@pytest.mark.parametrize("name", list(MODELS))
def test_config_round_trip(name):
    cfg = config_from_json(MODELS[name])
    back = config_to_json(cfg)
    assert config_from_json(back) == cfg and back == MODELS[name]
    assert (cfg.rms_eps, cfg.residual_mult, cfg.embed_scale) == tuple(
        v for v in (MODELS[name]["norm"]["eps"], MODELS[name]["residual_mult"], MODELS[name]["embedding"]["scale"]))


def test_cache_planes_and_states():
    """A layer on another one's keys has no cache of its own; a recurrence carries its padded channels and the last inputs."""
    cfg = config_from_json(ODD)
    assert [l.attention.cache_elems for l in cfg.layer_specs] == [2 * 3 * 64, 2 * 2 * 64, 2 * 1 * 64, 0]
    assert cfg.kv_bytes_per_token() == 2 * (384 + 256 + 128) == cfg.kv_bytes_per_token(4) // 2
    assert [l.state_elems(cfg.hidden) for l in cfg.layer_specs] == [0, 4 * 16 * 3, 2 * 24 * 4, 0]
    assert cfg.recurrent_state_bytes() == 4 * (192 + 192) and cfg.has_recurrent_state
    only = config_from_json(model(64, 50, [(windowed(2, 1, 8, 8, 0.3, 5, rotation(4, 10.0)), 16)]))
    assert not only.has_recurrent_state and only.recurrent_state_bytes() == 0


def _change(i, **kw):
    c = copy.deepcopy(ODD)
    for k, v in kw.items():
        c["layers"][i]["mixer"][k] = v
    return {"layers": c["layers"]}


@pytest.mark.parametrize("bad", [
    {"layers": []},
    {"layers": [{"type": "recurrent", "mixer": {}, "mlp": None}]},
    {"layers": [{**ODD["layers"][0], "mlp": {"kind": "moe"}}]},
    _change(0, kv_heads=4),
    _change(0, dim=600),
    _change(0, rot=rotation(22, 10.0)),
    _change(0, rot=rotation(9, 10.0)),
    _change(0, rot=rotation(10, 10.0, {"factor": 2.0})),
    _change(3, kv_from=3),
    _change(3, kv_from=1),
    _change(3, kv_from=7),
    _change(3, kv_heads=2),
    _change(1, right={"width": 61, "blocks": 4, "conv": 3}),
    _change(1, right={"width": 60, "blocks": 4, "conv": 0}),
    _change(1, left={**ODD["layers"][1]["mixer"]["left"], "vdim": 20}),
])
def test_impossible_configurations_are_refused(bad):
    with pytest.raises(ValueError):
        config_from_json({**ODD, **bad})


def test_checkpoint_folder(tmp_path):
    w, _, t = build(ODD)
    _write(tmp_path, ODD, t)
    got = load_model(tmp_path)
    assert got.config == w.config and set(got.tensors) == set(t) == set(tensor_shapes(w.config))
    assert "l2.norm2" not in t and "l3.mix.k" not in t and "l3.mix.k.norm" not in t and "l1.mix.left.v" not in t
    assert t["l1.mix.right.ra"].shape == (4, 15, 15) and t["l2.mix.right.conv"].shape == (44, 4)
    for n, x in t.items():
        assert torch.equal(got[n].dequant().to(torch.bfloat16), x), n
    d = describe_model_source(tmp_path)
    assert d["arch"] == "banelix" and d["source"] == "safetensors" and "error" not in d
    assert d["family"]["ffn"] == {"dense": 3, "none": 1} and d["family"]["layers"] == {"full+recurrent": 2, "sliding": 2}
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.loading.admission import admit
    report = admit(got, EngineConfig(), free_bytes=1 << 40)
    assert report["admitted"] and report["memory"]["recurrent_state_bytes"] > 0
    _write(tmp_path, ODD, {n: x for n, x in t.items() if n != "l1.mix.right.lam"})
    with pytest.raises(KeyError, match="lam"):
        load_model(tmp_path)
    _write(tmp_path, ODD, {**t, "l1.mix.right.ra": torch.ones(2, 30, 30, dtype=torch.bfloat16)})
    with pytest.raises(KeyError, match="ra"):
        load_model(tmp_path)


def test_registry_entries():
    p = plugin_for("banelix")
    assert p is folder_plugin("Banelix") and "banelix" in supported_architectures()
    assert p.compute_dtypes == ("bfloat16", "float32") and not p.tensor_parallel
    assert p.describe(TINY_BANELIX)["layers"] == {"full+recurrent": 2, "sliding": 2}
    from hipengine_b200.core import build as B
    assert set(p.native_sources) <= {s.name for s in B.sources()}
    assert load_object(p.executor).__name__ == "BanelixExecutor" and load_object(p.reference) is R.BanelixRef
    assert all(c in NAMED_CONFIGS for c in ("tiny-banelix", "banelix-8b"))
    from hipengine_b200.server.readiness import kv_capability
    from hipengine_b200.config import EngineConfig
    d = kv_capability(TINY_BANELIX, EngineConfig().kv)
    assert d["sliding_window"] and d["recurrent_state_snapshots"] and "[k|v]" in d["layout"]


@pytest.mark.parametrize("dims,base,s", [(2, 100.0, None), (12, 3000.0, ("y", 6.0, 256.0, 16.0, 1.0)), (64, 1e6, ("b", 8.0, 1.0, 4.0, 8192.0)),
                                         (4, 500.0, ("y", 3.0, 64.0, 8.0, 2.0)), (16, 10000.0, ("y", 1.0, 4096.0, 32.0, 1.0)),
                                         (40, 50.0, ("b", 3.0, 0.5, 7.0, 100.0)), (20, 9000.0, ("b", 1.0, 1.0, 4.0, 512.0))])
def test_rotation_table(dims, base, s):
    spec = None if s is None else YarnSpec(*s[1:]) if s[0] == "y" else BandSpec(*s[1:])
    freq, amp = RotarySpec(dims, base, spec, halves=True).table()
    want, want_amp = R.rotation(rotation(dims, base, None if s is None else (yarn if s[0] == "y" else bands)(*s[1:])))
    assert torch.allclose(torch.tensor(freq, dtype=torch.float64), want, rtol=1e-12) and abs(amp - want_amp) < 1e-12


# ----------------------------------------------------------------------------- the oracle, mechanism by mechanism
def test_oracle_rotation_turns_halves_and_passes_the_rest():
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 7.0]]])
    f = torch.tensor([math.pi / 2, math.pi / 6], dtype=torch.float64)
    y = R.rotate_halves(x, torch.tensor([1]), f, 1.5)[0, 0]                 # pairs (0, 2) and (1, 3)
    assert torch.allclose(y, torch.tensor([0.0, -1.5, 1.5, 1.5 * math.sqrt(3.0), 7.0]), atol=1e-6)
    assert torch.equal(R.rotate_halves(x, torch.tensor([0]), f), x)


def test_oracle_bands_keep_fast_waves_and_slow_down_long_ones():
    f = torch.tensor(R.plain_freqs(64, 5e5), dtype=torch.float64)
    g = torch.tensor(R.banded_freqs(f.tolist(), bands(8.0, 1.0, 4.0, 8192.0)), dtype=torch.float64)
    turns = f * 8192.0 / (2 * math.pi)
    assert torch.equal(g[turns > 4], f[turns > 4]) and torch.allclose(g[turns < 1], f[turns < 1] / 8)
    mid = (turns > 1) & (turns < 4)
    assert bool(mid.any()) and bool(((g < f) & (g > f / 8))[mid].all())


def test_oracle_extra_unit_and_window():
    s, seen = torch.tensor([[0.3, -0.2, 5.0]]), torch.tensor([[True, True, False]])
    e = [math.exp(0.3), math.exp(-0.2), 1.0]
    assert torch.allclose(R.weights_over(s, seen, True), torch.tensor([[e[0] / sum(e), e[1] / sum(e), 0.0]]))
    assert torch.allclose(R.weights_over(s - 200.0, seen, True), torch.zeros(1, 3), atol=1e-30)
    assert torch.allclose(R.weights_over(s, seen, False).sum(), torch.tensor(1.0))
    assert R.visible_keys(torch.tensor([4]), 6, 3)[0].tolist() == [False, False, True, True, True, False]


def test_oracle_convolution_and_blocks():
    x, before, w = torch.tensor([[1.0], [2.0]]), torch.tensor([[5.0], [7.0]]), torch.tensor([[100.0, 10.0, 1.0]])
    assert R.causal_conv(x, before, w, torch.tensor([0.5])).flatten().tolist() == [571.5, 712.5]
    assert R.causal_conv(x, torch.zeros(0, 1), torch.tensor([[3.0]]), torch.tensor([0.0])).flatten().tolist() == [3.0, 6.0]
    y = R.block_product(torch.tensor([[1.0, 2.0, 3.0, 4.0]]), torch.tensor([[[1.0, 10.0], [0.0, 1.0]], [[2.0, 0.0], [1.0, 1.0]]]),
                        torch.zeros(2, 2))
    assert y.tolist() == [[21.0, 2.0, 6.0, 7.0]]


def test_oracle_recurrence_step_by_step():
    u, r, i, lam = torch.tensor([[2.0], [3.0]]), torch.tensor([[0.5], [0.25]]), torch.tensor([[1.0], [0.5]]), torch.tensor([-2.0])
    sp, S, want = math.log1p(math.exp(-2.0)), 0.7, []
    for k in range(2):
        a = math.exp(-8 * float(r[k]) * sp)
        S = a * S + math.sqrt(1 - a * a) * float(i[k] * u[k])
        want.append(S)
    out, last = R.gated_recurrence(u, r, i, lam, torch.tensor([0.7]))
    assert torch.allclose(out.flatten(), torch.tensor(want)) and torch.equal(last, out[-1])


@pytest.mark.parametrize("name", list(MODELS))
def test_oracle_does_not_depend_on_the_cut(name):
    _, ref, _ = build(MODELS[name])
    ids = torch.tensor(tokens(30, MODELS[name]["vocab"], 3))
    whole, _ = ref.forward(ids)
    st, parts, at = ref.new_state(), [], 0
    for n in (2, 7, 1, 1, 10, 9):
        lg, st = ref.forward(ids[at:at + n], st)
        parts.append(lg)
        at += n
    assert logit_error(torch.cat(parts), whole) < 1e-5


def _mutants():
    """(what is wrong) -> configuration and tensors with a mistake that the whole-model tests must be able to see."""
    def cfg(f):
        def run(c, t):
            c = copy.deepcopy(c)
            for l in c["layers"]:
                f(l, c)
            return c, t
        return run

    def part(l):
        return l["mixer"]["left"] if l["type"] == "parallel" else l["mixer"]

    def ten(f):
        return lambda c, t: (c, {n: f(n, x) for n, x in t.items()})
    ones = lambda suffix: ten(lambda n, x: torch.ones_like(x) if n.endswith(suffix) else x)
    zero = lambda suffix: ten(lambda n, x: torch.zeros_like(x) if n.endswith(suffix) else x)
    swap = lambda x: x.reshape(-1, 2).flip(1).reshape(x.shape)
    right = lambda **kw: cfg(lambda l, c: l["mixer"].update(kw) if l["type"] == "parallel" else None)
    return {
        "no query bias": zero("mix.q.b"), "no key bias": zero("mix.k.b"), "no value bias": zero("mix.v.b"),
        "no query bias (left)": zero("left.q.b"), "no key bias (left)": zero("left.k.b"),
        "no query gain": ones("q.norm"), "no key gain": ones("k.norm"),
        "no gain 1": ones("norm1"), "no gain 2": ones("norm2"), "no final gain": ones("final.norm"),
        "head gate always half": zero("left.g"),
        "no bias of the output gate": zero("right.y.b"), "no bias of the recurrence": zero("right.x.b"),
        "no convolution bias": zero("conv.b"), "no gate bias r": zero("ra.b"), "no gate bias i": zero("ri.b"),
        "gates swapped": lambda c, t: (c, {n: t[n.replace("t.ra", "t.rX").replace("t.ri", "t.ra").replace("t.rX", "t.ri")] for n in t}),
        "taps reversed": ten(lambda n, x: x.flip(1) if n.endswith(".conv") else x),
        "lambda zero": zero(".lam"),
        "no residual factor": cfg(lambda l, c: c.update(residual_mult=1.0)),
        "no embedding factor": cfg(lambda l, c: c["embedding"].update(scale=1.0)),
        "left not scaled": right(left_scale=1.0), "right not scaled": right(right_scale=1.0),
        "no scaling of the rotation": cfg(lambda l, c: part(l)["rot"].pop("scaling", None)),
        "other base": cfg(lambda l, c: part(l)["rot"].update(base=part(l)["rot"]["base"] * 3)),
        "scores not scaled": cfg(lambda l, c: part(l).update(scale=1.0)),
        "window longer": lambda c, t: (with_windows(c, 1), t),
        "window shorter": lambda c, t: (with_windows(c, -1), t),
        "heads swapped": ten(lambda n, x: swap(x) if n.endswith("mix.o") else x),
        "blocks swapped": ten(lambda n, x: x.flip(0) if n.endswith((".ra", ".ri")) else x),
    }


@pytest.mark.parametrize("what", list(_mutants()))
def test_mistakes_show_in_the_test_models(what):
    """A mechanism left out of the oracle moves the logits by several times the bfloat16 tolerance of the GPU tests."""
    t = random_tensors(ODD, 0)
    ids = torch.tensor(tokens(60, ODD["vocab"], 5))
    want = R.BanelixRef(ODD, t).forward(ids)[0]
    c2, t2 = _mutants()[what](ODD, t)
    assert logit_error(R.BanelixRef(c2, t2).forward(ids)[0], want) > 4 * TOL["bfloat16"]


@pytest.mark.parametrize("what", ["unit", "keys", "rotated values", "extra"])
def test_mistakes_in_the_mixers_show(what, monkeypatch):
    t = random_tensors(ODD, 0)
    ids = torch.tensor(tokens(60, ODD["vocab"], 5))
    want = R.BanelixRef(ODD, t).forward(ids)[0]
    ref = R.BanelixRef(ODD, t)
    if what == "unit":                                     # queries and keys not brought to unit length
        real = R.rms
        monkeypatch.setattr(R, "rms", lambda x, eps: x if x.dim() == 3 else real(x, eps))
    elif what == "keys":                                   # the last layer on keys of its own rows' order: shifted by one
        real_att = ref.windowed_attention

        def shifted(i, h, st, pos):
            keep = st.k[0]
            if i == 3:
                st.k[0] = keep.roll(1, 0)
            out = real_att(i, h, st, pos)
            if i == 3:
                st.k[0] = keep
            return out
        ref.windowed_attention = lambda i, h, st, pos: shifted(i, h, st, pos) if 0 in st.k else real_att(i, h, st, pos)
    elif what == "rotated values":
        real_ext = ref.extend
        ref.extend = lambda i, st, k, v: real_ext(i, st, k, k if ODD["layers"][i]["type"] == "parallel" else v)
    else:
        real_w = R.weights_over
        monkeypatch.setattr(R, "weights_over", lambda s, seen, extra: real_w(s, seen, False))
    assert logit_error(ref.forward(ids)[0], want) > 4 * TOL["bfloat16"]


def test_lost_state_shows_after_a_cut():
    _, ref, _ = build(ODD)
    ids = torch.tensor(tokens(40, ODD["vocab"], 5))
    want = ref.forward(ids)[0][25:]
    for lost in ("S", "conv", "k", "v"):
        _, st = ref.forward(ids[:25], ref.new_state())
        for i, x in getattr(st, lost).items():
            getattr(st, lost)[i] = torch.zeros_like(x)
        assert logit_error(ref.forward(ids[25:], st)[0], want) > 4 * TOL["bfloat16"], lost


def test_needle_model_shows_the_key_and_the_window_edge():
    c = model(96, 160, [(both(4, 2, 24, 0.4, rotation(8, 500.0), 32, 2, 3, 1.0, 0.3), 64)])
    _, ref, _ = needle(c, 2.0)
    base = [3 + x for x in tokens(40, 157, 1)]
    base[-1] = 1
    for p in (0, 15, 16, 38):
        ids = list(base)
        ids[p] = 2
        assert logit_error(last_logits(ref, ids), last_logits(ref, base)) > 0.2
    c = model(96, 160, [(windowed(4, 2, 24, 16, 0.2, 12, rotation(8, 500.0)), 64)])
    _, ref, _ = needle(c, 2.0)
    err = {}
    for d in (10, 11, 12, 13):                             # distance from the asking token
        ids = list(base)
        ids[39 - d] = 2
        err[d] = logit_error(last_logits(ref, ids), last_logits(ref, base))
    assert min(err[10], err[11]) > 0.2 and max(err[12], err[13]) < 1e-5


# ----------------------------------------------------------------------------- host backend and scheduler
def test_reference_backend_generates_greedily(tmp_path):
    from hipengine_b200.config import EngineConfig
    _, ref, t = build(HEADS)
    _write(tmp_path, HEADS, t)
    prompts = [tokens(n, HEADS["vocab"], n) for n in (1, 5, 18)]
    base = EngineConfig()
    for policy in ("protect_decode", "mixed"):
        eng = replace(base, scheduler=replace(base.scheduler, policy=policy, max_prefill_chunk_tokens=4))
        with LLM(str(tmp_path), backend="cpu_reference", engine_config=eng) as llm:
            got = llm.generate_token_ids(prompts, SamplingParams(max_tokens=5, ignore_eos=True))
        for p, g in zip(prompts, got):
            seq = list(p)
            for tok in g:
                assert int(last_logits(ref, seq)[0].argmax()) == tok
                seq.append(tok)


def test_random_models_have_finite_states():
    from hipengine_b200.loading.synth import build_random_model
    w = build_random_model(TINY_BANELIX, seed=1)
    ref = R.BanelixRef(w.metadata["config"], {n: q.dequant() for n, q in w.tensors.items()})
    lg, st = ref.forward(torch.tensor(tokens(20, 1024, 0)))
    assert bool(torch.isfinite(lg).all()) and all(bool(torch.isfinite(s).all()) for s in st.S.values()) and len(st.S) == 2
