"""Mepatar on the host: configuration and checkpoint folders, the oracle's own consistency, the reference backend."""
import copy
import json
import math
from dataclasses import replace

import pytest
import torch

from hipengine_b200.llm import LLM, SamplingParams
from hipengine_b200.loading import safetensors_dir as S
from hipengine_b200.loading.mepatar import config_from_json, config_to_json, tensor_shapes
from hipengine_b200.loading.model_loader import describe_model_source, load_model
from hipengine_b200.models.config import NAMED_CONFIGS, TINY_MEPATAR
from hipengine_b200.models.registry import folder_plugin, load_object, plugin_for, supported_architectures
from hipengine_b200.ref import mepatar as R

from mepatar_models import (EXACT_MODELS, HEADS, ODD, TOL, attention, build, decided, delta, dense, last_logits, logit_error, model, moe,
                            needle, random_tensors, retention, tokens, with_masks)


def _write(path, cfg_json, t):
    (path / "config.json").write_text(json.dumps(cfg_json))
    S.write_tensors(path / "model.safetensors", t)


# ----------------------------------------------------------------------------- configuration, checkpoint folders
@pytest.mark.parametrize("name", list(EXACT_MODELS))
def test_config_round_trip(name):
    c = EXACT_MODELS[name]
    cfg = config_from_json(c)
    back = config_to_json(cfg)
    assert config_from_json(back) == cfg and back == c
    assert (cfg.rms_eps, cfg.norm_groups, cfg.embed_scale) == (c["norm"]["eps"], c["norm"]["groups"], c["embedding"]["scale"])


def test_cache_planes_and_states():
    """Only attention has a cache; states are the matrices, a ring of the convolution's inputs and the rows ahead of the mixer."""
    cfg = config_from_json(ODD)
    assert [l.mixer.cache_elems for l in cfg.layer_specs] == [0, 2 * 3 * 64, 0, 0, 0]
    assert cfg.kv_bytes_per_token() == 2 * 384
    conv = 2 * 64 + 168                                     # query, key, value columns, each padded to eight
    assert [l.state_elems(cfg.hidden) - 3 * 136 for l in cfg.layer_specs] == [6 * 20 * 32 + 3 * conv, 0, 3 * 33 * 24, 5 * 12 * 32,
                                                                             2 * 44 * 16 + 5 * (2 * 88 + 24)]
    assert cfg.has_recurrent_state and cfg.layer_specs[0].attention is None
    none = config_from_json(model(64, 50, [(attention(2, 1, 8, 8, 0.3, 5, 1, 4, 10.0), None)], taps=1))
    assert not none.has_recurrent_state and none.recurrent_state_bytes() == 0


def _change(i, part="mixer", **kw):
    c = copy.deepcopy(ODD)
    c["layers"][i][part].update(kw)
    return {"layers": c["layers"]}


@pytest.mark.parametrize("bad", [
    {"layers": []},
    {"norm": {"eps": 1e-5, "groups": 5}},
    {"canon": {"taps": 0}},
    {"canon": {"taps": 40}},
    {"width": 13200, "norm": {"eps": 1e-5, "groups": 1}},
    {"layers": [{"type": "recurrent", "mixer": {"heads": 1, "dim": 8, "vdim": 8}, "mlp": None}]},
    {"layers": [{**ODD["layers"][0], "mlp": {"kind": "sparse"}}]},
    _change(0, kv_heads=4), _change(0, dim=600), _change(0, vdim=513), _change(0, conv=0),
    _change(1, kv_heads=4), _change(1, rot={"dims": 9, "base": 10.0}), _change(1, rot={"dims": 22, "base": 10.0}),
    _change(1, mask={"size": 0, "keep_first": 3}), _change(1, mask={"size": 4, "keep_first": -1}), _change(1, dim=600),
    _change(1, "mlp", router={"experts": 4, "top": 5}), _change(1, "mlp", router={"experts": 600, "top": 2}),
    _change(2, decay=[0.9, 0.8]), _change(2, decay=[0.9, 0.8, 1.5]), _change(2, decay=[0.9, 0.0, 0.5]),
    _change(2, rot={"dims": 40, "base": 10.0}),
])
def test_impossible_configurations_are_refused(bad):
    with pytest.raises(ValueError):
        config_from_json({**ODD, **bad})


def test_checkpoint_folder(tmp_path):
    w, _, t = build(ODD)
    _write(tmp_path, ODD, t)
    got = load_model(tmp_path)
    assert got.config == w.config and set(got.tensors) == set(t) == set(tensor_shapes(w.config))
    assert "l2.norm2" not in t and "l2.mlp.gate" not in t and "l3.mlp.e6.down" in t and "l2.canon1" in t
    assert t["l0.mix.q.conv"].shape == (60, 3) and t["l4.mix.v.conv"].shape == (20, 5) and t["l1.mix.temp"].shape == (6,)
    for n, x in t.items():
        assert torch.equal(got[n].dequant().to(torch.bfloat16), x), n
    d = describe_model_source(tmp_path)
    assert d["arch"] == "mepatar" and d["source"] == "safetensors" and "error" not in d
    assert d["family"]["ffn"] == {"dense": 1, "moe": 2, "none": 2} and d["family"]["layers"] == {"linear": 2, "retention": 2, "sliding": 1}
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.loading.admission import admit
    report = admit(got, EngineConfig(), free_bytes=1 << 40)
    assert report["admitted"] and report["memory"]["recurrent_state_bytes"] > 0
    _write(tmp_path, ODD, {n: x for n, x in t.items() if n != "l4.mix.A_log"})
    with pytest.raises(KeyError, match="A_log"):
        load_model(tmp_path)
    _write(tmp_path, ODD, {**t, "l0.canon1": torch.ones(132, 3, dtype=torch.bfloat16)})
    with pytest.raises(KeyError, match="canon1"):
        load_model(tmp_path)


def test_registry_entries():
    p = plugin_for("mepatar")
    assert p is folder_plugin("Mepatar") and "mepatar" in supported_architectures()
    assert p.compute_dtypes == ("bfloat16", "float32") and not p.tensor_parallel
    assert p.describe(TINY_MEPATAR)["layers"] == {"linear": 2, "retention": 1, "sliding": 1}
    from hipengine_b200.core import build as B
    assert set(p.native_sources) <= {s.name for s in B.sources()}
    assert load_object(p.executor).__name__ == "MepatarExecutor" and load_object(p.reference) is R.MepatarRef
    assert all(c in NAMED_CONFIGS for c in ("tiny-mepatar", "mepatar-8b", "mepatar-30b-moe"))
    from hipengine_b200.server.readiness import kv_capability
    from hipengine_b200.config import EngineConfig
    d = kv_capability(TINY_MEPATAR, EngineConfig().kv)
    assert d["sliding_window"] and d["recurrent_state_snapshots"] and "[k|v]" in d["layout"]


# ----------------------------------------------------------------------------- the oracle, mechanism by mechanism
def test_oracle_norms():
    x = torch.tensor([[3.0, 4.0, 0.5, 0.0]])
    y = R.grouped_norm(x, torch.tensor([1.0, 2.0, 1.0, 1.0]), 2, 0.0)
    assert torch.allclose(y, torch.tensor([[3.0, 8.0, 1.0, 0.0]]) / torch.tensor([12.5 ** 0.5, 12.5 ** 0.5, 0.125 ** 0.5 / 0.5, 1.0]))
    assert torch.allclose(R.rms(torch.zeros(1, 3), 1e-4), torch.zeros(1, 3))
    assert torch.allclose(R.unit(torch.tensor([3.0, 4.0])), torch.tensor([0.6, 0.8]))


def test_oracle_convolution_keeps_the_newest_tap_last():
    x, before, w = torch.tensor([[1.0], [2.0]]), torch.tensor([[5.0], [7.0]]), torch.tensor([[100.0, 10.0, 1.0]])
    y, kept = R.causal_conv(x, before, w)
    assert y.flatten().tolist() == [571.0, 712.0] and kept.flatten().tolist() == [1.0, 2.0]
    y, kept = R.causal_conv(x[:1], before, w)
    assert y.flatten().tolist() == [571.0] and kept.flatten().tolist() == [7.0, 1.0]
    assert R.causal_conv(x, torch.zeros(0, 1), torch.tensor([[3.0]]))[0].flatten().tolist() == [3.0, 6.0]


def test_oracle_rotations():
    pos, base = torch.tensor([1]), 4.0                                   # frequencies 1 and 1/2
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 7.0]]])
    c, s = [math.cos(1.0), math.cos(0.5)], [math.sin(1.0), math.sin(0.5)]
    assert torch.allclose(R.rotate_halves(x, pos, 4, base)[0, 0], torch.tensor([c[0], -2 * s[1], s[0], 2 * c[1], 7.0]), atol=1e-6)
    assert torch.allclose(R.rotate_neighbours(x, pos, 4, base)[0, 0], torch.tensor([c[0], s[0], -2 * s[1], 2 * c[1], 7.0]), atol=1e-6)
    assert torch.equal(R.rotate_halves(x, torch.tensor([0]), 4, base), x)


def test_oracle_mask():
    assert R.visible_keys(torch.tensor([6]), 8, 3, 2)[0].tolist() == [True, True, False, False, True, True, True, False]
    assert R.visible_keys(torch.tensor([0]), 3, 1, 2)[0].tolist() == [True, False, False]     # kept tokens are not seen early
    assert R.visible_keys(torch.tensor([2]), 3, 1, 0)[0].tolist() == [False, False, True]


def test_oracle_recurrences_step_by_step():
    q, k, v = (torch.tensor([[[a]], [[b]]]) for a, b in ((2.0, 3.0), (0.5, 1.0), (4.0, 6.0)))
    o, S = R.retention(q, k, v, torch.tensor([0.5]), torch.tensor([[[8.0]]]))
    s1 = 0.5 * 8 + 0.5 * 4
    assert o.flatten().tolist() == [2 * s1, 3 * (0.5 * s1 + 6)] and float(S) == 0.5 * s1 + 6
    o, S = R.delta_rule(q, k, v, torch.tensor([[0.5], [1.0]]), torch.tensor([[1.0], [0.25]]), torch.tensor([[[8.0]]]))
    s1 = 4.0 + 0.5 * (4.0 - 0.5 * 4.0)
    s2 = s1 + 0.25 * (6.0 - s1)
    assert o.flatten().tolist() == [2 * s1, 3 * s2] and float(S) == s2


def test_oracle_experts_and_routing():
    ids, w = R.routing(torch.log(torch.tensor([[1.0, 4.0, 3.0, 2.0]])), 2)
    assert ids.tolist() == [[1, 2]] and torch.allclose(w, torch.tensor([[0.4, 0.3]]))
    eye = torch.eye(2)
    h = torch.tensor([[3.0, -0.5]])
    y = R.clamped_expert(h, eye, -eye, eye, 1.0)[0]                      # gates 1, -0.5; ups -1, 0.5
    sg = lambda x: 1 / (1 + math.exp(-1.702 * x))
    assert torch.allclose(y, torch.tensor([0.0, -0.5 * sg(-0.5) * 1.5]))


@pytest.mark.parametrize("name", list(EXACT_MODELS))
def test_oracle_does_not_depend_on_the_cut(name):
    _, ref, _ = build(EXACT_MODELS[name])
    ids = torch.tensor(tokens(30, EXACT_MODELS[name]["vocab"], 3))
    whole, _ = ref.forward(ids)
    st, parts, at = ref.new_state(), [], 0
    for n in (2, 7, 1, 1, 10, 9):
        lg, st = ref.forward(ids[at:at + n], st)
        parts.append(lg)
        at += n
    assert logit_error(torch.cat(parts), whole) < 1e-4


def _mutants():
    """(what is wrong) -> configuration and tensors with a mistake that the whole-model tests must be able to see."""
    def cfg(f):
        def run(c, t):
            c = copy.deepcopy(c)
            for l in c["layers"]:
                f(l, c)
            return c, t
        return run

    def ten(f):
        return lambda c, t: (c, {n: f(n, x) for n, x in t.items()})
    ones = lambda suffix: ten(lambda n, x: torch.ones_like(x) if n.endswith(suffix) else x)
    zero = lambda suffix: ten(lambda n, x: torch.zeros_like(x) if n.endswith(suffix) else x)
    of = lambda kind, **kw: cfg(lambda l, c: l["mixer"].update(kw) if l["type"] == kind else None)
    turned = lambda f: cfg(lambda l, c: l["mixer"]["rot"].update(f(l["mixer"]["rot"])) if "rot" in l["mixer"] else None)
    return {
        "no query bias": zero("mix.q.b"), "no key bias": zero("mix.k.b"), "no value bias": zero("mix.v.b"), "no output bias": zero("mix.o.b"),
        "no query gain": ones("q.norm"), "no key gain": ones("k.norm"), "no factor on the scores": ones(".temp"),
        "no gain 1": ones("norm1"), "no gain 2": ones("norm2"), "no final gain": ones("final.norm"), "no gain of the delta rule": ones("mix.norm"),
        "no input convolution": zero("canon1"), "input taps reversed": ten(lambda n, x: x.flip(1) if n.endswith("canon1") else x),
        "taps reversed": ten(lambda n, x: x.flip(1) if n.endswith(".conv") else x),
        "no step sizes": zero(".mix.b"), "decays not by the token": zero(".mix.a"), "no decay bias": zero("dt_bias"), "no rates": zero("A_log"),
        "no output gate": zero(".mix.g"),
        "one group": cfg(lambda l, c: c["norm"].update(groups=1)), "no embedding factor": cfg(lambda l, c: c["embedding"].update(scale=1.0)),
        "other eps": cfg(lambda l, c: c["norm"].update(eps=0.3)),
        "scores not scaled": of("attention", scale=1.0), "window longer": lambda c, t: (with_masks(c, size=1), t),
        "window shorter": lambda c, t: (with_masks(c, size=-1), t), "one more kept": lambda c, t: (with_masks(c, keep=1), t),
        "none kept": lambda c, t: (with_masks(c, keep=-100), t),
        "other base": turned(lambda r: {"base": r["base"] * 3}), "fewer dimensions turned": turned(lambda r: {"dims": r["dims"] - 2}),
        "slower decay": cfg(lambda l, c: l["mixer"].update(decay=[1 - (1 - d) / 2 for d in l["mixer"]["decay"]]) if "decay" in l["mixer"] else None),
        "no limit": cfg(lambda l, c: l["mlp"]["expert"].update(limit=100.0) if l["mlp"] and l["mlp"]["kind"] == "moe" else None),
        "one expert less": cfg(lambda l, c: l["mlp"]["router"].update(top=l["mlp"]["router"]["top"] - 1) if l["mlp"] and l["mlp"]["kind"] == "moe" else None),
        "heads swapped": ten(lambda n, x: x.reshape(-1, 2).flip(1).reshape(x.shape) if n.endswith("mix.o") else x),
    }


@pytest.mark.parametrize("what", list(_mutants()))
def test_mistakes_show_in_the_test_models(what):
    """A mechanism left out of the oracle moves the logits by several times the bfloat16 tolerance of the GPU tests."""
    t = decided(ODD, random_tensors(ODD, 0))
    ids = torch.tensor(tokens(60, ODD["vocab"], 5))
    want = R.MepatarRef(ODD, t).forward(ids)[0]
    c2, t2 = _mutants()[what](ODD, t)
    assert logit_error(R.MepatarRef(c2, t2).forward(ids)[0], want) > 4 * TOL["bfloat16"]


@pytest.mark.parametrize("what", ["normalised weights", "keys not scaled", "read before write", "no unit length", "halves", "shared norm"])
def test_mistakes_in_the_mechanisms_show(what, monkeypatch):
    t = decided(ODD, random_tensors(ODD, 0))
    ids = torch.tensor(tokens(60, ODD["vocab"], 5))
    ref = R.MepatarRef(ODD, t)
    want = ref.forward(ids)[0]
    if what == "normalised weights":
        real = R.routing
        monkeypatch.setattr(R, "routing", lambda lg, top: (real(lg, top)[0], real(lg, top)[1] / real(lg, top)[1].sum(-1, keepdim=True)))
    elif what == "keys not scaled":                        # the output is normalised, but eps is not
        real = R.retention
        monkeypatch.setattr(R, "retention", lambda q, k, v, d, S: real(q, k * 1e-3, v, d, S))
    elif what == "read before write":
        def early(q, k, v, g, beta, S):
            out = []
            for i in range(q.shape[0]):
                S = g[i][:, None, None] * S
                out.append(torch.einsum("hkv,hk->hv", S, q[i]))
                S = S + k[i][:, :, None] * (beta[i][:, None] * (v[i] - torch.einsum("hkv,hk->hv", S, k[i])))[:, None, :]
            return torch.stack(out), S
        monkeypatch.setattr(R, "delta_rule", early)
    elif what == "no unit length":
        monkeypatch.setattr(R, "unit", lambda x: 0.3 * torch.tanh(x))
    elif what == "halves":
        monkeypatch.setattr(R, "rotate_neighbours", R.rotate_halves)
    else:
        t2 = {n: t[n.replace("norm2", "norm1")] for n in t}
        ref = R.MepatarRef(ODD, t2)
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


def test_needle_model_shows_the_key_and_the_edges():
    c = model(96, 160, [(attention(4, 2, 24, 16, 1.0, 12, 6, 8, 500.0), dense(64))])
    _, ref, _ = needle(c, 2.0)
    base = [3 + x for x in tokens(40, 157, 1)]
    base[-1] = 1
    err = {}
    for p in (2, 5, 6, 20, 25, 28, 38):                    # 26 and 27 read 25 through the input convolution, 28 does not
        ids = list(base)
        ids[p] = 2
        err[p] = logit_error(last_logits(ref, ids), last_logits(ref, base))
    assert min(err[2], err[5], err[28], err[38]) > 0.16 and max(err[6], err[20], err[25]) < 1e-5


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
    w = build_random_model(TINY_MEPATAR, seed=1)
    ref = R.MepatarRef(w.metadata["config"], {n: q.dequant() for n, q in w.tensors.items()})
    lg, st = ref.forward(torch.tensor(tokens(20, 1024, 0)))
    assert bool(torch.isfinite(lg).all()) and all(bool(torch.isfinite(s).all()) for s in st.S.values()) and len(st.S) == 3
