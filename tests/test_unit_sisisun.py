"""Sisisun on the host: configuration and checkpoint folders, the oracle's own consistency, the reference backend."""
import json
import struct

import pytest
import torch

from hipengine_b200.llm import LLM, SamplingParams
from hipengine_b200.loading import safetensors_dir as S
from hipengine_b200.loading.model_loader import describe_model_source, load_model
from hipengine_b200.loading.sisisun import config_from_json, config_to_json, tensor_shapes
from hipengine_b200.models.config import NAMED_CONFIGS, TINY_SISISUN, padded_head_width
from hipengine_b200.models.registry import plugin_for, supported_architectures
from hipengine_b200.ref import sisisun as R

from sisisun_models import LOOPED, MODELS, WIDE, build, logit_error, model, moe, needle, tokens


def _write(path, cfg_json, t):
    (path / "config.json").write_text(json.dumps(cfg_json))
    S.write_tensors(path / "model.safetensors", t)


# ----------------------------------------------------------------------------- configuration, checkpoint folders
@pytest.mark.parametrize("name", list(MODELS))
def test_config_round_trip(name):
    cfg = config_from_json(MODELS[name])
    back = config_to_json(cfg)
    assert config_from_json(back) == cfg
    assert back["layers"] == MODELS[name]["layers"] and back["loop"] == MODELS[name]["loop"]
    assert cfg.rms_eps == MODELS[name]["norm"]["eps"]


def test_layer_runs_own_their_cache():
    cfg = config_from_json(WIDE)
    assert cfg.layer_runs() == ((0, -1), (1, 0), (2, 0), (3, 0), (1, 1), (2, 1), (3, 1), (4, -1))
    per_layer = [2 * l.mixer.kv_heads * l.mixer.width * 2 for l in cfg.layer_specs]
    assert cfg.kv_bytes_per_token() == sum(per_layer[i] for i, _ in cfg.layer_runs())
    assert cfg.kv_bytes_per_token(4) == 2 * cfg.kv_bytes_per_token()
    assert config_from_json(model(64, 32, [(WIDE["layers"][0]["mixer"], None)])).layer_runs() == ((0, -1),)
    assert [padded_head_width(d) for d in (1, 64, 65, 200, 257)] == [64, 64, 128, 256, 512]
    cut = cfg.with_layers(3)
    assert cut.layer_runs() == ((0, -1), (1, 0), (2, 0), (1, 1), (2, 1)) and cfg.with_layers(1).loop is None


@pytest.mark.parametrize("bad", [
    {"loop": {"start": 1, "stop": 6, "times": 2}},
    {"layers": [{"type": "recurrent", "mixer": {}, "mlp": None}]},
    {"layers": [{"type": "attention", "mixer": WIDE["layers"][0]["mixer"], "mlp": moe(12, 3, 8, 5, 2, 1.0)}]},
    {"layers": [{"type": "attention", "mixer": WIDE["layers"][0]["mixer"], "mlp": moe(12, 5, 8, 4, 1, 1.0)}]},
    {"layers": [{"type": "attention", "mixer": dict(WIDE["layers"][0]["mixer"], kv_heads=4), "mlp": None}]},
])
def test_impossible_configurations_are_refused(bad):
    with pytest.raises(ValueError):
        config_from_json({**WIDE, **bad})


def test_checkpoint_folder(tmp_path):
    w, _, t = build(WIDE)
    _write(tmp_path, WIDE, t)
    got = load_model(tmp_path)
    assert got.config == w.config and set(got.tensors) == set(t) == set(tensor_shapes(w.config))
    for n, x in t.items():
        assert torch.equal(got[n].dequant().to(torch.bfloat16), x), n
    d = describe_model_source(tmp_path)
    assert d["arch"] == "sisisun" and d["source"] == "safetensors" and "error" not in d
    assert d["family"]["ffn"] == {"dense": 2, "moe": 2, "none": 1} and d["family"]["layer_runs"] == 8
    # an odd header length leaves the data at an address no bfloat16 view may start at
    raw = (tmp_path / "model.safetensors").read_bytes()
    n = struct.unpack("<Q", raw[:8])[0]
    (tmp_path / "model.safetensors").write_bytes(struct.pack("<Q", n + 1) + raw[8:8 + n] + b" " + raw[8 + n:])
    assert torch.equal(load_model(tmp_path)["embed"].dequant().to(torch.bfloat16), t["embed"])


def test_checkpoint_folder_errors(tmp_path):
    _, _, t = build(LOOPED)
    _write(tmp_path, LOOPED, {n: x for n, x in t.items() if n != "loop.step"})
    with pytest.raises(KeyError, match="loop.step"):
        load_model(tmp_path)
    _write(tmp_path, LOOPED, {**t, "head": t["head"][:, :-1].contiguous()})
    with pytest.raises(KeyError, match="head"):
        load_model(tmp_path)
    (tmp_path / "config.json").write_text(json.dumps({**LOOPED, "architecture": "Other"}))
    with pytest.raises(ValueError, match="Other"):
        load_model(tmp_path)
    assert "error" in describe_model_source(tmp_path)
    (tmp_path / "model.safetensors").write_bytes(b"\x10\x00\x00\x00\x00\x00\x00\x00{}")
    with pytest.raises(ValueError):
        S.read_header(tmp_path / "model.safetensors")


def test_registry_entry():
    p = plugin_for("sisisun")
    assert "sisisun" in supported_architectures() and p.compute_dtypes == ("bfloat16", "float32")
    from hipengine_b200.core import build as B
    names = {s.name for s in B.sources()}
    assert set(p.native_sources) <= names
    assert p.describe(TINY_SISISUN)["layers"] == {"full": 4}
    assert all(c in NAMED_CONFIGS for c in ("tiny-sisisun", "sisisun-8b", "sisisun-30b-moe"))


# ----------------------------------------------------------------------------- the oracle, mechanism by mechanism
def test_oracle_sinusoid():
    s = R.sinusoid(torch.tensor([0, 3]), 6)
    assert torch.equal(s[0], torch.tensor([0., 1., 0., 1., 0., 1.]))
    want = [v for i in range(3) for v in (torch.tensor(3.0 * 10000 ** (-i / 3)).sin(),
                                          torch.tensor(3.0 * 10000 ** (-i / 3)).cos())]
    assert torch.allclose(s[1], torch.stack(want), atol=1e-6)


def test_oracle_attention_is_causal_grouped_and_capped():
    g = torch.Generator().manual_seed(0)
    q, k, v = torch.randn(3, 4, 8, generator=g), torch.randn(5, 2, 8, generator=g), torch.randn(5, 2, 3, generator=g)
    o = R.attention(q, k, v, torch.tensor([2, 3, 4]), 0.3, 2.0)
    s = 2.0 * torch.tanh(torch.tensor([float(q[0, 3] @ k[j, 1]) * 0.3 for j in range(3)]) / 2.0)
    assert torch.allclose(o[0, 3], torch.softmax(s, 0) @ v[:3, 1], atol=1e-6)
    k2 = k.clone()
    k2[4] += 100.0
    assert torch.equal(R.attention(q, k2, v, torch.tensor([2, 3, 4]), 0.3, 2.0)[:2], o[:2])


def test_oracle_clamped_glu():
    g, u = torch.tensor([5.0, -5.0, 1.0]), torch.tensor([9.0, -9.0, 0.5])
    y = R.clamped_glu(g, u, 2.0)
    f = lambda a, b: a / (1 + torch.exp(torch.tensor(-1.702 * a))) * (b + 1)
    assert torch.allclose(y, torch.stack([f(2.0, 2.0), f(-5.0, -2.0), f(1.0, 0.5)]))


def test_oracle_route_prefers_groups():
    # group 1 holds the single best expert, groups 0 and 2 the best pairs: with two groups kept expert 3 is out
    z = torch.tensor([1.0, 1.0, -9.0, 2.0, -9.0, -9.0, 0.9, 0.9, -9.0])
    ids, wts = R.route(z, 3, 3, 2, 2.0)
    assert ids == [0, 1, 6] and abs(sum(wts) - 2.0) < 1e-6 and wts[0] == wts[1] > wts[2]
    assert R.route(z, 1, 3, 3, 1.0)[0] == [3]


@pytest.mark.parametrize("name", list(MODELS))
def test_oracle_does_not_depend_on_the_cut(name):
    _, ref, _ = build(MODELS[name])
    ids = torch.tensor(tokens(21, MODELS[name]["vocab"], 3))
    whole, _ = ref.forward(ids)
    st, parts, at = ref.new_state(), [], 0
    for n in (2, 7, 1, 1, 10):
        lg, st = ref.forward(ids[at:at + n], st)
        parts.append(lg)
        at += n
    assert logit_error(torch.cat(parts), whole) < 1e-5


def test_needle_model_shows_the_far_key():
    _, ref, _ = needle(LOOPED)
    ids = tokens(40, LOOPED["vocab"] - 3, 1)
    ids = [3 + t for t in ids]
    ids[-1] = 1
    plain = ref.forward(torch.tensor(ids))[0][-1:]
    for p in (0, 15, 16, 38):
        with_needle = list(ids)
        with_needle[p] = 2
        assert logit_error(ref.forward(torch.tensor(with_needle))[0][-1:], plain) > 0.2


# ----------------------------------------------------------------------------- host backend and scheduler
def test_reference_backend_generates_greedily(tmp_path):
    _, ref, t = build(LOOPED)
    _write(tmp_path, LOOPED, t)
    prompts = [tokens(n, LOOPED["vocab"], n) for n in (1, 5, 18)]
    for policy in ("protect_decode", "mixed"):
        from dataclasses import replace
        from hipengine_b200.config import EngineConfig
        base = EngineConfig()
        eng = replace(base, scheduler=replace(base.scheduler, policy=policy, max_prefill_chunk_tokens=4))
        with LLM(str(tmp_path), backend="cpu_reference", engine_config=eng) as llm:
            got = llm.generate_token_ids(prompts, SamplingParams(max_tokens=6, ignore_eos=True))
        for p, g in zip(prompts, got):
            seq = list(p)
            for tok in g:
                assert int(ref.forward(torch.tensor(seq))[0][-1].argmax()) == tok
                seq.append(tok)


def test_float32_is_refused_where_it_is_not_built():
    from hipengine_b200.models import make_executor
    from hipengine_b200.loading.synth import build_random_model
    with pytest.raises(ValueError, match="float32"):
        make_executor(build_random_model(NAMED_CONFIGS["tiny-dense"]), dtype="float32")
    with pytest.raises(ValueError):
        LLM("tiny-sisisun", dtype="float8")
    assert LLM("tiny-sisisun", dtype="fp32").config.compute_dtype == "float32"


def test_trace_engine_is_sized_by_live_tokens():
    from hipengine_b200.generation.trace_replay import trace_engine_config
    c = trace_engine_config(130, "float32")
    assert c.kv.pool_pages == 192 // c.kv.page_tokens + 1 and c.max_sequence_length == 192
    assert c.scheduler.max_active_requests == 4 and c.kv.prefix_cache == "off" and c.compute_dtype == "float32"


def test_library_of_a_subset_of_the_sources(tmp_path, monkeypatch):
    """`ensure` links only the named sources on a fresh checkout and hands out the full library when that is current."""
    from hipengine_b200.core import build as B
    calls = []
    monkeypatch.delenv("HE_NATIVE_VARIANT", raising=False)
    monkeypatch.setattr(B, "nvcc_path", lambda: "/usr/bin/true")
    monkeypatch.setattr(B, "build", lambda name="", only=(), **kw: calls.append((name, tuple(only))) or B.lib_path(name))
    monkeypatch.setattr(B, "_up_to_date", lambda: False)
    assert B.ensure(["layers.cu"]).name == "libhe_b200_subset.so" and calls == [("subset", ("layers.cu",))]
    monkeypatch.delenv("HE_NATIVE_VARIANT", raising=False)
    monkeypatch.setattr(B, "_up_to_date", lambda: True)
    assert B.ensure(["layers.cu"]).name == "libhe_b200.so" and len(calls) == 1
