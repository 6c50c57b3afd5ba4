"""Milutar on the host: configuration and checkpoint folders, the oracle's own consistency, the reference backend."""
import copy
import json
import math
from dataclasses import replace

import pytest
import torch

from hipengine_b200.llm import LLM, SamplingParams
from hipengine_b200.loading import safetensors_dir as S
from hipengine_b200.loading.milutar import config_from_json, config_to_json, tensor_shapes
from hipengine_b200.loading.model_loader import describe_model_source, load_model
from hipengine_b200.models.config import NAMED_CONFIGS, TINY_MILUTAR, RotarySpec, YarnSpec
from hipengine_b200.models.registry import PLUGINS, folder_plugin, load_object, plugin_for, supported_architectures
from hipengine_b200.ref import milutar as R

from milutar_models import (LOOPED, MODELS, ODD, TOL, build, full, last_logits, logit_error, model, needle, random_tensors,
                            tokens, windowed, with_windows, yarn)


def _write(path, cfg_json, t):
    (path / "config.json").write_text(json.dumps(cfg_json))
    S.write_tensors(path / "model.safetensors", t)


# ----------------------------------------------------------------------------- configuration, checkpoint folders
@pytest.mark.parametrize("name", list(MODELS))
def test_config_round_trip(name):
    cfg = config_from_json(MODELS[name])
    back = config_to_json(cfg)
    assert config_from_json(back) == cfg and back == MODELS[name]
    assert cfg.rms_eps == MODELS[name]["norm"]["eps"] and cfg.residual_mult == MODELS[name]["residual_mult"]


def test_layer_runs_own_their_cache_and_state():
    cfg = config_from_json(ODD)
    assert cfg.layer_runs() == ((0, -1), (1, 0), (2, 0), (1, 1), (2, 1), (3, -1))
    rows = [l.mixer.row_cols for l in cfg.layer_specs]
    assert rows == [64, 64, 64, 96] and [l.mixer.rank_cols for l in cfg.layer_specs] == [48, 32, 32, 64]
    assert cfg.kv_bytes_per_token() == 2 * (64 + 64 + 64 + 64 + 64 + 96) == cfg.kv_bytes_per_token(4) // 2
    assert cfg.recurrent_state_bytes() == 6 * 4 * 136 and cfg.has_recurrent_state and not cfg.is_hybrid
    assert not NAMED_CONFIGS["tiny-sisisun"].has_recurrent_state and NAMED_CONFIGS["tiny-hybrid"].has_recurrent_state


@pytest.mark.parametrize("bad", [
    {"loop": {"start": 1, "stop": 5, "times": 2}},
    {"layers": []},
    {"layers": [{"type": "recurrent", "mixer": {}, "mlp": None}]},
    {"layers": [{**ODD["layers"][0], "mlp": {"kind": "moe"}}]},
    {"layers": [{**ODD["layers"][0], "mixer": {**ODD["layers"][0]["mixer"], "rot_dim": 5}}]},
    {"layers": [{**ODD["layers"][0], "mixer": {**ODD["layers"][0]["mixer"], "rot_dim": 8}}]},
    {"layers": [{**ODD["layers"][0], "mixer": {**ODD["layers"][0]["mixer"], "kv_rank": 1100}}]},
])
def test_impossible_configurations_are_refused(bad):
    with pytest.raises(ValueError):
        config_from_json({**ODD, **bad})


def test_checkpoint_folder(tmp_path):
    w, _, t = build(ODD)
    _write(tmp_path, ODD, t)
    got = load_model(tmp_path)
    assert got.config == w.config and set(got.tensors) == set(t) == set(tensor_shapes(w.config))
    assert got["final.norm"].shape == () and "l2.ls2" not in t and "l2.mlp.up" not in t and "l1.mix.sink" in t
    for n, x in t.items():
        assert torch.equal(got[n].dequant().to(torch.bfloat16), x), n
    d = describe_model_source(tmp_path)
    assert d["arch"] == "milutar" and d["source"] == "safetensors" and "error" not in d
    assert d["family"]["ffn"] == {"dense": 3, "none": 1} and d["family"]["layers"] == {"full": 2, "sliding": 2}
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.loading.admission import admit
    report = admit(got, EngineConfig(), free_bytes=1 << 40)
    assert report["admitted"] and report["memory"]["recurrent_state_bytes"] > 0
    _write(tmp_path, ODD, {n: x for n, x in t.items() if n != "l0.shift"})
    with pytest.raises(KeyError, match="l0.shift"):
        load_model(tmp_path)
    _write(tmp_path, ODD, {**t, "l0.norm1": torch.ones(132, dtype=torch.bfloat16)})
    with pytest.raises(KeyError, match="norm1"):
        load_model(tmp_path)


def test_registry_entries():
    p = plugin_for("milutar")
    assert p is folder_plugin("Milutar") and "milutar" in supported_architectures()
    assert p.compute_dtypes == ("bfloat16", "float32") and not p.tensor_parallel
    assert p.describe(TINY_MILUTAR)["layers"] == {"full": 2, "sliding": 2}
    from hipengine_b200.core import build as B
    assert set(p.native_sources) <= {s.name for s in B.sources()}
    with pytest.raises(KeyError, match="Milutar"):
        folder_plugin("Other")
    for q in PLUGINS:                      # every name in the registry can be imported
        assert load_object(q.executor).__name__.endswith("Executor")
        if q.folder_reader:
            assert load_object(q.folder_reader + ".tensor_shapes") and load_object(q.reference)
    assert all(c in NAMED_CONFIGS for c in ("tiny-milutar", "milutar-8b"))


def test_readiness_describes_the_latent_cache():
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.server.readiness import kv_capability
    d = kv_capability(TINY_MILUTAR, EngineConfig().kv)
    assert "latent" in d["layout"] and "latent" in d["decode_kernel"] and "expanded" in d["prefill_kernel"]
    assert d["sliding_window"] and d["recurrent_state_snapshots"]
    plain = kv_capability(NAMED_CONFIGS["tiny-sisisun"], EngineConfig().kv)
    assert "[k|v]" in plain["layout"] and not plain["sliding_window"]


@pytest.mark.parametrize("dims,base,y", [(2, 100.0, None), (12, 3000.0, (6.0, 256.0, 16.0, 1.0)), (64, 1e6, (32.0, 8192.0, 32.0, 1.0)),
                                         (4, 500.0, (3.0, 64.0, 8.0, 2.0)), (16, 10000.0, (1.0, 4096.0, 32.0, 1.0)),
                                         (8, 50.0, (4.0, 2.0, 32.0, 30.0))])
def test_rotation_table(dims, base, y):
    freq, amp = RotarySpec(dims, base, YarnSpec(*y) if y else None).table()
    want, want_amp = R.rotation_freqs(dims, base, yarn(*y) if y else None)
    assert torch.allclose(torch.tensor(freq, dtype=torch.float64), want, rtol=1e-12) and abs(amp - want_amp) < 1e-12


# ----------------------------------------------------------------------------- the oracle, mechanism by mechanism
def test_oracle_token_shift():
    h, s = torch.tensor([[1.0, 2.0], [3.0, 5.0]]), torch.tensor([0.25, 1.0])
    out = R.token_shift(h, torch.tensor([9.0, -1.0]), s)
    assert torch.equal(out, torch.tensor([[1 + 8 * 0.25, -1.0], [3 - 2 * 0.25, 2.0]]))


def test_oracle_rotation_turns_neighbouring_pairs():
    x = torch.tensor([[1.0, 0.0, 0.0, 2.0]])
    f = torch.tensor([math.pi / 2, math.pi / 6], dtype=torch.float64)
    y = R.rotate_pairs(x, torch.tensor([1]), f, 1.5)
    assert torch.allclose(y, 1.5 * torch.tensor([[0.0, 1.0, -1.0, math.sqrt(3.0)]]), atol=1e-6)
    assert torch.equal(R.rotate_pairs(x, torch.tensor([0]), f, 1.0), x)


def test_oracle_yarn_keeps_fast_pairs_and_slows_slow_ones():
    plain, _ = R.rotation_freqs(64, 1e4)
    f, amp = R.rotation_freqs(64, 1e4, yarn(8.0, 4096.0, 32.0, 1.0))
    turns = plain * 4096.0 / (2 * math.pi)
    assert torch.equal(f[turns > 60], plain[turns > 60]) and torch.allclose(f[turns < 0.5], plain[turns < 0.5] / 8.0)
    mid = (turns < 25) & (turns > 1.5)
    assert bool(((f < plain) & (f > plain / 8.0))[mid].all()) and abs(amp - (0.1 * math.log(8.0) + 1.0)) < 1e-12


def test_oracle_window_and_sink():
    seen = R.visible_keys(torch.tensor([4]), 6, 3)[0]
    assert seen.tolist() == [False, False, True, True, True, False]
    assert R.visible_keys(torch.tensor([4]), 6)[0].tolist() == [True] * 5 + [False]
    s = torch.tensor([[0.3, -0.2, 5.0]])
    p = R.softmax_with_sink(s, torch.tensor([[True, True, False]]), torch.tensor(0.7))
    e = [math.exp(0.3), math.exp(-0.2), math.exp(0.7)]
    assert torch.allclose(p, torch.tensor([[e[0] / sum(e), e[1] / sum(e), 0.0]]))


def test_oracle_latent_attention_is_attention_over_expanded_rows():
    g = torch.Generator().manual_seed(0)
    T, S, H, d, rd, dv, r = 2, 5, 3, 4, 2, 3, 6
    q, lat, rot = torch.randn(T, H, d + rd, generator=g), torch.randn(S, r, generator=g), torch.randn(S, rd, generator=g)
    wk, wv = torch.randn(H * d, r, generator=g), torch.randn(H * dv, r, generator=g)
    o = R.latent_attention(q, lat, rot, wk, wv, torch.tensor([3, 4]), H, 0.3)
    k = [torch.cat([wk[d:2 * d] @ lat[j], rot[j]]) for j in range(4)]
    p = torch.softmax(torch.stack([q[0, 1] @ x * 0.3 for x in k]), 0)
    want = sum(p[j] * (wv[dv:2 * dv] @ lat[j]) for j in range(4))
    assert torch.allclose(o[0, dv:2 * dv], want, atol=1e-5)


def test_oracle_schedule():
    c = lambda n, loop: R.MilutarRef({"layers": [None] * n, "loop": loop, "norm": {"eps": 1}, "residual_mult": 1}, {}).schedule()
    assert c(2, None) == [(0, None), (1, None)]
    assert c(4, {"start": 1, "stop": 3, "times": 2}) == [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (3, None)]
    assert c(2, {"start": 0, "stop": 2, "times": 1}) == [(0, 0), (1, 0)]
    assert c(2, {"start": 1, "stop": 2, "times": 3}) == [(0, None), (1, 0), (1, 1), (1, 2)]


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
    """(what is wrong, configuration change, tensor change) of mistakes the whole-model tests must be able to see."""
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
    swap = lambda x: x.reshape(-1, 2).flip(1).reshape(x.shape)
    return {
        "no sink": ten(lambda n, x: torch.full_like(x, -1e30) if n.endswith(".sink") else x),
        "no token shift": zero(".shift"),
        "no layer scale (mixer)": ones(".ls1"),
        "no layer scale (feed-forward)": ones(".ls2"),
        "no residual factor": cfg(lambda l, c: c.update(residual_mult=1.0)),
        "no gain": ones(".norm1"),
        "no latent gain": ones(".dkv.norm"),
        "no query latent gain": ones(".dq.norm"),
        "no loop step": zero("loop.step"),
        "no scaling of the rotation": cfg(lambda l, c: l["mixer"]["rot"].pop("scaling", None)),
        "other base": cfg(lambda l, c: l["mixer"]["rot"].update(base=l["mixer"]["rot"]["base"] * 3)),
        "scores not scaled": cfg(lambda l, c: l["mixer"].update(scale=1.0)),
        "window longer": lambda c, t: (with_windows(c, 1), t),
        "window shorter": lambda c, t: (with_windows(c, -1), t),
        "heads swapped": ten(lambda n, x: swap(x) if n.endswith("mix.o") else x),
    }


@pytest.mark.parametrize("what", list(_mutants()))
def test_mistakes_show_in_the_test_models(what):
    """A mechanism left out of the oracle moves the logits by several times the bfloat16 tolerance of the GPU tests."""
    t = random_tensors(ODD, 0)
    ids = torch.tensor(tokens(60, ODD["vocab"], 5))
    want = R.MilutarRef(ODD, t).forward(ids)[0]
    c2, t2 = _mutants()[what](ODD, t)
    assert logit_error(R.MilutarRef(c2, t2).forward(ids)[0], want) > 4 * TOL["bfloat16"]


def test_lost_state_shows_after_a_cut():
    _, ref, _ = build(ODD)
    ids = torch.tensor(tokens(40, ODD["vocab"], 5))
    want = ref.forward(ids)[0][25:]
    for lost in ("last", "lat"):
        _, st = ref.forward(ids[:25], ref.new_state())
        for run, x in getattr(st, lost).items():
            getattr(st, lost)[run] = torch.zeros_like(x)
        assert logit_error(ref.forward(ids[25:], st)[0], want) > 4 * TOL["bfloat16"]


def test_needle_model_shows_the_key_and_the_window_edge():
    _, ref, t = needle(LOOPED)
    base = [3 + x for x in tokens(40, LOOPED["vocab"] - 3, 1)]
    base[-1] = 1
    plain = last_logits(ref, base)
    for p in (0, 15, 16, 38):
        ids = list(base)
        ids[p] = 2
        assert logit_error(last_logits(ref, ids), plain) > 0.2
    c = model(96, 160, [(windowed(4, 24, 8, 40, 32, 0.2, 12), 64)])
    _, ref, t = needle(c)
    err = {}
    for d in (10, 11, 12, 13):                             # distance from the asking token
        ids = list(base)
        ids[39 - d] = 2
        err[d] = logit_error(last_logits(ref, ids), last_logits(ref, base))
    assert min(err[10], err[11]) > 0.2 and max(err[12], err[13]) < 1e-5


# ----------------------------------------------------------------------------- host backend and scheduler
def test_reference_backend_generates_greedily(tmp_path):
    from hipengine_b200.config import EngineConfig
    _, ref, t = build(LOOPED)
    _write(tmp_path, LOOPED, t)
    prompts = [tokens(n, LOOPED["vocab"], n) for n in (1, 5, 18)]
    base = EngineConfig()
    for policy in ("protect_decode", "mixed"):
        eng = replace(base, scheduler=replace(base.scheduler, policy=policy, max_prefill_chunk_tokens=4))
        with LLM(str(tmp_path), backend="cpu_reference", engine_config=eng) as llm:
            got = llm.generate_token_ids(prompts, SamplingParams(max_tokens=6, ignore_eos=True))
        for p, g in zip(prompts, got):
            seq = list(p)
            for tok in g:
                assert int(last_logits(ref, seq)[0].argmax()) == tok
                seq.append(tok)


def test_failing_prompt_beside_decoding_leaves_the_others_alone():
    """Policy 'mixed' on a runner that cannot pack: the decode step is committed before the prompt's chunk fails."""
    from hipengine_b200.config import EngineConfig
    from hipengine_b200.generation.engine_loop import EngineLoop
    from hipengine_b200.generation.runner import CpuReferenceRunner, ExecutionFailure
    from hipengine_b200.generation.types import GenerationRequest
    w, ref, _ = build(LOOPED)
    base = EngineConfig()
    conf = replace(base, scheduler=replace(base.scheduler, policy="mixed", max_prefill_chunk_tokens=8,
                                           max_active_requests=2))
    loop = EngineLoop(CpuReferenceRunner(w, conf), conf)
    real, bad = loop.runner.prefill, []

    def prefill(work):
        fail = [rs.rid for rs, _ in work if rs.rid in bad]
        if fail:
            raise ExecutionFailure(fail, "prefill", "planted", "none")
        return real(work)
    loop.runner.prefill = prefill
    prompt = tokens(5, LOOPED["vocab"], 1)
    a = loop.submit(GenerationRequest(prompt_token_ids=prompt, max_tokens=8, ignore_eos=True))
    loop.tick()
    loop.tick()
    b = loop.submit(GenerationRequest(prompt_token_ids=tokens(6, LOOPED["vocab"], 2), max_tokens=4, ignore_eos=True))
    bad.append(b.rid)
    for _ in range(20):
        loop.tick()
    want, seq = [], list(prompt)
    for _ in range(8):
        want.append(int(last_logits(ref, seq)[0].argmax()))
        seq.append(want[-1])
    assert a.generated == want and b.error
