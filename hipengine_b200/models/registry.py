"""Model family declarations: what each supported ``general.architecture`` is, which executor runs it, what its layer
schedule looks like, which speculative providers and KV storage modes it admits.

Pure metadata (the role of the reference's model plugins, ``hipengine/models/registry.py``, ``models/qwen35.py``,
``models/gemma4.py``: name, architectures, default quantisation, layer sequence, MTP serving and KV capability
declarations).  Used by the server's capability route and by error messages that must say what IS supported.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .config import LinearAttentionSpec, ModelConfig, MoeMlpSpec, SideBySideSpec


@dataclass(frozen=True)
class ModelPlugin:
    name: str
    architectures: Tuple[str, ...]
    executor: str                               # import path of the GPU executor class
    default_quant: str = "gguf_q4_k_m"
    native_block_types: Tuple[str, ...] = ("Q4_K", "Q6_K", "Q8_0", "F32", "F16", "BF16")
    widened_block_types: Tuple[str, ...] = ("Q4_0", "Q4_1", "Q5_0", "Q5_1", "Q5_K")
    chat_template: str = "chatml"
    speculative_providers: Tuple[str, ...] = ("prompt_lookup", "ngram")
    kv_storage: Tuple[str, ...] = ("bf16",)
    tensor_parallel: bool = True
    expert_parallel: bool = False
    compute_dtypes: Tuple[str, ...] = ("bfloat16",)
    native_sources: Tuple[str, ...] = ()        # csrc files a build for this family alone needs (empty: all of them)
    folder_architecture: str = ""               # ``architecture`` of its checkpoint folders (config.json), if it has any
    folder_reader: str = ""                     # module with their configuration reader and tensor list
    reference: str = ""                         # plain reference of a folder family: class over (config.json, tensors)
    notes: str = ""

    def layer_sequence(self, cfg: ModelConfig) -> List[str]:
        """One word per layer of ``cfg``: ``linear`` (Gated-DeltaNet), ``retention``, ``full``, ``sliding`` or ``global``; with
        ``+recurrent`` where a recurrence runs beside the attention."""
        out = []
        for i in range(cfg.n_layers):
            if cfg.layer_specs:
                m = cfg.layer_specs[i].mixer
                word = "sliding" if getattr(m, "window", 0) else "full"
                if isinstance(m, LinearAttentionSpec):
                    word = "linear" if m.delta else "retention"
                out.append(word + "+recurrent" if isinstance(m, SideBySideSpec) else word)
            elif cfg.arch == "gemma4":
                out.append("global" if cfg.is_global_layer(i) else "sliding")
            elif cfg.is_hybrid:
                out.append("full" if cfg.is_full_attention_layer(i) else "linear")
            else:
                out.append("full")
        return out

    def describe(self, cfg: Optional[ModelConfig] = None) -> Dict[str, Any]:
        d: Dict[str, Any] = {"name": self.name, "architectures": list(self.architectures), "executor": self.executor,
                             "default_quant": self.default_quant, "native_block_types": list(self.native_block_types),
                             "widened_block_types": list(self.widened_block_types), "chat_template": self.chat_template,
                             "speculative_providers": list(self.speculative_providers),
                             "kv_storage": list(self.kv_storage), "tensor_parallel": self.tensor_parallel,
                             "expert_parallel": self.expert_parallel, "compute_dtypes": list(self.compute_dtypes),
                             "notes": self.notes}
        if cfg is not None:
            seq = self.layer_sequence(cfg)
            d["layers"] = {k: seq.count(k) for k in sorted(set(seq))}
            d["ffn"] = "moe" if cfg.is_moe else "dense"
            if cfg.layer_specs:
                kinds = ["none" if l.mlp is None else "moe" if isinstance(l.mlp, MoeMlpSpec) else "dense"
                         for l in cfg.layer_specs]
                d["ffn"] = {k: kinds.count(k) for k in sorted(set(kinds))}
                d["layer_runs"] = len(cfg.layer_runs())
            providers = list(self.speculative_providers)
            if "mtp" in providers and cfg.arch != "gemma4" and cfg.nextn_layers == 0:
                providers.remove("mtp")                         # this checkpoint carries no NextN block
            d["speculative_providers"] = providers
        return d


_HYBRID = "hipengine_b200.models.executor.HybridExecutor"
PLUGINS: Tuple[ModelPlugin, ...] = (
    ModelPlugin("qwen35-dense-hybrid", ("qwen35",), _HYBRID,
                speculative_providers=("mtp", "prompt_lookup", "ngram"),
                notes="3 Gated-DeltaNet layers : 1 gated full-attention layer; optional trailing NextN block"),
    ModelPlugin("qwen35-moe-hybrid", ("qwen35moe",), _HYBRID, expert_parallel=True,
                speculative_providers=("mtp", "prompt_lookup", "ngram"),
                notes="hybrid schedule with top-k routed experts and a gated shared expert"),
    ModelPlugin("dense-decoder", ("qwen3", "llama"), _HYBRID, notes="full attention in every layer"),
    ModelPlugin("moe-decoder", ("qwen3moe",), _HYBRID, expert_parallel=True),
    ModelPlugin("gemma4-moe", ("gemma4",), "hipengine_b200.models.gemma4.Gemma4Executor", default_quant="gguf_q4_k_xl",
                chat_template="gemma", speculative_providers=("gemma4_mtp", "prompt_lookup", "ngram"),
                tensor_parallel=False,
                notes="5 sliding-window layers : 1 global layer, dense GeGLU branch beside top-k experts; the MTP "
                      "drafter is the separate gemma4-assistant artifact"),
    ModelPlugin("sisisun", ("sisisun",), "hipengine_b200.models.sisisun.SisisunExecutor", default_quant="bf16",
                native_block_types=("BF16",), widened_block_types=(), kv_storage=("bf16", "f32"),
                tensor_parallel=False, compute_dtypes=("bfloat16", "float32"),
                native_sources=("attn_decode.cu", "attn_prefill.cu", "exact_f32.cu", "gemm_sm100.cu", "gemv_float.cu",
                                "layers.cu", "moe.cu", "quant_util.cu", "runtime.cpp", "sampling.cu"),
                folder_architecture="Sisisun", folder_reader="hipengine_b200.loading.sisisun",
                reference="hipengine_b200.ref.sisisun.SisisunRef",
                notes="layers listed one by one: attention without rotation, soft-capped scores, dense (clamped GLU) or "
                      "group-limited sigmoid-routed experts; a range of layers may run several times; checkpoints are "
                      "folders with config.json and model.safetensors"),
    ModelPlugin("milutar", ("milutar",), "hipengine_b200.models.milutar.MilutarExecutor", default_quant="bf16",
                native_block_types=("BF16",), widened_block_types=(), kv_storage=("bf16", "f32"),
                tensor_parallel=False, compute_dtypes=("bfloat16", "float32"),
                native_sources=("gemm_sm100.cu", "gemv_float.cu", "latent_attn.cu", "latent_prefill.cu", "latent_prefill_tc.cu",
                                "layers.cu", "quant_util.cu", "runtime.cpp", "sampling.cu"),
                folder_architecture="Milutar", folder_reader="hipengine_b200.loading.milutar",
                reference="hipengine_b200.ref.milutar.MilutarRef",
                notes="layers listed one by one: latent attention (windowed, or causal with a softmax sink and a query "
                      "latent) beside a squared-ReLU feed-forward on one norm, token shift, layer scale; a range of layers "
                      "may run several times; checkpoints are folders with config.json and model.safetensors"),
    ModelPlugin("banelix", ("banelix",), "hipengine_b200.models.banelix.BanelixExecutor", default_quant="bf16",
                native_block_types=("BF16",), widened_block_types=(), kv_storage=("bf16", "f32"),
                tensor_parallel=False, compute_dtypes=("bfloat16", "float32"),
                native_sources=("attn_decode.cu", "attn_prefill.cu", "exact_f32.cu", "gemm_sm100.cu", "gemv_float.cu",
                                "layers.cu", "mixer_post.cu", "quant_util.cu", "rglru.cu", "runtime.cpp", "sampling.cu"),
                folder_architecture="Banelix", folder_reader="hipengine_b200.loading.banelix",
                reference="hipengine_b200.ref.banelix.BanelixRef",
                notes="layers listed one by one: windowed attention with one more unit in the softmax denominator (a layer may "
                      "attend to an earlier layer's keys and values), or attention over unit keys whose values are the plain "
                      "keys beside a real-gated linear recurrence; dense SiLU feed-forward or none; checkpoints are folders "
                      "with config.json and model.safetensors"),
    ModelPlugin("mepatar", ("mepatar",), "hipengine_b200.models.mepatar.MepatarExecutor", default_quant="bf16",
                native_block_types=("BF16",), widened_block_types=(), kv_storage=("bf16", "f32"),
                tensor_parallel=False, compute_dtypes=("bfloat16", "float32"),
                native_sources=("attn_decode.cu", "attn_prefill.cu", "exact_f32.cu", "gemm_sm100.cu", "gemv_float.cu",
                                "layers.cu", "linear_attn.cu", "linear_chunk.cu", "mixer_post.cu", "moe.cu", "norm_conv.cu",
                                "quant_util.cu", "runtime.cpp", "sampling.cu"),
                folder_architecture="Mepatar", folder_reader="hipengine_b200.loading.mepatar",
                reference="hipengine_b200.ref.mepatar.MepatarRef",
                notes="layers listed one by one, mixer and feed-forward side by side under grouped norms, a convolution ahead of "
                      "the mixer; mixers: attention over a window and the sequence's first tokens, retention, gated delta rule; "
                      "feed-forwards: dense, softmax-routed clamped experts or none; checkpoints are folders with config.json "
                      "and model.safetensors"),
)


def plugin_for(arch: str) -> ModelPlugin:
    for p in PLUGINS:
        if arch in p.architectures:
            return p
    known = sorted(a for p in PLUGINS for a in p.architectures)
    raise KeyError(f"no model plugin for architecture {arch!r}; supported: {known}")


def folder_plugin(architecture: str) -> ModelPlugin:
    """Family of a checkpoint folder by its ``architecture``."""
    for p in PLUGINS:
        if p.folder_architecture and p.folder_architecture == architecture:
            return p
    known = [p.folder_architecture for p in PLUGINS if p.folder_architecture]
    raise KeyError(f"unsupported architecture {architecture!r}; supported: {known}")


def load_object(path: str):
    """The class a plugin names by its import path."""
    from importlib import import_module
    mod, name = path.rsplit(".", 1)
    return getattr(import_module(mod), name)


def supported_architectures() -> List[str]:
    return sorted(a for p in PLUGINS for a in p.architectures)
