"""Model table: every family the framework knows, what serves it, and its state.  Reference: the
``sparkflash models`` subcommand (crates/sparkflash-cli/src/models.rs) and crates/sparkflash-model
architecture descriptors."""
from __future__ import annotations

import importlib
import json
import os
from dataclasses import dataclass


@dataclass(frozen=True)
class ModelEntry:
    name: str
    family: str
    status: str          # "device" = serves on the GPU engine, "oracle" = CPU reference + kernels, "planned"
    summary: str
    module: str


MODELS = {m.name: m for m in [
    ModelEntry("deepseek-v4.1-flash", "deepseek", "device", "CSA2 attention, mHC, 384-expert W4A8 MoE, DSpark drafter, Engram", "sparkflash_b200.models.deepseek_v41"),
    ModelEntry("tiny-csa2", "deepseek", "device", "6-layer test model with every layer mode of the flagship", "sparkflash_b200.models.deepseek_v41"),
    ModelEntry("tiny-mla-v3", "deepseek", "oracle", "classic MLA attention with absorbed decode, CPU oracle timing config", "sparkflash_b200.models.mla_v3"),
    ModelEntry("glm-5.3-flash", "glm", "oracle", "MLA with indexer-selected keys, noaux sigmoid router, shared expert; cached decode", "sparkflash_b200.models.glm"),
    ModelEntry("qwen3.8-flash-next", "qwen", "oracle", "gated delta-net / KDA linear attention + gated softmax attention + MoE; device rows step on the state kernels", "sparkflash_b200.models.qwen"),
    ModelEntry("inkling-2-small", "inkling", "oracle", "short conv, soft-capped windowed attention and SwiGLU, MoE with expert / intermediate / row splits; device rows step", "sparkflash_b200.models.inkling"),
    ModelEntry("dory-1.0-4b", "dory", "oracle", "latent-recurrence model, loops split over a ring pipeline of ranks", "sparkflash_b200.models.dory"),
    ModelEntry("fanodra", "fanodra", "device", "gated linear recurrence, alone or beside attention with a distance bias; looped layers, input convolution; layered engine (bf16 or 32-bit)", "sparkflash_b200.models.fanodra"),
    ModelEntry("gudutar", "gudutar", "device", "state-space duality, retention and latent attention in a window; norms on sublayer outputs, layers that share weights; layered engine (bf16 or 32-bit)", "sparkflash_b200.models.gudutar"),
    ModelEntry("lifulorn", "lifulorn", "device", "gated delta rule and windowed attention with sinks, capped scores and mixed values; mixture of experts, per-layer token input; layered engine (bf16 or 32-bit)", "sparkflash_b200.models.lifulorn"),
    ModelEntry("dironex", "dironex", "device", "latent attention with a latent for the queries and an output gate, windowed attention with normed heads; several residual streams, looped layers, grouped experts; layered engine (bf16 or 32-bit)", "sparkflash_b200.models.dironex"),
    ModelEntry("dflash-block-drafter", "drafter", "oracle", "one-forward block drafter over a ring of captured target features", "sparkflash_b200.models.dflash"),
]}

# config.json "architecture" -> (module, class) of the models that run on the layered engine (models/layered.py)
LAYERED = {"Fanodra": ("sparkflash_b200.models.fanodra", "Fanodra"), "Gudutar": ("sparkflash_b200.models.gudutar", "Gudutar"),
           "Lifulorn": ("sparkflash_b200.models.lifulorn", "Lifulorn"), "Dironex": ("sparkflash_b200.models.dironex", "Dironex")}


def architecture(path: str) -> str:
    """What a model folder's config.json says it is."""
    with open(os.path.join(path, "config.json")) as f:
        d = json.load(f)
    return d.get("architecture") or d.get("model_type") or (d.get("architectures") or ["unknown"])[0]


def layered_class(arch: str):
    if arch not in LAYERED:
        raise ValueError(f"architecture {arch!r} does not run on the layered engine; known: {sorted(LAYERED)}")
    module, cls = LAYERED[arch]
    return getattr(importlib.import_module(module), cls)


def layered_engine(path: str, dtype: str = "bfloat16", device: str = "cuda", max_context: int = 4096, **engine):
    """The layered engine over the model folder ``path`` (config.json + safetensors)."""
    import torch

    from .layered import LayeredEngine
    model = layered_class(architecture(path)).from_dir(path, {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype], device, max_context)
    return LayeredEngine(model, max_context=max_context, **engine)
