"""AR / generation model registry: ``model_arch`` (+ ``model_stage``) -> stage model class
(vllm_omni/model_executor/models/registry.py)."""
from __future__ import annotations

import importlib

_MODELS: dict[str, tuple[str, str]] = {
    "Qwen3OmniMoeForConditionalGeneration": ("vllm_omni_b200.models.qwen3_omni.model", "build_qwen3_omni_stage"),
    "Qwen2_5OmniForConditionalGeneration": ("vllm_omni_b200.models.qwen2_5_omni.model", "build_qwen2_5_omni_stage"),
    "Qwen3TTSForConditionalGeneration": ("vllm_omni_b200.models.qwen3_tts.model", "build_qwen3_tts_stage"),
    "Qwen3ForCausalLM": ("vllm_omni_b200.models.text", "build_text_model"),
    "Qwen2ForCausalLM": ("vllm_omni_b200.models.text", "build_text_model"),
    "Qwen3MoeForCausalLM": ("vllm_omni_b200.models.text", "build_text_model"),
    "Tavulix": ("vllm_omni_b200.models.tavulix.model", "build_tavulix"),
    "Nidilix": ("vllm_omni_b200.models.nidilix.model", "build_nidilix"),
    "Milivik": ("vllm_omni_b200.models.milivik.model", "build_milivik"),
    "Fikizen": ("vllm_omni_b200.models.fikizen.model", "build_fikizen"),
    "BagelForConditionalGeneration": ("vllm_omni_b200.models.text", "build_text_model"),
}


def register_model(arch: str, module: str, factory: str) -> None:
    _MODELS[arch] = (module, factory)


def native_libs(arch: str) -> tuple[str, ...] | None:
    """Libraries under csrc/ that serving ``arch`` loads (the model module's ``NATIVE_LIBS``), None = not declared."""
    return getattr(importlib.import_module(_MODELS[arch][0]), "NATIVE_LIBS", None)


def arch_from_config(cfg: dict) -> str | None:
    """Architecture name of a ``config.json``: first of ``architectures``, or ``architecture``."""
    archs = cfg.get("architectures") or [cfg.get("architecture")]
    return archs[0] if isinstance(archs, list) else archs


def supported_archs() -> list[str]:
    return sorted(_MODELS)


def build_stage_model(model_arch: str, model_stage: str | None, hf_config: dict, dtype, device, **kw):
    if model_arch not in _MODELS:
        raise ValueError(f"unknown model_arch {model_arch!r}; supported: {supported_archs()}")
    mod, fn = _MODELS[model_arch]
    return getattr(importlib.import_module(mod), fn)(model_stage, hf_config, dtype, device, **kw)
