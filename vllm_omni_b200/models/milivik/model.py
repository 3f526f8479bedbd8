"""Stage model of the Milivik decoder (a plain causal-LM stage)."""
from __future__ import annotations

import torch

from ..base import StageModel
from .config import MilivikConfig, tiny_config_dict
from .decoder import MilivikDecoder

# libraries under csrc/ that serving this model loads on a GPU
NATIVE_LIBS = ("gemm_sm100", "gemm_f32", "lm_ops", "stream_ops", "elementwise", "moe", "latent_attn", "attn_window",
               "attn_window_sm100", "sampler", "rt_host", "io_host")


class MilivikForCausalLM(StageModel):
    def __init__(self, cfg: MilivikConfig, dtype=torch.bfloat16, device=None):
        super().__init__(cfg, dtype, device)
        self.decoder = MilivikDecoder(cfg, dtype, device)

    def load_weights(self, weights) -> set:
        return self.decoder.load_weights(weights)


def build_milivik(model_stage, hf_config: dict, dtype, device, **kw) -> MilivikForCausalLM:
    d = hf_config if hf_config.get("layers") else tiny_config_dict(**(kw.get("config") or {}))
    model = MilivikForCausalLM(MilivikConfig.from_dict(d), dtype, device)
    model.decoder.load_weights(model.decoder.random_weights())      # replaced when a checkpoint is loaded
    return model
