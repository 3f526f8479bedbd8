"""Stage model of the Fikizen decoder (a plain causal-LM stage)."""
from __future__ import annotations

import torch

from ..base import StageModel
from .config import FikizenConfig, tiny_config_dict
from .decoder import FikizenDecoder

# libraries under csrc/ that serving this model loads on a GPU
NATIVE_LIBS = ("gemm_sm100", "gemm_f32", "lm_ops", "stream_ops", "attn_window", "attn_window_sm100", "short_conv", "delta_rule",
               "delta_chunks", "sampler", "rt_host", "io_host")


class FikizenForCausalLM(StageModel):
    def __init__(self, cfg: FikizenConfig, dtype=torch.bfloat16, device=None):
        super().__init__(cfg, dtype, device)
        self.decoder = FikizenDecoder(cfg, dtype, device)

    def load_weights(self, weights) -> set:
        return self.decoder.load_weights(weights)


def build_fikizen(model_stage, hf_config: dict, dtype, device, **kw) -> FikizenForCausalLM:
    d = hf_config if hf_config.get("layers") else tiny_config_dict(**(kw.get("config") or {}))
    model = FikizenForCausalLM(FikizenConfig.from_dict(d), dtype, device)
    model.decoder.load_weights(model.decoder.random_weights())      # replaced when a checkpoint is loaded
    return model
