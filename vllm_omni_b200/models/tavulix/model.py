"""Stage model of the Tavulix decoder (a plain causal-LM stage)."""
from __future__ import annotations

import torch

from ..base import StageModel
from .config import TavulixConfig, tiny_config_dict
from .decoder import TavulixDecoder

# libraries under csrc/ that serving this model loads on a GPU
NATIVE_LIBS = ("gemm_sm100", "gemm_f32", "lm_ops", "attn_window", "attn_window_sm100", "sampler", "rt_host", "io_host")


class TavulixForCausalLM(StageModel):
    def __init__(self, cfg: TavulixConfig, dtype=torch.bfloat16, device=None):
        super().__init__(cfg, dtype, device)
        self.decoder = TavulixDecoder(cfg, dtype, device)

    def load_weights(self, weights) -> set:
        return self.decoder.load_weights(weights)


def build_tavulix(model_stage, hf_config: dict, dtype, device, **kw) -> TavulixForCausalLM:
    d = hf_config if hf_config.get("layers") else tiny_config_dict(**(kw.get("config") or {}))
    model = TavulixForCausalLM(TavulixConfig.from_dict(d), dtype, device)
    model.decoder.load_weights(model.decoder.random_weights())      # replaced when a checkpoint is loaded
    return model
