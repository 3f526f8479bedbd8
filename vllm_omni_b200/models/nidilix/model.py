"""Stage model of the Nidilix decoder (a plain causal-LM stage)."""
from __future__ import annotations

import torch

from ..base import StageModel
from .config import NidilixConfig, tiny_config_dict
from .decoder import NidilixDecoder

# libraries under csrc/ that serving this model loads on a GPU
NATIVE_LIBS = ("gemm_sm100", "gemm_f32", "lm_ops", "stream_ops", "moe", "latent_attn", "attn_window", "attn_window_sm100",
               "short_conv", "gated_scan", "gated_scan_sm100", "sampler", "rt_host", "io_host")


class NidilixForCausalLM(StageModel):
    def __init__(self, cfg: NidilixConfig, dtype=torch.bfloat16, device=None):
        super().__init__(cfg, dtype, device)
        self.decoder = NidilixDecoder(cfg, dtype, device)

    def load_weights(self, weights) -> set:
        return self.decoder.load_weights(weights)


def build_nidilix(model_stage, hf_config: dict, dtype, device, **kw) -> NidilixForCausalLM:
    d = hf_config if hf_config.get("layers") else tiny_config_dict(**(kw.get("config") or {}))
    model = NidilixForCausalLM(NidilixConfig.from_dict(d), dtype, device)
    model.decoder.load_weights(model.decoder.random_weights())      # replaced when a checkpoint is loaded
    return model
