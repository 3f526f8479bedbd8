"""Weight packing shared by decoders whose checkpoint tensors are copied into padded, fused layouts: a decoder says
where every checkpoint tensor goes (``targets``) and which shape it must have (``cfg.tensor_shapes()``)."""
from __future__ import annotations

import torch
from torch import nn

from ..diffusion.layers.linear import FusedLinear


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def zeros_param(*shape, dtype, device) -> nn.Parameter:
    return nn.Parameter(torch.zeros(*shape, dtype=dtype, device=device), requires_grad=False)


def packed_linear(n_in: int, n_out: int, dtype, device, bias: bool = False) -> FusedLinear:
    """Zero weights at sizes padded for the GEMM; checkpoint rows and columns are copied into place."""
    m = FusedLinear(round_up(n_in, 8), round_up(n_out, 8), bias=bias, dtype=dtype, device="meta")
    m.weight = zeros_param(round_up(n_out, 8), round_up(n_in, 8), dtype=dtype, device=device)
    if bias:
        m.bias = zeros_param(round_up(n_out, 8), dtype=dtype, device=device)
    return m


class PackedDecoder(nn.Module):
    uses_seq_table = True            # the runner hands a SeqTable with every batch

    def targets(self) -> dict:
        """Checkpoint name -> list of (destination view, selection of the checkpoint tensor that goes there)."""
        raise NotImplementedError

    def resize(self, name: str, shape: tuple[int, ...]) -> None:
        """Makes room for a checkpoint tensor whose size only the checkpoint tells (None in ``cfg.tensor_shapes()``)."""
        raise NotImplementedError

    def weights_loaded(self) -> None:
        """Called when every tensor is in place: values derived from the weights are computed here."""

    @torch.no_grad()
    def load_weights(self, weights) -> set:
        """Copies (name, tensor) pairs into the packed layout; a missing or misshapen tensor is an error."""
        targets, shapes, loaded = self.targets(), self.cfg.tensor_shapes(), set()
        for name, w in weights:
            if name not in targets:
                continue
            if None in shapes[name]:
                if len(w.shape) != len(shapes[name]) or any(b not in (None, a) for a, b in zip(w.shape, shapes[name])):
                    raise ValueError(f"{name}: shape {tuple(w.shape)}, expected {shapes[name]}")
                self.resize(name, tuple(w.shape))
                targets = self.targets()
            elif tuple(w.shape) != shapes[name]:
                raise ValueError(f"{name}: shape {tuple(w.shape)}, expected {shapes[name]}")
            w = w.reshape(1) if w.dim() == 0 else w
            if any(sel != slice(None) for _, sel in targets[name]):
                w = w.to(targets[name][0][0].device)        # one transfer, then copies per part
            for dst, sel in targets[name]:
                dst.copy_(w[sel].to(dst.dtype))
            loaded.add(name)
        missing = sorted(set(targets) - loaded)
        if missing:
            raise ValueError(f"checkpoint lacks {len(missing)} tensors: {', '.join(missing[:8])}")
        self.weights_loaded()
        return loaded
