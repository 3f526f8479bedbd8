"""Tavulix decoder: attention layers with a short causal convolution on q, k and v, head norms, bounded
scores, a logarithmic distance bias, a sliding window that keeps the first tokens, a softmax sink, values
mixed with those of the first mixing layer, and a per-head output gate; PolyNorm feed-forward; RMS norms
with one gain before and after every sublayer; learned positions; bounded logits.

One step over a mixed batch (portions of prompts and decoded tokens), per layer:

    qkvg GEMM -> conv + head norms + value mixing + pages (one kernel) -> windowed paged attention with
    the gate in its epilogue -> output GEMM -> residual add of the normed branch + next norm (one kernel)
    -> up GEMM -> PolyNorm -> down GEMM -> residual add + next norm

The residual stream is fp32; activations are bf16 (serving) or fp32 (exact mode, every product in true
fp32).  A sequence's convolution history lives in the runner's state pool (third tensor of a layer's cache
entry).  Heads are padded to 16 channels, rows to 8, both with zeros."""
from __future__ import annotations

import torch
import torch.nn.functional as F
from torch import nn

from ...ops import lm
from ...ops.window_attention import ScoreRule, bounded_scores, window_attention
from ..packed_decoder import PackedDecoder, packed_linear as _linear, zeros_param as _zeros
from ..qwen_decoder import ModelBatch
from .config import LayerConfig, TavulixConfig


class TavulixLayer(nn.Module):
    def __init__(self, cfg: TavulixConfig, lc: LayerConfig, dtype, device):
        super().__init__()
        f32 = lambda *s: _zeros(*s, dtype=torch.float32, device=device)
        D, m = cfg.hidden_size, lc.mixer
        self.lc, self.hs = lc, lc.mixer.head_shape
        self.bounded = False         # whether the score bound may serve as softmax reference; set with the weights
        hs = self.hs
        self.norm1, self.norm1b = f32(1), f32(1)
        self.qkvg = _linear(D, hs.channels + m.heads, dtype, device)
        self.conv = f32(m.conv, hs.channels) if m.conv else None
        self.q_norm, self.k_norm = f32(hs.dp), f32(hs.dp)
        self.vmix = f32(1)
        self.r1, self.r2, self.sink = f32(m.heads), f32(m.heads), f32(m.heads)
        self.o = _linear(m.heads * hs.vp, D, dtype, device)
        if lc.ff is not None:
            self.norm2, self.norm2b = f32(1), f32(1)
            self.up, self.down = _linear(D, lc.ff, dtype, device), _linear(lc.ff, D, dtype, device)
            self.act = f32(4)

    def rule(self) -> ScoreRule:
        m = self.lc.mixer
        return ScoreRule(m.scale, m.softcap, self.r1, self.r2, self.sink, m.window, m.keep_first, self.bounded)


class TavulixDecoder(PackedDecoder):
    def __init__(self, cfg: TavulixConfig, dtype=torch.bfloat16, device=None):
        super().__init__()
        self.cfg, self.dtype_ = cfg, dtype
        Dp = cfg.padded_width
        self.embed_tokens = _zeros(cfg.vocab_size, Dp, dtype=dtype, device=device)
        self.pos_table = _zeros(cfg.max_position_embeddings, Dp, dtype=dtype, device=device)
        self.layers = nn.ModuleList([TavulixLayer(cfg, l, dtype, device) for l in cfg.layers])
        mixing = [i for i, l in enumerate(cfg.layers) if l.mixer.v_mix]
        self.first_mix = mixing[0] if mixing else None
        self.final_norm = _zeros(1, dtype=torch.float32, device=device)
        self.lm_head = _linear(cfg.hidden_size, cfg.vocab_size, dtype, device)

    # ------------------------------------------------------------------ forward
    def _mixer(self, li: int, layer: TavulixLayer, xn, batch: ModelBatch, cache, v_first):
        hs, T = layer.hs, xn.shape[0]
        proj = layer.qkvg(xn)
        mode = "plain" if not layer.lc.mixer.v_mix else ("save" if li == self.first_mix else "mix")
        q = lm.conv_heads(proj, hs, batch.seqs, batch.slot_mapping, cache[0], cache[1], conv=layer.conv,
                          state=cache[2] if len(cache) > 2 else None, q_norm=layer.q_norm, k_norm=layer.k_norm,
                          eps=self.cfg.norm_eps, v_first=v_first, v_mode=mode, lam=layer.vmix)
        attn = torch.empty(T, hs.heads * hs.vp, dtype=xn.dtype, device=xn.device)
        window_attention(q, cache[0], cache[1], batch.seqs, layer.rule(), attn,
                         gate=proj[:, hs.channels:hs.channels + hs.heads])
        return layer.o(attn)

    def forward(self, batch: ModelBatch, kv_caches, capture_layers=(), deepstack=None):
        """Returns (rows after the final norm [T, padded width], {i: fp32 stream after layer i - 1})."""
        cfg = self.cfg
        D, eps = cfg.hidden_size, cfg.norm_eps
        overlay = batch.input_embeds
        if overlay is not None:
            overlay = overlay.to(self.dtype_)
            if overlay.shape[1] < cfg.padded_width:
                overlay = F.pad(overlay, (0, cfg.padded_width - overlay.shape[1]))
        x, xn = lm.embed_norm(batch.input_ids, batch.positions, self.embed_tokens, self.pos_table,
                              self.layers[0].norm1 if len(self.layers) else self.final_norm, D, eps, overlay=overlay,
                              overlay_mask=batch.embeds_mask if overlay is not None else None)
        T = x.shape[0]
        captured = {0: x.clone()} if 0 in capture_layers else {}
        v_first = None
        if self.first_mix is not None:
            hs = self.layers[self.first_mix].hs
            v_first = torch.empty(T, hs.kv_heads * hs.vp, dtype=xn.dtype, device=xn.device)
        for li, layer in enumerate(self.layers):
            after = self.layers[li + 1].norm1 if li + 1 < len(self.layers) else self.final_norm
            y = self._mixer(li, layer, xn, batch, kv_caches[li], v_first)
            if layer.lc.ff is None:
                lm.add_norm_(x, y, layer.norm1b, D, eps, xn, after)
            else:
                lm.add_norm_(x, y, layer.norm1b, D, eps, xn, layer.norm2)
                z = layer.up(xn)
                y = layer.down(lm.poly_norm(z, layer.act, layer.lc.ff, eps, out=z))
                lm.add_norm_(x, y, layer.norm2b, D, eps, xn, after)
            if (li + 1) in capture_layers:
                captured[li + 1] = x.clone()
        return xn, captured

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits [rows, vocab]."""
        return lm.logit_softcap(self.lm_head(hidden), self.cfg.logit_softcap, self.cfg.vocab_size)

    # ------------------------------------------------------------------ weights
    def targets(self) -> dict:
        cfg, D = self.cfg, self.cfg.hidden_size
        whole = slice(None)
        t = {"embed": [(self.embed_tokens[:, :D], whole)], "pos": [(self.pos_table[:, :D], whole)],
             "final.norm": [(self.final_norm, whole)], "head": [(self.lm_head.weight[:cfg.vocab_size, :D], whole)]}
        for i, layer in enumerate(self.layers):
            p, m, hs = f"l{i}.", layer.lc.mixer, layer.hs
            W = layer.qkvg.weight
            off = 0
            for n, heads, d, pad in (("q", m.heads, m.dim, hs.dp), ("k", m.kv_heads, m.dim, hs.dp),
                                     ("v", m.kv_heads, m.vdim, hs.vp)):
                src = [slice(h * d, (h + 1) * d) for h in range(heads)]
                dst = [slice(off + h * pad, off + h * pad + d) for h in range(heads)]
                t[f"{p}mix.{n}"] = [(W[b, :D], a) for a, b in zip(src, dst)]
                if m.conv:
                    t[f"{p}mix.{n}.conv"] = [(layer.conv[:, b].t(), a) for a, b in zip(src, dst)]
                off += heads * pad
            t[p + "mix.g"] = [(W[off:off + m.heads, :D], whole)]
            t[p + "mix.q.norm"] = [(layer.q_norm[:m.dim], whole)]
            t[p + "mix.k.norm"] = [(layer.k_norm[:m.dim], whole)]
            if m.v_mix:
                t[p + "mix.vmix"] = [(layer.vmix, whole)]
            for n in ("r1", "r2", "sink"):
                t[f"{p}mix.{n}"] = [(getattr(layer, n), whole)]
            t[p + "mix.o"] = [(layer.o.weight[:D, h * hs.vp:h * hs.vp + m.vdim],
                               (whole, slice(h * m.vdim, (h + 1) * m.vdim))) for h in range(m.heads)]
            t[p + "norm1"], t[p + "norm1b"] = [(layer.norm1, whole)], [(layer.norm1b, whole)]
            if layer.lc.ff is not None:
                t[p + "norm2"], t[p + "norm2b"] = [(layer.norm2, whole)], [(layer.norm2b, whole)]
                t[p + "mlp.up"] = [(layer.up.weight[:layer.lc.ff, :D], whole)]
                t[p + "mlp.down"] = [(layer.down.weight[:D, :layer.lc.ff], whole)]
                t[p + "mlp.act"] = [(layer.act, whole)]
        return t

    def weights_loaded(self) -> None:
        for layer in self.layers:
            layer.bounded = bounded_scores(layer.lc.mixer.softcap, layer.r1, layer.r2)

    def random_weights(self, seed: int | None = None):
        """(name, tensor) pairs of a random checkpoint (runs without weights)."""
        dev = self.embed_tokens.device
        g = torch.Generator(device=dev).manual_seed(torch.initial_seed() if seed is None else seed)
        rnd = lambda s: torch.randn(s, generator=g, device=dev)
        for name, shape in self.cfg.tensor_shapes().items():
            last = name.split(".")[-1]
            if last in ("norm1", "norm1b", "norm2", "norm2b", "norm"):
                w = torch.ones(shape, device=dev)
            elif last == "conv":
                w = 0.3 * rnd(shape)
                w[:, -1] += 1.0
            elif last in ("r1", "r2"):
                w = 0.2 + 0.1 * rnd(shape).abs()
            elif last == "vmix":
                w = torch.full(shape, 0.3, device=dev)
            elif last == "act":
                w = torch.tensor([0.6, 0.3, 0.1, 0.0], device=dev)
            elif last == "sink":
                w = rnd(shape)
            else:
                w = rnd(shape) * (0.02 if name in ("embed", "pos") else shape[-1] ** -0.5)
            yield name, w
