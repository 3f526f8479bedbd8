"""Fikizen decoder: windowed attention with a zero sink and a gate per head, gated delta-rule recurrences, and layers whose
mixer is attention and a delta rule with decays per channel side by side, in any order; some layers use another layer's
weights; xIELU feed-forward, bounded logits.

One step over a mixed batch (portions of prompts and decoded tokens), per layer:

    attention          q | k | v | gate GEMM -> rotation, pages (one kernel) -> windowed paged attention with sink and gate in
                       its epilogue -> output GEMM
    gated delta        q | k | v | gate | step size | decay GEMM -> prompts: convolution and silu, chunk matrices, chunked
                       recurrence, norm and gate; decoded tokens: all of it in one kernel -> output GEMM
    parallel           q | k | v | r | k | v | a | gate | low-rank decay GEMM -> tanh, GEMM; row norms, rotation, value norm,
                       pages (one kernel) -> attention; channel delta rule; both write one row -> output GEMM
    stream step        x += branch, next norm (one kernel)
    feed-forward       up GEMM with xIELU in its epilogue -> down GEMM

The residual stream, norms, angles, scores, decays and recurrent state are fp32; activations are bf16 (serving) or fp32
(exact mode, every product in true fp32).  Heads are padded to 16 channels, rows to 8, both with zeros.  Rotated channels
are stored in interleaved order: pair i, channels (i, i + n / 2) of the checkpoint, is channels (2 i, 2 i + 1) of queries
and keys."""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F
from torch import nn

from ...ops import lm, stream
from ...ops.delta_rule import ChannelDelta, DeltaShape, GatedDelta, delta_rule
from ...ops.stream import RmsRows
from ...ops.window_attention import ScoreRule, window_attention
from ..packed_decoder import PackedDecoder, packed_linear as _linear, round_up, zeros_param as _zeros
from ..qwen_decoder import ModelBatch
from .config import AttentionMixer, DeltaMixer, FikizenConfig, LayerConfig, ParallelMixer

_WHOLE = slice(None)
_DECAY = -math.exp(-0.5)         # log decay of a fully open channel
_RANK = 16                       # of the decay's low-rank projection until a checkpoint tells


def _heads(n: int, count: int, pad: int, first: int = 0) -> list[tuple[slice, slice]]:
    """(checkpoint rows, packed rows) of every head."""
    return [(slice(h * n, (h + 1) * n), slice(first + h * pad, first + h * pad + n)) for h in range(count)]


def _interleaved(n: int, count: int, pad: int, first: int, rot: int) -> list[tuple[slice, slice]]:
    """The same where the halves of the first ``rot`` channels become interleaved pairs."""
    out, half = [], rot // 2
    for h in range(count):
        a, b = h * n, first + h * pad
        if half:
            out += [(slice(a, a + half), slice(b, b + rot, 2)), (slice(a + half, a + rot), slice(b + 1, b + rot, 2))]
        if rot < n:
            out.append((slice(a + rot, a + n), slice(b + rot, b + n)))
    return out


class _Heads:
    """Where q, k and v of an attention mixer go in packed rows that start at ``first``."""

    def __init__(self, m: AttentionMixer, first: int = 0):
        hs = m.head_shape
        k0, v0 = m.heads * hs.dp, (m.heads + m.kv_heads) * hs.dp
        self.parts = {"q": _interleaved(m.dim, m.heads, hs.dp, first, m.rot_dims),
                      "k": _interleaved(m.dim, m.kv_heads, hs.dp, first + k0, m.rot_dims),
                      "v": _heads(m.vdim, m.kv_heads, hs.vp, first + v0)}
        self.k0 = first + k0

    def rows(self, p: str, W, D: int, suffix: str = "") -> dict:
        return {p + n + suffix: [(W[d, :D] if W.dim() == 2 else W[d], a) for a, d in parts] for n, parts in self.parts.items()}


class _Attention(nn.Module):
    """Windowed attention with a zero sink and a gate per head."""

    def __init__(self, cfg: FikizenConfig, m: AttentionMixer, dtype, device):
        super().__init__()
        self.m, self.hs = m, m.head_shape
        self.proj = _linear(cfg.hidden_size, self.hs.channels + m.heads, dtype, device)
        self.sink = _zeros(m.heads, dtype=torch.float32, device=device)
        self.o = _linear(m.heads * self.hs.vp, cfg.hidden_size, dtype, device)

    def targets(self, p: str, D: int) -> dict:
        m, hs, W = self.m, self.hs, self.proj.weight
        return {**_Heads(m).rows(p, W, D), p + "g": [(W[hs.channels:hs.channels + m.heads, :D], _WHOLE)],
                p + "o": [(self.o.weight[:D, d], (_WHOLE, a)) for a, d in _heads(m.vdim, m.heads, hs.vp)]}

    def weights_loaded(self):
        pass

    def forward(self, xn, batch: ModelBatch, cache, turns):
        m, hs = self.m, self.hs
        proj = self.proj(xn)
        q = lm.rotary_heads(proj, hs, batch.slot_mapping, cache[0], cache[1], turns(m), m.rot_dims)
        out = torch.empty(xn.shape[0], m.heads * hs.vp, dtype=xn.dtype, device=xn.device)
        window_attention(q, cache[0], cache[1], batch.seqs, ScoreRule(m.scale, sink=self.sink, window=m.window), out,
                         gate=proj[:, hs.channels:hs.channels + m.heads])
        return self.o(out)


class _Delta(nn.Module):
    """Gated delta rule."""

    def __init__(self, cfg: FikizenConfig, m: DeltaMixer, dtype, device):
        super().__init__()
        self.s = s = m.shape
        f32 = lambda *sh: _zeros(*sh, dtype=torch.float32, device=device)
        self.proj = _linear(cfg.hidden_size, s.channels + s.v_cols + 2 * s.heads, dtype, device)
        self.a_log = f32(s.heads)
        self.rule = GatedDelta(f32(s.taps, s.channels), f32(s.heads), f32(s.heads), f32(s.vp), cfg.norm_eps)
        self.conv, self.rate, self.dt_bias, self.gain = self.rule.conv, self.rule.rate, self.rule.dt_bias, self.rule.gain
        self.o = _linear(s.v_cols, cfg.hidden_size, dtype, device)

    def targets(self, p: str, D: int) -> dict:
        s, W, t = self.s, self.proj.weight, {}
        values = _heads(s.vdim, s.heads, s.vp)
        for n, parts in (("q", _heads(s.dim, s.kv_heads, s.dp)), ("k", _heads(s.dim, s.kv_heads, s.dp, s.q_cols)),
                         ("v", _heads(s.vdim, s.heads, s.vp, 2 * s.q_cols))):
            t[p + n] = [(W[d, :D], a) for a, d in parts]
            t[f"{p}{n}.conv"] = [(self.conv[:, d].t(), a) for a, d in parts]
        t[p + "g"] = [(W[d, :D], a) for a, d in _heads(s.vdim, s.heads, s.vp, s.channels)]
        at = s.channels + s.v_cols
        t[p + "b"], t[p + "a"] = [(W[at:at + s.heads, :D], _WHOLE)], [(W[at + s.heads:at + 2 * s.heads, :D], _WHOLE)]
        t[p + "A_log"], t[p + "dt_bias"] = [(self.a_log, _WHOLE)], [(self.dt_bias, _WHOLE)]
        t[p + "norm"] = [(self.gain[:s.vdim], _WHOLE)]
        t[p + "o"] = [(self.o.weight[:D, d], (_WHOLE, a)) for a, d in values]
        return t

    def weights_loaded(self):
        self.rate.copy_(-torch.exp(self.a_log.double()))

    def forward(self, xn, batch: ModelBatch, cache, turns):
        s = self.s
        out = torch.empty(xn.shape[0], s.v_cols, dtype=xn.dtype, device=xn.device)
        delta_rule(self.proj(xn), s, batch.seqs, self.rule, cache[2], out, hist=cache[3] if s.taps > 1 else None)
        return self.o(out)


class _Parallel(nn.Module):
    """Attention over normed rows and a delta rule with decays per channel, side by side."""

    def __init__(self, cfg: FikizenConfig, m: ParallelMixer, dtype, device):
        super().__init__()
        self.m, self.hs, self.s, self.eps = m, m.left.head_shape, m.right, cfg.norm_eps
        hs, s, D = self.hs, self.s, cfg.hidden_size
        self.make = lambda n_in, n_out, **kw: _linear(n_in, n_out, dtype, device, **kw)
        self.width, self.low_col = D, hs.channels + 5 * s.q_cols
        f32 = lambda *sh: _zeros(*sh, dtype=torch.float32, device=device)
        self.q_gain, self.k_gain = f32(hs.heads * hs.dp), f32(hs.kv_heads * hs.dp)
        self.sink = f32(hs.heads)
        self.norm, self.removal = f32(s.v_cols), f32(s.q_cols)
        self.rule = ChannelDelta(f32(s.q_cols), self.removal, _DECAY, f32(s.v_cols), cfg.norm_eps)
        self.decay_bias, self.gain = self.rule.decay_bias, self.rule.gain
        self.set_rank(_RANK)
        self.left_cols = hs.heads * hs.vp
        self.o = _linear(self.left_cols + s.v_cols, D, dtype, device)

    @torch.no_grad()
    def set_rank(self, n: int):
        """Sizes of the low-rank decay: the last rows of the projection, and the matrix behind the tanh."""
        old = getattr(self, "proj", None)
        self.rank, self.rank_p, self.proj = n, round_up(n, 8), self.make(self.width, self.low_col + n, bias=True)
        if old is not None:
            self.proj.weight[:self.low_col].copy_(old.weight[:self.low_col])
            self.proj.bias[:self.low_col].copy_(old.bias[:self.low_col])
        self.w2 = self.make(n, self.s.q_cols)

    def targets(self, p: str, D: int) -> dict:
        m, hs, s, W = self.m, self.hs, self.s, self.proj.weight
        left = _Heads(m.left)
        t = {**left.rows(p + "left.", W, D), **left.rows(p + "left.", self.proj.bias, D, ".b")}
        t[p + "left.q.norm"] = [(self.q_gain[d], a) for a, d in left.parts["q"]]
        t[p + "left.k.norm"] = [(self.k_gain[d.start - left.k0:d.stop - left.k0:d.step], a) for a, d in left.parts["k"]]
        t[p + "left.o"] = [(self.o.weight[:D, d], (_WHOLE, a)) for a, d in _heads(m.left.vdim, m.left.heads, hs.vp)]
        p += "right."
        for i, n in enumerate("rkvag"):
            t[p + n] = [(W[d, :D], a) for a, d in _heads(s.dim, s.heads, s.dp, hs.channels + i * s.q_cols)]
        parts = _heads(s.dim, s.heads, s.dp)
        for n, w in (("a.b", self.removal), ("w0", self.decay_bias), ("norm", self.norm)):
            t[p + n] = [(w[d], a) for a, d in parts]
        t[p + "w1"] = [(W[self.low_col:self.low_col + self.rank, :D], _WHOLE)]
        t[p + "w2"] = [(self.w2.weight[d, :self.rank], a) for a, d in parts]
        t[p + "o"] = [(self.o.weight[:D, self.left_cols + d.start:self.left_cols + d.stop], (_WHOLE, a)) for a, d in parts]
        return t

    def weights_loaded(self):
        self.gain.copy_(self.norm * self.m.right_scale)

    def forward(self, xn, batch: ModelBatch, cache, turns):
        m, hs, s = self.m, self.hs, self.s
        proj = self.proj(xn)
        decay = self.w2(lm.tanh_cols(proj[:, self.low_col:self.low_col + self.rank_p]))
        out = torch.empty(xn.shape[0], self.left_cols + s.v_cols, dtype=xn.dtype, device=xn.device)
        # the constant on the left branch rides on its values: the sink has none, so the result is linear in them
        q = lm.rotary_heads(proj, hs, batch.slot_mapping, cache[0], cache[1], turns(m.left), m.left.rot_dims, q_gain=self.q_gain,
                            k_gain=self.k_gain, v_norm=True, v_mult=m.left_scale, eps=self.eps)
        window_attention(q, cache[0], cache[1], batch.seqs, ScoreRule(m.left.scale, sink=self.sink, window=m.left.window),
                         out[:, :self.left_cols])
        delta_rule(proj[:, hs.channels:self.low_col], s, batch.seqs, self.rule, cache[2], out[:, self.left_cols:], decay=decay)
        return self.o(out)


_MODULES = {AttentionMixer: _Attention, DeltaMixer: _Delta, ParallelMixer: _Parallel}


class _Dense(nn.Module):
    """Two matrices around an xIELU."""

    def __init__(self, cfg: FikizenConfig, ff: int, dtype, device):
        super().__init__()
        self.ff = ff
        self.up, self.down = _linear(cfg.hidden_size, ff, dtype, device), _linear(ff, cfg.hidden_size, dtype, device)
        self.act = _zeros(2, dtype=torch.float32, device=device)
        self.coef = (0.0, 0.5)                              # set with the weights

    def targets(self, p: str, D: int) -> dict:
        return {p + "up": [(self.up.weight[:self.ff, :D], _WHOLE)], p + "down": [(self.down.weight[:D, :self.ff], _WHOLE)],
                p + "act": [(self.act, _WHOLE)]}

    def weights_loaded(self):
        above, below = F.softplus(self.act.double(), threshold=1e9).tolist()
        self.coef = (above, 0.5 + below)

    def forward(self, xn):
        return self.down(self.up(xn, act="xielu", coef=self.coef))


class FikizenLayer(nn.Module):
    def __init__(self, cfg: FikizenConfig, lc: LayerConfig, dtype, device):
        super().__init__()
        norm = lambda: RmsRows(_zeros(cfg.padded_width, dtype=torch.float32, device=device), cfg.norm_eps, cfg.hidden_size)
        self.norm1, self.norm2 = norm(), norm() if lc.ff is not None else None
        self.gain1, self.gain2 = self.norm1.gain, self.norm2.gain if self.norm2 else None
        self.mix = _MODULES[type(lc.mixer)](cfg, lc.mixer, dtype, device)
        self.mlp = _Dense(cfg, lc.ff, dtype, device) if lc.ff is not None else None

    def targets(self, p: str, D: int) -> dict:
        t = {p + "norm1": [(self.gain1[:D], _WHOLE)], **self.mix.targets(p + "mix.", D)}
        if self.mlp is not None:
            t.update({p + "norm2": [(self.gain2[:D], _WHOLE)], **self.mlp.targets(p + "mlp.", D)})
        return t


class FikizenDecoder(PackedDecoder):
    def __init__(self, cfg: FikizenConfig, dtype=torch.bfloat16, device=None):
        super().__init__()
        self.cfg, self.dtype_ = cfg, dtype
        Dp = cfg.padded_width
        self.embed_tokens = _zeros(cfg.vocab_size, Dp, dtype=dtype, device=device)
        # one module per layer that has weights
        self.owners = nn.ModuleDict({str(i): FikizenLayer(cfg, l, dtype, device) for i, l in enumerate(cfg.layers) if l.owner == i})
        self.final_gain = _zeros(Dp, dtype=torch.float32, device=device)
        self.final_norm = RmsRows(self.final_gain, cfg.norm_eps, cfg.hidden_size)
        self.lm_head = _linear(cfg.hidden_size, cfg.vocab_size, dtype, device)

    def layer(self, i: int) -> FikizenLayer:
        return self.owners[str(self.cfg.layers[i].owner)]

    # ------------------------------------------------------------------ forward
    def forward(self, batch: ModelBatch, kv_caches, capture_layers=(), deepstack=None):
        """Returns (rows after the final norm [T, padded width], {i: fp32 stream after layer i - 1})."""
        cfg, n = self.cfg, len(self.cfg.layers)
        overlay = batch.input_embeds
        if overlay is not None:
            overlay = overlay.to(self.dtype_)
            if overlay.shape[1] < cfg.padded_width:
                overlay = F.pad(overlay, (0, cfg.padded_width - overlay.shape[1]))
        layers = [self.layer(i) for i in range(n)]
        x, xn = stream.embed_rows(batch.input_ids, self.embed_tokens, layers[0].norm1 if n else self.final_norm,
                                  overlay=overlay, overlay_mask=batch.embeds_mask if overlay is not None else None)
        captured = {0: x.clone()} if 0 in capture_layers else {}
        angles: dict = {}

        def turns(m: AttentionMixer):                       # rows of cos and sin, shared by the layers that turn alike
            key = (m.rot_base, m.rot_dims)
            if key not in angles:
                angles[key] = stream.rotary_rows(batch.positions, *key) if m.rot_dims else None
            return angles[key]
        for i, layer in enumerate(layers):
            after = layers[i + 1].norm1 if i + 1 < n else self.final_norm
            y = layer.mix(xn, batch, kv_caches[i], turns)
            stream.add_branch_(x, y, 1.0, xn, after if layer.mlp is None else layer.norm2)
            if layer.mlp is not None:
                stream.add_branch_(x, layer.mlp(xn), 1.0, xn, after)
            if (i + 1) in capture_layers:
                captured[i + 1] = x.clone()
        return xn, captured

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits [rows, vocab]."""
        return lm.logit_softcap(self.lm_head(hidden), self.cfg.logit_softcap, self.cfg.vocab_size)

    # ------------------------------------------------------------------ weights
    def targets(self) -> dict:
        cfg, D = self.cfg, self.cfg.hidden_size
        t = {"embed": [(self.embed_tokens[:, :D], _WHOLE)], "head": [(self.lm_head.weight[:cfg.vocab_size, :D], _WHOLE)],
             "final.norm": [(self.final_gain[:D], _WHOLE)]}
        for i, layer in self.owners.items():
            t.update(layer.targets(f"l{i}.", D))
        return t

    def load_weights(self, weights) -> set:
        self._ranked = {}                                       # layers whose rank a tensor of this checkpoint has told
        return super().load_weights(weights)

    def resize(self, name: str, shape) -> None:
        i = name.split(".")[0][1:]
        n = shape[0] if name.endswith("w1") else shape[1]
        if self._ranked.setdefault(i, n) != n:
            raise ValueError(f"{name}: rank {n}, but {self._ranked[i]} in the other tensor")
        if n != self.owners[i].mix.rank:
            self.owners[i].mix.set_rank(n)

    def weights_loaded(self) -> None:
        for layer in self.owners.values():
            layer.mix.weights_loaded()
            if layer.mlp is not None:
                layer.mlp.weights_loaded()

    def random_weights(self, seed: int | None = None):
        """(name, tensor) pairs of a random checkpoint (runs without weights)."""
        dev = self.embed_tokens.device
        g = torch.Generator(device=dev).manual_seed(torch.initial_seed() if seed is None else seed)
        rnd = lambda s: torch.randn(s, generator=g, device=dev)
        for name, shape in self.cfg.tensor_shapes().items():
            shape = tuple(_RANK if n is None else n for n in shape)
            last = name.split(".")[-1]
            if last in ("norm1", "norm2", "norm"):
                w = torch.ones(shape, device=dev)
            elif last in ("A_log", "w0"):
                w = rnd(shape)
            elif last in ("b", "dt_bias") and len(shape) == 1:
                w = 0.1 * rnd(shape)
            elif last == "act":
                w = torch.tensor([0.5, 0.2], device=dev)
            elif last == "conv":
                w = 0.3 * rnd(shape)
                w[:, -1] += 1.0
            else:
                w = rnd(shape) * (1.0 if name == "embed" else shape[-1] ** -0.5)
            yield name, w
