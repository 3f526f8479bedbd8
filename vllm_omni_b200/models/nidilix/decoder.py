"""Nidilix decoder: latent attention (some layers read another layer's latents) and gated linear recurrences in any
order, a mixture of squared-ReLU experts with a shared one, an input per layer and token from a side table, norms
without statistics (a scaled tanh), and a constant on every branch.

One step over a mixed batch (portions of prompts and decoded tokens), per layer:

    latent attention   q | latent | rotated key | gate GEMM -> rotation, latent norm, pages (one kernel) ->
                       prompts: up-projection of the latents, tcgen05 attention with the gate in its epilogue;
                       decoded tokens: queries taken to the latent space, attention over the latent pages,
                       values taken back with the gate -> output GEMM
    recurrence         y | x GEMM -> convolution, gates, scan and output branch (fused) -> output GEMM
    stream step        x += m * branch, next norm (one kernel)
    experts            router + choice (one kernel) -> grouped up GEMM, squared ReLU in its epilogue -> grouped
                       down GEMM; shared expert -> x += m * (weighted sum + shared) (one kernel)
    side input         gate GEMM -> gelu * table row -> GEMM -> x += m * norm(.), next norm (one kernel)

The residual stream, norms, angles, scores, routers and recurrent state are fp32; activations are bf16 (serving) or
fp32 (exact mode, every product in true fp32).  Heads are padded to 16 channels, rows to 8, both with zeros."""
from __future__ import annotations

import torch
import torch.nn.functional as F
from torch import nn

from ...ops import gemm, latent_attention as LA, moe, recurrent, stream
from ...ops.lm import logit_softcap
from ..packed_decoder import PackedDecoder, packed_linear as _linear, round_up, zeros_param as _zeros
from ..qwen_decoder import ModelBatch
from .config import ExpertsConfig, LatentMixer, LayerConfig, NidilixConfig, ScanMixer

_WHOLE = slice(None)


class _TanhNorm(nn.Module):
    def __init__(self, width: int, device):
        super().__init__()
        f32 = lambda n: _zeros(n, dtype=torch.float32, device=device)
        self.alpha, self.w, self.b = f32(1), f32(width), f32(width)

    def targets(self, name: str, n: int) -> dict:
        return {name: [(self.w[:n], _WHOLE)], name + ".b": [(self.b[:n], _WHOLE)], name + ".alpha": [(self.alpha, _WHOLE)]}


class _Latent(nn.Module):
    """Latent attention mixer."""

    def __init__(self, cfg: NidilixConfig, m: LatentMixer, dtype, device):
        super().__init__()
        self.m, self.s, self.own = m, m.shape, m.kv_from is None
        s = self.s
        z = lambda *sh, dt=dtype: _zeros(*sh, dtype=dt, device=device)
        self.proj = _linear(cfg.hidden_size, s.q_cols + (s.row if self.own else 0) + s.heads, dtype, device)
        if self.own:
            self.c_norm = z(s.rank_p, dt=torch.float32)
        self.uk_t = z(s.heads, s.rank_p, s.dim_p)                   # query side: latent <- head channels
        self.kv_up = z(s.heads * (s.dim_p + s.vdim_p), s.rank_p)    # key rows of all heads, then value rows
        self.o = _linear(s.heads * s.vdim_p, cfg.hidden_size, dtype, device)

    @property
    def gate_col(self) -> int:
        return self.s.q_cols + (self.s.row if self.own else 0)

    def targets(self, p: str, D: int) -> dict:
        s, W = self.s, self.proj.weight
        q = []
        for h in range(s.heads):
            a, b = h * (s.dim + s.rot), h * s.head_cols
            q += [(W[b:b + s.dim, :D], slice(a, a + s.dim)),
                  (W[b + s.dim_p:b + s.dim_p + s.rot, :D], slice(a + s.dim, a + s.dim + s.rot))]
        t = {p + "q": q, p + "g": [(W[self.gate_col:self.gate_col + s.heads, :D], _WHOLE)]}
        if self.own:
            c = s.q_cols
            t[p + "dkv"] = [(W[c:c + s.rank, :D], slice(0, s.rank)),
                            (W[c + s.rank_p:c + s.rank_p + s.rot, :D], slice(s.rank, s.rank + s.rot))]
            t[p + "dkv.norm"] = [(self.c_norm[:s.rank], _WHOLE)]
        nk, U = s.heads * s.dim_p, self.kv_up
        head = lambda n: [slice(h * n, (h + 1) * n) for h in range(s.heads)]
        t[p + "uk"] = [(U[h * s.dim_p:h * s.dim_p + s.dim, :s.rank], a) for h, a in enumerate(head(s.dim))] + \
                      [(self.uk_t[h, :s.rank, :s.dim].t(), a) for h, a in enumerate(head(s.dim))]
        t[p + "uv"] = [(U[nk + h * s.vdim_p:nk + h * s.vdim_p + s.vdim, :s.rank], a) for h, a in enumerate(head(s.vdim))]
        t[p + "o"] = [(self.o.weight[:D, h * s.vdim_p:h * s.vdim_p + s.vdim], (_WHOLE, a)) for h, a in enumerate(head(s.vdim))]
        return t

    def forward(self, xn, batch: ModelBatch, cache, turns, eps):
        s = self.s
        proj = self.proj(xn)
        LA.latent_rows(proj, s, turns, batch.slot_mapping, cache[0], self.c_norm if self.own else None, eps)
        out = torch.empty(xn.shape[0], s.heads * s.vdim_p, dtype=xn.dtype, device=xn.device)
        LA.latent_attention(proj, s, cache[0], batch.seqs, self.uk_t, self.kv_up, self.m.scale, out,
                            gate=proj[:, self.gate_col:self.gate_col + s.heads])
        return self.o(out)


class _Scan(nn.Module):
    """Gated linear recurrence mixer."""

    def __init__(self, cfg: NidilixConfig, m: ScanMixer, dtype, device):
        super().__init__()
        self.s = s = m.shape
        f32 = lambda *sh: _zeros(*sh, dtype=torch.float32, device=device)
        self.proj = _linear(cfg.hidden_size, 2 * s.channels, dtype, device, bias=True)
        self.conv, self.conv_b = f32(s.taps, s.channels), f32(s.channels)
        self.gates = _zeros(2, s.blocks, s.part_p, s.part_p, dtype=dtype, device=device)
        self.gates_b = f32(2, s.channels)
        self.lam, self.decay = f32(s.channels), f32(s.channels)
        self.o = _linear(s.channels, cfg.hidden_size, dtype, device)

    def targets(self, p: str, D: int) -> dict:
        s = self.s
        parts = [(slice(b * s.part, (b + 1) * s.part), slice(b * s.part_p, b * s.part_p + s.part)) for b in range(s.blocks)]
        W, B = self.proj.weight, self.proj.bias
        t = {}
        for n, off in (("y", 0), ("x", s.channels)):
            t[p + n] = [(W[off:off + s.channels][d, :D], a) for a, d in parts]
            t[p + n + ".b"] = [(B[off:off + s.channels][d], a) for a, d in parts]
        t[p + "conv"] = [(self.conv[:, d].t(), a) for a, d in parts]
        t[p + "conv.b"] = [(self.conv_b[d], a) for a, d in parts]
        for g, n in enumerate(("ra", "ri")):
            t[p + n] = [(self.gates[g, :, :s.part, :s.part], _WHOLE)]
            t[p + n + ".b"] = [(self.gates_b[g].view(s.blocks, s.part_p)[:, :s.part], _WHOLE)]
        t[p + "lam"] = [(self.lam[d], a) for a, d in parts]
        t[p + "o"] = [(self.o.weight[:D, d], (_WHOLE, a)) for a, d in parts]
        return t

    def weights_loaded(self):
        self.decay.copy_(-8.0 * F.softplus(self.lam.double(), threshold=1e9))

    def forward(self, xn, batch: ModelBatch, cache):
        out = recurrent.gated_scan(self.proj(xn), self.s, batch.seqs, self.conv, self.conv_b, self.gates, self.gates_b,
                                   self.decay, cache[2], cache[3])
        return self.o(out)


class _Experts(nn.Module):
    def __init__(self, cfg: NidilixConfig, m: ExpertsConfig, dtype, device):
        super().__init__()
        self.m = m
        D, ff = cfg.padded_width, round_up(m.ff, 8)
        self.router = _zeros(round_up(m.experts, 8), D, dtype=dtype, device=device)
        self.router_b = _zeros(round_up(m.experts, 8), dtype=torch.float32, device=device)
        self.up = _zeros(m.experts, ff, D, dtype=dtype, device=device)
        self.down = _zeros(m.experts, D, ff, dtype=dtype, device=device)
        if m.shared_ff:
            self.shared_up = _linear(cfg.hidden_size, m.shared_ff, dtype, device)
            self.shared_down = _linear(m.shared_ff, cfg.hidden_size, dtype, device)
        self.ws = moe.MoEWorkspace()

    def targets(self, p: str, D: int) -> dict:
        m = self.m
        t = {p + "router": [(self.router[:m.experts, :D], _WHOLE)], p + "router.b": [(self.router_b[:m.experts], _WHOLE)]}
        for e in range(m.experts):
            t[f"{p}e{e}.up"] = [(self.up[e, :m.ff, :D], _WHOLE)]
            t[f"{p}e{e}.down"] = [(self.down[e, :D, :m.ff], _WHOLE)]
        if m.shared_ff:
            t[p + "shared.up"] = [(self.shared_up.weight[:m.shared_ff, :D], _WHOLE)]
            t[p + "shared.down"] = [(self.shared_down.weight[:D, :m.shared_ff], _WHOLE)]
        return t

    def forward(self, xn):
        """(rows of the chosen experts with their weights, shared expert's rows or None)."""
        shared = self.shared_down(self.shared_up(xn, act="relu2")) if self.m.shared_ff else None
        return moe.expert_rows(xn, self.router, self.router_b, self.m.router, self.up, self.down, act="relu2", ws=self.ws), shared


class NidilixLayer(nn.Module):
    def __init__(self, cfg: NidilixConfig, lc: LayerConfig, dtype, device):
        super().__init__()
        Dp = cfg.padded_width
        self.norm1 = _TanhNorm(Dp, device)
        self.mix = (_Latent if isinstance(lc.mixer, LatentMixer) else _Scan)(cfg, lc.mixer, dtype, device)
        self.norm2 = _TanhNorm(Dp, device) if lc.mlp is not None else None
        self.mlp = _Experts(cfg, lc.mlp, dtype, device) if lc.mlp is not None else None
        self.side_gate = self.side_proj = None
        if cfg.side_dim:
            self.side_gate, self.side_proj = _linear(cfg.hidden_size, cfg.side_dim, dtype, device), \
                _linear(cfg.side_dim, cfg.hidden_size, dtype, device)
            self.side_norm = _zeros(Dp, dtype=torch.float32, device=device)

    def targets(self, p: str, cfg: NidilixConfig) -> dict:
        D = cfg.hidden_size
        t = {**self.norm1.targets(p + "norm1", D), **self.mix.targets(p + "mix.", D)}
        if self.mlp is not None:
            t.update(self.norm2.targets(p + "norm2", D))
            t.update(self.mlp.targets(p + "mlp.", D))
        if self.side_gate is not None:
            t[p + "side.gate"] = [(self.side_gate.weight[:cfg.side_dim, :D], _WHOLE)]
            t[p + "side.proj"] = [(self.side_proj.weight[:D, :cfg.side_dim], _WHOLE)]
            t[p + "side.norm"] = [(self.side_norm[:D], _WHOLE)]
        return t


class NidilixDecoder(PackedDecoder):
    def __init__(self, cfg: NidilixConfig, dtype=torch.bfloat16, device=None):
        super().__init__()
        self.cfg, self.dtype_ = cfg, dtype
        self.embed_tokens = _zeros(cfg.vocab_size, cfg.padded_width, dtype=dtype, device=device)
        self.side_table = _zeros(cfg.vocab_size, cfg.side_dim * len(cfg.layers), dtype=dtype, device=device) \
            if cfg.side_dim else None
        self.layers = nn.ModuleList([NidilixLayer(cfg, l, dtype, device) for l in cfg.layers])
        self.final_norm = _TanhNorm(cfg.padded_width, device)
        self.lm_head = _linear(cfg.hidden_size, cfg.vocab_size, dtype, device)

    # ------------------------------------------------------------------ forward
    def forward(self, batch: ModelBatch, kv_caches, capture_layers=(), deepstack=None):
        """Returns (rows after the final norm [T, padded width], {i: fp32 stream after layer i - 1})."""
        cfg = self.cfg
        D, eps, mult, ids = cfg.hidden_size, cfg.norm_eps, cfg.residual_mult, batch.input_ids
        overlay = batch.input_embeds
        if overlay is not None:
            overlay = overlay.to(self.dtype_)
            if overlay.shape[1] < cfg.padded_width:
                overlay = F.pad(overlay, (0, cfg.padded_width - overlay.shape[1]))
        x, xn = stream.embed_rows(ids, self.embed_tokens, self.layers[0].norm1 if len(self.layers) else self.final_norm,
                                  overlay=overlay, overlay_mask=batch.embeds_mask if overlay is not None else None)
        captured = {0: x.clone()} if 0 in capture_layers else {}
        turns: dict = {}
        for li, (lc, layer) in enumerate(zip(cfg.layers, self.layers)):
            after = self.layers[li + 1].norm1 if li + 1 < len(self.layers) else self.final_norm
            plain = stream.CAST if cfg.side_dim else after              # the side input reads the stream itself
            if isinstance(lc.mixer, LatentMixer):
                key = (lc.mixer.rot_base, lc.mixer.shape.rot)
                if key not in turns:
                    turns[key] = stream.rotary_rows(batch.positions, *key)
                src = li if lc.mixer.kv_from is None else lc.mixer.kv_from
                y = layer.mix(xn, batch, kv_caches[src], turns[key], eps)
            else:
                y = layer.mix(xn, batch, kv_caches[li])
            if layer.mlp is None:
                stream.add_branch_(x, y, mult, xn, plain)
            else:
                stream.add_branch_(x, y, mult, xn, layer.norm2)
                rows, shared = layer.mlp(xn)
                stream.add_expert_rows_(x, rows, shared, mult, xn, plain)
            if layer.side_gate is not None:
                z = stream.gelu_lookup_(layer.side_gate(xn), self.side_table, ids, li * cfg.side_dim, cfg.side_dim)
                stream.add_branch_(x, layer.side_proj(z), mult, xn, after, gain=layer.side_norm, eps=eps, n=D)
            if (li + 1) in capture_layers:
                captured[li + 1] = x.clone()
        return xn, captured

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits [rows, vocab]."""
        return logit_softcap(self.lm_head(hidden), None, self.cfg.vocab_size)

    # ------------------------------------------------------------------ weights
    def targets(self) -> dict:
        cfg, D = self.cfg, self.cfg.hidden_size
        t = {"embed": [(self.embed_tokens[:, :D], _WHOLE)], "head": [(self.lm_head.weight[:cfg.vocab_size, :D], _WHOLE)],
             **self.final_norm.targets("final.norm", D)}
        if self.side_table is not None:
            t["side.embed"] = [(self.side_table, _WHOLE)]
        for i, layer in enumerate(self.layers):
            t.update(layer.targets(f"l{i}.", cfg))
        return t

    def weights_loaded(self) -> None:
        for layer in self.layers:
            if isinstance(layer.mix, _Scan):
                layer.mix.weights_loaded()

    def random_weights(self, seed: int | None = None):
        """(name, tensor) pairs of a random checkpoint (runs without weights)."""
        dev = self.embed_tokens.device
        g = torch.Generator(device=dev).manual_seed(torch.initial_seed() if seed is None else seed)
        rnd = lambda s: torch.randn(s, generator=g, device=dev)
        for name, shape in self.cfg.tensor_shapes().items():
            last = name.split(".")[-1]
            if last in ("norm1", "norm2", "norm"):
                w = torch.ones(shape, device=dev)
            elif last == "alpha":
                w = torch.full(shape, 0.7, device=dev)
            elif last == "b":
                w = 0.1 * rnd(shape)
            elif last == "lam":                                # a^(1/r) between 0.9 and 0.999
                a = 0.9 + 0.099 * torch.rand(shape, generator=g, device=dev)
                w = torch.log(torch.expm1(-torch.log(a) / 8.0))
            elif last == "conv":
                w = 0.3 * rnd(shape)
                w[:, -1] += 1.0
            else:
                w = rnd(shape) * (1.0 if name in ("embed", "side.embed") else shape[-1] ** -0.5)
            yield name, w
