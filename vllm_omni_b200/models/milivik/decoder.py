"""Milivik decoder: latent attention with a sliding window and a latent on the query side, and differential attention, in any
order; dense or mixture-of-experts feed-forward with a gated shared expert; norms on the sublayers' results only.

One step over a mixed batch (portions of prompts and decoded tokens), per layer:

    latent attention   query latent | latent | rotated key | gate GEMM -> both norms, rotation, pages (one kernel) -> query
                       GEMM -> rotation -> prompts: up-projection of the latents in the window, tcgen05 attention;
                       decoded tokens: attention over the latent pages; the gate in either epilogue -> output GEMM
    differential       q | k | v | gate GEMM -> head norms, query growth, pages (one kernel) -> attention of both maps with
      attention        their difference, its norm and the gate in the epilogue (one kernel) -> output GEMM
    stream step        x += norm(branch), x in the activations' type (one kernel)
    feed-forward       gate | up GEMM -> SwiGLU -> down GEMM -> stream step
    experts            router + choice (one kernel) -> grouped GEMMs around SwiGLU; shared expert, whose own gate is one more
                       row of its first GEMM -> x += norm(weighted sum + gate * shared), cast (one kernel)

The residual stream, norms, angles, scores and routers are fp32; activations are bf16 (serving) or fp32 (exact mode,
every product in true fp32).  Heads are padded to 16 channels, rows to 8, both with zeros.  Rotated channels are stored in
interleaved order: pair i, channels (i, i + n / 2) of the checkpoint, is channels (2 i, 2 i + 1) of queries and keys."""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F
from torch import nn

from ...ops import fused, gemm, latent_attention as LA, lm, moe, stream
from ...ops.window_attention import DiffRule, ScoreRule, window_attention
from ..packed_decoder import PackedDecoder, packed_linear as _linear, round_up, zeros_param as _zeros
from ..qwen_decoder import ModelBatch
from .config import DenseConfig, DiffMixer, ExpertsConfig, LatentMixer, LayerConfig, MilivikConfig

_WHOLE = slice(None)


def _heads(n: int, count: int) -> list[slice]:
    return [slice(h * n, (h + 1) * n) for h in range(count)]


class _Gain(nn.Module):
    """Gain of a norm whose checkpoint tensor is the gain less one."""

    def __init__(self, n: int, padded: int, device):
        super().__init__()
        self.n, self.w = n, _zeros(padded, dtype=torch.float32, device=device)
        self.gain = _zeros(padded, dtype=torch.float32, device=device)

    def targets(self, name: str) -> dict:
        return {name: [(self.w[:self.n], _WHOLE)]}

    def weights_loaded(self):
        self.gain[:self.n] = 1.0 + self.w[:self.n]


class _Latent(nn.Module):
    """Latent attention mixer."""

    def __init__(self, cfg: MilivikConfig, m: LatentMixer, dtype, device):
        super().__init__()
        self.m, self.s = m, m.shape
        s = self.s
        z = lambda *sh, dt=dtype: _zeros(*sh, dtype=dt, device=device)
        self.gate_col = m.q_rank_p + s.row
        self.proj = _linear(cfg.hidden_size, self.gate_col + s.heads * s.vdim_p, dtype, device)
        self.q_norm, self.c_norm = z(m.q_rank_p, dt=torch.float32), z(s.rank_p, dt=torch.float32)
        self.uq = _linear(m.q_rank_p, s.q_cols, dtype, device)
        self.uk_t = z(s.heads, s.rank_p, s.dim_p)                   # query side: latent <- head channels
        self.kv_up = z(s.heads * (s.dim_p + s.vdim_p), s.rank_p)    # key rows of all heads, then value rows
        self.o = _linear(s.heads * s.vdim_p, cfg.hidden_size, dtype, device)

    def _interleaved(self, rows, first: int) -> list:
        """``rows``: destination of the rot rotated rows; checkpoint rows from ``first`` on."""
        half = self.s.rot // 2
        return [(rows[0::2], slice(first, first + half)), (rows[1::2], slice(first + half, first + 2 * half))]

    def targets(self, p: str, D: int) -> dict:
        m, s, W, U = self.m, self.s, self.proj.weight, self.kv_up
        q = []
        for h in range(s.heads):
            a, b = h * (s.dim + s.rot), h * s.head_cols
            q.append((self.uq.weight[b:b + s.dim, :m.q_rank], slice(a, a + s.dim)))
            q += self._interleaved(self.uq.weight[b + s.dim_p:b + s.dim_p + s.rot, :m.q_rank], a + s.dim)
        c, k, g, nk = m.q_rank_p, m.q_rank_p + s.rank_p, self.gate_col, s.heads * s.dim_p
        return {
            p + "dq": [(W[:m.q_rank, :D], _WHOLE)], p + "dq.norm": [(self.q_norm[:m.q_rank], _WHOLE)], p + "uq": q,
            p + "dkv": [(W[c:c + s.rank, :D], slice(0, s.rank))] + self._interleaved(W[k:k + s.rot, :D], s.rank),
            p + "dkv.norm": [(self.c_norm[:s.rank], _WHOLE)],
            p + "uk": [(U[h * s.dim_p:h * s.dim_p + s.dim, :s.rank], a) for h, a in enumerate(_heads(s.dim, s.heads))]
                      + [(self.uk_t[h, :s.rank, :s.dim].t(), a) for h, a in enumerate(_heads(s.dim, s.heads))],
            p + "uv": [(U[nk + h * s.vdim_p:nk + h * s.vdim_p + s.vdim, :s.rank], a) for h, a in enumerate(_heads(s.vdim, s.heads))],
            p + "g": [(W[g + h * s.vdim_p:g + h * s.vdim_p + s.vdim, :D], a) for h, a in enumerate(_heads(s.vdim, s.heads))],
            p + "o": [(self.o.weight[:D, h * s.vdim_p:h * s.vdim_p + s.vdim], (_WHOLE, a)) for h, a in enumerate(_heads(s.vdim, s.heads))]}

    def weights_loaded(self):
        pass

    def forward(self, xn, batch: ModelBatch, cache, turns, eps):
        m, s = self.m, self.s
        proj = self.proj(xn)
        qc = proj[:, :m.q_rank_p]
        LA.cache_rows(proj[:, m.q_rank_p:], s, turns, batch.slot_mapping, cache[0], self.c_norm, eps, query_latent=qc,
                      query_norm=self.q_norm, query_rank=m.q_rank)
        q = self.uq(qc)
        LA.rotate_queries(q, s, turns)
        out = torch.empty(xn.shape[0], s.heads * s.vdim_p, dtype=xn.dtype, device=xn.device)
        LA.latent_attention(q, s, cache[0], batch.seqs, self.uk_t, self.kv_up, m.scale, out,
                            gate=proj[:, self.gate_col:self.gate_col + s.heads * s.vdim_p], window=m.window)
        return self.o(out)


class _Diff(nn.Module):
    """Differential attention mixer."""

    def __init__(self, cfg: MilivikConfig, m: DiffMixer, dtype, device):
        super().__init__()
        self.m, self.hs, self.eps = m, m.head_shape, cfg.norm_eps
        hs = self.hs
        f32 = lambda n: _zeros(n, dtype=torch.float32, device=device)
        self.proj = _linear(cfg.hidden_size, hs.channels + m.heads, dtype, device)
        self.q_norm, self.k_norm = f32(hs.dp), f32(hs.dp)
        self.lq1, self.lk1, self.lq2, self.lk2 = (f32(m.dim) for _ in range(4))
        self.o = _linear(m.heads * hs.vp, cfg.hidden_size, dtype, device)
        self.rule = None                                            # set with the weights

    def targets(self, p: str, D: int) -> dict:
        m, hs, W = self.m, self.hs, self.proj.weight
        R, k0, v0 = m.heads // m.kv_heads, 2 * m.heads * hs.dp, 2 * (m.heads + m.kv_heads) * hs.dp
        q = []
        for h in range(m.heads):
            g, r = divmod(h, R)
            for n in range(2):                                      # (KV head, map, head of the group)
                b = ((2 * g + n) * R + r) * hs.dp
                q.append((W[b:b + m.dim, :D], slice((2 * h + n) * m.dim, (2 * h + n + 1) * m.dim)))
        t = {p + "q": q,
             p + "k": [(W[k0 + h * hs.dp:k0 + h * hs.dp + m.dim, :D], a) for h, a in enumerate(_heads(m.dim, 2 * m.kv_heads))],
             p + "v": [(W[v0 + h * hs.vp:v0 + h * hs.vp + m.vdim, :D], a) for h, a in enumerate(_heads(m.vdim, m.kv_heads))],
             p + "g": [(W[hs.channels:hs.channels + m.heads, :D], _WHOLE)],
             p + "q.norm": [(self.q_norm[:m.dim], _WHOLE)], p + "k.norm": [(self.k_norm[:m.dim], _WHOLE)],
             p + "o": [(self.o.weight[:D, h * hs.vp:h * hs.vp + m.vdim], (_WHOLE, a)) for h, a in enumerate(_heads(m.vdim, m.heads))]}
        t.update({p + n: [(getattr(self, n), _WHOLE)] for n in ("lq1", "lk1", "lq2", "lk2")})
        return t

    def weights_loaded(self):
        m = self.m
        dot = lambda a, b: float((a.double() * b.double()).sum())
        lam = math.exp(dot(self.lq1, self.lk1)) - math.exp(dot(self.lq2, self.lk2)) + m.diff
        self.rule = ScoreRule(m.scale, diff=DiffRule(lam, 1.0 - m.diff, self.eps, m.vdim))

    def forward(self, xn, batch: ModelBatch, cache):
        m, hs = self.m, self.hs
        proj = self.proj(xn)
        q = lm.conv_heads(proj, hs, batch.seqs, batch.slot_mapping, cache[0], cache[1], q_norm=self.q_norm, k_norm=self.k_norm,
                          eps=self.eps, growth=m.growth)
        out = torch.empty(xn.shape[0], m.heads * hs.vp, dtype=xn.dtype, device=xn.device)
        window_attention(q, cache[0], cache[1], batch.seqs, self.rule, out, gate=proj[:, hs.channels:hs.channels + m.heads])
        return self.o(out)


class _Gated(nn.Module):
    """down(silu(gate x) * (up x)); with ``extra`` one more row of the first product, whose result is returned beside it."""

    def __init__(self, cfg: MilivikConfig, ff: int, dtype, device, extra: bool = False):
        super().__init__()
        self.ff, self.ff_p, self.extra = ff, round_up(ff, 8), extra
        self.up = _linear(cfg.hidden_size, 2 * self.ff_p + (1 if extra else 0), dtype, device)
        self.down = _linear(self.ff_p, cfg.hidden_size, dtype, device)

    def targets(self, p: str, D: int) -> dict:
        W = self.up.weight
        t = {p + "gate": [(W[:self.ff, :D], _WHOLE)], p + "up": [(W[self.ff_p:self.ff_p + self.ff, :D], _WHOLE)],
             p + "down": [(self.down.weight[:D, :self.ff], _WHOLE)]}
        if self.extra:
            t[p + "sg"] = [(W[2 * self.ff_p:2 * self.ff_p + 1, :D], _WHOLE)]
        return t

    def forward(self, xn):
        z = self.up(xn)
        y = self.down(fused.silu_mul(z[:, :2 * self.ff_p]))
        return (y, z[:, 2 * self.ff_p]) if self.extra else y


class _Experts(nn.Module):
    def __init__(self, cfg: MilivikConfig, m: ExpertsConfig, dtype, device):
        super().__init__()
        self.m = m
        D, E, self.ff_p = cfg.padded_width, m.router.experts, round_up(m.ff, 8)
        self.router = _zeros(round_up(E, 8), D, dtype=dtype, device=device)
        self.up = _zeros(E, 2 * self.ff_p, D, dtype=dtype, device=device)
        self.down = _zeros(E, D, self.ff_p, dtype=dtype, device=device)
        self.shared = _Gated(cfg, m.shared_ff, dtype, device, extra=True) if m.shared_ff else None
        self.ws = moe.MoEWorkspace()

    def targets(self, p: str, D: int) -> dict:
        m = self.m
        t = {p + "router": [(self.router[:m.router.experts, :D], _WHOLE)]}
        for e in range(m.router.experts):
            t[f"{p}e{e}.gate"] = [(self.up[e, :m.ff, :D], _WHOLE)]
            t[f"{p}e{e}.up"] = [(self.up[e, self.ff_p:self.ff_p + m.ff, :D], _WHOLE)]
            t[f"{p}e{e}.down"] = [(self.down[e, :D, :m.ff], _WHOLE)]
        if self.shared is not None:
            t.update(self.shared.targets(p + "shared.", D))
        return t

    def forward(self, xn):
        """(rows of the chosen experts with their weights, shared expert's rows, their gate logits)."""
        shared, gate = self.shared(xn) if self.shared is not None else (None, None)
        return moe.expert_rows(xn, self.router, None, self.m.router, self.up, self.down, act="swiglu", ws=self.ws), shared, gate


class MilivikLayer(nn.Module):
    def __init__(self, cfg: MilivikConfig, lc: LayerConfig, dtype, device):
        super().__init__()
        D, Dp = cfg.hidden_size, cfg.padded_width
        self.norm1 = _Gain(D, Dp, device)
        self.mix = (_Latent if isinstance(lc.mixer, LatentMixer) else _Diff)(cfg, lc.mixer, dtype, device)
        self.norm2 = _Gain(D, Dp, device) if lc.mlp is not None else None
        self.mlp = None
        if isinstance(lc.mlp, DenseConfig):
            self.mlp = _Gated(cfg, lc.mlp.ff, dtype, device)
        elif lc.mlp is not None:
            self.mlp = _Experts(cfg, lc.mlp, dtype, device)

    def targets(self, p: str, D: int) -> dict:
        t = {**self.norm1.targets(p + "norm1"), **self.mix.targets(p + "mix.", D)}
        if self.mlp is not None:
            t.update(self.norm2.targets(p + "norm2"))
            t.update(self.mlp.targets(p + "mlp.", D))
        return t


class MilivikDecoder(PackedDecoder):
    def __init__(self, cfg: MilivikConfig, dtype=torch.bfloat16, device=None):
        super().__init__()
        self.cfg, self.dtype_ = cfg, dtype
        # also the output projection, hence whole rows of eight
        self.embed_tokens = _zeros(round_up(cfg.vocab_size, 8), cfg.padded_width, dtype=dtype, device=device)
        self.layers = nn.ModuleList([MilivikLayer(cfg, l, dtype, device) for l in cfg.layers])
        self.final_norm = _Gain(cfg.hidden_size, cfg.padded_width, device)

    # ------------------------------------------------------------------ forward
    def forward(self, batch: ModelBatch, kv_caches, capture_layers=(), deepstack=None):
        """Returns (rows after the final norm [T, padded width], {i: fp32 stream after layer i - 1})."""
        cfg = self.cfg
        D, eps = cfg.hidden_size, cfg.norm_eps
        overlay = batch.input_embeds
        if overlay is not None:
            overlay = overlay.to(self.dtype_)
            if overlay.shape[1] < cfg.padded_width:
                overlay = F.pad(overlay, (0, cfg.padded_width - overlay.shape[1]))
        final = stream.RmsRows(self.final_norm.gain, eps, D)
        x, xn = stream.embed_rows(batch.input_ids, self.embed_tokens, stream.CAST if len(self.layers) else final, overlay=overlay,
                                  overlay_mask=batch.embeds_mask if overlay is not None else None, mult=cfg.embed_scale)
        captured = {0: x.clone()} if 0 in capture_layers else {}
        turns: dict = {}
        for li, (lc, layer) in enumerate(zip(cfg.layers, self.layers)):
            after = stream.CAST if li + 1 < len(self.layers) else final
            m = lc.mixer
            if isinstance(m, LatentMixer):
                key = (m.rot_base, m.shape.rot, m.yarn)
                if key not in turns:
                    turns[key] = stream.rotary_rows(batch.positions, *key)
                y = layer.mix(xn, batch, kv_caches[li], turns[key], eps)
            else:
                y = layer.mix(xn, batch, kv_caches[li])
            norm = dict(gain=layer.norm1.gain, eps=eps, n=D)
            stream.add_branch_(x, y, 1.0, xn, after if layer.mlp is None else stream.CAST, **norm)
            if layer.mlp is not None:
                norm["gain"] = layer.norm2.gain
                if isinstance(layer.mlp, _Experts):
                    rows, shared, gate = layer.mlp(xn)
                    stream.add_expert_rows_(x, rows, shared, 1.0, xn, after, shared_gate=gate, **norm)
                else:
                    stream.add_branch_(x, layer.mlp(xn), 1.0, xn, after, **norm)
            if (li + 1) in capture_layers:
                captured[li + 1] = x.clone()
        return xn, captured

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits [rows, vocab]."""
        return lm.logit_softcap(gemm.linear(hidden, self.embed_tokens), None, self.cfg.vocab_size, self.cfg.logit_scale)

    # ------------------------------------------------------------------ weights
    def targets(self) -> dict:
        D = self.cfg.hidden_size
        t = {"embed": [(self.embed_tokens[:self.cfg.vocab_size, :D], _WHOLE)], **self.final_norm.targets("final.norm")}
        for i, layer in enumerate(self.layers):
            t.update(layer.targets(f"l{i}.", D))
        return t

    def weights_loaded(self) -> None:
        for m in self.modules():
            if isinstance(m, (_Gain, _Latent, _Diff)):
                m.weights_loaded()

    def random_weights(self, seed: int | None = None):
        """(name, tensor) pairs of a random checkpoint (runs without weights)."""
        dev = self.embed_tokens.device
        g = torch.Generator(device=dev).manual_seed(torch.initial_seed() if seed is None else seed)
        rnd = lambda s: torch.randn(s, generator=g, device=dev)
        for name, shape in self.cfg.tensor_shapes().items():
            last = name.split(".")[-1]
            if last in ("norm1", "norm2") or name == "final.norm":
                w = 0.1 * rnd(shape)
            elif last == "norm":
                w = torch.ones(shape, device=dev)
            elif last in ("lq1", "lk1", "lq2", "lk2"):
                w = 0.1 * rnd(shape)
            else:
                w = rnd(shape) * shape[-1] ** -0.5
            yield name, w
