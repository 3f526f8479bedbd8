"""Delta-rule recurrences over a mixed batch (prompt portions and single decoded tokens).  Every head keeps a matrix S
(key channels x value channels) per sequence, in fp32, that a token decays, corrects and writes to; two forms:

    gated      S <- g S,  u = b (v - S^T k),  S <- S + k u^T,  o = S^T q      one decay g and step size b per head and token;
               q and k unit vectors; q, k, v from a short causal convolution per channel and silu; o / rms(o) * gain * silu(gate)
    channel    S <- diag(w) S - (a * u) (u^T S) + k v^T,  o = S^T r, u the unit key     decay w and removal rate a per key
               channel; o / rms(o) * gain * sigmoid(gate)

Kernels: csrc/delta_rule.cu (token by token: decoded tokens in one launch; every row in the exact mode and for sizes the
others do not take), csrc/delta_chunks.cu (prompt portions in chunks of 32 tokens on tensor cores).  Convolution history
and state live in the runner's pools.  CPU tensors take a PyTorch restatement."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _native as nv
from .short_conv import conv_rows

c_int, c_long, c_float, c_void_p = ctypes.c_int, ctypes.c_long, ctypes.c_float, ctypes.c_void_p

MAX_DIM = 256            # key channels the chunked kernels take


@dataclass(frozen=True)
class DeltaShape:
    heads: int
    kv_heads: int             # query / key heads; head h uses head h // (heads / kv_heads) of them
    dim: int                  # query / key channels per head
    vdim: int                 # value channels per head
    taps: int = 1             # of the convolution; the last one is the current token's

    @property
    def dp(self) -> int:      # padded with zeros
        return (self.dim + 15) // 16 * 16

    @property
    def vp(self) -> int:
        return (self.vdim + 15) // 16 * 16

    @property
    def q_cols(self) -> int:
        return self.kv_heads * self.dp

    @property
    def v_cols(self) -> int:
        return self.heads * self.vp

    @property
    def channels(self) -> int:           # q, k and v
        return 2 * self.q_cols + self.v_cols


@dataclass
class GatedDelta:
    """Columns of the packed projection: q | k | v | gate [heads * vp] | b [heads] | a [heads]."""
    conv: torch.Tensor        # fp32 [taps, channels]
    rate: torch.Tensor        # fp32 [heads], <= 0: ln g = rate * softplus(a + dt_bias)
    dt_bias: torch.Tensor     # fp32 [heads]
    gain: torch.Tensor        # fp32 [vp], shared by the heads
    eps: float
    unit_eps: float = 1e-6

    channel = False


@dataclass
class ChannelDelta:
    """Columns of the packed projection: r | k | v | a | gate, heads * dp each (vdim = dim).  The logits of the decay are
    an operand of their own."""
    decay_bias: torch.Tensor      # fp32 [heads * dp]
    removal_bias: torch.Tensor    # fp32 [heads * dp]
    decay_scale: float            # <= 0: ln w = decay_scale * sigmoid(logit + decay_bias)
    gain: torch.Tensor            # fp32 [heads * vp]
    eps: float
    unit_eps: float = 1e-6

    channel = True


class _Delta(ctypes.Structure):
    _fields_ = [("proj", c_void_p), ("ldp", c_long), ("T", c_int), ("H", c_int), ("G", c_int), ("dp", c_int), ("vp", c_int),
                ("d", c_int), ("dv", c_int), ("taps", c_int), ("q_col", c_int), ("k_col", c_int), ("v_col", c_int), ("g_col", c_int),
                ("b_col", c_int), ("a_col", c_int), ("conv", c_void_p), ("rate", c_void_p), ("dt_bias", c_void_p), ("z", c_void_p),
                ("ldz", c_long), ("decay_bias", c_void_p), ("removal_bias", c_void_p), ("decay_scale", c_float), ("q_mul", c_float),
                ("eps", c_float), ("unit_eps", c_float), ("gain", c_void_p), ("gain_hs", c_long), ("row_seq", c_void_p),
                ("q_start", c_void_p), ("context", c_void_p), ("state_in", c_void_p), ("state_out", c_void_p), ("hist", c_void_p),
                ("state", c_void_p), ("num_state", c_int), ("num_seqs", c_int), ("seq_list", c_void_p), ("n_list", c_int),
                ("out", c_void_p), ("ldo", c_long), ("raw", c_void_p), ("chunks", c_void_p), ("n_chunks", c_int),
                ("long_list", c_void_p), ("n_long", c_int), ("u", c_void_p), ("ldu", c_long), ("mats", c_void_p), ("coef", c_void_p),
                ("tiles", c_void_p), ("status", c_void_p)]


def _chunk(s: DeltaShape, rule, proj) -> int:
    """Tokens the chunked kernels take at a time, 0 where they do not take this.  Decays per channel are undone within a
    chunk, so their product must stay in range; their operands fill shared memory."""
    if proj.dtype != torch.bfloat16 or s.dp > MAX_DIM:
        return 0
    if not rule.channel:
        return 32
    n = 32 if s.dp <= 128 else 16
    return n if -rule.decay_scale * n <= 40.0 else 0


def delta_rule(proj, s: DeltaShape, seqs, rule, state, out, *, hist=None, decay=None, impl: str | None = None):
    """``proj`` [T, columns of ``rule``]; ``state`` fp32 [rows, heads, dp, vp] and ``hist`` [rows, taps - 1, channels], read
    at ``seqs.state_in`` and written at ``seqs.state_out`` (distinct rows; < 0 = not written); ``decay`` [T, heads * dp]
    logits of a ``ChannelDelta``; ``out`` [T, heads * vp] (a column view is fine).

    ``impl="steps"`` forces the token-by-token kernel for every row."""
    T = proj.shape[0]
    if not proj.is_cuda:
        return _cpu(proj, s, seqs, rule, state, out, hist, decay)
    assert proj.stride(1) == 1 and out.stride(1) == 1 and out.shape == (T, s.v_cols) and out.dtype == proj.dtype
    assert state.is_contiguous() and state.dtype == torch.float32 and state.shape[1:] == (s.heads, s.dp, s.vp)
    a = _Delta()
    P = lambda t: 0 if t is None else t.data_ptr()
    a.proj, a.ldp, a.T, a.H, a.G, a.dp, a.vp, a.d, a.dv, a.taps = P(proj), proj.stride(0), T, s.heads, s.kv_heads, s.dp, s.vp, \
        s.dim, s.vdim, s.taps
    a.q_col, a.k_col, a.v_col = 0, s.q_cols, 2 * s.q_cols
    a.gain, a.eps, a.unit_eps, a.q_mul = P(rule.gain), rule.eps, rule.unit_eps, 1.0
    if rule.channel:
        assert s.dp == s.vp and s.heads == s.kv_heads and s.taps == 1 and decay.stride(1) == 1 and decay.shape[1] >= s.q_cols
        a.a_col, a.g_col, a.gain_hs = 3 * s.q_cols, 4 * s.q_cols, s.vp
        a.z, a.ldz, a.decay_bias, a.removal_bias, a.decay_scale = P(decay), decay.stride(0), P(rule.decay_bias), P(rule.removal_bias), \
            rule.decay_scale
    else:
        a.g_col, a.b_col, a.a_col = s.channels, s.channels + s.v_cols, s.channels + s.v_cols + s.heads
        a.conv, a.rate, a.dt_bias, a.q_mul = P(rule.conv), P(rule.rate), P(rule.dt_bias), s.dim ** -0.5
        assert s.taps == 1 or (hist.is_contiguous() and hist.shape[1:] == (s.taps - 1, s.channels) and hist.dtype == proj.dtype)
    a.row_seq, a.q_start, a.context = P(seqs.row_seq), P(seqs.q_start), P(seqs.context)
    a.state_in, a.state_out, a.hist, a.state = P(seqs.state_in), P(seqs.state_out), P(hist), P(state)
    a.num_state, a.num_seqs, a.out, a.ldo = state.shape[0], seqs.n_seqs, P(out), out.stride(0)
    a.status = P(nv.status_word(proj.device))
    bf, kind, st = c_int(proj.dtype == torch.bfloat16), c_int(rule.channel), nv.stream_ptr()
    lib = nv.lib("delta_rule")
    size = _chunk(s, rule, proj) if seqs.n_decode < seqs.n_seqs and impl != "steps" else 0
    chunked = size > 0
    wide = s.dp * s.vp > 16384                              # a head's state does not fit the registers of one block
    raw = torch.empty(T, s.v_cols, dtype=proj.dtype, device=proj.device) if chunked or wide else None
    a.raw = P(raw)
    finish = lambda: nv.check_rc(lib.omni_delta_finish(ctypes.byref(a), kind, bf, st), "omni_delta_finish")
    if chunked:
        chunks = seqs.chunks(size)
        a.chunks, a.n_chunks, a.long_list, a.n_long = P(chunks.table), chunks.n, P(chunks.seqs), chunks.n_seqs
        dev, n = proj.device, chunks.n * s.heads
        lower = 512 * (3 if size == 32 else 1)              # lower tiles of a chunk's matrix, high and low parts
        if rule.channel:
            mats, coef = torch.empty(n, 4 * lower, dtype=torch.bfloat16, device=dev), torch.empty(n, s.dp, device=dev)
            tiles = torch.empty(n, 8, size, s.dp + 8, dtype=torch.bfloat16, device=dev)
            a.tiles = P(tiles)
        else:
            mats, coef = torch.empty(n, 2 * lower, dtype=torch.bfloat16, device=dev), torch.empty(n, 4 * size + 4, device=dev)
            u = conv_rows(proj, seqs, s.taps, s.channels, rule.conv, hist, act="silu", skip_single=True)
            a.u, a.ldu = P(u), u.stride(0)
        a.mats, a.coef = P(mats), P(coef)
        nv.check_rc(nv.lib("delta_chunks").omni_delta_chunks(ctypes.byref(a), kind, c_int(size), st), "omni_delta_chunks")
        if not wide:
            finish()                                        # rows of single tokens are written over below
    if not chunked or seqs.n_decode:
        a.n_list = seqs.n_decode if chunked else seqs.n_seqs
        a.seq_list = P(seqs.decode_list) if chunked else 0  # none: every sequence
        nv.check_rc(lib.omni_delta_steps(ctypes.byref(a), kind, bf, c_int(wide), st), "omni_delta_steps")
    if wide:
        finish()
    return out


def _unit(x, eps):
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + eps)


def _cpu(proj, s, seqs, rule, state, out, hist, decay):
    H, G, dp, vp, h = s.heads, s.kv_heads, s.dp, s.vp, s.taps - 1
    f = proj.float()
    for n in range(seqs.n_seqs):
        a, b, ctx = int(seqs.q_start[n]), int(seqs.q_start[n + 1]), int(seqs.context[n])
        sin, sout, m = int(seqs.state_in[n]), int(seqs.state_out[n]), b - a
        x = f[a:b, :s.channels]
        if not rule.channel:
            past = hist[sin].float().clone() if h else x.new_zeros(0, s.channels)
            past[:max(0, h - ctx)] = 0
            ext = torch.cat([past, x])
            x = F.silu(sum(ext[j:j + m] * rule.conv[j] for j in range(s.taps)))
            if h and sout >= 0:
                hist[sout] = ext[ext.shape[0] - h:].to(hist.dtype)
        q, k = x[:, :s.q_cols].view(m, G, dp), x[:, s.q_cols:2 * s.q_cols].view(m, G, dp)
        v = x[:, 2 * s.q_cols:].reshape(m, H, vp)
        S = state[sin].clone() if ctx else torch.zeros(H, dp, vp)
        o = torch.empty(m, H, vp)
        if rule.channel:
            rest = f[a:b, s.channels:].view(m, -1, H, dp)
            kill = torch.sigmoid(rest[:, 0] + rule.removal_bias.view(H, dp))
            w = torch.exp(rule.decay_scale * torch.sigmoid(decay[a:b, :H * dp].float() + rule.decay_bias).view(m, H, dp))
            u, gate = _unit(k, rule.unit_eps), torch.sigmoid(rest[:, 1])
            for t in range(m):
                seen = torch.einsum("hcv,hc->hv", S, u[t])
                S = w[t][:, :, None] * S - (kill[t] * u[t])[:, :, None] * seen[:, None] + k[t][:, :, None] * v[t][:, None]
                o[t] = torch.einsum("hcv,hc->hv", S, q[t])
        else:
            rest = f[a:b, s.channels:]
            gate = F.silu(rest[:, :H * vp]).view(m, H, vp)
            beta = torch.sigmoid(rest[:, H * vp:H * vp + H])
            g = torch.exp(rule.rate * F.softplus(rest[:, H * vp + H:H * vp + 2 * H] + rule.dt_bias, threshold=1e9))
            q = (_unit(q, rule.unit_eps) * s.dim ** -0.5).repeat_interleave(H // G, 1)
            k = _unit(k, rule.unit_eps).repeat_interleave(H // G, 1)
            for t in range(m):
                S = g[t][:, None, None] * S
                u = beta[t][:, None] * (v[t] - torch.einsum("hcv,hc->hv", S, k[t]))
                S = S + k[t][:, :, None] * u[:, None]
                o[t] = torch.einsum("hcv,hc->hv", S, q[t])
        o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / s.vdim + rule.eps)
        gain = rule.gain.view(H, vp) if rule.channel else rule.gain
        out[a:b] = (o * gain * gate).reshape(m, -1).to(out.dtype)
        if sout >= 0:
            state[sout] = S
    return out
