"""Row-wise steps of decoders with an fp32 residual stream (csrc/lm_ops.cu), for bf16 or fp32
activations.  Gains are fp32 tensors: one element (the same number for every channel) or one per
channel.  Rows may be padded to a multiple of 8 channels (``n`` is the real width); padding channels
stay zero.  CPU tensors take a PyTorch restatement of the same step."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _native as nv

c_int, c_long, c_float, c_void_p = ctypes.c_int, ctypes.c_long, ctypes.c_float, ctypes.c_void_p


def _rms(x, n, eps):
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / n + eps)


def _gs(g):
    return 0 if g.numel() == 1 else 1


def _bf(t):
    assert t.dtype in (torch.bfloat16, torch.float32)
    return c_int(1 if t.dtype == torch.bfloat16 else 0)


def embed_norm(ids, positions, embed, pos_table, gain, n: int, eps: float, overlay=None, overlay_mask=None):
    """x = embed[ids] (+ pos_table[positions]) in fp32 and xn = rms(x) * gain in the table's dtype.
    ``overlay`` [T, D] replaces the embedding row where ``overlay_mask`` (all rows without one)."""
    T, Dp = ids.shape[0], embed.shape[1]
    if not embed.is_cuda:
        x = embed[ids.long().clamp(0, embed.shape[0] - 1)].float()
        if overlay is not None:
            o = overlay.float()
            x = o if overlay_mask is None else torch.where(overlay_mask[:, None], o, x)
        if pos_table is not None:
            x = x + pos_table[positions.long().clamp(0, pos_table.shape[0] - 1)].float()
        return x, (_rms(x, n, eps) * gain).to(embed.dtype)
    x = torch.empty(T, Dp, dtype=torch.float32, device=embed.device)
    xn = torch.empty(T, Dp, dtype=embed.dtype, device=embed.device)
    assert ids.dtype == torch.int64 and ids.is_contiguous() and embed.is_contiguous()
    if pos_table is not None:
        assert positions.dtype == torch.int64 and positions.is_contiguous() and pos_table.stride(0) == embed.stride(0)
    if overlay is not None:
        assert overlay.dtype == embed.dtype and overlay.is_contiguous() and overlay.shape == (T, Dp)
    rc = nv.lib("lm_ops").omni_embed_norm(
        nv.ptr(ids), nv.ptr(positions if pos_table is not None else None), nv.ptr(embed), c_int(embed.shape[0]),
        nv.ptr(pos_table), c_int(0 if pos_table is None else pos_table.shape[0]), nv.ptr(overlay), nv.ptr(overlay_mask),
        nv.ptr(x), nv.ptr(xn), nv.ptr(gain), c_int(_gs(gain)), c_int(T), c_int(n), c_int(Dp), c_int(embed.stride(0)),
        c_float(eps), _bf(embed), nv.stream_ptr())
    nv.check_rc(rc, "omni_embed_norm")
    return x, xn


def add_norm_(x, y, gain_y, n: int, eps: float, xn=None, gain_n=None):
    """x (fp32, in place) += rms(y) * gain_y; then xn = rms(x) * gain_n when ``xn`` is given."""
    if not x.is_cuda:
        x += _rms(y[:, :x.shape[1]].float(), n, eps) * gain_y
        if xn is not None:
            xn.copy_(_rms(x, n, eps) * gain_n)
        return x
    assert x.dtype == torch.float32 and x.is_contiguous() and y.stride(-1) == 1 and y.shape[1] >= x.shape[1]
    assert xn is None or (xn.is_contiguous() and xn.shape == x.shape and xn.dtype == y.dtype)
    rc = nv.lib("lm_ops").omni_add_norm(
        nv.ptr(x), nv.ptr(y), c_int(y.stride(0)), nv.ptr(gain_y), c_int(_gs(gain_y)), nv.ptr(xn), nv.ptr(gain_n),
        c_int(0 if gain_n is None else _gs(gain_n)), c_int(x.shape[0]), c_int(n), c_int(x.shape[1]), c_float(eps), _bf(y),
        nv.stream_ptr())
    nv.check_rc(rc, "omni_add_norm")
    return x


def poly_norm(z, coef, n: int, eps: float, out=None):
    """c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3 with N(u) = u / sqrt(mean(u^2) + eps) over each row."""
    if out is None:
        out = torch.empty_like(z)
    if not z.is_cuda:
        f = z.float()
        out.copy_(coef[0] * _rms(f, n, eps) + coef[1] * _rms(f * f, n, eps) + coef[2] * _rms(f * f * f, n, eps) + coef[3])
        return out
    assert z.stride(1) == 1 and out.stride(1) == 1 and out.dtype == z.dtype and coef.dtype == torch.float32
    rc = nv.lib("lm_ops").omni_poly_norm(nv.ptr(z), c_int(z.stride(0)), nv.ptr(out), c_int(out.stride(0)), nv.ptr(coef),
                                         c_int(z.shape[0]), c_int(n), c_int(z.shape[1]), c_float(eps), _bf(z),
                                         nv.stream_ptr())
    nv.check_rc(rc, "omni_poly_norm")
    return out


def tanh_cols(x):
    """tanh of a column view [T, n] (n a multiple of 8), packed."""
    if not x.is_cuda:
        return torch.tanh(x.float()).to(x.dtype)
    assert x.stride(1) == 1
    out = torch.empty(x.shape[0], x.shape[1], dtype=x.dtype, device=x.device)
    nv.check_rc(nv.lib("lm_ops").omni_tanh_cols(nv.ptr(x), c_long(x.stride(0)), nv.ptr(out), c_long(x.shape[0]), c_int(x.shape[1]), _bf(x),
                                                nv.stream_ptr()), "omni_tanh_cols")
    return out


def logit_softcap(logits, cap: float | None, n: int, mult: float = 1.0):
    """``mult`` times the first ``n`` columns of ``logits`` as fp32, bounded to cap * tanh(. / cap) when ``cap`` is set."""
    if not logits.is_cuda:
        f = mult * logits[:, :n].float()
        return f if not cap else cap * torch.tanh(f / cap)
    out = torch.empty(logits.shape[0], n, dtype=torch.float32, device=logits.device)
    rc = nv.lib("lm_ops").omni_logit_softcap(nv.ptr(logits), c_long(logits.stride(0)), nv.ptr(out), c_long(n),
                                             c_long(logits.shape[0]), c_int(n), c_float(cap or 0.0), c_float(mult), _bf(logits),
                                             nv.stream_ptr())
    nv.check_rc(rc, "omni_logit_softcap")
    return out


# ------------------------------------------------------------------ conv + head norms + pages
class _ConvHeads(ctypes.Structure):
    _fields_ = [("proj", c_void_p), ("ldp", c_long), ("T", c_int), ("H", c_int), ("G", c_int), ("dp", c_int),
                ("vp", c_int), ("d", c_int), ("taps", c_int), ("conv", c_void_p), ("q_norm", c_void_p),
                ("k_norm", c_void_p), ("eps", c_float), ("row_seq", c_void_p), ("q_start", c_void_p),
                ("context", c_void_p), ("slots", c_void_p), ("state", c_void_p), ("state_in", c_void_p),
                ("state_out", c_void_p), ("q_out", c_void_p), ("k_cache", c_void_p), ("v_cache", c_void_p),
                ("v_first", c_void_p), ("v_mode", c_int), ("lam", c_void_p), ("num_slots", c_long),
                ("num_state", c_int), ("num_seqs", c_int), ("status", c_void_p), ("lph", c_int), ("GV", c_int),
                ("q_coef", c_float), ("q_every", c_float)]


@dataclass
class HeadShape:
    """Attention heads of one layer; ``dp`` / ``vp`` are ``dim`` / ``vdim`` padded to what the kernels take."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    dp: int
    vp: int
    taps: int = 0                     # convolution taps, 0 = no convolution
    v_heads: int = 0                  # value heads where they are fewer than key heads, 0 = kv_heads

    @property
    def values(self) -> int:
        return self.v_heads or self.kv_heads

    @property
    def channels(self) -> int:        # convolved channels: q, k and v
        return (self.heads + self.kv_heads) * self.dp + self.values * self.vp


@dataclass(frozen=True)
class QueryGrowth:
    """Queries at position p are multiplied by 1 + coef ln(floor((p + 1) / every) + 1)."""
    coef: float
    every: float


def conv_heads(proj, hs: HeadShape, seqs, slots, k_cache, v_cache, *, conv=None, state=None, q_norm=None, k_norm=None,
               eps: float = 1e-6, v_first=None, v_mode: str = "plain", lam=None, growth: QueryGrowth | None = None):
    """One pass over the packed projection ``proj`` [T, >= channels] (columns q | k | v): causal convolution
    over time per channel, RMS norm of every q and k head, ``growth`` of q, value mixing, K/V to their pages,
    convolution history to the state pool.  Returns q [T, H, dp].

    ``conv``: fp32 [taps, channels]; ``state``: [rows, taps - 1, channels], read at ``seqs.state_in`` and
    written at ``seqs.state_out`` (distinct rows; < 0 = not written).  ``v_mode``: "plain", "save" (the
    values are also stored in ``v_first`` [T, G * vp]) or "mix" (v <- (1 - lam) v + lam v_first)."""
    T = proj.shape[0]
    H, G, dp, vp = hs.heads, hs.kv_heads, hs.dp, hs.vp
    taps = conv.shape[0] if conv is not None else 1
    q_out = torch.empty(T, H, dp, dtype=proj.dtype, device=proj.device)
    if not proj.is_cuda:
        return _conv_heads_cpu(proj, hs, seqs, slots, k_cache, v_cache, conv, state, q_norm, k_norm, eps, v_first, v_mode,
                               lam, q_out, taps, growth)
    assert proj.stride(1) == 1 and slots.dtype == torch.int32 and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert k_cache.shape[2:].numel() == G * dp and v_cache.shape[2:] == (hs.values, vp) and k_cache.dtype == proj.dtype
    a = _ConvHeads()
    P = lambda t: 0 if t is None else t.data_ptr()
    a.proj, a.ldp, a.T, a.H, a.G, a.dp, a.vp, a.d, a.taps = P(proj), proj.stride(0), T, H, G, dp, vp, hs.dim, taps
    a.conv, a.q_norm, a.k_norm, a.eps = P(conv), P(q_norm), P(k_norm), eps
    a.row_seq, a.q_start, a.context, a.slots = P(seqs.row_seq), P(seqs.q_start), P(seqs.context), P(slots)
    if taps > 1:
        assert state is not None and state.is_contiguous() and state.shape[1:] == (taps - 1, hs.channels)
        a.state, a.state_in, a.state_out, a.num_state = P(state), P(seqs.state_in), P(seqs.state_out), state.shape[0]
    a.q_out, a.k_cache, a.v_cache = P(q_out), P(k_cache), P(v_cache)
    a.v_first, a.v_mode, a.lam = P(v_first), {"plain": 0, "save": 1, "mix": 2}[v_mode], P(lam)
    a.num_slots, a.num_seqs, a.GV = k_cache.shape[0] * k_cache.shape[1], seqs.n_seqs, hs.values
    if growth is not None:
        a.q_coef, a.q_every = growth.coef, growth.every
    a.status = P(nv.status_word(proj.device))
    nv.check_rc(nv.lib("lm_ops").omni_conv_heads(ctypes.byref(a), _bf(proj), nv.stream_ptr()), "omni_conv_heads")
    return q_out


class _RotaryHeads(ctypes.Structure):
    _fields_ = [("proj", c_void_p), ("ldp", c_long), ("T", c_int), ("H", c_int), ("G", c_int), ("dp", c_int), ("vp", c_int),
                ("rot", c_int), ("turns", c_void_p), ("q_gain", c_void_p), ("k_gain", c_void_p), ("nq", c_int), ("nk", c_int),
                ("vdim", c_int), ("v_norm", c_int), ("v_mult", c_float), ("eps", c_float), ("slots", c_void_p), ("q_out", c_void_p),
                ("k_cache", c_void_p), ("v_cache", c_void_p), ("num_slots", c_long), ("status", c_void_p)]


def rotary_heads(proj, hs: HeadShape, slots, k_cache, v_cache, turns, rot: int, *, q_gain=None, k_gain=None, v_norm: bool = False,
                 v_mult: float = 1.0, eps: float = 1e-6):
    """One pass over the packed projection ``proj`` [T, >= channels] (columns q | k | v): where gains are given, RMS norm of
    the whole query row and of the whole key row (all heads' channels at once); rotation of the first ``rot`` channels of
    every q and k head in interleaved pairs; with ``v_norm`` every value head over its root mean square, times
    ``v_mult``; K/V to their pages.  Returns q [T, H, dp].

    ``turns``: fp32 [T, rot / 2, 2] (ops/stream.py rotary_rows); ``q_gain`` fp32 [H * dp], ``k_gain`` [G * dp]."""
    T, H, G, dp, vp = proj.shape[0], hs.heads, hs.kv_heads, hs.dp, hs.vp
    q_out = torch.empty(T, H, dp, dtype=proj.dtype, device=proj.device)
    if not proj.is_cuda:
        f = proj.float()
        q, k, v = f[:, :H * dp], f[:, H * dp:(H + G) * dp], f[:, (H + G) * dp:hs.channels].reshape(T, G, vp)
        if q_gain is not None:
            q = _rms(q, H * hs.dim, eps) * q_gain
        if k_gain is not None:
            k = _rms(k, G * hs.dim, eps) * k_gain
        if v_norm:
            v = _rms(v, hs.vdim, eps)
        if rot:
            c, s = turns[:, None, :, 0], turns[:, None, :, 1]

            def turn(x):
                x = x.clone()
                a, b = x[..., 0:rot:2].clone(), x[..., 1:rot:2].clone()
                x[..., 0:rot:2], x[..., 1:rot:2] = a * c - b * s, b * c + a * s
                return x
            q, k = turn(q.reshape(T, H, dp)), turn(k.reshape(T, G, dp))
        q_out.copy_(q.reshape(T, H, dp))
        ok = slots >= 0
        where = slots[ok].long()
        k_cache.view(-1, G * dp)[where] = k.reshape(T, -1)[ok].to(k_cache.dtype)
        v_cache.view(-1, G * vp)[where] = (v_mult * v).reshape(T, -1)[ok].to(v_cache.dtype)
        return q_out
    assert proj.stride(1) == 1 and slots.dtype == torch.int32 and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert k_cache.shape[2:] == (G, dp) and v_cache.shape[2:] == (G, vp) and k_cache.dtype == proj.dtype and rot % 2 == 0
    assert not rot or (turns.is_contiguous() and turns.shape == (T, rot // 2, 2))
    a = _RotaryHeads()
    P = lambda t: 0 if t is None else t.data_ptr()
    a.proj, a.ldp, a.T, a.H, a.G, a.dp, a.vp, a.rot, a.turns = P(proj), proj.stride(0), T, H, G, dp, vp, rot, P(turns) if rot else 0
    a.q_gain, a.k_gain, a.nq, a.nk, a.vdim = P(q_gain), P(k_gain), H * hs.dim, G * hs.dim, hs.vdim
    a.v_norm, a.v_mult, a.eps, a.slots, a.q_out = int(v_norm), v_mult, eps, P(slots), P(q_out)
    a.k_cache, a.v_cache, a.num_slots = P(k_cache), P(v_cache), k_cache.shape[0] * k_cache.shape[1]
    a.status = P(nv.status_word(proj.device))
    nv.check_rc(nv.lib("lm_ops").omni_rotary_heads(ctypes.byref(a), _bf(proj), nv.stream_ptr()), "omni_rotary_heads")
    return q_out


def _conv_heads_cpu(proj, hs, seqs, slots, k_cache, v_cache, conv, state, q_norm, k_norm, eps, v_first, v_mode, lam,
                    q_out, taps, growth):
    H, G, dp, vp, C = hs.heads, hs.kv_heads, hs.dp, hs.vp, hs.channels
    T, hist = proj.shape[0], taps - 1
    u = proj[:, :C].float()
    y = torch.empty_like(u)
    for s in range(seqs.n_seqs):
        a, b, ctx = int(seqs.q_start[s]), int(seqs.q_start[s + 1]), int(seqs.context[s])
        if conv is None:
            y[a:b] = u[a:b]
            continue
        past = torch.zeros(hist, C)
        if hist:
            past.copy_(state[int(seqs.state_in[s])])
            past[: max(0, hist - ctx)] = 0
        ext = torch.cat([past, u[a:b]])
        y[a:b] = sum(ext[j:j + b - a] * conv[j] for j in range(taps))
        if hist and int(seqs.state_out[s]) >= 0:
            state[int(seqs.state_out[s])] = ext[ext.shape[0] - hist:].to(state.dtype)
    q, k = y[:, :H * dp].view(T, H, dp), y[:, H * dp:(H + G) * dp].view(T, G, dp)
    v = y[:, (H + G) * dp:]
    if q_norm is not None:
        q = _rms(q, hs.dim, eps) * q_norm
    if k_norm is not None:
        k = _rms(k, hs.dim, eps) * k_norm
    if growth is not None:
        pos = torch.cat([torch.arange(int(c), int(c) + int(b - a)) for a, b, c in zip(seqs.q_start, seqs.q_start[1:], seqs.context)])
        q = q * (1 + growth.coef * torch.log(torch.floor((pos + 1).double() / growth.every) + 1)).float()[:, None, None]
    if v_mode == "save":
        v_first.copy_(v)
    elif v_mode == "mix":
        v = (1 - lam) * v + lam * v_first.float()
    q_out.copy_(q)
    ok = slots >= 0
    where = slots[ok].long()
    k_cache.view(-1, G * dp)[where] = k.reshape(T, -1)[ok].to(k_cache.dtype)
    v_cache.view(-1, hs.values * vp)[where] = v[ok].to(v_cache.dtype)
    return q_out
