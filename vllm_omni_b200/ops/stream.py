"""Steps on an fp32 residual stream that takes scaled branches (csrc/stream_ops.cu), for bf16 or fp32 activations:
``x += mult * branch`` fused with the rows the next GEMM reads.  What those rows are is an argument: ``None``
(nothing), ``CAST`` (the stream in the activations' type), a norm without statistics, w tanh(alpha x) + b (any
object with fp32 tensors ``alpha`` [1], ``w`` and ``b`` [D]), or an ``RmsRows`` norm.  Rows may be padded to a multiple of 8 channels
(``n`` is the real width) with zeros.  CPU tensors take a PyTorch restatement of the same step."""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _native as nv

c_int, c_long, c_float, c_void_p = ctypes.c_int, ctypes.c_long, ctypes.c_float, ctypes.c_void_p

CAST = "cast"
_EMBED, _ROW, _NORMED, _EXPERTS, _EXPERTS_NORMED = range(5)


@dataclass
class RmsRows:
    """x / sqrt(<x^2> + eps) * gain over the first ``n`` channels; ``gain``: fp32 [D]."""
    gain: torch.Tensor
    eps: float
    n: int


class _StreamStep(ctypes.Structure):
    _fields_ = [("x", c_void_p), ("rows", c_int), ("D", c_int), ("Dp", c_int), ("source", c_int), ("out_mode", c_int),
                ("mult", c_float), ("eps", c_float), ("y", c_void_p), ("ldy", c_long), ("y_rows", c_long), ("gain", c_void_p),
                ("row_of_pair", c_void_p), ("weights", c_void_p), ("k", c_int), ("shared", c_void_p), ("lds", c_long),
                ("ids", c_void_p), ("embed", c_void_p), ("vocab", c_int), ("overlay", c_void_p), ("overlay_mask", c_void_p),
                ("out", c_void_p), ("alpha", c_void_p), ("w", c_void_p), ("b", c_void_p), ("status", c_void_p), ("shared_gate", c_void_p),
                ("ldsg", c_long), ("out_eps", c_float)]


def _finish_cpu(x, out, rows):
    if rows is None:
        return
    if isinstance(rows, RmsRows):
        out.copy_(_rms(x, rows.n, rows.eps) * rows.gain)
    else:
        out.copy_(x if isinstance(rows, str) else rows.w * torch.tanh(rows.alpha * x) + rows.b)


def _rms(x, n, eps):
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / n + eps)


def _launch(x, source, out, rows, n=None, dtype=None, **kw):
    T, Dp = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous()
    a = _StreamStep()
    a.x, a.rows, a.D, a.Dp, a.source = x.data_ptr(), T, n or Dp, Dp, source
    for k, v in kw.items():
        setattr(a, k, v.data_ptr() if isinstance(v, torch.Tensor) else v)
    if rows is not None:
        assert out.is_contiguous() and out.shape == x.shape and out.dtype == dtype
        a.out, a.out_mode = out.data_ptr(), 1
        if isinstance(rows, RmsRows):
            assert n is None or n == rows.n
            a.out_mode, a.w, a.out_eps, a.D = 3, rows.gain.data_ptr(), rows.eps, rows.n
        elif not isinstance(rows, str):
            a.out_mode, a.alpha, a.w, a.b = 2, rows.alpha.data_ptr(), rows.w.data_ptr(), rows.b.data_ptr()
    a.status = nv.status_word(x.device).data_ptr()
    nv.check_rc(nv.lib("stream_ops").omni_stream_step(ctypes.byref(a), c_int(1 if dtype == torch.bfloat16 else 0),
                                                      nv.stream_ptr()), "omni_stream_step")


def embed_rows(ids, embed, rows, overlay=None, overlay_mask=None, mult: float = 1.0):
    """x = mult * embed[ids] in fp32 and what ``rows`` asks for in the table's type.  ``overlay`` [T, D] replaces the
    scaled embedding row where ``overlay_mask`` (all rows without one)."""
    T, Dp = ids.shape[0], embed.shape[1]
    x = torch.empty(T, Dp, dtype=torch.float32, device=embed.device)
    out = torch.empty(T, Dp, dtype=embed.dtype, device=embed.device)
    if not embed.is_cuda:
        x.copy_(embed[ids.long().clamp(0, embed.shape[0] - 1)])
        x *= mult
        if overlay is not None:
            x.copy_(overlay.float() if overlay_mask is None else torch.where(overlay_mask[:, None], overlay.float(), x))
        _finish_cpu(x, out, rows)
        return x, out
    assert ids.dtype == torch.int64 and ids.is_contiguous() and embed.is_contiguous()
    kw = {}
    if overlay is not None:
        assert overlay.dtype == embed.dtype and overlay.is_contiguous() and overlay.shape == (T, Dp)
        kw["overlay"] = overlay
        if overlay_mask is not None:
            kw["overlay_mask"] = overlay_mask
    _launch(x, _EMBED, out, rows, dtype=embed.dtype, ids=ids, embed=embed, vocab=embed.shape[0], mult=mult, **kw)
    return x, out


def add_branch_(x, y, mult: float, out, rows, *, gain=None, eps: float = 0.0, n: int | None = None):
    """x (fp32, in place) += mult * y, or mult * y / sqrt(<y^2> + eps) * gain with a ``gain`` [D]; ``rows`` -> ``out``."""
    if not x.is_cuda:
        b = y[:, :x.shape[1]].float()
        if gain is not None:
            b = _rms(b, n or b.shape[1], eps) * gain
        x += mult * b
        _finish_cpu(x, out, rows)
        return x
    assert y.stride(-1) == 1 and y.shape[1] >= x.shape[1]
    kw = {} if gain is None else dict(gain=gain, eps=eps)
    _launch(x, _ROW if gain is None else _NORMED, out, rows, n, y.dtype, y=y, ldy=y.stride(0), mult=mult, **kw)
    return x


def add_expert_rows_(x, er, shared, mult: float, out, rows, *, shared_gate=None, gain=None, eps: float = 0.0,
                     n: int | None = None):
    """x += mult * b for b = the sum over a token's chosen experts of weight * row, plus ``shared`` (times
    sigmoid(``shared_gate``) with logits [T], a column view is fine); with a ``gain`` [D], b / sqrt(<b^2> + eps) * gain
    instead of b.  ``er``: ops/moe.py ExpertRows."""
    T, k = er.weights.shape
    if not x.is_cuda:
        y = er.y.float()
        pick = y.view(T, k, -1) if er.row_of_pair is None else y[er.row_of_pair.long()].view(T, k, -1)
        b = (er.weights[:, :, None] * pick).sum(1)
        if shared is not None:
            b = b + (shared.float() if shared_gate is None else shared.float() * torch.sigmoid(shared_gate.float())[:, None])
        if gain is not None:
            b = _rms(b, n or b.shape[1], eps) * gain
        x += mult * b
        _finish_cpu(x, out, rows)
        return x
    assert er.y.stride(1) == 1 and er.weights.is_contiguous()
    kw = {}
    if er.row_of_pair is not None:
        kw["row_of_pair"] = er.row_of_pair
    if shared is not None:
        kw.update(shared=shared, lds=shared.stride(0))
        if shared_gate is not None:
            assert shared_gate.dtype == er.y.dtype
            kw.update(shared_gate=shared_gate, ldsg=shared_gate.stride(0))
    if gain is not None:
        kw.update(gain=gain, eps=eps)
    _launch(x, _EXPERTS if gain is None else _EXPERTS_NORMED, out, rows, n, er.y.dtype, y=er.y, ldy=er.y.stride(0), y_rows=er.y.shape[0], weights=er.weights,
            k=k, mult=mult, **kw)
    return x


@dataclass(frozen=True)
class Yarn:
    """Frequencies for contexts ``factor`` times the ``original`` length: pairs that turn more than ``fast`` times over that
    length keep theirs, pairs below ``slow`` turns are slowed by ``factor``, with a linear ramp between; cos and sin grow
    by 0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float

    @property
    def magnitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0

    def frequencies(self, f: torch.Tensor, base: float, dims: int) -> torch.Tensor:
        at = lambda turns: dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
        lo, hi = max(math.floor(at(self.fast)), 0), min(math.ceil(at(self.slow)), dims - 1)
        ramp = ((torch.arange(f.numel(), dtype=f.dtype) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / self.factor * ramp + f * (1.0 - ramp)


_freqs: dict = {}


def rotary_rows(positions, base: float | None, dims: int, yarn: Yarn | None = None):
    """fp32 [T, dims / 2, 2]: cos and sin of position * base^(-2 i / dims), with ``yarn``'s frequencies and magnitude where
    given; ``base`` None: no rotation."""
    half = dims // 2
    key = (base, dims, yarn, positions.device)
    f = _freqs.get(key)
    if f is None:
        f = torch.zeros(half, dtype=torch.float64)
        if base is not None:
            f = float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
            if yarn is not None:
                f = yarn.frequencies(f, float(base), dims)
        f = _freqs[key] = f.to(positions.device)
    T = positions.shape[0]
    mag = 1.0 if yarn is None else yarn.magnitude
    if not positions.is_cuda:
        a = positions.double()[:, None] * f
        return (mag * torch.stack([a.cos(), a.sin()], -1)).float()
    out = torch.empty(T, half, 2, dtype=torch.float32, device=positions.device)
    assert positions.dtype == torch.int64 and positions.is_contiguous()
    nv.check_rc(nv.lib("stream_ops").omni_rotary_rows(nv.ptr(positions), nv.ptr(f), c_float(mag), nv.ptr(out), c_int(T), c_int(half),
                                                      nv.stream_ptr()), "omni_rotary_rows")
    return out


def gelu_lookup_(z, table, ids, col: int, n: int):
    """z[:, :n] = gelu_tanh(z[:, :n]) * table[ids, col:col + n], in place."""
    if not z.is_cuda:
        e = table[ids.long().clamp(0, table.shape[0] - 1), col:col + n].float()
        z[:, :n] = (F.gelu(z[:, :n].float(), approximate="tanh") * e).to(z.dtype)
        return z
    assert z.stride(1) == 1 and table.stride(1) == 1 and z.dtype == table.dtype
    nv.check_rc(nv.lib("stream_ops").omni_gelu_lookup(
        nv.ptr(z), c_long(z.stride(0)), nv.ptr(table), c_long(table.stride(0)), nv.ptr(ids), c_int(table.shape[0]), c_int(col),
        c_int(n), c_int(z.shape[0]), c_int(1 if z.dtype == torch.bfloat16 else 0), nv.stream_ptr()), "omni_gelu_lookup")
    return z
