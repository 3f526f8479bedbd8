"""Steps on an fp32 residual stream that takes scaled branches (csrc/stream_ops.cu), for bf16 or fp32 activations:
``x += mult * branch`` fused with the rows the next GEMM reads.  What those rows are is an argument: ``None``
(nothing), ``CAST`` (the stream in the activations' type) or a norm without statistics, w tanh(alpha x) + b (any
object with fp32 tensors ``alpha`` [1], ``w`` and ``b`` [D]).  Rows may be padded to a multiple of 8 channels
(``n`` is the real width) with zeros.  CPU tensors take a PyTorch restatement of the same step."""
from __future__ import annotations

import ctypes

import torch
import torch.nn.functional as F

from . import _native as nv

c_int, c_long, c_float, c_void_p = ctypes.c_int, ctypes.c_long, ctypes.c_float, ctypes.c_void_p

CAST = "cast"
_EMBED, _ROW, _NORMED, _EXPERTS = range(4)


class _StreamStep(ctypes.Structure):
    _fields_ = [("x", c_void_p), ("rows", c_int), ("D", c_int), ("Dp", c_int), ("source", c_int), ("out_mode", c_int),
                ("mult", c_float), ("eps", c_float), ("y", c_void_p), ("ldy", c_long), ("y_rows", c_long), ("gain", c_void_p),
                ("row_of_pair", c_void_p), ("weights", c_void_p), ("k", c_int), ("shared", c_void_p), ("lds", c_long),
                ("ids", c_void_p), ("embed", c_void_p), ("vocab", c_int), ("overlay", c_void_p), ("overlay_mask", c_void_p),
                ("out", c_void_p), ("alpha", c_void_p), ("w", c_void_p), ("b", c_void_p), ("status", c_void_p)]


def _finish_cpu(x, out, rows):
    if rows is None:
        return
    out.copy_(x if isinstance(rows, str) else rows.w * torch.tanh(rows.alpha * x) + rows.b)


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
        if not isinstance(rows, str):
            a.out_mode, a.alpha, a.w, a.b = 2, rows.alpha.data_ptr(), rows.w.data_ptr(), rows.b.data_ptr()
    a.status = nv.status_word(x.device).data_ptr()
    nv.check_rc(nv.lib("stream_ops").omni_stream_step(ctypes.byref(a), c_int(1 if dtype == torch.bfloat16 else 0),
                                                      nv.stream_ptr()), "omni_stream_step")


def embed_rows(ids, embed, rows, overlay=None, overlay_mask=None):
    """x = embed[ids] in fp32 and what ``rows`` asks for in the table's type.  ``overlay`` [T, D] replaces the
    embedding row where ``overlay_mask`` (all rows without one)."""
    T, Dp = ids.shape[0], embed.shape[1]
    x = torch.empty(T, Dp, dtype=torch.float32, device=embed.device)
    out = torch.empty(T, Dp, dtype=embed.dtype, device=embed.device)
    if not embed.is_cuda:
        x.copy_(embed[ids.long().clamp(0, embed.shape[0] - 1)])
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
    _launch(x, _EMBED, out, rows, dtype=embed.dtype, ids=ids, embed=embed, vocab=embed.shape[0], **kw)
    return x, out


def add_branch_(x, y, mult: float, out, rows, *, gain=None, eps: float = 0.0, n: int | None = None):
    """x (fp32, in place) += mult * y, or mult * y / sqrt(<y^2> + eps) * gain with a ``gain`` [D]; ``rows`` -> ``out``."""
    if not x.is_cuda:
        b = y[:, :x.shape[1]].float()
        if gain is not None:
            b = b * torch.rsqrt(b.pow(2).sum(-1, keepdim=True) / (n or b.shape[1]) + eps) * gain
        x += mult * b
        _finish_cpu(x, out, rows)
        return x
    assert y.stride(-1) == 1 and y.shape[1] >= x.shape[1]
    kw = {} if gain is None else dict(gain=gain, eps=eps)
    _launch(x, _ROW if gain is None else _NORMED, out, rows, n, y.dtype, y=y, ldy=y.stride(0), mult=mult, **kw)
    return x


def add_expert_rows_(x, er, shared, mult: float, out, rows):
    """x += mult * (sum over a token's chosen experts of weight * row, plus ``shared``); ``er``: ops/moe.py ExpertRows."""
    T, k = er.weights.shape
    if not x.is_cuda:
        y = er.y.float()
        pick = y.view(T, k, -1) if er.row_of_pair is None else y[er.row_of_pair.long()].view(T, k, -1)
        b = (er.weights[:, :, None] * pick).sum(1)
        x += mult * (b if shared is None else b + shared.float())
        _finish_cpu(x, out, rows)
        return x
    assert er.y.stride(1) == 1 and er.weights.is_contiguous()
    kw = {}
    if er.row_of_pair is not None:
        kw["row_of_pair"] = er.row_of_pair
    if shared is not None:
        kw.update(shared=shared, lds=shared.stride(0))
    _launch(x, _EXPERTS, out, rows, None, er.y.dtype, y=er.y, ldy=er.y.stride(0), y_rows=er.y.shape[0], weights=er.weights,
            k=k, mult=mult, **kw)
    return x


_freqs: dict = {}


def rotary_rows(positions, base: float | None, dims: int):
    """fp32 [T, dims / 2, 2]: cos and sin of position * base^(-2 i / dims); ``base`` None: no rotation."""
    half = dims // 2
    key = (base, dims, positions.device)
    f = _freqs.get(key)
    if f is None:
        f = torch.zeros(half, dtype=torch.float64)
        if base is not None:
            f = float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
        f = _freqs[key] = f.to(positions.device)
    T = positions.shape[0]
    if not positions.is_cuda:
        a = positions.double()[:, None] * f
        return torch.stack([a.cos(), a.sin()], -1).float()
    out = torch.empty(T, half, 2, dtype=torch.float32, device=positions.device)
    assert positions.dtype == torch.int64 and positions.is_contiguous()
    nv.check_rc(nv.lib("stream_ops").omni_rotary_rows(nv.ptr(positions), nv.ptr(f), nv.ptr(out), c_int(T), c_int(half),
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
