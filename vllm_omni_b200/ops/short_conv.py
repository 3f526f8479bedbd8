"""Short causal convolution over time, per channel, of a mixed batch's rows (csrc/short_conv.cu, bf16): the rows before a
portion come from the history pool of its sequence."""
from __future__ import annotations

import ctypes

import torch

from . import _native as nv

c_int, c_long, c_void_p = ctypes.c_int, ctypes.c_long, ctypes.c_void_p
ACT = {None: 0, "silu": 1}


class _ConvRows(ctypes.Structure):
    _fields_ = [("x", c_void_p), ("ldx", c_long), ("T", c_int), ("C", c_int), ("taps", c_int), ("conv", c_void_p), ("bias", c_void_p),
                ("act", c_int), ("skip_single", c_int), ("row_seq", c_void_p), ("q_start", c_void_p), ("context", c_void_p),
                ("state_in", c_void_p), ("state_out", c_void_p), ("hist", c_void_p), ("num_state", c_int), ("num_seqs", c_int),
                ("out", c_void_p), ("status", c_void_p)]


def conv_rows(x, seqs, taps: int, channels: int, conv, hist, *, bias=None, act: str | None = None, skip_single: bool = False):
    """act(bias + sum_j conv[j] x_(t - taps + 1 + j)) of the first ``channels`` columns of ``x`` [T, >= channels]: bf16
    [T, channels].  ``conv`` fp32 [taps, channels]; ``hist`` [rows, taps - 1, channels], read at ``seqs.state_in`` and
    written at ``seqs.state_out`` (distinct rows).  ``skip_single``: sequences with one row are left to another kernel, their
    results here are not used and their history is not written."""
    T = x.shape[0]
    assert x.is_cuda and x.dtype == torch.bfloat16 and x.stride(1) == 1 and x.shape[1] >= channels
    assert taps == 1 or (hist.dtype == x.dtype and hist.is_contiguous() and hist.shape[1:] == (taps - 1, channels))
    out = torch.empty(T, channels, dtype=x.dtype, device=x.device)
    a = _ConvRows()
    P = lambda t: 0 if t is None else t.data_ptr()
    a.x, a.ldx, a.T, a.C, a.taps, a.conv, a.bias, a.act = P(x), x.stride(0), T, channels, taps, P(conv), P(bias), ACT[act]
    a.skip_single, a.row_seq, a.q_start, a.context = int(skip_single), P(seqs.row_seq), P(seqs.q_start), P(seqs.context)
    a.state_in, a.state_out, a.hist = P(seqs.state_in), P(seqs.state_out), P(hist) if taps > 1 else 0
    a.num_state, a.num_seqs, a.out, a.status = 0 if hist is None else hist.shape[0], seqs.n_seqs, P(out), P(nv.status_word(x.device))
    nv.check_rc(nv.lib("short_conv").omni_conv_rows(ctypes.byref(a), nv.stream_ptr()), "omni_conv_rows")
    return out
