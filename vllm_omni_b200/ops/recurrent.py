"""Gated linear recurrence over a mixed batch (prompt portions and single decoded tokens): a causal convolution per
channel, block-diagonal gates on its result, the scan S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with
ln a_t = decay r_t, and the product with a gelu branch.  Convolution history and state live in the runner's pools.

Kernels: csrc/short_conv.cu and csrc/gated_scan_sm100.cu (tcgen05, portions of two tokens and more), csrc/gated_scan.cu (single tokens on
tensor cores; and plain kernels for fp32 and block sizes the tensor-core kernels do not take)."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _native as nv
from . import gemm
from .short_conv import conv_rows

c_int, c_long, c_float, c_void_p = ctypes.c_int, ctypes.c_long, ctypes.c_float, ctypes.c_void_p


@dataclass(frozen=True)
class GatedScanShape:
    width: int
    blocks: int              # equal parts of the width that the gates mix within
    taps: int                # convolution taps, the last one is the current token's

    @property
    def part(self) -> int:
        return self.width // self.blocks

    @property
    def part_p(self) -> int:             # channels of a part, padded with zeros
        return (self.part + 15) // 16 * 16

    @property
    def channels(self) -> int:
        return self.blocks * self.part_p


class _Scan(ctypes.Structure):
    _fields_ = [("proj", c_void_p), ("ldp", c_long), ("T", c_int), ("C", c_int), ("blocks", c_int), ("part", c_int), ("taps", c_int),
                ("conv", c_void_p), ("conv_b", c_void_p), ("gates", c_void_p), ("gates_b", c_void_p), ("decay", c_void_p),
                ("row_seq", c_void_p), ("q_start", c_void_p), ("context", c_void_p), ("state_in", c_void_p), ("state_out", c_void_p),
                ("hist", c_void_p), ("state", c_void_p), ("num_state", c_int), ("num_seqs", c_int), ("seq_list", c_void_p),
                ("n_list", c_int), ("runs", c_void_p), ("n_runs", c_int), ("sums", c_void_p), ("u", c_void_p), ("z", c_void_p),
                ("out", c_void_p), ("status", c_void_p)]


_STREAMS = 4             # runs a block of the prompt kernel walks side by side


def run_length(lens, channel_tiles: int, sms: int = 148) -> int:
    """Tokens of a run for portions of ``lens`` tokens: fills the SMs evenly, 64 runs per portion at most."""
    most = max(lens)
    best, best_cost = None, None
    for n in range(64, 4096 + 1, 64):
        if n * 64 < most and n < 4096:
            continue
        runs = sum(-(-k // n) for k in lens)
        waves = -(-channel_tiles * -(-runs // _STREAMS) // sms)
        cost = waves * (min(n, -(-most // 64) * 64) + 64) * (1 if most <= n else 2)       # several runs: two passes
        if best_cost is None or cost < best_cost:
            best, best_cost = n, cost
        if n >= most:
            break
    return best if best * 64 >= most else -(-most // 4096) * 64


def gated_scan(proj, s: GatedScanShape, seqs, conv, conv_b, gates, gates_b, decay, hist, state, impl: str | None = None):
    """``proj`` [T, 2 C]: gelu branch before its activation | convolution input; ``conv`` fp32 [taps, C], ``conv_b``
    [C]; ``gates`` [2, blocks, part_p, part_p] ([out, in]; decay gate r, then input gate i), ``gates_b`` fp32 [2, C];
    ``decay`` fp32 [C] (<= 0); ``hist`` [rows, taps - 1, C] and ``state`` fp32 [rows, C], read at ``seqs.state_in``
    and written at ``seqs.state_out`` (distinct rows; < 0 = not written).  Returns [T, C].

    ``impl="plain"`` forces the plain kernels for every row."""
    T, C = proj.shape[0], s.channels
    out = torch.empty(T, C, dtype=proj.dtype, device=proj.device)
    if not proj.is_cuda:
        return _cpu(proj, s, seqs, conv, conv_b, gates, gates_b, decay, hist, state, out)
    assert proj.stride(1) == 1 and hist.is_contiguous() and state.is_contiguous() and gates.is_contiguous()
    assert state.dtype == torch.float32 and hist.dtype == proj.dtype and hist.shape[1:] == (s.taps - 1, C)
    a = _Scan()
    P = lambda t: 0 if t is None else t.data_ptr()
    a.proj, a.ldp, a.T, a.C, a.blocks, a.part, a.taps = P(proj), proj.stride(0), T, C, s.blocks, s.part_p, s.taps
    a.conv, a.conv_b, a.gates, a.gates_b, a.decay = P(conv), P(conv_b), P(gates), P(gates_b), P(decay)
    a.row_seq, a.q_start, a.context = P(seqs.row_seq), P(seqs.q_start), P(seqs.context)
    a.state_in, a.state_out, a.hist, a.state = P(seqs.state_in), P(seqs.state_out), P(hist), P(state)
    a.num_state, a.num_seqs, a.out, a.status = state.shape[0], seqs.n_seqs, P(out), P(nv.status_word(proj.device))
    bf = proj.dtype == torch.bfloat16
    lib = nv.lib("gated_scan")
    if impl == "plain" or not bf or s.part_p > 256:
        u = torch.empty(T, C, dtype=torch.float32, device=proj.device)
        z = torch.empty(2, T, C, dtype=torch.float32, device=proj.device)
        a.u, a.z = P(u), P(z)
        nv.check_rc(lib.omni_scan_conv(ctypes.byref(a), c_int(bf), nv.stream_ptr()), "omni_scan_conv")
        w, n = gates.float(), s.part_p
        for g in range(2):
            gemm.batched_f32(u[:, :n], w[g, 0], z[g], bias=gates_b[g], batch=s.blocks, a_stride=n, w_stride=n * n, c_stride=n,
                             bias_stride=n)
        nv.check_rc(lib.omni_scan_plain(ctypes.byref(a), c_int(bf), nv.stream_ptr()), "omni_scan_plain")
        return out
    if seqs.n_decode:
        a.seq_list, a.n_list = P(seqs.decode_list), seqs.n_decode
        nv.check_rc(lib.omni_scan_step(ctypes.byref(a), nv.stream_ptr()), "omni_scan_step")
    if seqs.n_decode < seqs.n_seqs:
        u = conv_rows(proj[:, C:], seqs, s.taps, C, conv, hist, bias=conv_b, skip_single=True)
        a.u = P(u)
        tiles = s.blocks * ((s.part_p + 127) // 128)
        runs, a.n_runs, several = seqs.time_runs(tiles, lambda lens: run_length(lens, tiles))
        a.runs = P(runs)
        sums = torch.empty(a.n_runs, 2, C, dtype=torch.float32, device=proj.device) if several else None
        a.sums = P(sums)
        nv.check_rc(nv.lib("gated_scan_sm100").omni_scan_runs(ctypes.byref(a), nv.stream_ptr()), "omni_scan_runs")
    return out


def _cpu(proj, s, seqs, conv, conv_b, gates, gates_b, decay, hist, state, out):
    C, h, taps = s.channels, s.taps - 1, s.taps
    f = proj.float()
    y, x = F.gelu(f[:, :C], approximate="tanh"), f[:, C:2 * C]
    for n in range(seqs.n_seqs):
        a, b, ctx = int(seqs.q_start[n]), int(seqs.q_start[n + 1]), int(seqs.context[n])
        sin, sout = int(seqs.state_in[n]), int(seqs.state_out[n])
        past = hist[sin].float().clone()
        past[:max(0, h - ctx)] = 0
        ext = torch.cat([past, x[a:b]])
        u = conv_b + sum(ext[j:j + b - a] * conv[j] for j in range(taps))
        z = torch.einsum("tbk,gbnk->gtbn", u.view(b - a, s.blocks, s.part_p), gates.float()).reshape(2, b - a, C)
        r, i = torch.sigmoid(z + gates_b[:, None])
        log_a = decay * r
        add = torch.sqrt(-torch.expm1(2 * log_a)) * i * u
        S = state[sin].clone() if ctx else torch.zeros(C)
        for t in range(b - a):
            S = torch.exp(log_a[t]) * S + add[t]
            out[a + t] = (S * y[a + t]).to(out.dtype)
        if sout >= 0:
            state[sout] = S
            if h:
                hist[sout] = ext[ext.shape[0] - h:].to(hist.dtype)
    return out
