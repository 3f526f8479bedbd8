"""Causal attention over a paged cache of latents, optionally with a sliding window: a token leaves one row (its normed
latent c and a rotated key part) that all heads share, head h has keys [W_uk[h] c, rotated part] and values W_uv[h] c.
The output gate has one logit per head or one per channel.

Two ways to the same sums.  Portions of more than ``SHORT`` tokens expand the latents of their sequence to keys and
values with one GEMM and run on the tcgen05 kernel (csrc/attn_window_sm100.cu).  Single tokens and short portions take
their queries to the latent space instead (W_uk[h]^T q) and attend to the latent rows themselves, so a row is read
once for all heads (csrc/latent_attn.cu).  fp32 and sizes the tensor-core kernels do not take use the second way on
the row-per-block kernel of csrc/attn_window.cu."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _native as nv
from . import gemm
from . import window_attention as WA

c_int, c_long, c_float, c_void_p = ctypes.c_int, ctypes.c_long, ctypes.c_float, ctypes.c_void_p

SHORT = 4                   # portions up to this many tokens attend in the latent space
MAX_KEYS = 1 << 16          # keys expanded at a time


def _up16(n: int) -> int:
    return (n + 15) // 16 * 16


@dataclass(frozen=True)
class LatentShape:
    heads: int
    dim: int                # unrotated query / key channels per head
    rot: int                # rotated ones (one key part for all heads)
    vdim: int
    rank: int               # channels of the latent

    @property
    def dim_p(self) -> int:
        return _up16(self.dim)

    @property
    def rot_p(self) -> int:
        return _up16(self.rot)

    @property
    def vdim_p(self) -> int:
        return _up16(self.vdim)

    @property
    def rank_p(self) -> int:
        return _up16(self.rank)

    @property
    def head_cols(self) -> int:         # a head's query channels in the packed projection
        return self.dim_p + self.rot_p

    @property
    def q_cols(self) -> int:
        return self.heads * self.head_cols

    @property
    def row(self) -> int:               # channels of a cached row
        return self.rank_p + self.rot_p


class _LatentRows(ctypes.Structure):
    _fields_ = [("q", c_void_p), ("ldq", c_long), ("T", c_int), ("H", c_int), ("dim_p", c_int), ("rot", c_int), ("rot_p", c_int),
                ("z", c_void_p), ("ldz", c_long), ("rank", c_int), ("rank_p", c_int), ("turns", c_void_p), ("slots", c_void_p),
                ("pages", c_void_p), ("num_slots", c_long), ("norm", c_void_p), ("eps", c_float), ("status", c_void_p),
                ("qc", c_void_p), ("ldqc", c_long), ("q_rank", c_int), ("q_rank_p", c_int), ("q_norm", c_void_p)]


class _HeadGemm(ctypes.Structure):
    _fields_ = [("A", c_void_p), ("a_row", c_long), ("a_head", c_long), ("a_rows", c_void_p), ("W", c_void_p), ("C", c_void_p),
                ("c_row", c_long), ("c_head", c_long), ("c_rows", c_void_p), ("gate", c_void_p), ("g_row", c_long), ("M", c_int),
                ("N", c_int), ("K", c_int), ("H", c_int), ("rows_a", c_int), ("rows_c", c_int), ("g_head", c_long), ("g_col", c_int)]


class _LatentDecode(ctypes.Structure):
    _fields_ = [("q_lat", c_void_p), ("proj", c_void_p), ("ldp", c_long), ("head_cols", c_int), ("dim_p", c_int),
                ("pages", c_void_p), ("rank_p", c_int), ("rot_p", c_int), ("block_tables", c_void_p), ("bt_stride", c_int),
                ("block_size", c_int), ("num_blocks", c_int), ("rows", c_void_p), ("n", c_int), ("row_seq", c_void_p),
                ("q_start", c_void_p), ("context", c_void_p), ("num_seqs", c_int), ("T", c_int), ("scale", c_float),
                ("out", c_void_p), ("H", c_int), ("splits", c_int), ("part_o", c_void_p), ("part_ml", c_void_p),
                ("status", c_void_p), ("window", c_int)]


def _P(t):
    return 0 if t is None else t.data_ptr()


# ------------------------------------------------------------------ rows and pages
def latent_rows(proj, s: LatentShape, turns, slots, pages, norm, eps: float):
    """Rotates the query heads of ``proj`` [T, q | latent | rotated key | ...] in place (``turns``: cos / sin rows of
    ops/stream.py rotary_rows); with ``norm`` (fp32 [rank_p]) also norms and rotates each token's latent row and writes
    it to its page slot (< 0: not written).  ``norm`` None: the layer reads another layer's pages."""
    _rows_step(s, turns, q=proj, z=None if norm is None else proj[:, s.q_cols:], slots=slots, pages=pages, norm=norm, eps=eps)


def rotate_queries(q, s: LatentShape, turns):
    """Rotates the query heads of ``q`` [T, >= q_cols] in place."""
    _rows_step(s, turns, q=q)


def cache_rows(z, s: LatentShape, turns, slots, pages, norm, eps: float, query_latent=None, query_norm=None, query_rank: int = 0):
    """Norms and rotates each token's latent row ``z`` [T, latent | rotated key | ...] and writes it to its page slot (< 0: not
    written); norms ``query_latent`` [T, n] (``query_rank`` of its channels are real) in place with ``query_norm`` (fp32 [n])."""
    _rows_step(s, turns, z=z, slots=slots, pages=pages, norm=norm, eps=eps, qc=query_latent, q_norm=query_norm, q_rank=query_rank)


def _rows_step(s, turns, q=None, z=None, slots=None, pages=None, norm=None, eps=0.0, qc=None, q_norm=None, q_rank=0):
    some = q if q is not None else z
    T = some.shape[0]
    if not some.is_cuda:
        if q is not None:
            part = q[:, :s.q_cols].view(T, s.heads, s.head_cols)[:, :, s.dim_p:s.dim_p + s.rot]
            part.copy_(_turn(part.float(), turns[:, None]))
        rms = lambda x, n: x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / n + eps)
        if qc is not None:
            qc.copy_(rms(qc.float(), q_rank) * q_norm)
        if z is not None:
            z = z[:, :s.row].float()
            row = torch.zeros(T, s.row)
            row[:, :s.rank] = rms(z[:, :s.rank], s.rank) * norm[:s.rank]
            row[:, s.rank_p:s.rank_p + s.rot] = _turn(z[:, s.rank_p:s.rank_p + s.rot], turns)
            ok = slots >= 0
            pages.view(-1, s.row)[slots[ok].long()] = row[ok].to(pages.dtype)
        return
    assert turns.is_contiguous() and turns.shape == (T, s.rot // 2, 2)
    a = _LatentRows()
    a.T, a.H, a.dim_p, a.rot, a.rot_p, a.rank, a.rank_p = T, s.heads, s.dim_p, s.rot, s.rot_p, s.rank, s.rank_p
    a.turns, a.eps, a.status = _P(turns), eps, _P(nv.status_word(some.device))
    if q is not None:
        assert q.stride(1) == 1
        a.q, a.ldq = _P(q), q.stride(0)
    if z is not None:
        assert z.stride(1) == 1 and slots.dtype == torch.int32 and pages.is_contiguous()
        assert pages.shape[2:] == (1, s.row) and pages.dtype == z.dtype
        a.z, a.ldz, a.slots, a.pages, a.norm = _P(z), z.stride(0), _P(slots), _P(pages), _P(norm)
        a.num_slots = pages.shape[0] * pages.shape[1]
    if qc is not None:
        assert qc.stride(1) == 1 and qc.dtype == some.dtype and q_norm.numel() == qc.shape[1]
        a.qc, a.ldqc, a.q_rank, a.q_rank_p, a.q_norm = _P(qc), qc.stride(0), q_rank, qc.shape[1], _P(q_norm)
    nv.check_rc(nv.lib("latent_attn").omni_latent_rows(ctypes.byref(a), c_int(1 if some.dtype == torch.bfloat16 else 0),
                                                       nv.stream_ptr()), "omni_latent_rows")


def _turn(x, turns):
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * turns[..., 0] - v * turns[..., 1], v * turns[..., 0] + u * turns[..., 1]], -1).flatten(-2)


# ------------------------------------------------------------------ attention
def latent_attention(proj, s: LatentShape, pages, seqs, uk_t, kv_up, scale: float, out, gate=None, impl: str | None = None,
                     window: int | None = None):
    """``proj`` [T, >= q_cols] with rotated queries (``latent_rows``); ``pages`` [num_blocks, block_size, 1, row] that
    already hold this step's tokens; ``seqs``: the batch's ``SeqTable``; ``uk_t`` [H, rank_p, dim_p]; ``kv_up``
    [H dim_p key rows | H vdim_p value rows, rank_p]; ``out`` [T, H vdim_p]; ``gate`` [T, H] or [T, H vdim_p] logits (a
    view is fine); ``window``: a row sees itself and the window - 1 positions before it.

    ``impl``: "latent" attends in the latent space for every row, "rows" also forces the row-per-block kernel."""
    if not proj.is_cuda:
        return _cpu(proj, s, pages, seqs, kv_up, scale, out, gate, window)
    assert proj.stride(1) == 1 and out.is_contiguous() and uk_t.is_contiguous() and kv_up.is_contiguous()
    bf = proj.dtype == torch.bfloat16
    if impl == "rows" or not bf or not nv.lib("latent_attn").omni_latent_decode_heads(s.heads, s.rank_p, s.rot_p):
        return _rows(proj, s, pages, seqs, uk_t, kv_up, scale, out, gate, window)
    short = 1 << 30 if impl == "latent" or not _expands(s) else SHORT
    rows, n, keys = seqs.short_rows(short)
    if n:
        _latent_space(proj, s, pages, seqs, uk_t, kv_up, scale, out, gate, rows, n, keys, window)
    if seqs.lens:
        for group in seqs.long_groups(short, MAX_KEYS, _rows_per_block(s), window):
            _expanded(proj, s, pages, seqs, kv_up, scale, out, gate, group, window)
    return out


def _boxes(s: LatentShape) -> int:
    return (s.dim_p + 63) // 64 + (s.rot_p + 63) // 64


def _expands(s: LatentShape) -> bool:
    """Do a head's keys and values fit the prompt kernel?"""
    return _boxes(s) <= 4 and s.vdim_p <= 128


def _rows_per_block(s: LatentShape) -> int:
    return 256 if _boxes(s) <= 3 else 128


def _expanded(proj, s, pages, seqs, kv_up, scale, out, gate, group, window=None):
    nb, bs = pages.shape[:2]
    rows = torch.empty(group.keys, s.row, dtype=proj.dtype, device=proj.device)
    nv.check_rc(nv.lib("latent_attn").omni_latent_gather(
        nv.ptr(pages), c_int(s.row * pages.element_size()), nv.ptr(seqs.block_tables), c_int(seqs.block_tables.stride(0)), c_int(bs),
        c_int(nb), nv.ptr(group.members), c_int(group.n_members), nv.ptr(group.key_start), nv.ptr(rows), c_long(group.keys), nv.stream_ptr()),
        "omni_latent_gather")
    expanded_attention(proj, s, rows, gemm.linear(rows[:, :s.rank_p], kv_up), seqs, scale, out, gate, group, window)


def expanded_attention(proj, s, rows, kv, seqs, scale, out, gate, group, window=None):
    """Attention of a group's portions over expanded keys and values ``kv`` [keys, H dim_p | H vdim_p]; the shared key
    parts are the last channels of ``rows`` [keys, row]."""
    nk = s.heads * s.dim_p
    a = WA._WinAttn()
    a.q, a.q_rs, a.k_cache, a.v_cache = _P(proj), proj.stride(0), _P(kv), _P(kv[:, nk:])
    a.block_tables, a.bt_stride = _P(seqs.block_tables), seqs.block_tables.stride(0)
    a.q_start, a.context, a.row_seq = _P(seqs.q_start), _P(seqs.context), _P(seqs.row_seq)
    a.items, a.n_items, a.block_tokens = _P(group.items), group.n_items, group.rows_per_block
    a.out, a.o_rs, a.window, a.maps = _P(out), out.stride(0), window or 0, 1
    a.set_gate(gate, s.heads)
    a.scale, a.T, a.H, a.G, a.dp, a.vp = scale, proj.shape[0], s.heads, s.heads, s.head_cols, s.vdim_p
    a.num_seqs, a.num_blocks, a.block_size, a.splits, a.status = seqs.n_seqs, 1, 32, 1, _P(nv.status_word(proj.device))
    a.k_ts = a.v_ts = kv.stride(0)
    a.dp_u, a.k_shared, a.ks_ts = s.dim_p, _P(rows[:, s.rank_p:]), rows.stride(0)
    a.key_start, a.key_rows = _P(group.key_start), group.keys
    nv.check_rc(nv.lib("attn_window_sm100").omni_attn_window_prefill(ctypes.byref(a), nv.stream_ptr()),
                "omni_attn_window_prefill")


def decode_splits(blocks: int, keys: int, sms: int = 148) -> int:
    """Blocks that share one row's keys: fills the SMs evenly, about 256 keys each at least."""
    best, best_cost = 1, None
    for n in range(1, max(1, min(64, (keys + 255) // 256)) + 1):
        waves = -(-blocks * n // sms)
        cost = waves * (-(-keys // (32 * n)) + 6)           # key tiles of a block and its start-up, per wave
        if best_cost is None or cost < best_cost:
            best, best_cost = n, cost
    return best


def head_gemm(a, a_row: int, a_head: int, w, c, c_row: int, c_head: int, M: int, H: int, *, a_rows=None, c_rows=None, gate=None):
    """c[m, h, :] = w[h] a[m, h, :] for bf16 operands at the given element strides, times sigmoid(gate[row of c, h]) or, with a
    gate of N logits per head, channel by channel."""
    p = _HeadGemm()
    N, K = w.shape[-2:]
    p.A, p.a_row, p.a_head, p.a_rows, p.W, p.C = _P(a), a_row, a_head, _P(a_rows), _P(w), _P(c)
    p.c_row, p.c_head, p.c_rows, p.gate, p.g_row = c_row, c_head, _P(c_rows), _P(gate), 0 if gate is None else gate.stride(0)
    p.M, p.N, p.K, p.H, p.rows_a, p.rows_c = M, N, K, H, a.shape[0], c.shape[0]
    if gate is not None:
        assert gate.stride(1) == 1 and gate.shape[1] in (H, H * N)
        p.g_head, p.g_col = gate.shape[1] // H, 0 if gate.shape[1] == H else 1
    nv.check_rc(nv.lib("latent_attn").omni_head_gemm(ctypes.byref(p), nv.stream_ptr()), "omni_head_gemm")


def _latent_space(proj, s, pages, seqs, uk_t, kv_up, scale, out, gate, rows, n, keys, window=None):
    H = s.heads
    q_lat = torch.empty(n, H, s.rank_p, dtype=proj.dtype, device=proj.device)
    head_gemm(proj, proj.stride(0), s.head_cols, uk_t, q_lat, H * s.rank_p, s.rank_p, n, H, a_rows=rows)
    o_lat = latent_decode(q_lat, proj, s, pages, seqs, rows, n, keys, scale, window)
    head_gemm(o_lat, H * s.rank_p, s.rank_p, kv_up[H * s.dim_p:].view(H, s.vdim_p, s.rank_p), out, out.stride(0), s.vdim_p, n, H,
              c_rows=rows, gate=gate)


def latent_decode(q_lat, proj, s, pages, seqs, rows, n, keys, scale, window=None):
    """Weighted sums of latent rows [n, H, rank_p] for ``n`` batch ``rows`` that see ``keys`` keys at most (of those, the last
    ``window``)."""
    keys = keys if window is None else min(keys, window)
    H, dev = s.heads, proj.device
    o_lat = torch.empty_like(q_lat)
    lib = nv.lib("latent_attn")
    hb = lib.omni_latent_decode_heads(H, s.rank_p, s.rot_p)
    a = _LatentDecode()
    a.q_lat, a.proj, a.ldp, a.head_cols, a.dim_p = _P(q_lat), _P(proj), proj.stride(0), s.head_cols, s.dim_p
    a.pages, a.rank_p, a.rot_p = _P(pages), s.rank_p, s.rot_p
    a.block_tables, a.bt_stride, a.block_size, a.num_blocks = _P(seqs.block_tables), seqs.block_tables.stride(0), pages.shape[1], \
        pages.shape[0]
    a.rows, a.n, a.row_seq, a.q_start, a.context = _P(rows), n, _P(seqs.row_seq), _P(seqs.q_start), _P(seqs.context)
    a.num_seqs, a.T, a.scale, a.out, a.H = seqs.n_seqs, proj.shape[0], scale, _P(o_lat), H
    a.window = window or 0
    a.splits, a.status = decode_splits(n * -(-H // hb), keys), _P(nv.status_word(dev))
    if a.splits > 1:
        po, pml = WA._parts(dev, n * H * a.splits, s.rank_p)
        a.part_o, a.part_ml = _P(po), _P(pml)
    nv.check_rc(lib.omni_latent_decode(ctypes.byref(a), nv.stream_ptr()), "omni_latent_decode")
    return o_lat


def _rows(proj, s, pages, seqs, uk_t, kv_up, scale, out, gate, window=None):
    """Every row in the latent space on the row-per-block kernel."""
    T, H, dev = proj.shape[0], s.heads, proj.device
    bf = proj.dtype == torch.bfloat16
    uv = kv_up[H * s.dim_p:].view(H, s.vdim_p, s.rank_p)
    q = torch.empty(T, H, s.row, dtype=proj.dtype, device=dev)
    o = torch.empty(T, H, s.rank_p, dtype=proj.dtype, device=dev)
    q[:, :, s.rank_p:] = proj[:, :s.q_cols].view(T, H, s.head_cols)[:, :, s.dim_p:]
    if bf:
        head_gemm(proj, proj.stride(0), s.head_cols, uk_t, q, H * s.row, s.row, T, H)
    else:
        gemm.batched_f32(proj, uk_t[0], q.view(T, H * s.row), batch=H, a_stride=s.head_cols, w_stride=s.rank_p * s.dim_p,
                         c_stride=s.row)
    a = WA._WinAttn()
    a.q, a.q_rs, a.k_cache, a.v_cache = _P(q), q.stride(0), _P(pages), _P(pages)
    a.block_tables, a.bt_stride = _P(seqs.block_tables), seqs.block_tables.stride(0)
    a.q_start, a.context, a.row_seq = _P(seqs.q_start), _P(seqs.context), _P(seqs.row_seq)
    per_head = gate is not None and gate.shape[1] == H
    a.out, a.o_rs, a.window, a.maps = _P(o), o.stride(0), window or 0, 1
    a.set_gate(gate if per_head else None, H)
    a.scale, a.T, a.H, a.G, a.dp, a.vp, a.num_seqs = scale, T, H, 1, s.row, s.rank_p, seqs.n_seqs
    a.num_blocks, a.block_size, a.splits = pages.shape[0], pages.shape[1], 1
    a.k_ts = a.v_ts = a_row = s.row
    a.dp_u, a.status = a_row, _P(nv.status_word(dev))
    nv.check_rc(nv.lib("attn_window").omni_attn_window_rows(ctypes.byref(a), c_int(1 if bf else 0), nv.stream_ptr()),
                "omni_attn_window_rows")
    if bf:
        head_gemm(o, H * s.rank_p, s.rank_p, uv, out, out.stride(0), s.vdim_p, T, H, gate=None if per_head else gate)
    else:
        gemm.batched_f32(o.view(T, H * s.rank_p), uv[0], out, batch=H, a_stride=s.rank_p, w_stride=s.vdim_p * s.rank_p,
                         c_stride=s.vdim_p)
        if gate is not None and not per_head:
            gate_channels_(out, gate)
    return out


def gate_channels_(out, gate):
    """out *= sigmoid(gate), channel by channel: [T, n] each (views with unit column stride are fine)."""
    if not out.is_cuda:
        return out.copy_(out.float() * torch.sigmoid(gate.float()))
    assert out.shape == gate.shape and out.dtype == gate.dtype and out.stride(1) == 1 and gate.stride(1) == 1
    nv.check_rc(nv.lib("latent_attn").omni_gate_channels(
        nv.ptr(out), c_long(out.stride(0)), nv.ptr(gate), c_long(gate.stride(0)), c_long(out.shape[0]), c_int(out.shape[1]),
        c_int(1 if out.dtype == torch.bfloat16 else 0), nv.stream_ptr()), "omni_gate_channels")
    return out


def _cpu(proj, s, pages, seqs, kv_up, scale, out, gate, window=None):
    T, H = proj.shape[0], s.heads
    q = proj[:, :s.q_cols].float().view(T, H, s.head_cols)
    flat, bs = pages.view(-1, s.row), pages.shape[1]
    o = torch.empty(T, H, s.vdim_p)
    for n in range(seqs.n_seqs):
        a, b, ctx = int(seqs.q_start[n]), int(seqs.q_start[n + 1]), int(seqs.context[n])
        j = torch.arange(ctx + b - a)
        row = flat[seqs.block_tables[n].long()[j // bs] * bs + j % bs].float()
        kv = F.linear(row[:, :s.rank_p], kv_up.float())
        k = kv[:, :H * s.dim_p].view(-1, H, s.dim_p)
        v = kv[:, H * s.dim_p:].view(-1, H, s.vdim_p)
        sc = torch.einsum("thd,jhd->htj", q[a:b, :, :s.dim_p], k) + torch.einsum("thd,jd->htj", q[a:b, :, s.dim_p:], row[:, s.rank_p:])
        dist = torch.arange(ctx, ctx + b - a)[:, None] - j[None, :]
        see = dist >= 0 if window is None else (dist >= 0) & (dist < window)
        w = (sc * scale).masked_fill(~see, float("-inf")).softmax(-1)
        o[a:b] = torch.einsum("htj,jhd->thd", w, v)
    if gate is not None:
        o = o * torch.sigmoid(gate.float()).view(T, H, -1)
    out.copy_(o.reshape(T, H * s.vdim_p))
    return out
