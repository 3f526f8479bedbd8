"""Attention of a mixed batch (prompt portions and single decoded tokens) over the paged cache, with a
sliding window that keeps the first tokens, bounded scores, a logarithmic distance bias, a softmax sink,
two maps per head whose results are subtracted, and an output gate — each optional.  Kernels: csrc/attn_window_sm100.cu (tcgen05, portions of two
tokens and more), csrc/attn_window.cu (single tokens; and one block per row for fp32 and head sizes the
tensor-core kernels do not take)."""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from . import _native as nv

c_int, c_long, c_float, c_void_p = ctypes.c_int, ctypes.c_long, ctypes.c_float, ctypes.c_void_p


class _WinAttn(ctypes.Structure):
    _fields_ = [("q", c_void_p), ("q_rs", c_long), ("k_cache", c_void_p), ("v_cache", c_void_p),
                ("block_tables", c_void_p), ("bt_stride", c_int), ("q_start", c_void_p), ("context", c_void_p),
                ("row_seq", c_void_p), ("seq_list", c_void_p), ("n_list", c_int), ("items", c_void_p), ("n_items", c_int),
                ("block_tokens", c_int),
                ("out", c_void_p), ("o_rs", c_long), ("gate", c_void_p), ("g_rs", c_long), ("r1", c_void_p),
                ("r2", c_void_p), ("sink", c_void_p), ("scale", c_float), ("cap", c_float), ("bounded", c_int), ("window", c_int),
                ("keep_first", c_int), ("T", c_int), ("H", c_int), ("G", c_int), ("dp", c_int), ("vp", c_int),
                ("num_seqs", c_int), ("num_blocks", c_int), ("block_size", c_int), ("splits", c_int),
                ("part_o", c_void_p), ("part_ml", c_void_p), ("status", c_void_p), ("k_ts", c_long), ("v_ts", c_long),
                ("k_shared", c_void_p), ("ks_ts", c_long), ("dp_u", c_int), ("key_start", c_void_p), ("key_rows", c_long),
                ("g_hs", c_long), ("g_cs", c_int), ("maps", c_int), ("lam", c_float), ("out_mul", c_float), ("out_eps", c_float),
                ("vdim", c_int)]

    def set_gate(self, gate, heads: int):
        """``gate``: logits [T, heads] or [T, heads * channels of a head], a view with unit column stride."""
        if gate is None:
            return
        assert gate.stride(1) == 1 and gate.shape[1] % heads == 0
        self.gate, self.g_rs, self.g_hs = gate.data_ptr(), gate.stride(0), gate.shape[1] // heads
        self.g_cs = 0 if gate.shape[1] == heads else 1


@dataclass(frozen=True)
class DiffRule:
    """Differential attention: head h's result is u / sqrt(<u^2> + eps) * mult for u = a1 - lam a2, a1 and a2 the results of
    its two maps over the same values; ``vdim``: real channels of a value head."""
    lam: float
    mult: float
    eps: float
    vdim: int


@dataclass
class ScoreRule:
    """What turns q . k into an attention weight.  None / 0 switches a step off."""
    scale: float
    softcap: float | None = None
    r1: torch.Tensor | None = None        # fp32 [H]: distance bias r1 ln(1 + r2 dist)
    r2: torch.Tensor | None = None
    sink: torch.Tensor | None = None      # fp32 [H]
    window: int | None = None
    keep_first: int = 0
    bounded: bool = False                 # see ``bounded_scores``
    diff: DiffRule | None = None          # two maps per head; not together with a bias or a sink


def bounded_scores(softcap, r1=None, r2=None) -> bool:
    """May the cap stand in for the row maximum?  A row always sees its own position, where the bias is zero and the
    score at least -cap: relative to the cap its weight is at least 2^-(2 cap log2 e), and what lies far below that
    does not count.  True when this is well inside fp32's range and the bias never raises a score.  Reads r1 / r2
    on the host."""
    if not softcap:
        return False
    if r1 is not None and (bool((r1 < 0).any()) or bool((r2 < 0).any())):
        return False
    return 2.0 * softcap * math.log2(math.e) <= 90.0


def prefill_rows_per_block(heads: int, kv_heads: int, dp: int, maps: int = 1) -> int:
    """Tokens one block of the tcgen05 kernel serves: two 128-row tiles of (token, head of the KV group) rows,
    one when two tiles of the widest heads do not fit in shared memory or the second one is the second map."""
    return (1 if dp > 192 or maps == 2 else 2) * (128 // (heads // kv_heads))


def prefill_kernel_ok(heads: int, kv_heads: int, dp: int, vp: int, block_size: int) -> bool:
    return heads // kv_heads <= 128 and dp <= 256 and vp <= 128 and block_size >= 8 and block_size % 8 == 0 \
        and 128 % block_size == 0


def decode_splits(n: int, kv_heads: int, group: int, max_keys: int, heads_per_block: int = 16) -> int:
    """Blocks that share one sequence's visible keys: enough for about two blocks per SM, at least 64 keys each."""
    blocks = n * kv_heads * -(-group // heads_per_block)
    want = max(1, (2 * 148) // max(1, blocks))
    return max(1, min(want, 32, (max_keys + 63) // 64))


_scratch: dict = {}


def _parts(device, n: int, vp: int):
    """fp32 scratch of the split decode; grows, and is never freed: captured graphs hold its address."""
    key = (device.index, n, vp)
    t = _scratch.get(key)
    if t is None:
        t = (torch.empty(n * vp, dtype=torch.float32, device=device), torch.empty(n * 2, dtype=torch.float32, device=device))
        _scratch[key] = t
    return t


def window_attention(q, k_cache, v_cache, seqs, rule: ScoreRule, out, gate=None, impl: str | None = None):
    """q [T, H, dp]; caches [num_blocks, block_size, G, dp | vp] that already hold this step's tokens;
    ``seqs``: the batch's ``SeqTable``; ``out`` [T, H * vp]; ``gate`` [T, H] or [T, H * vp] logits (a view is fine).
    With ``rule.diff`` q is [T, 2 H, dp], heads ordered (KV head, map, head of the group), and a cached key has
    2 dp channels, its two maps side by side.

    ``impl="rows"`` forces the row-per-block kernel for every row."""
    maps = 1 if rule.diff is None else 2
    T, H, dp = q.shape[0], q.shape[1] // maps, q.shape[2]
    nb, bs, G, _ = k_cache.shape
    vp = v_cache.shape[3]
    assert k_cache.shape[3] == maps * dp and out.shape[1] == H * vp
    if not q.is_cuda:
        return _cpu(q, k_cache, v_cache, seqs, rule, out, gate)
    assert q.is_contiguous() and out.stride(1) == 1 and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert seqs.block_tables.dtype == torch.int32 and seqs.block_tables.stride(1) == 1
    a = _WinAttn()
    P = lambda t: 0 if t is None else t.data_ptr()
    a.q, a.q_rs, a.k_cache, a.v_cache = P(q), q.stride(0), P(k_cache), P(v_cache)
    a.block_tables, a.bt_stride = P(seqs.block_tables), seqs.block_tables.stride(0)
    a.q_start, a.context, a.row_seq = P(seqs.q_start), P(seqs.context), P(seqs.row_seq)
    a.out, a.o_rs = P(out), out.stride(0)
    a.set_gate(gate, H)
    a.r1, a.r2, a.sink = P(rule.r1), P(rule.r2), P(rule.sink)
    a.scale, a.cap = rule.scale, rule.softcap or 0.0
    a.bounded, a.window, a.keep_first = int(rule.bounded), rule.window or 0, rule.keep_first
    a.T, a.H, a.G, a.dp, a.vp, a.num_seqs, a.num_blocks, a.block_size = T, H, G, dp, vp, seqs.n_seqs, nb, bs
    a.k_ts, a.v_ts, a.dp_u, a.maps = G * maps * dp, G * vp, dp, maps
    if rule.diff is not None:
        a.lam, a.out_mul, a.out_eps, a.vdim = rule.diff.lam, rule.diff.mult, rule.diff.eps, rule.diff.vdim
    a.splits = 1
    a.status = P(nv.status_word(q.device))
    bf = q.dtype == torch.bfloat16
    rows_only = impl == "rows" or not bf or dp > (256 if maps == 1 else 128) or vp > 256 or (maps == 2 and rule.softcap) or not (
        seqs.n_decode == seqs.n_seqs or prefill_kernel_ok(H, G, dp, vp, bs))
    if rows_only:
        rc = nv.lib("attn_window").omni_attn_window_rows(ctypes.byref(a), c_int(1 if bf else 0), nv.stream_ptr())
        nv.check_rc(rc, "omni_attn_window_rows")
        return out
    if seqs.n_decode < seqs.n_seqs:
        a.block_tokens = prefill_rows_per_block(H, G, dp, maps)
        items, a.n_items = seqs.prefill_items(a.block_tokens)
        a.items = P(items)
        rc = nv.lib("attn_window_sm100").omni_attn_window_prefill(ctypes.byref(a), nv.stream_ptr())
        nv.check_rc(rc, "omni_attn_window_prefill")
    if seqs.n_decode:
        a.seq_list, a.n_list = P(seqs.decode_list), seqs.n_decode
        keys = seqs.max_context + 1
        if rule.window:
            keys = min(keys, rule.window + rule.keep_first)
        a.splits = decode_splits(seqs.n_decode, G, H // G, keys, 16 // maps)
        if a.splits > 1:
            po, pml = _parts(q.device, seqs.n_decode * H * maps * a.splits, vp)
            a.part_o, a.part_ml = P(po), P(pml)
        nv.check_rc(nv.lib("attn_window").omni_attn_window_decode(ctypes.byref(a), nv.stream_ptr()),
                    "omni_attn_window_decode")
    return out


def _cpu(q, k_cache, v_cache, seqs, rule, out, gate):
    maps = 1 if rule.diff is None else 2
    T, H, dp = q.shape[0], q.shape[1] // maps, q.shape[2]
    nb, bs, G, _ = k_cache.shape
    vp, R = v_cache.shape[3], H // G
    qm = q.float().view(T, G, maps, R, dp).permute(2, 0, 1, 3, 4).reshape(maps, T, H, dp)
    kf, vf = k_cache.view(nb * bs, G, maps, dp), v_cache.view(nb * bs, G, vp)
    o = torch.empty(maps, T, H, vp)
    for s in range(seqs.n_seqs):
        a, b, ctx = int(seqs.q_start[s]), int(seqs.q_start[s + 1]), int(seqs.context[s])
        j = torch.arange(ctx + b - a)
        i = torch.arange(ctx, ctx + b - a)[:, None]
        slot = seqs.block_tables[s].long()[j // bs] * bs + j % bs
        k = kf[slot].float().repeat_interleave(R, 1)
        v = vf[slot].float().repeat_interleave(R, 1)
        sc = torch.einsum("mthd,jhmd->mhtj", qm[:, a:b], k) * rule.scale
        if rule.softcap:
            sc = rule.softcap * torch.tanh(sc / rule.softcap)
        dist = (i - j).float()
        if rule.r1 is not None:
            sc = sc - rule.r1[:, None, None] * torch.log1p(rule.r2[:, None, None] * dist.clamp_min(0))
        see = dist >= 0
        if rule.window:
            see &= (dist < rule.window) | (j < rule.keep_first)
        sc = sc.masked_fill(~see, float("-inf"))
        if rule.sink is not None:
            sc = torch.cat([sc, rule.sink.float()[:, None, None].expand(maps, H, b - a, 1)], -1)
        w = sc.softmax(-1)[..., : j.numel()]
        o[:, a:b] = torch.einsum("mhtj,jhd->mthd", w, v)
    if rule.diff is None:
        o = o[0]
    else:
        u = o[0] - rule.diff.lam * o[1]
        o = u * torch.rsqrt(u.pow(2).sum(-1, keepdim=True) / rule.diff.vdim + rule.diff.eps) * rule.diff.mult
    if gate is not None:
        o = o * torch.sigmoid(gate.float()).view(T, H, -1)
    out.copy_(o.reshape(T, H * vp))
    return out
