"""Decoder-layer throughput: the Milivik decoder beside the Qwen3-MoE and Nidilix decoders at equal size.

    python bench.py --workload lm --lm-design milivik [--steps K --warmup W] [--lm-sizes 2048,4096]

The same two tables as lm_layers.py.  Equal size: same width, heads, experts and expert width; a token uses one expert less
beside the shared one.  Three of the four layers are latent attention with a window of 1024 and a query latent three quarters
as wide as the stream, the fourth is differential attention whose two maps together are as wide as a Qwen3 head."""
from __future__ import annotations

import ctypes
from types import SimpleNamespace

import torch

from .kernel_cases import _peaks
from .lm_layers import BS, DIM, VOCAB, WINDOW, Timer, step_table
from .lm_nidilix import RANK, ROT, SIZES, _decoders as _nidilix_decoders

GROUPS, KEEP = 8, 4


def milivik_config(width: int) -> dict:
    s = SIZES[width]
    mlp = {"kind": "moe", "expert": {"ff": s["ff"]}, "shared": {"ff": s["ff"]},
           "router": {"experts": s["experts"], "top": s["top"] - 1, "scale": 2.0, "groups": {"count": GROUPS, "keep": KEEP}}}
    latent = {"heads": s["heads"], "dim": DIM, "rot_dim": ROT, "vdim": DIM, "kv_rank": RANK, "q_rank": width * 3 // 4,
              "scale": (DIM + ROT) ** -0.5, "mask": {"size": WINDOW},
              "rot": {"base": 10000.0, "dims": ROT, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    diff = {"heads": s["heads"], "kv_heads": s["kv"], "dim": DIM // 2, "vdim": DIM, "scale": (DIM // 2) ** -0.5, "diff": 0.5,
            "q_temp": {"coef": 0.1, "every": 4096}}
    layer = lambda t, m: {"type": t, "mixer": m, "mlp": mlp}
    return {"architecture": "Milivik", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5},
            "logit_scale": 0.5, "layers": [layer("latent_attention", latent)] * 3 + [layer("attention", diff)]}


def _decoders(width: int, dev):
    from ..models.milivik import MilivikConfig, MilivikDecoder
    yield from _nidilix_decoders(width, dev)
    m = MilivikDecoder(MilivikConfig.from_dict(milivik_config(width)), torch.bfloat16, dev)
    m.load_weights(m.random_weights(0))
    yield "milivik", m


@torch.no_grad()
def kernel_rows(width: int, timer: Timer) -> list[dict]:
    from ..models.seq_table import SeqTable
    from ..ops import _native as nv, fused, gemm, kv_cache as KC, latent_attention as LA, lm, moe, stream
    from ..ops.attention import attention
    from ..ops.window_attention import DiffRule, ScoreRule, window_attention
    dev, bf = torch.device("cuda"), torch.bfloat16
    tf, gbs, _ = _peaks()
    s = SIZES[width]
    H, G, T, E, F_ = s["heads"], s["kv"], 8192, s["experts"], s["ff"]
    k2, QR = s["top"] - 1, width * 3 // 4
    out = []

    def row(name, like, fn, flops=0.0, bytes_=0.0):
        ms = timer(fn)
        a, b = flops / tf / 1e9, bytes_ / gbs / 1e6                 # milliseconds at either roofline
        out.append({"width": width, "kernel": name, "like": like, "us": round(ms * 1e3, 1),
                    "bound": "tensor" if a >= b else "memory", "of_measured": round(max(a, b) / ms, 3)})

    rnd = lambda *sh, dt=bf: torch.randn(*sh, dtype=dt, device=dev)
    one, tiny = torch.zeros(1, dtype=torch.int64, device=dev), torch.zeros(1, 8, dtype=bf, device=dev)
    row("timing floor", "an 8-channel lookup", lambda: stream.gelu_lookup_(tiny, tiny, one, 0, 8), bytes_=48.0)
    # ---- attention of a prompt
    q, k, v, o = rnd(1, T, H, DIM), rnd(1, T, G, DIM), rnd(1, T, G, DIM), rnd(T, H * DIM)
    pairs = T * (T + 1) / 2
    near = float(sum(min(i + 1, WINDOW) for i in range(T)))
    row("attention prompt", "qwen3_moe", lambda: attention(q, k, v, causal=True, out=o.view(1, T, H, DIM)), flops=4.0 * H * DIM * pairs)
    nb = T // BS
    seqs = SeqTable.build([T], [0], [list(range(nb))], [(0, 1)], dev)
    kc, vc, qd = k.view(nb, BS, G, DIM), v.view(nb, BS, G, DIM), q.view(T, 2 * H, DIM // 2)
    hg = rnd(T, H)
    rule = ScoreRule(DIM ** -0.5, diff=DiffRule(0.6, 0.5, 1e-6, DIM))
    row("attention prompt", "milivik differential", lambda: window_attention(qd, kc, vc, seqs, rule, o, gate=hg), flops=6.0 * H * DIM * pairs)
    plain = ScoreRule(DIM ** -0.5, window=WINDOW)
    row("attention prompt", f"tavulix w{WINDOW}, no cap / bias / sink / gate", lambda: window_attention(q[0], kc, vc, seqs, plain, o),
        flops=4.0 * H * DIM * near)
    ls = LA.LatentShape(H, DIM, ROT, DIM, RANK)
    pages, qp, gate, hgate = rnd(nb, BS, 1, ls.row), rnd(T, ls.q_cols), rnd(T, H * DIM), rnd(T, H)
    uk_t, kv_up = rnd(H, RANK, DIM) * RANK ** -0.5, rnd(2 * H * DIM, RANK) * RANK ** -0.5
    per_pair, up = 2.0 * H * (2 * DIM + ROT), 4.0 * T * RANK * H * DIM
    rows, kv = rnd(T, ls.row), rnd(T, 2 * H * DIM)
    for name, g, w, n in (("nidilix", hgate, None, pairs), ("milivik latent, no window", gate, None, pairs),
                          (f"milivik latent w{WINDOW}", gate, WINDOW, near)):
        group = seqs.long_groups(LA.SHORT, LA.MAX_KEYS, LA._rows_per_block(ls), w)[0]
        row("attention prompt", name, lambda: LA.expanded_attention(qp, ls, rows, kv, seqs, 0.07, o, g, group, w), flops=per_pair * n)
        row("attention prompt, with gather and up-projection", name, lambda: LA.latent_attention(
            qp, ls, pages, seqs, uk_t, kv_up, 0.07, o, gate=g, window=w), flops=per_pair * n + up)
    del q, k, v, rows, kv, kc, vc, qd
    # ---- attention of decoded tokens
    B, ctx = 64, 4095
    nb = B * 4096 // BS
    kc, vc = rnd(nb, BS, G, DIM), rnd(nb, BS, G, DIM)
    tables = torch.randperm(nb).view(B, -1)
    seqs = SeqTable.build([1] * B, [ctx] * B, tables.tolist(), None, dev)
    qd, od, gd = rnd(B, H, DIM), rnd(B, H * DIM), rnd(B, H * DIM)
    lens = torch.full((B,), ctx + 1, dtype=torch.int32, device=dev)
    kvb = 4.0 * B * G * DIM * (ctx + 1)
    row("attention decode", "qwen3_moe", lambda: KC.paged_decode(qd, kc, vc, seqs.block_tables, lens, out=od.view(B, H, DIM)), bytes_=kvb)
    row("attention decode", "milivik differential", lambda: window_attention(qd.view(B, 2 * H, DIM // 2), kc, vc, seqs, rule, od,
                                                                             gate=gd[:, :H]), bytes_=kvb)
    del kc, vc
    pages, pd, q_lat = rnd(nb, BS, 1, ls.row), rnd(B, ls.q_cols), rnd(B, H, RANK)
    rows, n, keys = seqs.short_rows(LA.SHORT)
    for name, w in (("nidilix", None), (f"milivik latent w{WINDOW}", WINDOW)):
        row("attention decode", name, lambda: LA.latent_decode(q_lat, pd, ls, pages, seqs, rows, n, keys, 0.07, w),
            bytes_=2.0 * B * ls.row * (w or ctx + 1))
    w = rnd(width, H * DIM)
    row("small product, 64 rows", "qwen3_moe (output projection)", lambda: gemm.linear(od, w), bytes_=2.0 * w.numel() + 4.0 * od.numel())
    uv = kv_up[H * DIM:].view(H, DIM, RANK)
    for name, g in (("nidilix (values out of the latent space)", gd[:, :H]), ("milivik (the same, gate per channel)", gd)):
        row("small product, 64 rows", name, lambda: LA.head_gemm(q_lat, H * RANK, RANK, uv, od, H * DIM, DIM, B, H, c_rows=rows, gate=g),
            bytes_=2.0 * H * DIM * RANK + 2.0 * B * H * (RANK + DIM))
    wu, cq = rnd(ls.q_cols, QR), rnd(B, QR)
    row("small product, 64 rows", "milivik (queries from their latent)", lambda: gemm.linear(cq, wu),
        bytes_=2.0 * wu.numel() + 2.0 * B * (QR + ls.q_cols))
    del pages
    # ---- projection to heads and pages
    C = (H + 2 * G) * DIM
    nb = T // BS
    qkv, wn, cs = rnd(1, T, C), rnd(DIM), rnd(T, DIM // 2, dt=torch.float32)
    kc, vc = rnd(nb, BS, G, DIM), rnd(nb, BS, G, DIM)
    slots = torch.arange(T, dtype=torch.int32, device=dev)
    seqs = SeqTable.build([T], [0], [list(range(nb))], None, dev)

    def dense_heads():
        fused.qk_norm_rope_(qkv, H, G, DIM, wq=wn, wk=wn, cos=cs, sin=cs, interleaved=False)
        x = qkv.view(T, C)
        KC.kv_write(x[:, H * DIM:(H + G) * DIM].view(T, G, DIM), x[:, (H + G) * DIM:].view(T, G, DIM), kc, vc, slots)
    row("heads and pages", "qwen3_moe (two kernels)", dense_heads, bytes_=4.0 * T * C)
    hs, nrm = lm.HeadShape(2 * H, 2 * G, DIM // 2, DIM, DIM // 2, DIM, v_heads=G), rnd(DIM // 2, dt=torch.float32)
    proj = rnd(T, C + H)
    row("heads and pages", "milivik differential", lambda: lm.conv_heads(proj, hs, seqs, slots, kc, vc, q_norm=nrm, k_norm=nrm,
                                                                         growth=lm.QueryGrowth(0.1, 4096)), bytes_=4.0 * T * C)
    pages, cn, qn = rnd(nb, BS, 1, ls.row), rnd(RANK, dt=torch.float32), rnd(QR, dt=torch.float32)
    turns = stream.rotary_rows(torch.arange(T, device=dev), 10000.0, ROT)
    pn, pm = rnd(T, ls.q_cols + ls.row + H), rnd(T, QR + ls.row + H * DIM)
    moved = 4.0 * T * (H * ROT + ls.row) + 4.0 * T * ROT
    row("heads and pages", "nidilix", lambda: LA.latent_rows(pn, ls, turns, slots, pages, cn, 1e-5), bytes_=moved)
    row("heads and pages", "milivik latent (norms, pages)", lambda: LA.cache_rows(
        pm[:, QR:], ls, turns, slots, pages, cn, 1e-6, query_latent=pm[:, :QR], query_norm=qn, query_rank=QR),
        bytes_=4.0 * T * (QR + ls.row) + 4.0 * T * ROT)
    row("heads and pages", "milivik latent (query rotation)", lambda: LA.rotate_queries(qp, ls, turns), bytes_=4.0 * T * (H + 1) * ROT)
    del qkv, kc, vc, pages, proj, pn, pm
    # ---- stream steps
    x, y, xn = rnd(T, width, dt=torch.float32), rnd(T, width), rnd(T, width)
    wv, g32 = rnd(width), rnd(width, dt=torch.float32)
    tn = SimpleNamespace(alpha=rnd(1, dt=torch.float32), w=g32, b=g32)
    kw = dict(gain=g32, eps=1e-6)
    row("norm", "qwen3_moe", lambda: fused.norm_modulate(y, weight=wv, rms=True, out=xn), bytes_=4.0 * T * width)
    row("norm", "nidilix (branch norm + add + tanh norm)", lambda: stream.add_branch_(x, y, 0.5, xn, tn, **kw), bytes_=12.0 * T * width)
    row("norm", "milivik (branch norm + add + cast)", lambda: stream.add_branch_(x, y, 1.0, xn, stream.CAST, **kw), bytes_=12.0 * T * width)
    row("norm", "milivik (branch norm + add + final norm)", lambda: stream.add_branch_(
        x, y, 1.0, xn, stream.RmsRows(g32, 1e-6, width), **kw), bytes_=12.0 * T * width)
    # ---- experts
    lib, P, ci = nv.lib("moe"), nv.ptr, LA.c_int
    soft, best = moe.Router(E, k2), moe.Router(E, k2, True, GROUPS, KEEP, 2.0)
    for rows_, tag in ((T, "prompt"), (64, "64 rows")):
        xr, rw = rnd(rows_, width), rnd(E, width) * width ** -0.5
        idb, wtb = torch.empty(rows_, 8, dtype=torch.int32, device=dev), torch.empty(rows_, 8, device=dev)

        def dense_router():
            lg = gemm.linear(xr, rw)
            lib.omni_moe_route(P(lg), ci(E), ci(rows_), ci(E), ci(s["top"]), ci(1), P(idb), P(wtb), nv.stream_ptr())
        cost = dict(bytes_=2.0 * xr.numel() + 2.0 * rw.numel(), flops=2.0 * rows_ * E * width)
        row(f"router, {tag}", "qwen3_moe (two kernels)", dense_router, **cost)
        for name, r in (("nidilix", soft), ("milivik (sigmoid, groups)", best)):
            row(f"router, {tag}", name, lambda: lib.omni_moe_router(
                P(xr), LA.c_long(width), P(rw), LA.c_long(width), P(None), ci(rows_), ci(width), ci(E), ci(E), ci(k2),
                ctypes.byref(r.rule), P(idb), P(wtb), nv.stream_ptr()), **cost)
        w13, w2 = rnd(E, 2 * F_, width) * 0.02, rnd(E, width, F_) * 0.02
        ws, ws_q = moe.MoEWorkspace(), moe.MoEWorkspace()
        er = moe.expert_rows(xr, rw, None, best, w13, w2, act="swiglu", ws=ws)
        n_used = ws.ids.unique().numel()                            # experts whose weights are read
        row(f"experts, {tag}", "milivik (router to expert rows)", lambda: moe.expert_rows(xr, rw, None, best, w13, w2, act="swiglu", ws=ws),
            flops=6.0 * rows_ * k2 * width * F_, bytes_=6.0 * n_used * width * F_)
        lg = gemm.linear(xr, rw)
        moe.moe_forward(xr, lg, w13, w2, s["top"], ws=ws_q)
        n_used = ws_q.ids.unique().numel()
        row(f"experts, {tag}", "qwen3_moe (route to combined rows)", lambda: moe.moe_forward(
            xr, lg, w13, w2, s["top"], ws=ws_q, residual=xr, out=torch.empty_like(xr)),
            flops=6.0 * rows_ * s["top"] * width * F_, bytes_=6.0 * n_used * width * F_)
        if rows_ == T:
            sh, sg = rnd(T, width), rnd(T, 8)
            row("experts' sum", "milivik (sum + gated shared + norm + add + cast)", lambda: stream.add_expert_rows_(
                x, er, sh, 1.0, xn, stream.CAST, shared_gate=sg[:, 0], **kw), bytes_=T * width * (2.0 * k2 + 2 + 8 + 2))
            row("experts' sum", "nidilix (sum + shared + add + cast)", lambda: stream.add_expert_rows_(x, er, sh, 0.5, xn, stream.CAST),
                bytes_=T * width * (2.0 * k2 + 2 + 8 + 2))
            yk, rp = rnd(T * s["top"], width), torch.arange(T * s["top"], dtype=torch.int32, device=dev)
            wt = torch.rand(T, s["top"], device=dev)
            row("experts' sum", "qwen3_moe (sum + residual)", lambda: lib.omni_moe_combine(
                P(yk), P(rp), P(wt), ci(T), ci(s["top"]), ci(width), P(y), LA.c_long(width), P(xn), LA.c_long(width), nv.stream_ptr()),
                bytes_=T * width * (2.0 * s["top"] + 4))
            gu = rnd(T, 2 * F_ + 8)
            row("activation", "qwen3_moe (SwiGLU of the chosen experts)", lambda a=rnd(T * s["top"], 2 * F_), h=rnd(T * s["top"], F_):
                fused.silu_mul(a, out=h), bytes_=6.0 * T * s["top"] * F_)
            row("activation", "milivik (SwiGLU of the shared expert)", lambda h=rnd(T, F_): fused.silu_mul(gu[:, :2 * F_], out=h),
                bytes_=6.0 * T * F_)
        del w13, w2
    emb, ids = rnd(VOCAB, width), torch.randint(0, VOCAB, (T,), device=dev)
    row("embedding", "nidilix (table + tanh norm)", lambda: stream.embed_rows(ids, emb, tn), bytes_=8.0 * T * width)
    row("embedding", "milivik (scaled table + cast)", lambda: stream.embed_rows(ids, emb, stream.CAST, mult=45.0), bytes_=8.0 * T * width)
    return out


def step_rows(width: int, timer: Timer) -> list[dict]:
    return step_table(width, timer, _decoders)
