"""Decoder-layer throughput: the Nidilix decoder beside the Qwen3-MoE decoder at equal size.

    python bench.py --workload lm --lm-design nidilix [--steps K --warmup W] [--lm-sizes 2048,4096]

The same two tables as lm_layers.py.  Equal size: same width, heads, head channels and experts; the two-matrix experts are
1.5 times as wide as the three-matrix ones and a token uses one expert less beside the shared one, so both hold about the
same number of weights and use the same number per token.  Of the four Nidilix layers two are latent attention (the
second reads the first one's latents) and two are recurrences as wide as the stream, in parts of 256 channels."""
from __future__ import annotations

import ctypes

import torch

from .kernel_cases import _peaks
from .lm_layers import BS, DIM, LAYERS, VOCAB, Timer, step_table

SIZES = {2048: dict(heads=16, kv=4, experts=64, top=5, ff=768), 4096: dict(heads=32, kv=8, experts=64, top=5, ff=1536)}
ROT, RANK, SIDE, TAPS, PART = 64, 512, 256, 4, 256


def nidilix_config(width: int) -> dict:
    s = SIZES[width]
    ff = s["ff"] * 3 // 2
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": s["experts"], "top": s["top"] - 1}, "shared": {"ff": ff}}

    def attention(**kw):
        return {"type": "latent_attention", "mlp": mlp,
                "mixer": {"heads": s["heads"], "dim": DIM, "rot_dim": ROT, "vdim": DIM, "kv_rank": RANK,
                          "scale": (DIM + ROT) ** -0.5, "rot": {"base": 10000.0, "dims": ROT}, **kw}}
    scan = {"type": "rglru", "mlp": mlp, "mixer": {"width": width, "blocks": width // PART, "conv": TAPS}}
    return {"architecture": "Nidilix", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-5}, "residual_mult": 0.5,
            "token_side": {"dim": SIDE}, "layers": [attention(), scan, attention(kv_from=0), scan]}


def _decoders(width: int, dev):
    from ..models.nidilix import NidilixConfig, NidilixDecoder
    from ..models.qwen_decoder import DecoderConfig, QwenDecoderModel
    s = SIZES[width]
    yield "qwen3_moe", QwenDecoderModel(
        DecoderConfig(vocab_size=VOCAB, hidden_size=width, num_hidden_layers=LAYERS, num_attention_heads=s["heads"],
                      num_key_value_heads=s["kv"], head_dim=DIM, num_experts=s["experts"], num_experts_per_tok=s["top"],
                      moe_intermediate_size=s["ff"]), torch.bfloat16, dev)
    m = NidilixDecoder(NidilixConfig.from_dict(nidilix_config(width)), torch.bfloat16, dev)
    m.load_weights(m.random_weights(0))
    yield "nidilix", m


@torch.no_grad()
def kernel_rows(width: int, timer: Timer) -> list[dict]:
    from ..models.seq_table import SeqTable
    from ..ops import _native as nv, fused, gemm, kv_cache as KC, latent_attention as LA, lm, moe, recurrent, stream
    from ..ops.attention import attention
    from types import SimpleNamespace
    dev, bf = torch.device("cuda"), torch.bfloat16
    tf, gbs, _ = _peaks()
    s = SIZES[width]
    H, G, T, E, F_ = s["heads"], s["kv"], 8192, s["experts"], s["ff"]
    F2, k2 = F_ * 3 // 2, s["top"] - 1
    router = moe.Router(E, k2)
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
    q, k, v = rnd(1, T, H, DIM), rnd(1, T, G, DIM), rnd(1, T, G, DIM)
    o = rnd(T, H * DIM)
    pairs = T * (T + 1) / 2
    row("attention prompt", "qwen3_moe", lambda: attention(q, k, v, causal=True, out=o.view(1, T, H, DIM)), flops=4.0 * H * DIM * pairs)
    ls = LA.LatentShape(H, DIM, ROT, DIM, RANK)
    nb = T // BS
    cols = ls.q_cols + ls.row + H
    proj, pages = rnd(T, cols), rnd(nb, BS, 1, ls.row)
    uk_t, kv_up = rnd(H, RANK, DIM) * RANK ** -0.5, rnd(2 * H * DIM, RANK) * RANK ** -0.5
    seqs = SeqTable.build([T], [0], [list(range(nb))], [(0, 1)], dev)
    gate = proj[:, ls.q_cols + ls.row:]
    fl = 2.0 * H * (2 * DIM + ROT) * pairs
    row("attention prompt", "nidilix with gather and up-projection", lambda: LA.latent_attention(
        proj, ls, pages, seqs, uk_t, kv_up, 0.07, o, gate=gate), flops=fl + 4.0 * T * RANK * H * DIM)
    group = seqs.long_groups(LA.SHORT, LA.MAX_KEYS, LA._rows_per_block(ls))[0]
    rows, kv = rnd(T, ls.row), rnd(T, 2 * H * DIM)
    row("attention prompt", "nidilix", lambda: LA.expanded_attention(proj, ls, rows, kv, seqs, 0.07, o, gate, group), flops=fl)
    del q, k, v, rows, kv
    # ---- attention of decoded tokens
    B, ctx = 64, 4095
    nb = B * 4096 // BS
    kc, vc = rnd(nb, BS, G, DIM), rnd(nb, BS, G, DIM)
    tables = torch.randperm(nb).view(B, -1)
    seqs = SeqTable.build([1] * B, [ctx] * B, tables.tolist(), None, dev)
    qd, od = rnd(B, H, DIM), rnd(B, H * DIM)
    lens = torch.full((B,), ctx + 1, dtype=torch.int32, device=dev)
    row("attention decode", "qwen3_moe", lambda: KC.paged_decode(qd, kc, vc, seqs.block_tables, lens, out=od.view(B, H, DIM)),
        bytes_=4.0 * B * G * DIM * (ctx + 1))
    del kc, vc
    pages, pd, q_lat = rnd(nb, BS, 1, ls.row), rnd(B, cols), rnd(B, H, RANK)
    rows, n, keys = seqs.short_rows(LA.SHORT)
    row("attention decode", "nidilix", lambda: LA.latent_decode(q_lat, pd, ls, pages, seqs, rows, n, keys, 0.07),
        bytes_=2.0 * B * ls.row * (ctx + 1))
    w = rnd(width, H * DIM)
    row("small product, 64 rows", "qwen3_moe (output projection)", lambda: gemm.linear(od, w), bytes_=2.0 * w.numel() + 4.0 * od.numel())
    row("small product, 64 rows", "nidilix (queries to the latent space)", lambda: LA.head_gemm(
        pd, cols, ls.head_cols, uk_t, q_lat, H * RANK, RANK, B, H, a_rows=rows), bytes_=2.0 * uk_t.numel() + 2.0 * B * H * (RANK + DIM))
    row("small product, 64 rows", "nidilix (values out of it)", lambda: LA.head_gemm(
        q_lat, H * RANK, RANK, kv_up[H * DIM:].view(H, DIM, RANK), od, H * DIM, DIM, B, H, c_rows=rows),
        bytes_=2.0 * H * DIM * RANK + 2.0 * B * H * (RANK + DIM))
    del pages
    # ---- projection to heads and pages
    C = (H + 2 * G) * DIM
    nb = T // BS
    qkv, wn, cs = rnd(1, T, C), rnd(DIM), rnd(T, DIM // 2, dt=torch.float32)
    kc, vc = rnd(nb, BS, G, DIM), rnd(nb, BS, G, DIM)
    slots = torch.arange(T, dtype=torch.int32, device=dev)

    def dense_heads():
        fused.qk_norm_rope_(qkv, H, G, DIM, wq=wn, wk=wn, cos=cs, sin=cs, interleaved=False)
        x = qkv.view(T, C)
        KC.kv_write(x[:, H * DIM:(H + G) * DIM].view(T, G, DIM), x[:, (H + G) * DIM:].view(T, G, DIM), kc, vc, slots)
    row("heads and pages", "qwen3_moe (two kernels)", dense_heads, bytes_=4.0 * T * C)
    pages, cn = rnd(nb, BS, 1, ls.row), rnd(RANK, dt=torch.float32)
    turns = stream.rotary_rows(torch.arange(T, device=dev), 10000.0, ROT)
    row("heads and pages", "nidilix", lambda: LA.latent_rows(proj, ls, turns, slots, pages, cn, 1e-5),
        bytes_=4.0 * T * (H * ROT + ls.row) + 4.0 * T * ROT)
    del qkv, kc, vc, pages, proj
    # ---- stream steps
    x, y, xn = rnd(T, width, dt=torch.float32), rnd(T, width), rnd(T, width)
    wv, g32 = rnd(width), rnd(width, dt=torch.float32)
    tn = SimpleNamespace(alpha=rnd(1, dt=torch.float32), w=g32, b=g32)
    row("norm", "qwen3_moe", lambda: fused.norm_modulate(y, weight=wv, rms=True, out=xn), bytes_=4.0 * T * width)
    row("norm", "nidilix (add + tanh norm)", lambda: stream.add_branch_(x, y, 0.5, xn, tn), bytes_=12.0 * T * width)
    row("norm", "nidilix (branch norm + add + tanh norm)", lambda: stream.add_branch_(x, y, 0.5, xn, tn, gain=g32, eps=1e-5),
        bytes_=12.0 * T * width)
    z, table, ids = rnd(T, SIDE), rnd(VOCAB, LAYERS * SIDE), torch.randint(0, VOCAB, (T,), device=dev)
    row("activation", "qwen3_moe (SwiGLU)", lambda gu=rnd(T * s["top"], 2 * F_), h=rnd(T * s["top"], F_): fused.silu_mul(gu, out=h),
        bytes_=6.0 * T * s["top"] * F_)
    row("activation", "nidilix (side gate: gelu times table row)", lambda: stream.gelu_lookup_(z, table, ids, SIDE, SIDE), bytes_=6.0 * T * SIDE)
    # ---- experts
    lib = nv.lib("moe")
    for rows_, tag in ((T, "prompt"), (64, "64 rows")):
        xr = rnd(rows_, width)
        rw, rb = rnd(E, width) * width ** -0.5, rnd(E, dt=torch.float32)
        idb, wtb = torch.empty(rows_, 8, dtype=torch.int32, device=dev), torch.empty(rows_, 8, device=dev)
        P, ci = nv.ptr, LA.c_int

        def dense_router():
            lg = gemm.linear(xr, rw)
            lib.omni_moe_route(P(lg), ci(E), ci(rows_), ci(E), ci(s["top"]), ci(1), P(idb), P(wtb), nv.stream_ptr())
        rbytes = 2.0 * xr.numel() + 2.0 * rw.numel()
        row(f"router, {tag}", "qwen3_moe (two kernels)", dense_router, bytes_=rbytes, flops=2.0 * rows_ * E * width)
        row(f"router, {tag}", "nidilix", lambda: lib.omni_moe_router(P(xr), LA.c_long(width), P(rw), LA.c_long(width), P(rb), ci(rows_),
            ci(width), ci(E), ci(E), ci(k2), ctypes.byref(router.rule), P(idb), P(wtb), nv.stream_ptr()), bytes_=rbytes, flops=2.0 * rows_ * E * width)
        up, down = rnd(E, F2, width) * 0.02, rnd(E, width, F2) * 0.02
        er = moe.expert_rows(xr, rw, rb, router, up, down, act="relu2")
        ws, ws_q = moe.MoEWorkspace(), moe.MoEWorkspace()
        moe.expert_rows(xr, rw, rb, router, up, down, act="relu2", ws=ws)
        n_used = ws.ids.unique().numel()                            # experts whose weights are read
        row(f"experts, {tag}", "nidilix (router to expert rows)", lambda: moe.expert_rows(xr, rw, rb, router, up, down, act="relu2", ws=ws),
            flops=4.0 * rows_ * k2 * width * F2, bytes_=4.0 * n_used * width * F2)
        w13, w2 = rnd(E, 2 * F_, width) * 0.02, rnd(E, width, F_) * 0.02
        lg = gemm.linear(xr, rw)
        moe.moe_forward(xr, lg, w13, w2, s["top"], ws=ws_q)
        n_used_q = ws_q.ids.unique().numel()
        row(f"experts, {tag}", "qwen3_moe (route to combined rows)", lambda: moe.moe_forward(xr, lg, w13, w2, s["top"], ws=ws_q, residual=xr, out=torch.empty_like(xr)),
            flops=6.0 * rows_ * s["top"] * width * F_, bytes_=6.0 * n_used_q * width * F_)
        if rows_ == T:
            sh = rnd(T, width)
            row("experts' sum", "nidilix (sum + shared + add + cast)", lambda: stream.add_expert_rows_(x, er, sh, 0.5, xn, stream.CAST),
                bytes_=T * width * (2.0 * k2 + 2 + 8 + 2))
            yk, rp = rnd(T * s["top"], width), torch.arange(T * s["top"], dtype=torch.int32, device=dev)
            wt = torch.rand(T, s["top"], device=dev)
            row("experts' sum", "qwen3_moe (sum + residual)", lambda: lib.omni_moe_combine(
                P(yk), P(rp), P(wt), ci(T), ci(s["top"]), ci(width), P(y), LA.c_long(width), P(xn), LA.c_long(width), nv.stream_ptr()),
                bytes_=T * width * (2.0 * s["top"] + 4))
        del up, down, w13, w2
    # ---- recurrence
    sc = recurrent.GatedScanShape(width, width // PART, TAPS)
    conv, gates = rnd(TAPS, width, dt=torch.float32), rnd(2, sc.blocks, PART, PART) * PART ** -0.5
    b1, b2, dec = rnd(width, dt=torch.float32), rnd(2, width, dt=torch.float32), -0.3 * torch.rand(width, device=dev)
    hs = lm.HeadShape(H, G, DIM, DIM, DIM, DIM, 3)
    projq, convq, nrm = rnd(T, hs.channels + H), rnd(3, hs.channels, dt=torch.float32), rnd(DIM, dt=torch.float32)
    kc, vc = rnd(nb, BS, G, DIM), rnd(nb, BS, G, DIM)
    seqs = SeqTable.build([T], [0], [list(range(nb))], [(0, 1)], dev)
    stq = rnd(2, 2, hs.channels)
    row("recurrence prompt", "tavulix (convolution + head norms + pages)", lambda: lm.conv_heads(
        projq, hs, seqs, slots, kc, vc, conv=convq, state=stq, q_norm=nrm, k_norm=nrm), bytes_=4.0 * T * hs.channels)
    px = rnd(T, 2 * width)
    hist, state = rnd(128, TAPS - 1, width), rnd(128, width, dt=torch.float32)
    row("recurrence prompt", "nidilix", lambda: recurrent.gated_scan(px, sc, seqs, conv, b1, gates, b2, dec, hist, state),
        bytes_=6.0 * T * width, flops=4.0 * T * width * PART)
    seqs8 = SeqTable.build([1024] * 8, [0] * 8, [[0]] * 8, [(2 * i, 2 * i + 1) for i in range(8)], dev)
    row("recurrence prompt, 8 x 1024", "nidilix", lambda: recurrent.gated_scan(px, sc, seqs8, conv, b1, gates, b2, dec, hist, state),
        bytes_=6.0 * T * width, flops=4.0 * T * width * PART)
    seqs1 = SeqTable.build([1] * B, [100] * B, [[0]] * B, [(2 * i, 2 * i + 1) for i in range(B)], dev)
    p1 = rnd(B, 2 * width)
    row("recurrence decode", "nidilix", lambda: recurrent.gated_scan(p1, sc, seqs1, conv, b1, gates, b2, dec, hist, state),
        bytes_=2.0 * gates.numel() + B * width * (6.0 + 8 + 4 * (TAPS - 1)))
    emb = rnd(VOCAB, width)
    row("embedding", "nidilix (table + tanh norm)", lambda: stream.embed_rows(ids, emb, tn), bytes_=8.0 * T * width)
    return out


def step_rows(width: int, timer: Timer) -> list[dict]:
    return step_table(width, timer, _decoders)
