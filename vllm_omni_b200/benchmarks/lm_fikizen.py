"""Decoder-layer throughput: the Fikizen decoder beside the Tavulix decoder at equal size.

    python bench.py --workload lm --lm-design fikizen [--steps K --warmup W] [--lm-sizes 2048,4096]

The same two tables as lm_layers.py.  Equal size: same width, attention heads, window and feed-forward; of the four Fikizen
layers one is attention beside a delta rule with decays per channel (heads of 64 channels, a quarter of the width), two are
attention (the second on the first one's weights) and one is a gated delta rule (heads of 128 channels as many as the
attention's, half as many key heads).  The recurrences stand beside Nidilix's, the other recurrence there is."""
from __future__ import annotations

import torch

from .kernel_cases import _peaks
from .lm_layers import BS, DIM, SIZES, VOCAB, WINDOW, Timer, step_table, tavulix_config

TAPS, RDIM, RANK = 4, 64, 64


def fikizen_config(width: int, window: int = WINDOW) -> dict:
    s = SIZES[width]
    attn = {"heads": s["heads"], "kv_heads": s["kv"], "dim": DIM, "vdim": DIM, "scale": DIM ** -0.5, "mask": {"size": window},
            "rot": {"base": 10000.0, "dims": DIM}}
    mlp = {"kind": "dense", "ff": s["ff"] * 3 // 2}
    layers = [{"type": "parallel", "mlp": mlp, "mixer": {"left": attn, "left_scale": 1.0, "right_scale": 1.0,
                                                         "right": {"heads": width // 4 // RDIM, "dim": RDIM}}},
              {"type": "attention", "mlp": mlp, "mixer": attn},
              {"type": "delta", "mlp": mlp, "mixer": {"heads": s["heads"], "kv_heads": s["heads"] // 2, "dim": DIM, "vdim": DIM, "conv": TAPS}}]
    layers.append(dict(layers[1], weights_of=1))
    return {"architecture": "Fikizen", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-5}, "logit_softcap": 30.0, "layers": layers}


def _decoders(width: int, dev):
    from ..models.fikizen import FikizenConfig, FikizenDecoder
    from ..models.tavulix import TavulixConfig, TavulixDecoder
    m = TavulixDecoder(TavulixConfig.from_dict(tavulix_config(width, WINDOW)), torch.bfloat16, dev)
    m.load_weights(m.random_weights(0))
    yield f"tavulix_w{WINDOW}", m
    m = FikizenDecoder(FikizenConfig.from_dict(fikizen_config(width)), torch.bfloat16, dev)
    m.load_weights(m.random_weights(0))
    yield f"fikizen_w{WINDOW}", m


@torch.no_grad()
def kernel_rows(width: int, timer: Timer) -> list[dict]:
    from ..models.seq_table import SeqTable
    from ..ops import fused, gemm, kv_cache as KC, lm, recurrent, stream
    from ..ops import delta_rule as DR
    from ..ops.attention import attention
    from ..ops.short_conv import conv_rows
    from ..ops.window_attention import ScoreRule, window_attention
    dev, bf = torch.device("cuda"), torch.bfloat16
    tf, gbs, _ = _peaks()
    s = SIZES[width]
    H, G, T, F_ = s["heads"], s["kv"], 8192, s["ff"] * 3 // 2
    out = []

    def row(name, like, fn, flops=0.0, bytes_=0.0):
        ms = timer(fn)
        a, b = flops / tf / 1e9, bytes_ / gbs / 1e6                 # milliseconds at either roofline
        out.append({"width": width, "kernel": name, "like": like, "us": round(ms * 1e3, 1),
                    "bound": "tensor" if a >= b else "memory", "of_measured": round(max(a, b) / ms, 3)})

    rnd = lambda *sh, dt=bf: torch.randn(*sh, dtype=dt, device=dev)
    f32 = lambda *sh: rnd(*sh, dt=torch.float32)
    one, sink = torch.ones(1, device=dev), torch.zeros(H, device=dev)
    # ---- attention of a prompt
    q, k, v, o, gate = rnd(T, H, DIM), rnd(T, G, DIM), rnd(T, G, DIM), rnd(T, H * DIM), rnd(T, H)
    pairs, nwin = T * (T + 1) / 2, sum(min(i + 1, WINDOW) for i in range(T))
    nb = T // BS
    kc, vc = k.view(nb, BS, G, DIM), v.view(nb, BS, G, DIM)
    seqs = SeqTable.build([T], [0], [list(range(nb))], [(0, 1)], dev)
    vecs = dict(r1=torch.rand(H, device=dev), r2=0.2 * torch.rand(H, device=dev), sink=f32(H))
    row("attention prompt", "dense, no window", lambda: attention(q[None], k[None], v[None], causal=True, out=o.view(1, T, H, DIM)),
        flops=4.0 * H * DIM * pairs)
    row("attention prompt", f"tavulix w{WINDOW}", lambda: window_attention(
        q, kc, vc, seqs, ScoreRule(DIM ** -0.5, 20.0, window=WINDOW, keep_first=4, bounded=True, **vecs), o, gate=gate), flops=4.0 * H * DIM * nwin)
    row("attention prompt", f"fikizen w{WINDOW}", lambda: window_attention(
        q, kc, vc, seqs, ScoreRule(DIM ** -0.5, sink=sink, window=WINDOW), o, gate=gate), flops=4.0 * H * DIM * nwin)
    row("attention prompt", "fikizen, no window", lambda: window_attention(q, kc, vc, seqs, ScoreRule(DIM ** -0.5, sink=sink), o, gate=gate),
        flops=4.0 * H * DIM * pairs)
    # ---- attention of decoded tokens
    B, ctx = 64, 4095
    nb = B * 4096 // BS
    kc, vc = rnd(nb, BS, G, DIM), rnd(nb, BS, G, DIM)
    seqs = SeqTable.build([1] * B, [ctx] * B, torch.randperm(nb).view(B, -1).tolist(), None, dev)
    qd, od, gd = rnd(B, H, DIM), rnd(B, H * DIM), rnd(B, H)
    row("attention decode", f"tavulix w{WINDOW}", lambda: window_attention(
        qd, kc, vc, seqs, ScoreRule(DIM ** -0.5, 20.0, window=WINDOW, keep_first=4, bounded=True, **vecs), od, gate=gd),
        bytes_=4.0 * B * G * DIM * (WINDOW + 4))
    row("attention decode", f"fikizen w{WINDOW}", lambda: window_attention(
        qd, kc, vc, seqs, ScoreRule(DIM ** -0.5, sink=sink, window=WINDOW), od, gate=gd), bytes_=4.0 * B * G * DIM * WINDOW)
    del kc, vc
    # ---- projection to heads and pages
    for rows_, tag in ((T, "prompt"), (B, "64 rows")):
        C = (H + 2 * G) * DIM
        nb = max(1, rows_ // BS)
        proj, kc, vc = rnd(rows_, C + H), rnd(nb, BS, G, DIM), rnd(nb, BS, G, DIM)
        slots, wn, cs = torch.arange(rows_, dtype=torch.int32, device=dev), rnd(DIM), f32(rows_, DIM // 2)
        qkv = rnd(1, rows_, C)

        def dense_heads():
            fused.qk_norm_rope_(qkv, H, G, DIM, wq=wn, wk=wn, cos=cs, sin=cs, interleaved=False)
            x = qkv.view(rows_, C)
            KC.kv_write(x[:, H * DIM:(H + G) * DIM].view(rows_, G, DIM), x[:, (H + G) * DIM:].view(rows_, G, DIM), kc, vc, slots)
        row(f"heads and pages, {tag}", "dense (two kernels)", dense_heads, bytes_=4.0 * rows_ * C)
        lens = [rows_] if rows_ == T else [1] * B
        seqs = SeqTable.build(lens, [0] * len(lens), [[0]] * len(lens), [(2 * i, 2 * i + 1) for i in range(len(lens))], dev)
        hs = lm.HeadShape(H, G, DIM, DIM, DIM, DIM, 3)
        conv, nrm, state, vf = f32(3, C), f32(DIM), rnd(2 * B, 2, C), rnd(rows_, G * DIM)
        row(f"heads and pages, {tag}", "tavulix", lambda: lm.conv_heads(proj, hs, seqs, slots, kc, vc, conv=conv, state=state, q_norm=nrm,
            k_norm=nrm, v_first=vf, v_mode="mix", lam=one), bytes_=4.0 * rows_ * C + 2.0 * rows_ * G * DIM)
        turns = stream.rotary_rows(torch.arange(rows_, device=dev), 10000.0, DIM)
        bytes_ = 4.0 * rows_ * C + 4.0 * rows_ * DIM
        row(f"heads and pages, {tag}", "fikizen (rotation)", lambda: lm.rotary_heads(proj, hs, slots, kc, vc, turns, DIM), bytes_=bytes_)
        qg, kg = f32(H * DIM), f32(G * DIM)
        row(f"heads and pages, {tag}", "fikizen (row norms, rotation, value norms)", lambda: lm.rotary_heads(
            proj, hs, slots, kc, vc, turns, DIM, q_gain=qg, k_gain=kg, v_norm=True), bytes_=bytes_)
    del proj, qkv, kc, vc
    # ---- stream steps
    x, y, xn, g32 = f32(T, width), rnd(T, width), rnd(T, width), f32(width)
    row("norm", "tavulix (branch norm + add + norm)", lambda: lm.add_norm_(x, y, one, width, 1e-5, xn, one), bytes_=12.0 * T * width)
    nxt = stream.RmsRows(g32, 1e-5, width)
    row("norm", "fikizen (add + norm)", lambda: stream.add_branch_(x, y, 1.0, xn, nxt), bytes_=12.0 * T * width)
    ids, emb = torch.randint(0, VOCAB, (T,), device=dev), rnd(VOCAB, width)
    row("embedding", "fikizen (table + norm)", lambda: stream.embed_rows(ids, emb, nxt), bytes_=8.0 * T * width)
    # ---- feed-forward
    coef, up = (0.9, 1.3), rnd(F_, width) * width ** -0.5
    coef4 = torch.tensor([0.5, 0.3, 0.1, 0.0], device=dev)
    z = rnd(T, F_)
    for rows_, tag in ((T, "prompt"), (B, "64 rows")):
        xr = rnd(rows_, width)
        fl, by = 2.0 * rows_ * width * F_, 2.0 * width * F_ + 2.0 * rows_ * (F_ + width)
        row(f"up and activation, {tag}", "GEMM alone", lambda: gemm.linear(xr, up, out=z[:rows_]), flops=fl, bytes_=by)
        row(f"up and activation, {tag}", "tavulix (GEMM, PolyNorm)", lambda: lm.poly_norm(gemm.linear(xr, up, out=z[:rows_]), coef4, F_, 1e-5, out=z[:rows_]),
            flops=fl, bytes_=by)
        row(f"up and activation, {tag}", "fikizen (GEMM with xIELU)", lambda: gemm.linear(xr, up, act="xielu", coef=coef, out=z[:rows_]),
            flops=fl, bytes_=by)
    del z, up
    # ---- recurrences
    P_ = 256
    sc = recurrent.GatedScanShape(width, width // P_, TAPS)
    conv, gates = f32(TAPS, width), rnd(2, sc.blocks, P_, P_) * P_ ** -0.5
    b1, b2, dec = f32(width), f32(2, width), -0.3 * torch.rand(width, device=dev)
    hist_n, state_n = rnd(2 * B, TAPS - 1, width), f32(2 * B, width)
    gs, rs = DR.DeltaShape(H, H // 2, DIM, DIM, TAPS), DR.DeltaShape(width // 4 // RDIM, width // 4 // RDIM, RDIM, RDIM)
    gated = DR.GatedDelta(0.4 * f32(TAPS, gs.channels), -torch.rand(H, device=dev), f32(H), f32(DIM), 1e-5)
    chan = DR.ChannelDelta(f32(rs.q_cols), f32(rs.q_cols), -0.6065, f32(rs.v_cols), 1e-5)
    hist = rnd(2 * B, TAPS - 1, gs.channels)
    st_g, st_c = torch.zeros(2 * B, H, DIM, DIM, device=dev), torch.zeros(2 * B, rs.heads, RDIM, RDIM, device=dev)
    for lens, tag in (([T], "prompt 1 x 8192"), ([1024] * 8, "prompt 8 x 1024"), ([1] * B, "decode 64"), ([1] * 8, "decode 8")):
        rows_, S = sum(lens), len(lens)
        seqs = SeqTable.build(lens, [0 if lens[0] > 1 else 100] * S, [[0]] * S, [(2 * i, 2 * i + 1) for i in range(S)], dev)
        px, pg, pc = rnd(rows_, 2 * width), rnd(rows_, gs.channels + gs.v_cols + 2 * H), rnd(rows_, 5 * rs.q_cols)
        og, oc, zc = rnd(rows_, gs.v_cols), rnd(rows_, rs.v_cols), rnd(rows_, rs.q_cols)
        one_tok = lens[0] == 1
        sb = lambda st: (2.0 if one_tok else 1.0) * S * st[0].numel() * 4
        row(f"recurrence, {tag}", "nidilix", lambda: recurrent.gated_scan(px, sc, seqs, conv, b1, gates, b2, dec, hist_n, state_n),
            bytes_=6.0 * rows_ * width + sb(state_n) + (2.0 * gates.numel() if one_tok else 0), flops=4.0 * rows_ * width * P_)
        gb = 2.0 * rows_ * (gs.channels + 2 * gs.v_cols) + sb(st_g)
        row(f"recurrence, {tag}", "fikizen gated", lambda: DR.delta_rule(pg, gs, seqs, gated, st_g, og, hist=hist), bytes_=gb)
        cb = 2.0 * rows_ * (6 * rs.q_cols + rs.v_cols) + sb(st_c)
        row(f"recurrence, {tag}", "fikizen channel", lambda: DR.delta_rule(pc, rs, seqs, chan, st_c, oc, decay=zc), bytes_=cb)
        if not one_tok:
            row(f"of it, {tag}", "fikizen gated: convolution", lambda: conv_rows(pg, seqs, TAPS, gs.channels, gated.conv, hist, act="silu",
                skip_single=True), bytes_=4.0 * rows_ * gs.channels)
    # ---- low-rank decay
    low, w2 = rnd(T, 4096 + RANK), rnd(rs.q_cols, RANK) * RANK ** -0.5
    for rows_, tag in ((T, "prompt"), (B, "64 rows")):
        row(f"decay logits, {tag}", "fikizen (tanh, GEMM)", lambda: gemm.linear(lm.tanh_cols(low[:rows_, 4096:]), w2),
            bytes_=2.0 * (rows_ * (3 * RANK + rs.q_cols) + w2.numel()), flops=2.0 * rows_ * RANK * rs.q_cols)
        small = rnd(width, H * DIM)
        row(f"decay logits, {tag}", "output GEMM", lambda a=rnd(rows_, H * DIM): gemm.linear(a, small),
            bytes_=2.0 * (rows_ * (width + H * DIM) + small.numel()), flops=2.0 * rows_ * width * H * DIM)
    return out


def step_rows(width: int, timer: Timer) -> list[dict]:
    return step_table(width, timer, _decoders)
