"""Decoder-layer throughput: the Tavulix decoder beside the dense Qwen3 decoder at equal size.

    python bench.py --workload lm [--steps K --warmup W] [--lm-sizes 2048,4096]

Two parts, one JSON line.  ``steps``: whole engine-style steps (random weights, four layers, no sampling) — prompts
in tokens/s, decoding in tokens/s with the step replayed from a captured graph.  ``kernels``: every kernel of the
new decoder next to the like kernel of the dense one, with the fraction of its roofline.  CUDA events, L2 flushed
(256 MB written) before every timed launch or step; fractions are of the measured peaks in MEASURED_PEAKS.json.

Equal size: same width, heads, KV heads and head size; the two-matrix feed-forward is 1.5 times as wide as the
three-matrix one, so both hold the same number of weights.  The windowed decoder runs once with a window that never
cuts (the dense decoder's attention work) and once with a window of 1024."""
from __future__ import annotations

import torch

from ..models.seq_table import layer_caches
from .kernel_cases import _peaks

LAYERS = 4
SIZES = {2048: dict(heads=16, kv=4, ff=6144), 4096: dict(heads=32, kv=8, ff=12288)}
DIM, VOCAB, WINDOW, BS = 128, 32768, 1024, 16
FULL = 1 << 20        # a window no context reaches


class Timer:
    def __init__(self, steps: int, warmup: int):
        self.steps, self.warmup = steps, max(3, warmup)
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def __call__(self, fn) -> float:
        """Median milliseconds of ``fn`` with a cold L2."""
        for _ in range(self.warmup):
            fn()
        torch.cuda.synchronize()
        ts = []
        for _ in range(self.steps):
            self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        return sorted(ts)[len(ts) // 2]


def tavulix_config(width: int, window: int, layers: int = LAYERS, positions: int = 16384) -> dict:
    s = SIZES[width]
    layer = {"type": "attention", "mlp": {"kind": "dense", "ff": s["ff"] * 3 // 2},
             "mixer": {"heads": s["heads"], "kv_heads": s["kv"], "dim": DIM, "vdim": DIM, "conv": 3, "scale": DIM ** -0.5,
                       "softcap": 20.0, "v_mix": True, "mask": {"size": window, "keep_first": 4}}}
    return {"architecture": "Tavulix", "vocab": VOCAB, "width": width, "max_positions": positions,
            "norm": {"eps": 1e-5}, "logit_softcap": 30.0, "layers": [layer] * layers}


def _decoders(width: int, dev):
    from ..models.qwen_decoder import DecoderConfig, QwenDecoderModel
    from ..models.tavulix import TavulixConfig, TavulixDecoder
    s = SIZES[width]
    dense = DecoderConfig(vocab_size=VOCAB, hidden_size=width, num_hidden_layers=LAYERS, num_attention_heads=s["heads"],
                          num_key_value_heads=s["kv"], head_dim=DIM, intermediate_size=s["ff"], num_experts=0)
    yield "dense_qwen3", QwenDecoderModel(dense, torch.bfloat16, dev)
    for name, window in (("tavulix_full", FULL), (f"tavulix_w{WINDOW}", WINDOW)):
        m = TavulixDecoder(TavulixConfig.from_dict(tavulix_config(width, window)), torch.bfloat16, dev)
        m.load_weights(m.random_weights(0))
        yield name, m


def _caches(model, blocks: int, dev, seqs: int):
    return layer_caches(model.cfg, blocks, BS, 2 * seqs, torch.bfloat16, dev, fill=torch.randn)


def _batch(lens, contexts, dev):
    """One step's batch of sequences with ``contexts`` tokens in the cache and ``lens`` new ones."""
    from ..models.qwen_decoder import ModelBatch, PrefillSeg
    from ..models.seq_table import SeqTable
    tables, nxt = [], 0
    for n, c in zip(lens, contexts):
        k = (n + c + BS - 1) // BS
        tables.append(list(range(nxt, nxt + k)))
        nxt += k
    pos = torch.cat([torch.arange(c, c + n) for n, c in zip(lens, contexts)])
    slots = torch.cat([torch.tensor(t)[torch.arange(c, c + n) // BS] * BS + torch.arange(c, c + n) % BS
                       for t, n, c in zip(tables, lens, contexts)])
    ids = torch.randint(0, VOCAB, (pos.numel(),))
    b = ModelBatch(ids.to(dev), pos.to(dev), slots.int().to(dev))
    b.seqs = SeqTable.build(lens, contexts, tables, [(2 * i, 2 * i + 1) for i in range(len(lens))], dev)
    if max(lens) > 1:
        row = 0
        for n, c, t in zip(lens, contexts, tables):
            b.prefills.append(PrefillSeg(row, n, c, torch.tensor(t, dtype=torch.int32, device=dev)))
            row += n
    else:
        b.decode_rows = torch.arange(len(lens), device=dev)
        b.decode_block_tables = b.seqs.block_tables
        b.decode_seq_lens = torch.tensor([c + 1 for c in contexts], dtype=torch.int32, device=dev)
    return b, nxt


def step_rows(width: int, timer: Timer) -> list[dict]:
    return step_table(width, timer, _decoders)


@torch.no_grad()
def step_table(width: int, timer: Timer, decoders) -> list[dict]:
    """Prompt and decode steps of every (name, model) that ``decoders`` yields."""
    from ..engine.graph_runner import DecodeGraphRunner
    dev = torch.device("cuda")
    rows = []
    for name, model in decoders(width, dev):
        r = {"width": width, "decoder": name}
        for label, lens in (("prefill_1x8192", [8192]), ("prefill_8x1024", [1024] * 8)):
            b, nb = _batch(lens, [0] * len(lens), dev)
            kv = _caches(model, nb, dev, len(lens))
            ms = timer(lambda: model(b, kv))
            r[label] = {"ms": round(ms, 3), "tokens_s": round(sum(lens) / ms * 1e3)}
        for n in (8, 64):
            b, nb = _batch([1] * n, [4000] * n, dev)
            kv = _caches(model, nb, dev, n)
            g = DecodeGraphRunner(model, kv, 4096 // BS, buckets=(n,))
            ms = timer(lambda: g.run(b))
            r[f"decode_{n}x4000"] = {"ms": round(ms, 3), "tokens_s": round(n / ms * 1e3)}
            del g, kv
        rows.append(r)
        del model
        torch.cuda.empty_cache()
    return rows


@torch.no_grad()
def kernel_rows(width: int, timer: Timer) -> list[dict]:
    from ..models.seq_table import SeqTable
    from ..ops import fused, kv_cache as KC, lm
    from ..ops.attention import attention
    from ..ops.window_attention import ScoreRule, window_attention
    dev, bf = torch.device("cuda"), torch.bfloat16
    tf, gbs, _ = _peaks()
    s = SIZES[width]
    H, G, T, F_ = s["heads"], s["kv"], 8192, s["ff"]
    out = []

    def row(name, like, fn, flops=0.0, bytes_=0.0):
        ms = timer(fn)
        frac = flops / ms / 1e9 / tf if flops else bytes_ / ms / 1e6 / gbs
        out.append({"width": width, "kernel": name, "like": like, "us": round(ms * 1e3, 1),
                    "bound": "tensor" if flops else "memory", "of_measured": round(frac, 3)})

    rnd = lambda *sh, dt=bf: torch.randn(*sh, dtype=dt, device=dev)
    one = torch.ones(1, device=dev)
    # ---- attention of a prompt
    q, k, v = rnd(1, T, H, DIM), rnd(1, T, G, DIM), rnd(1, T, G, DIM)
    o = rnd(T, H * DIM)
    full = 4.0 * H * DIM * T * (T + 1) / 2
    nwin = sum(min(i + 1, WINDOW) for i in range(T))
    row("attention prompt", "dense", lambda: attention(q, k, v, causal=True, out=o.view(1, T, H, DIM)), flops=full)
    nb = T // BS
    kc, vc = k.view(nb, BS, G, DIM), v.view(nb, BS, G, DIM)
    seqs = SeqTable.build([T], [0], [list(range(nb))], [(0, 1)], dev)
    vecs = dict(r1=torch.rand(H, device=dev), r2=0.2 * torch.rand(H, device=dev), sink=torch.randn(H, device=dev))
    gate = rnd(T, H)
    rule = lambda w: ScoreRule(DIM ** -0.5, 20.0, window=w, keep_first=4, bounded=True, **vecs)
    row("attention prompt", "tavulix full", lambda: window_attention(q[0], kc, vc, seqs, rule(FULL), o, gate=gate), flops=full)
    row("attention prompt", f"tavulix w{WINDOW}", lambda: window_attention(q[0], kc, vc, seqs, rule(WINDOW), o, gate=gate),
        flops=4.0 * H * DIM * nwin)
    plain = ScoreRule(DIM ** -0.5, window=FULL)
    row("attention prompt", "tavulix full, no cap / bias / sink / gate", lambda: window_attention(q[0], kc, vc, seqs, plain, o),
        flops=full)
    # ---- attention of decoded tokens
    B, ctx = 64, 4095
    nb = B * 4096 // BS
    kc, vc = rnd(nb, BS, G, DIM), rnd(nb, BS, G, DIM)
    tables = torch.randperm(nb).view(B, -1)
    seqs = SeqTable.build([1] * B, [ctx] * B, tables.tolist(), None, dev)
    qd, od, gd = rnd(B, H, DIM), rnd(B, H * DIM), rnd(B, H)
    lens = torch.full((B,), ctx + 1, dtype=torch.int32, device=dev)
    kvb = lambda n: 4.0 * B * G * DIM * n
    row("attention decode", "dense", lambda: KC.paged_decode(qd, kc, vc, seqs.block_tables, lens, out=od.view(B, H, DIM)), bytes_=kvb(ctx + 1))
    row("attention decode", "tavulix full", lambda: window_attention(qd, kc, vc, seqs, rule(FULL), od, gate=gd), bytes_=kvb(ctx + 1))
    row("attention decode", f"tavulix w{WINDOW}", lambda: window_attention(qd, kc, vc, seqs, rule(WINDOW), od, gate=gd),
        bytes_=kvb(WINDOW + 4))
    del kc, vc
    # ---- projection to heads and pages
    C = (H + 2 * G) * DIM
    nb = T // BS
    qkv = rnd(1, T, C)
    wn, cs = rnd(DIM), rnd(T, DIM // 2, dt=torch.float32)
    kc, vc = rnd(nb, BS, G, DIM), rnd(nb, BS, G, DIM)
    slots = torch.arange(T, dtype=torch.int32, device=dev)

    def dense_heads():
        fused.qk_norm_rope_(qkv, H, G, DIM, wq=wn, wk=wn, cos=cs, sin=cs, interleaved=False)
        x = qkv.view(T, C)
        KC.kv_write(x[:, H * DIM:(H + G) * DIM].view(T, G, DIM), x[:, (H + G) * DIM:].view(T, G, DIM), kc, vc, slots)
    row("heads and pages", "dense (two kernels)", dense_heads, bytes_=4.0 * T * C)
    hs = lm.HeadShape(H, G, DIM, DIM, DIM, DIM, 3)
    proj = rnd(T, C + H)
    seqs = SeqTable.build([T], [0], [list(range(nb))], [(0, 1)], dev)
    conv, nrm = rnd(3, C, dt=torch.float32), rnd(DIM, dt=torch.float32)
    state, vf = rnd(2, 2, C), rnd(T, G * DIM)
    row("heads and pages", "tavulix", lambda: lm.conv_heads(proj, hs, seqs, slots, kc, vc, conv=conv, state=state, q_norm=nrm,
                                                            k_norm=nrm, v_first=vf, v_mode="mix", lam=one),
        bytes_=4.0 * T * C + 2.0 * T * G * DIM)
    # ---- norms and activations
    x, y, xn = rnd(T, width, dt=torch.float32), rnd(T, width), rnd(T, width)
    wv = rnd(width)
    row("norm", "dense", lambda: fused.norm_modulate(y, weight=wv, rms=True, out=xn), bytes_=4.0 * T * width)
    row("norm", "tavulix (branch norm + add + norm, fp32 stream)", lambda: lm.add_norm_(x, y, one, width, 1e-5, xn, one),
        bytes_=12.0 * T * width)
    gu, z = rnd(T, 2 * F_), rnd(T, F_ * 3 // 2)
    h, z2 = rnd(T, F_), rnd(T, F_ * 3 // 2)
    row("activation", "dense (SwiGLU)", lambda: fused.silu_mul(gu, out=h), bytes_=6.0 * T * F_)
    coef = torch.tensor([0.5, 0.3, 0.1, 0.0], device=dev)
    row("activation", "tavulix (PolyNorm)", lambda: lm.poly_norm(z, coef, F_ * 3 // 2, 1e-5, out=z2), bytes_=6.0 * T * F_)
    ids, pos = torch.randint(0, VOCAB, (T,), device=dev), torch.arange(T, device=dev)
    emb, pt = rnd(VOCAB, width), rnd(T, width)
    row("embedding", "tavulix (table + position + norm)", lambda: lm.embed_norm(ids, pos, emb, pt, one, width, 1e-5),
        bytes_=10.0 * T * width)
    return out


def run(steps: int, warmup: int, widths, parts=("steps", "kernels"), design: str = "tavulix") -> dict:
    import importlib
    from ..ops import _native as nv
    tables = importlib.import_module({"nidilix": ".lm_nidilix", "milivik": ".lm_milivik", "fikizen": ".lm_fikizen"}.get(design, ".lm_layers"), __package__)
    timer = Timer(steps, warmup)
    n0 = nv.launch_count
    rec = {"metric": "lm_layers", "design": design, "unit": "tokens/s", "layers": LAYERS, "dtype": "bf16", "data": "synthetic (random weights)",
           "l2": "flushed (256 MB written) before every timed launch", "peaks": dict(zip(("bf16_tflops", "hbm_gbs", "source"), _peaks()))}
    if "kernels" in parts:
        rec["kernels"] = [r for w in widths for r in tables.kernel_rows(w, timer)]
    if "steps" in parts:
        rec["steps"] = [r for w in widths for r in tables.step_rows(w, timer)]
    rec["gpu_launches"] = nv.launch_count - n0
    nv.check_status()
    return rec
