"""Row-wise decoder steps (embedding + norm, branch add + norm, PolyNorm, convolution + head norms + pages, bounded
logits) against the plain restatements, one mechanism at a time."""
import pytest
import torch

import fikizen_oracle as F
import milivik_oracle as M
import tavulix_oracle as O
from vllm_omni_b200.models.seq_table import SeqTable
from vllm_omni_b200.ops import lm

DEVICES = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="fp32", marks=pytest.mark.gpu),
           pytest.param("cuda", torch.bfloat16, id="bf16", marks=pytest.mark.gpu)]


def _close(got, want, dtype, scale=1.0):
    tol = scale * (2e-5 if dtype == torch.float32 else 1.2e-2)
    err = (got.double().cpu() - want.double()).abs()
    assert (err <= tol * (1 + want.double().abs())).all(), float(err.max())


def _pad(t, n):
    return torch.nn.functional.pad(t, (0, n - t.shape[-1]))


@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("width", [24, 100, 520, 4096])
@pytest.mark.parametrize("per_channel", [False, True])
def test_embed_norm(device, dtype, width, per_channel):
    torch.manual_seed(1)
    Wp = (width + 7) // 8 * 8
    table, pos = torch.randn(30, width).to(dtype), torch.randn(50, width).to(dtype)
    ids, at = torch.tensor([0, 29, 7, 7]), torch.tensor([0, 49, 3, 31])
    g = torch.rand(width) + 0.5 if per_channel else torch.tensor([1.3])
    x, xn = lm.embed_norm(ids.to(device), at.to(device), _pad(table, Wp).to(device), _pad(pos, Wp).to(device),
                          (_pad(g, Wp) if per_channel else g).to(device), width, 1e-2)
    want = table[ids].double() + pos[at].double()
    assert x.dtype == torch.float32
    _close(x[:, :width], want, torch.float32)
    _close(xn[:, :width], O.rms_unit(want, 1e-2) * g.double(), dtype)
    assert not x[:, width:].any() and not xn[:, width:].any()


@pytest.mark.parametrize("device,dtype", DEVICES)
def test_embed_overlay_replaces_rows(device, dtype):
    torch.manual_seed(2)
    table, over = torch.randn(10, 16).to(dtype), torch.randn(3, 16).to(dtype)
    ids, mask = torch.tensor([1, 2, 3]), torch.tensor([False, True, False])
    x, _ = lm.embed_norm(ids.to(device), ids.to(device), table.to(device), None, torch.ones(1, device=device), 16, 1e-6,
                         overlay=over.to(device), overlay_mask=mask.to(device))
    _close(x, torch.where(mask[:, None], over.double(), table[ids].double()), torch.float32)


@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("width", [20, 264, 2048, 6000])
def test_add_norm(device, dtype, width):
    """The branch is normed before it is added; eps counts, also for rows of zeros."""
    torch.manual_seed(3)
    Wp = (width + 7) // 8 * 8
    x0, y = torch.randn(5, width) * 4, (torch.randn(5, width) * 0.05).to(dtype)
    y[2] = 0
    g1, g2 = torch.tensor([0.7]), torch.tensor([1.9])
    x = _pad(x0, Wp).to(device)
    yy = torch.zeros(5, Wp + 8, dtype=dtype)
    yy[:, :width] = y
    xn = torch.empty(5, Wp, dtype=dtype, device=device)
    lm.add_norm_(x, yy.to(device), g1.to(device), width, 1e-3, xn, g2.to(device))
    want = x0.double() + O.rms_unit(y.double(), 1e-3) * 0.7
    _close(x[:, :width], want, torch.float32)
    _close(xn[:, :width], O.rms_unit(want, 1e-3) * 1.9, dtype)
    assert not xn[:, width:].any()
    x2 = _pad(x0, Wp).to(device)
    lm.add_norm_(x2, yy.to(device), g1.to(device), width, 1e-3)         # without a second norm
    assert torch.equal(x2, x)


@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("width", [12, 160, 1100, 12288])
def test_poly_norm(device, dtype, width):
    torch.manual_seed(4)
    Wp = (width + 7) // 8 * 8
    z = (torch.randn(4, width) * torch.tensor([[0.02], [1.0], [3.0], [0.0]])).to(dtype)
    coef = torch.tensor([0.6, -0.4, 0.3, 0.25])
    out = lm.poly_norm(_pad(z, Wp).to(device), coef.to(device), width, 1e-4)
    _close(out[:, :width], O.poly_norm(z.double(), coef.double(), 1e-4), dtype, scale=2)


@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("cap", [None, 5.0])
def test_logit_softcap(device, dtype, cap):
    torch.manual_seed(5)
    z = (torch.randn(3, 304) * 8).to(dtype)
    got = lm.logit_softcap(z.to(device), cap, 300)
    assert got.dtype == torch.float32 and got.shape == (3, 300)
    _close(got, O.soft_cap(z[:, :300].double(), cap), torch.float32)


# ------------------------------------------------------------------ convolution + heads + pages
class ConvCase:
    def __init__(self, shape, taps, dtype, device, norms=True, seed=0):
        H, G, d, dv = shape
        up = lambda n: (n + 15) // 16 * 16
        self.hs = lm.HeadShape(H, G, d, dv, up(d), up(dv), taps)
        self.dtype, self.device = dtype, device
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        self.rnd = rnd
        self.conv = rnd(taps, (H + G) * d + G * dv) if taps else None
        self.qn, self.kn = (rnd(d), rnd(d)) if norms else (None, None)
        self.lam = torch.tensor([0.35])

    def columns(self):
        """Places of the real channels (q, k, v heads) among the padded ones."""
        h, cols, o = self.hs, [], 0
        for heads, d, p in ((h.heads, h.dim, h.dp), (h.kv_heads, h.dim, h.dp), (h.kv_heads, h.vdim, h.vp)):
            for _ in range(heads):
                cols += range(o, o + d)
                o += p
        return torch.tensor(cols)

    def expected(self, u, v_first=None):
        h, f = self.hs, u.double()
        y = f if self.conv is None else O.causal_conv(f, self.conv.double().T)
        T = y.shape[0]
        q, k, v = y.split([h.heads * h.dim, h.kv_heads * h.dim, h.kv_heads * h.vdim], 1)
        q, k = q.reshape(T, h.heads, h.dim), k.reshape(T, h.kv_heads, h.dim)
        if self.qn is not None:
            q, k = O.rms_unit(q, 1e-5) * self.qn.double(), O.rms_unit(k, 1e-5) * self.kn.double()
        own = v.reshape(T, h.kv_heads, h.vdim)
        return q, k, own, own if v_first is None else O.mix_values(own, v_first.double(), self.lam.double())

    def run(self, us, cuts, mode="plain", v_firsts=None, order=None):
        """Feeds sequence s in portions cuts[s] (lists of equal length; 0 = sits out), all sequences of a round in
        one batch, through pages and state rows given out in a scrambled order.  Returns q, k, v, saved values."""
        h, bs, dev = self.hs, 8, self.device
        S, C = len(us), h.channels
        pages = [(u.shape[0] + bs - 1) // bs for u in us]
        ids = iter(torch.randperm(sum(pages) + 2, generator=torch.Generator().manual_seed(9)).tolist())
        tables = [[next(ids) for _ in range(n)] for n in pages]
        nb = sum(pages) + 2
        kc = torch.zeros(nb, bs, h.kv_heads, h.dp, dtype=self.dtype, device=dev)
        vc = torch.zeros(nb, bs, h.kv_heads, h.vp, dtype=self.dtype, device=dev)
        taps = h.taps
        state = torch.full((2 * S, taps - 1, C), 5.0, dtype=self.dtype, device=dev) if taps > 1 else None   # stale
        conv = qn = kn = None
        if self.conv is not None:
            conv = torch.zeros(taps, C)
            conv[:, self.columns()] = self.conv
            conv = conv.to(dev)
        if self.qn is not None:
            qn, kn = _pad(self.qn, h.dp).to(dev), _pad(self.kn, h.dp).to(dev)
        at, phase = [0] * S, [0] * S
        qs, saved = [[] for _ in us], [[] for _ in us]
        for rnd in zip(*cuts):
            live = [s for s in range(S) if rnd[s]]
            T = sum(rnd[s] for s in live)
            proj = torch.zeros(T, C + 8, dtype=self.dtype)
            vf = torch.zeros(T, h.kv_heads * h.vp, dtype=self.dtype)
            slots, o = [], 0
            for s in live:
                n = rnd[s]
                proj[o:o + n, self.columns()] = us[s][at[s]:at[s] + n]
                if v_firsts is not None:
                    vf.view(T, h.kv_heads, h.vp)[o:o + n, :, :h.vdim] = v_firsts[s][at[s]:at[s] + n]
                slots += [tables[s][t // bs] * bs + t % bs for t in range(at[s], at[s] + n)]
                o += n
            seqs = SeqTable.build([rnd[s] for s in live], [at[s] for s in live], [tables[s] for s in live],
                                  [(2 * s + phase[s], 2 * s + 1 - phase[s]) for s in live] if taps > 1 else None, dev)
            vf = vf.to(dev)
            q = lm.conv_heads(proj.to(dev), h, seqs, torch.tensor(slots, dtype=torch.int32, device=dev), kc, vc, conv=conv,
                              state=state, q_norm=qn, k_norm=kn, eps=1e-5, v_first=vf, v_mode=mode, lam=self.lam.to(dev))
            o = 0
            for s in live:
                n = rnd[s]
                qs[s].append(q[o:o + n, :, :h.dim].float().cpu())
                saved[s].append(vf.view(T, h.kv_heads, h.vp)[o:o + n, :, :h.vdim].float().cpu())
                at[s], phase[s], o = at[s] + n, phase[s] ^ 1, o + n
        out = []
        for s, u in enumerate(us):
            slot = torch.tensor([tables[s][t // bs] * bs + t % bs for t in range(u.shape[0])])
            k = kc.view(nb * bs, h.kv_heads, h.dp).cpu()[slot].float()
            v = vc.view(nb * bs, h.kv_heads, h.vp).cpu()[slot].float()
            assert not k[:, :, h.dim:].any() and not v[:, :, h.vdim:].any()
            out.append((torch.cat(qs[s]), k[:, :, :h.dim], v[:, :, :h.vdim], torch.cat(saved[s])))
        return out

    def inputs(self, lens):
        h = self.hs
        C = (h.heads + h.kv_heads) * h.dim + h.kv_heads * h.vdim
        return [self.rnd(n, C).to(self.dtype) for n in lens]



@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("taps", [0, 1, 2, 4, 7])
@pytest.mark.parametrize("cuts", [[[23], [9]], [[2] * 11 + [1], [0, 2, 2, 0, 0, 1, 1, 1, 2, 0, 0, 0]],
                                  [[10, 1, 1, 3, 2, 6], [1, 1, 0, 3, 0, 4]]], ids=["whole", "pairs", "mixed"])
def test_conv_heads_portions(device, dtype, taps, cuts):
    """The same rows whatever the cut: history comes from the portion, the state pool or (before the start) is zero."""
    c = ConvCase((4, 2, 24, 40), taps, dtype, device, seed=taps)
    us = c.inputs([23, 9])
    for u, (q, k, v, _) in zip(us, c.run(us, cuts)):
        eq, ek, _, ev = c.expected(u)
        for got, want in ((q, eq), (k, ek), (v, ev)):
            _close(got, want, dtype, scale=4)


@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("shape", [(1, 1, 16, 16), (6, 3, 20, 72), (2, 1, 128, 128), (2, 2, 136, 48), (3, 1, 272, 300)])
def test_conv_heads_sizes_and_value_mixing(device, dtype, shape):
    c = ConvCase(shape, 3, dtype, device, seed=11)
    us = c.inputs([19, 5])
    vf = [c.rnd(u.shape[0], shape[1], shape[3]).to(dtype) for u in us]
    cuts = [[7, 1, 9, 2], [2, 0, 2, 1]]
    for u, f, (q, k, v, _) in zip(us, vf, c.run(us, cuts, "mix", vf)):
        eq, ek, own, ev = c.expected(u, f)
        for got, want in ((q, eq), (k, ek), (v, ev)):
            _close(got, want, dtype, scale=4)
    for u, (_, _, v, saved) in zip(us, c.run(us, cuts, "save")):
        own = c.expected(u)[2]
        _close(saved, own, dtype, scale=4)
        _close(v, own, dtype, scale=4)


@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5])
def test_conv_heads_long_batches(device, dtype, taps):
    """Batches long enough for the sliding-window kernel; sequences of one to many rows meet inside its runs."""
    c = ConvCase((3, 1, 40, 24), taps, dtype, device, seed=20 + taps)
    lens = [300, 1, 2, 5, 129, 3]
    us = c.inputs(lens)
    vf = [c.rnd(u.shape[0], 1, 24).to(dtype) for u in us]
    cuts = [[290, 3, 7], [1, 0, 0], [2, 0, 0], [1, 4, 0], [3, 125, 1], [0, 2, 1]]
    for mode, first in (("plain", None), ("mix", vf)):
        for u, f, (q, k, v, _) in zip(us, vf, c.run(us, cuts, mode, first)):
            eq, ek, _, ev = c.expected(u, f if mode == "mix" else None)
            for got, want in ((q, eq), (k, ek), (v, ev)):
                _close(got, want, dtype, scale=4)


@pytest.mark.parametrize("device,dtype", DEVICES)
def test_conv_heads_without_norms(device, dtype):
    c = ConvCase((2, 1, 32, 16), 2, dtype, device, norms=False)
    us = c.inputs([6])
    q, k, v, _ = c.run(us, [[4, 2]])[0]
    eq, ek, _, ev = c.expected(us[0])
    for got, want in ((q, eq), (k, ek), (v, ev)):
        _close(got, want, dtype, scale=4)


@pytest.mark.gpu
@pytest.mark.parametrize("m,n,k", [(1, 8, 8), (3, 70, 40), (130, 64, 300)])
def test_fp32_linear_is_exact(m, n, k):
    from vllm_omni_b200.ops.gemm import linear
    torch.manual_seed(0)
    x, w, b = torch.randn(m, k), torch.randn(n, k), torch.randn(n)
    got = linear(x.cuda(), w.cuda(), b.cuda())
    want = x.double() @ w.double().T + b.double()
    assert (got.cpu().double() - want).abs().max() < 1e-5 * k ** 0.5
    assert torch.equal(linear(x[:1].cuda(), w.cuda(), b.cuda()), got[:1])       # a row alone: the same bits


@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("taps", [0, 3])
@pytest.mark.parametrize("coef,every", [(0.35, 50), (0.5, 1), (0.2, 7.0), (-0.1, 300)])
def test_queries_grow_with_the_position(device, dtype, taps, coef, every):
    """Fewer value heads than key heads; positions at both sides of a whole period, in portions and one by one."""
    c = ConvCase((4, 2, 20, 36), taps, dtype, device)
    c.hs = lm.HeadShape(8, 4, 20, 36, 32, 48, taps, v_heads=2)
    h = c.hs
    cols, o = [], 0
    for heads, d, p in ((8, 20, 32), (4, 20, 32), (2, 36, 48)):
        for _ in range(heads):
            cols += range(o, o + d)
            o += p
    assert o == h.channels
    T = 330
    u = torch.randn(T, len(cols), generator=torch.Generator().manual_seed(4)).bfloat16()
    w = torch.randn(max(taps, 1), len(cols), generator=torch.Generator().manual_seed(5))
    conv = state = None
    if taps:
        conv = torch.zeros(taps, h.channels)
        conv[:, cols] = w
        conv, state = conv.to(device), torch.zeros(2, taps - 1, h.channels, dtype=dtype, device=device)
    qn, kn = torch.rand(20) + 0.5, torch.rand(20) + 0.5
    kc, vc = (torch.full((T // 8 + 2, 8, 2, n), 5.0, dtype=dtype, device=device) for n in (64, 48))
    pages = torch.randperm(T // 8 + 2, generator=torch.Generator().manual_seed(6)).tolist()
    at, qs, phase = 0, [], 0
    for n in [1, 1, 2, 5, 290] + [1] * 31:
        proj = torch.zeros(n, h.channels + 8, dtype=dtype)
        proj[:, cols] = u[at:at + n].to(dtype)
        t = torch.arange(at, at + n)
        slots = (torch.tensor(pages)[t // 8] * 8 + t % 8).int().to(device)
        seqs = SeqTable.build([n], [at], [pages], [(phase, 1 - phase)], device)
        qs.append(lm.conv_heads(proj.to(device), h, seqs, slots, kc, vc, conv=conv, state=state, q_norm=_pad(qn, 32).to(device),
                                k_norm=_pad(kn, 32).to(device), eps=1e-5, growth=lm.QueryGrowth(coef, every)).float().cpu())
        at, phase = at + n, phase ^ 1
    y = O.causal_conv(u.double(), w.double().T) if taps else u.double()
    q, k, v = y.split([160, 80, 72], 1)
    q = O.rms_unit(q.reshape(T, 8, 20), 1e-5) * qn.double() * M.query_temperature(range(T), coef, every)[:, None, None]
    _close(torch.cat(qs)[..., :20], q, dtype, scale=3)
    flat = (torch.tensor(pages)[torch.arange(T) // 8] * 8 + torch.arange(T) % 8).to(device)
    _close(kc.view(-1, 4, 32)[flat][..., :20], O.rms_unit(k.reshape(T, 4, 20), 1e-5) * kn.double(), dtype)
    _close(vc.view(-1, 2, 48)[flat][..., :36], v.reshape(T, 2, 36), dtype)


@pytest.mark.parametrize("device,dtype", DEVICES)
def test_scaled_logits(device, dtype):
    z = (torch.randn(3, 304) * 8).to(dtype)
    _close(lm.logit_softcap(z.to(device), None, 300, 0.4), 0.4 * z[:, :300].double(), torch.float32)
    _close(lm.logit_softcap(z.to(device), 5.0, 300, 0.4), O.soft_cap(0.4 * z[:, :300].double(), 5.0), torch.float32)


# ------------------------------------------------------------------------------ row norms, rotation, pages
@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("shape", [(4, 2, 24, 20, 16), (3, 1, 18, 34, 18), (16, 4, 128, 128, 64), (6, 6, 10, 12, 2), (2, 1, 40, 136, 0), (40, 8, 128, 128, 128),
                                   (1, 1, 2, 1, 2)])
@pytest.mark.parametrize("normed", [False, True])
def test_rotary_heads(device, dtype, shape, normed):
    """Norms over all heads' channels at once, halves rotated against each other (stored as interleaved pairs), value heads
    over their root mean square; rows without a slot leave no trace in the pages."""
    from vllm_omni_b200.ops import stream
    H, G, d, dv, rot = shape
    T, BS, up = 11, 4, lambda n: (n + 15) // 16 * 16
    hs = lm.HeadShape(H, G, d, dv, up(d), up(dv))
    torch.manual_seed(H + d)
    q, k, v = torch.randn(T, H, d).to(dtype), torch.randn(T, G, d).to(dtype), (0.3 * torch.randn(T, G, dv)).to(dtype)
    order = torch.cat([torch.arange(rot).view(2, -1).T.reshape(-1), torch.arange(rot, d)]).long()      # stored channel <- checkpoint channel
    pos = torch.arange(T) * 37
    qg, kg = torch.rand(H, d) + 0.5, torch.rand(G, d) + 0.5
    pad = lambda x, n: _pad(x.float(), n).reshape(x.shape[0], -1)
    proj = torch.cat([pad(q[..., order], hs.dp), pad(k[..., order], hs.dp), pad(v, hs.vp), torch.full((T, 8), 5.0)], 1).to(device, dtype)
    slots = torch.randperm(16)[:T].int()
    slots[3] = -1
    kc, vc = (torch.full((4, BS, G, n), 9.0, dtype=dtype, device=device) for n in (hs.dp, hs.vp))
    turns = stream.rotary_rows(pos.to(device), 500.0, rot) if rot else None
    kw = dict(q_gain=_pad(qg[:, order], hs.dp).reshape(-1).to(device), k_gain=_pad(kg[:, order], hs.dp).reshape(-1).to(device), v_norm=True,
              v_mult=1.3, eps=1e-3) if normed else {}
    out = lm.rotary_heads(proj, hs, slots.to(device), kc, vc, turns, rot, **kw)
    qw, kw_, vw = q.double(), k.double(), v.double()
    if normed:
        qw = (F.rms_unit(qw.reshape(T, -1), 1e-3) * qg.double().reshape(-1)).reshape(T, H, d)
        kw_ = (F.rms_unit(kw_.reshape(T, -1), 1e-3) * kg.double().reshape(-1)).reshape(T, G, d)
        vw = 1.3 * F.rms_unit(vw, 1e-3)
    qw, kw_ = (F.rotate_halves(x, pos.double(), 500.0, rot)[..., order] if rot else x for x in (qw, kw_))
    _close(out[..., :d], qw, dtype)
    assert not out[..., d:].any()
    for t in range(T):
        if slots[t] < 0:
            continue
        page, at = divmod(int(slots[t]), BS)
        _close(kc[page, at, :, :d], kw_[t], dtype)
        _close(vc[page, at, :, :dv], vw[t], dtype)
    used = set(slots.tolist())
    for s in set(range(16)) - used:
        assert (kc.view(16, -1)[s] == 9).all() and (vc.view(16, -1)[s] == 9).all()


@pytest.mark.parametrize("device,dtype", DEVICES)
@pytest.mark.parametrize("rows", [3, 300])
def test_xielu_of_a_product(device, dtype, rows):
    """Small, ordinary and large arguments on either side of zero."""
    from vllm_omni_b200.ops import gemm
    torch.manual_seed(rows)
    x, w = torch.randn(rows, 40).to(dtype), torch.randn(56, 40).to(dtype)
    w *= torch.logspace(-6, 1, 56)[:, None].to(dtype)
    p, q = torch.tensor(0.7), torch.tensor(-0.4)
    coef = (float(F.softplus(p)), 0.5 + float(F.softplus(q)))
    z = x.double() @ w.double().T
    want = F.xielu(z, p.double(), q.double())
    got = gemm.linear(x.to(device), w.to(device), act="xielu", coef=coef).double().cpu()
    err = (got - want).abs() / (want.abs() + 1e-2 * torch.minimum(z.abs().mean(0), torch.ones(56)))
    assert err.max() < (2e-4 if dtype == torch.float32 else 0.02), float(err.max())


@pytest.mark.parametrize("device,dtype", DEVICES)
def test_tanh_of_columns(device, dtype):
    torch.manual_seed(5)
    x = (torch.randn(37, 40) * torch.logspace(-5, 1.5, 40)).to(dtype)
    _close(lm.tanh_cols(x.to(device)[:, 8:32]), torch.tanh(x[:, 8:32].double()), dtype)
