"""Delta-rule recurrences (ops/delta_rule.py) against the plain restatement: mixed batches, pools with stale contents, sizes
that take each of the kernels, long memories, decays and keys at the ends of their ranges; the short convolution alone."""
import math

import pytest
import torch

import fikizen_oracle as O
from vllm_omni_b200.models.seq_table import SeqTable
from vllm_omni_b200.ops import delta_rule as D
from vllm_omni_b200.ops.short_conv import conv_rows

GPU = pytest.mark.gpu
MODES = [pytest.param(("cpu", torch.float32, 5e-5), id="cpu"), pytest.param(("cuda", torch.float32, 5e-5), id="fp32", marks=GPU),
         pytest.param(("cuda", torch.bfloat16, 0.02), id="bf16", marks=GPU)]
EPS = 1e-4
# heads, key heads, key channels, value channels, taps
GATED = {"base": (6, 3, 24, 40, 4), "keys64": (4, 2, 64, 56, 3), "keys96": (2, 1, 90, 72, 2), "keys128": (3, 3, 128, 128, 4),
         "no_history": (2, 1, 40, 24, 1), "many_taps": (4, 2, 20, 28, 7), "wide_state": (2, 1, 200, 136, 2), "one_key": (5, 1, 1, 17, 3),
         "wide_values": (1, 1, 32, 600, 2), "one_value": (2, 2, 30, 1, 2), "too_wide": (1, 1, 300, 32, 2)}
SIGNS = "one_value"           # a norm over one channel gives its sign, which bf16 may turn
# heads, channels
CHANNEL = {"base": (3, 20), "dim64": (5, 64), "dim96": (2, 96), "dim128": (2, 120), "small_chunks": (1, 200), "widest": (1, 256), "one": (2, 1)}


class Gated:
    """Random weights and the packed layout of a gated rule."""

    def __init__(self, size, dtype, dev, seed=0, rate=None):
        H, G, d, dv, taps = size
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *sh: torch.randn(*sh, generator=g)
        self.s = s = D.DeltaShape(H, G, d, dv, taps)
        self.conv = [(0.7 * rnd(n, taps)).bfloat16().double() for n in (G * d, G * d, H * dv)]
        self.a_log = (0.5 * rnd(H) if rate is None else torch.full((H,), math.log(rate))).double()
        self.dt = (0.5 * rnd(H)).bfloat16().double()
        self.gain = (0.5 + torch.rand(dv, generator=g)).bfloat16().double()
        q, v = self.slots(d, s.dp, G), self.slots(dv, s.vp, H)
        self.at = [q, s.q_cols + q, 2 * s.q_cols + v, s.channels + v, s.channels + s.v_cols + torch.arange(H),
                   s.channels + s.v_cols + H + torch.arange(H)]                       # columns of q, k, v, gate, b, a
        self.cols = (s.channels + s.v_cols + 2 * H + 7) // 8 * 8
        self.out_at = v
        conv = torch.zeros(taps, s.channels)
        for c, at in zip(self.conv, self.at):
            conv[:, at] = c.T.float()
        gain = torch.zeros(s.vp)
        gain[:dv] = self.gain.float()
        f = lambda t: t.float().to(dev)
        self.rule = D.GatedDelta(conv.to(dev), f(-torch.exp(self.a_log)), f(self.dt), gain.to(dev), EPS)
        self.sizes = [G * d, G * d, H * dv, H * dv, H, H]

    @staticmethod
    def slots(n, pad, heads):
        return torch.cat([torch.arange(h * pad, h * pad + n) for h in range(heads)])

    def rows(self, T, seed):
        g = torch.Generator().manual_seed(100 + seed)
        return [torch.randn(T, n, generator=g).bfloat16().double() for n in self.sizes]

    def expected(self, parts):
        s, T = self.s, parts[0].shape[0]
        q, k, v = (O.silu(O.causal_conv(x, c)) for x, c in zip(parts, self.conv))
        R = s.heads // s.kv_heads
        q = O.unit(q.reshape(T, s.kv_heads, -1)).repeat_interleave(R, 1) * s.dim ** -0.5
        k = O.unit(k.reshape(T, s.kv_heads, -1)).repeat_interleave(R, 1)
        g = torch.exp(-torch.exp(self.a_log) * O.softplus(parts[5] + self.dt))
        o = O.gated_delta(q, k, v.reshape(T, s.heads, -1), g, O.sigmoid(parts[4]))
        return (O.rms_unit(o, EPS) * self.gain * O.silu(parts[3]).reshape(o.shape)).reshape(T, -1)

    def operands(self, parts, dtype, dev):
        x = torch.zeros(parts[0].shape[0], self.cols)
        for p, at in zip(parts, self.at):
            x[:, at] = p.float()
        return dict(proj=x.to(dev, dtype))


class Channel:
    """The same for decays per channel."""

    def __init__(self, size, dtype, dev, seed=0):
        H, d = size
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *sh: torch.randn(*sh, generator=g).bfloat16().double()
        self.s = s = D.DeltaShape(H, H, d, d)
        self.w0, self.ab, self.gain = rnd(H * d), rnd(H * d), 0.5 + rnd(H * d).abs()
        at = Gated.slots(d, s.dp, H)
        self.out_at, self.col, self.cols, self.sizes = at, at, 5 * s.q_cols, [H * d] * 6

        def pad(x):
            out = torch.zeros(*x.shape[:-1], s.q_cols)
            out[..., at] = x.float()
            return out
        self.pad = pad
        self.rule = D.ChannelDelta(pad(self.w0).to(dev), pad(self.ab).to(dev), -math.exp(-0.5), pad(self.gain).to(dev), EPS)

    rows = Gated.rows

    def expected(self, parts):
        r, k, v, a, gate, z = parts
        heads = lambda x: x.reshape(x.shape[0], self.s.heads, -1)
        w = torch.exp(-math.exp(-0.5) * O.sigmoid(z + self.w0))
        o = O.channel_delta(heads(r), heads(k), heads(v), heads(w), heads(O.sigmoid(a + self.ab)))
        return O.rms_unit(o, EPS).reshape(r.shape) * self.gain * O.sigmoid(gate)

    def operands(self, parts, dtype, dev):
        return dict(proj=torch.cat([self.pad(p) for p in parts[:5]], dim=1).to(dev, dtype), decay=self.pad(parts[5]).to(dev, dtype))


LAYERS = [pytest.param(Gated, size, id=f"gated-{n}") for n, size in GATED.items()] + \
         [pytest.param(Channel, size, id=f"channel-{n}") for n, size in CHANNEL.items()]


def run(layer, data, rounds, mode, impl=None):
    """``rounds``: lists of {sequence: tokens of this step}; the pools start with NaN."""
    dev, dtype, _ = mode
    s, n = layer.s, len(data)
    hist = torch.full((2 * n, s.taps - 1, s.channels), float("nan"), dtype=dtype, device=dev)
    state = torch.full((2 * n, s.heads, s.dp, s.vp), float("nan"), device=dev)
    at, phase, got = [0] * n, [0] * n, [[] for _ in data]
    for step in rounds:
        seqs = sorted(step)
        ops = [layer.operands([t[at[i]:at[i] + step[i]] for t in data[i]], dtype, dev) for i in seqs]
        ops = {k: torch.cat([o[k] for o in ops]) for k in ops[0]}
        states = [(2 * i + phase[i], 2 * i + 1 - phase[i]) for i in seqs]
        tab = SeqTable.build([step[i] for i in seqs], [at[i] for i in seqs], [[0]] * len(seqs), states, dev)
        wide = torch.full((ops["proj"].shape[0], s.v_cols + 16), float("nan"), dtype=dtype, device=dev)
        out = D.delta_rule(ops.pop("proj"), s, tab, layer.rule, state, wide[:, 8:8 + s.v_cols], hist=hist, impl=impl, **ops)
        o = 0
        for i in seqs:
            got[i].append(out[o:o + step[i]][:, layer.out_at.to(dev)].cpu())
            at[i] += step[i]
            phase[i] ^= 1
            o += step[i]
        assert not wide[:, :8].isfinite().any() and not wide[:, 8 + s.v_cols:].isfinite().any()
    return [torch.cat(g) for g in got]


def compare(got, want, tol):
    got = got.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    err = (got - want).norm(dim=1) / want.norm(dim=1).mean()
    assert err.max() < tol, f"row {int(err.argmax())}: {float(err.max()):.4g}"


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("kind,size", LAYERS)
def test_portions_beside_single_tokens(mode, kind, size):
    if size is GATED[SIGNS] and mode[1] == torch.bfloat16:
        pytest.skip("signs")
    layer = kind(size, mode[1], mode[0])
    data = [layer.rows(T, i) for i, T in enumerate((70, 41, 52, 1, 9))]
    rounds = [{0: 35, 1: 1, 3: 1, 4: 2}, {0: 1, 1: 33, 2: 5}, {0: 2, 1: 1, 2: 46, 4: 4}, {0: 31, 1: 1, 4: 3}, {0: 1, 1: 5, 2: 1}]
    for g, d in zip(run(layer, data, rounds, mode), data):
        compare(g, layer.expected(d), mode[2])


CUTS = {"whole": [150], "tokens": [3] + [1] * 30 + [117], "chunk_edges": [32, 31, 33, 16, 17, 15, 2, 4], "pairs": [2] * 75}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("cut", sorted(CUTS))
@pytest.mark.parametrize("kind,size", [pytest.param(Gated, GATED["keys64"], id="gated"), pytest.param(Channel, CHANNEL["dim64"], id="channel")])
def test_cuts_of_a_prompt(mode, cut, kind, size):
    layer = kind(size, mode[1], mode[0])
    d = layer.rows(150, 3)
    compare(run(layer, [d], [{0: n} for n in CUTS[cut]], mode)[0], layer.expected(d), mode[2])


@pytest.mark.gpu
@pytest.mark.parametrize("kind,size", [p for p in LAYERS if p.values[1] is not GATED[SIGNS]])
def test_chunks_equal_steps(kind, size):
    """The chunked kernels and the token-by-token one agree to what bf16 convolution results leave."""
    mode = ("cuda", torch.bfloat16, 0.03 if kind is Gated else 0.006)
    layer = kind(size, mode[1], mode[0], seed=2)
    data = [layer.rows(T, 7 + T) for T in (67, 18)]
    rounds = [{0: 40, 1: 16}, {0: 27, 1: 2}]
    for a, b in zip(run(layer, data, rounds, mode), run(layer, data, rounds, mode, impl="steps")):
        compare(a, b.double(), mode[2])


@pytest.mark.gpu
@pytest.mark.parametrize("kind,size", [pytest.param(Gated, (4, 2, 128, 64, 2), id="gated"), pytest.param(Channel, (4, 64), id="channel")])
def test_many_portions_at_once(kind, size):
    """So many that a warp has its columns to itself; a few of them are alike and must stay so."""
    mode = ("cuda", torch.bfloat16, 0.02)
    layer = kind(size, mode[1], mode[0])
    data = [layer.rows(35 + i % 40, i % 50) for i in range(100)]
    got = run(layer, data, [{i: 20 + i % 7 for i in range(100)}, {i: 15 + i % 40 - i % 7 for i in range(100)}], mode)
    for i in (0, 13, 49, 99):
        compare(got[i], layer.expected(data[i]), mode[2])


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("cut", ["whole", "tokens", "chunks"])
def test_far_write_is_still_there(mode, cut):
    """A key that only token 5 and the last token use, decays near one: what the far token wrote is what the last one reads."""
    layer = Gated((2, 1, 32, 24, 2), mode[1], mode[0], rate=1e-4)
    T = 200
    for c in layer.conv:                                     # the convolution passes the current token
        c.zero_()
        c[:, -1] = 1
    layer.rule.conv[:-1] = 0
    layer.rule.conv[-1] = 1
    q, k, v, gate, b, a = layer.rows(T, 3)
    k = -30 + 0 * k                                          # silu leaves nothing
    k[:, :16] = 3 * torch.randn(T, 16, generator=torch.Generator().manual_seed(1)).abs().bfloat16().double()
    for t in (5, T - 1):
        k[t] = -30
        k[t, 20] = 6
    q[T - 1] = -30
    q[T - 1, 20] = 6
    b[:] = 4
    d = [q, k, v, gate, b, a]
    want = layer.expected(d)
    other = [x.clone() for x in d]
    other[2][5] = -other[2][5] + 1
    # the last token's own value is a small part of what it reads
    b[T - 1] = other[4][T - 1] = -6
    want, moved = layer.expected(d), layer.expected(other)
    assert (want[-1] - moved[-1]).norm() > 0.5 * want[-1].norm()
    cuts = {"whole": [T], "tokens": [6] + [1] * 40 + [153] + [1], "chunks": [5, 32, 64, 33, 50, 14, 2]}[cut]
    got = run(layer, [d], [{0: n} for n in cuts], mode)[0]
    compare(got, want, mode[2])
    assert (got[-1].double() - want[-1]).norm() < 2 * mode[2] * want[-1].norm()


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("rate", [1e-6, 200.0])
def test_slow_and_immediate_decay(mode, rate):
    layer = Gated(GATED["keys64"], mode[1], mode[0], rate=rate)
    d = layer.rows(80, 5)
    compare(run(layer, [d], [{0: 75}] + [{0: 1}] * 5, mode)[0], layer.expected(d), mode[2])


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("z", [-40.0, 40.0])
def test_closed_and_open_channel_decay(mode, z):
    """No decay at all, and the fastest one over several chunks; zero keys have no direction and must not divide by zero."""
    layer = Channel(CHANNEL["dim64"], mode[1], mode[0])
    d = layer.rows(100, 6)
    d[5] = torch.full_like(d[5], z)
    d[1][10:14] = 0
    d[3] -= 1                                                # removal rates well below one keep an undecayed state bounded
    compare(run(layer, [d], [{0: 97}] + [{0: 1}] * 3, mode)[0], layer.expected(d), mode[2])


@pytest.mark.gpu
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("act", [None, "silu"])
@pytest.mark.parametrize("biased", [False, True])
def test_short_convolution(taps, act, biased):
    C, lens, total = 40, [(9, 1, 20), (1, 12, 3)], 0
    g = torch.Generator().manual_seed(taps)
    w, bias = torch.randn(C, taps, generator=g), torch.randn(C, generator=g) if biased else None
    data = [torch.randn(sum(n), C, generator=g).bfloat16() for n in zip(*lens)]
    hist = torch.full((2 * len(data), taps - 1, C), float("nan"), dtype=torch.bfloat16, device="cuda")
    at, got = [0] * len(data), [[] for _ in data]
    for step, n in enumerate(lens):
        x = torch.cat([torch.nn.functional.pad(d[a:a + m], (0, 8)) for d, a, m in zip(data, at, n)]).cuda()
        tab = SeqTable.build(list(n), at, [[0]] * len(n), [(2 * i + step, 2 * i + 1 - step) for i in range(len(n))], "cuda")
        y = conv_rows(x, tab, taps, C, w.T.contiguous().cuda(), hist if taps > 1 else None, bias=None if bias is None else bias.cuda(), act=act)
        for i, part in enumerate(y.split(list(n))):
            got[i].append(part.cpu())
            at[i] += n[i]
    for d, parts in zip(data, got):
        want = O.causal_conv(d.double(), w.double()) + (0 if bias is None else bias.double())
        want = O.silu(want) if act else want
        assert (torch.cat(parts).double() - want).abs().max() < 0.02 * want.abs().max()


def test_single_rows_leave_history_alone():
    """With ``skip_single`` the decode kernel, not the convolution, moves a one-row sequence's history."""
    layer = Gated(GATED["base"], torch.float32, "cpu")
    d = layer.rows(30, 1)
    compare(run(layer, [d, d], [{0: 20, 1: 1}, {0: 1, 1: 20}, {0: 9, 1: 9}], ("cpu", torch.float32, 0))[1], layer.expected(d), 5e-5)
