"""Gated linear recurrence op (ops/recurrent.py) against the plain restatement: mixed batches, state pools with stale
contents, sizes that take each of its kernels, long memories."""
import pytest
import torch
import torch.nn.functional as F

import nidilix_oracle as O
from vllm_omni_b200.models.seq_table import SeqTable
from vllm_omni_b200.ops import recurrent as R

GPU = pytest.mark.gpu
MODES = [pytest.param(("cpu", torch.float32, 1e-4), id="cpu"), pytest.param(("cuda", torch.float32, 1e-4), id="fp32", marks=GPU),
         pytest.param(("cuda", torch.bfloat16, 0.02), id="bf16", marks=GPU)]
# width, blocks, taps
SIZES = {"base": (144, 3, 4), "one_block": (80, 1, 3), "full_part": (512, 2, 2), "no_history": (336, 4, 1), "many_taps": (48, 3, 6),
         "wide_part": (600, 2, 3), "padded_part": (36, 2, 3), "two_tiles": (340, 2, 4), "more_taps": (32, 2, 9)}


class Layer:
    def __init__(self, size, dtype, dev, seed=0, lam=None, bias=0.2):
        width, blocks, taps = size
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *sh: torch.randn(*sh, generator=g).bfloat16().double()
        self.s = s = R.GatedScanShape(width, blocks, taps)
        n = s.part
        self.w = (0.6 * rnd(width, taps), bias * rnd(width), (1.5 * n ** -0.5 * rnd(2, blocks, n, n)).bfloat16().double(),
                  rnd(2, blocks, n), rnd(width) - 2 if lam is None else torch.full((width,), lam).double())
        conv, conv_b, gates, gates_b, lam = self.w
        self.at = torch.cat([torch.arange(b * s.part_p, b * s.part_p + n) for b in range(blocks)])   # channels in the padded layout

        def pad(x):
            out = torch.zeros(*x.shape[:-1], s.channels)
            out[..., self.at] = x.float()
            return out.to(dev)
        self.pad = pad
        G = torch.zeros(2, blocks, s.part_p, s.part_p)
        G[:, :, :n, :n] = gates
        self.packed = (pad(conv.T), pad(conv_b), G.to(dev, dtype), pad(gates_b.reshape(2, -1)), pad(-8 * F.softplus(lam)))


def reference(layer, y, x):
    conv, conv_b, gates, gates_b, lam = layer.w
    u = O.causal_conv(x, conv, conv_b)
    r, i = (torch.sigmoid(O.block_linear(u, gates[k], gates_b[k])) for k in range(2))
    return O.rglru_scan(u, r, i, lam) * O.gelu_tanh(y)


def run(layer, data, rounds, mode, impl=None):
    dev, dtype, _ = mode
    s, n = layer.s, len(data)
    hist = torch.full((2 * n, s.taps - 1, s.channels), float("nan"), dtype=dtype, device=dev)       # stale contents
    state = torch.full((2 * n, s.channels), float("nan"), device=dev)
    at, phase, got = [0] * n, [0] * n, [[] for _ in data]
    for step in rounds:
        seqs = sorted(step)
        proj = torch.cat([torch.cat([layer.pad(t[at[i]:at[i] + step[i]]) for t in data[i]], dim=1) for i in seqs]).to(dev, dtype)
        states = [(2 * i + phase[i], 2 * i + 1 - phase[i]) for i in seqs]
        tab = SeqTable.build([step[i] for i in seqs], [at[i] for i in seqs], [[0]] * len(seqs), states, dev)
        out = R.gated_scan(proj, s, tab, *layer.packed, hist, state, impl=impl)
        o = 0
        for i in seqs:
            got[i].append(out[o:o + step[i]][:, layer.at.to(dev)].cpu())
            at[i] += step[i]
            phase[i] ^= 1
            o += step[i]
    return [torch.cat(g) for g in got]


def rows(layer, T, seed):
    g = torch.Generator().manual_seed(seed)
    return tuple(torch.randn(T, layer.s.width, generator=g).bfloat16().double() for _ in range(2))


def compare(got, want, tol):
    got = got.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    err = (got - want).norm(dim=1) / want.norm(dim=1).mean()
    assert err.max() < tol, f"row {int(err.argmax())}: {float(err.max()):.4g}"


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", sorted(SIZES))
def test_portions_beside_single_tokens(mode, name):
    layer = Layer(SIZES[name], mode[1], mode[0])
    data = [rows(layer, T, i) for i, T in enumerate((90, 41, 70, 1, 9))]
    rounds = [{0: 40, 1: 1, 3: 1, 4: 2}, {0: 1, 1: 33, 2: 5}, {0: 2, 1: 1, 2: 64, 4: 4}, {0: 46, 1: 1, 4: 3}, {0: 1, 1: 5, 2: 1}]
    for g, d in zip(run(layer, data, rounds, mode), data):
        compare(g, reference(layer, *d), mode[2])


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("cut", ["whole", "tokens", "runs"])
def test_several_runs(mode, cut):
    """Portions of several runs that hand their state on, and the same tokens cut otherwise."""
    layer = Layer(SIZES["base"], mode[1], mode[0], lam=-6.0)
    d = rows(layer, 700, 3)
    cuts = {"whole": [700], "tokens": [5] + [1] * 20 + [675], "runs": [128, 129, 2, 255, 31, 33, 122]}[cut]
    other = rows(layer, 300, 4)
    got = run(layer, [d, other], [{0: cuts[0], 1: 300}] + [{0: n} for n in cuts[1:]], mode)
    compare(got[0], reference(layer, *d), mode[2])
    compare(got[1], reference(layer, *other), mode[2])


@pytest.mark.parametrize("mode", MODES)
def test_long_memory(mode):
    """One large input early on, decays near one: what a far token left must still be there, across every border."""
    layer = Layer((64, 2, 3), mode[1], mode[0], lam=-9.5, bias=0.0)
    y, x = rows(layer, 520, 5)
    x = 0.02 * x
    x[3] = 8.0
    want = reference(layer, y, x)
    quiet = x.clone()
    quiet[3] = 0
    assert (want - reference(layer, y, quiet))[-20:].norm() > 0.7 * want[-20:].norm()     # the far token dominates
    for cuts in ([520], [2, 2, 124, 128, 200, 64], [4] + [1] * 60 + [456]):
        compare(run(layer, [(y, x)], [{0: n} for n in cuts], mode)[0], want, mode[2])


@pytest.mark.gpu
def test_many_tokens_and_plain_kernels():
    mode = ("cuda", torch.bfloat16, 0.02)
    layer = Layer((160, 2, 4), mode[1], mode[0])
    d = rows(layer, 4200, 6)                              # many runs
    want = reference(layer, *d)
    compare(run(layer, [d], [{0: 4199}, {0: 1}], mode)[0], want, mode[2])
    compare(run(layer, [d], [{0: 700}, {0: 3500}], mode, impl="plain")[0], want, mode[2])


@pytest.mark.gpu
def test_many_single_tokens():
    mode = ("cuda", torch.bfloat16, 0.02)
    layer = Layer((288, 2, 4), mode[1], mode[0])
    data = [rows(layer, 7, 10 + i) for i in range(37)]
    rounds = [{i: 1 for i in range(37)}] * 5 + [{i: 1 for i in range(0, 37, 2)}] * 2 + [{i: 2 for i in range(1, 37, 2)}]
    for g, d in zip(run(layer, data, rounds, mode), data):
        compare(g, reference(layer, *d), mode[2])


@pytest.mark.parametrize("mode", MODES)
def test_padding_rows_write_no_state(mode):
    dev, dtype, tol = mode
    layer = Layer((64, 2, 3), dtype, dev)
    s, d = layer.s, rows(layer, 1, 1)
    proj = torch.cat([layer.pad(t) for t in d], dim=1).repeat(3, 1).to(dev, dtype)
    hist = torch.zeros(4, 2, s.channels, dtype=dtype, device=dev)
    state = torch.zeros(4, s.channels, device=dev)
    tab = SeqTable.build([1, 1, 1], [0, 0, 0], [[0]] * 3, [(0, 1), (0, -1), (0, -1)], dev)
    out = R.gated_scan(proj, s, tab, *layer.packed, hist, state)
    assert torch.equal(out[0], out[1]) and torch.equal(out[0], out[2])
    assert state[1].abs().sum() > 0 and not state[[0, 2, 3]].any() and not hist[[0, 2, 3]].any()


def test_run_lengths():
    for lens in ([2], [31], [64], [65, 2], [4096], [4097], [9000], [100000], [1024] * 8, [300000, 5]):
        for tiles in (1, 16, 40, 200):
            L = R.run_length(lens, tiles)
            assert L % 64 == 0 and L >= 64 and -(-max(lens) // L) <= 64
    t = SeqTable.build([5, 1, 70], [0, 4, 9], [[0]] * 3, None, "cpu")
    runs, n, several = t.time_runs(0, lambda lens: 64)
    assert n == 3 and several and runs.tolist() == [[0, 0, 5, 0], [2, 0, 64, 1], [2, 64, 6, 1]]
