"""Windowed paged attention of mixed batches against the plain restatement: window edges, kept first tokens,
sinks, bounded scores, distance bias, gates, portions and decoded tokens, pages in any order."""
import pytest
import torch

import tavulix_oracle as O
from vllm_omni_b200.models.seq_table import SeqTable
from vllm_omni_b200.ops.window_attention import ScoreRule, bounded_scores, decode_splits, window_attention

BS = 16


def _up(n, m):
    return (n + m - 1) // m * m


class Case:
    """Sequences with random q / k / v; ``portions``: (tokens already in the cache, tokens of this step) each."""

    def __init__(self, shape, portions, window, keep, cap=None, bias=True, sink=True, gate=True, scale=None, seed=0,
                 block=BS):
        self.H, self.G, self.d, self.dv = shape
        self.portions, self.window, self.keep, self.cap, self.block = portions, window, keep, cap, block
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        self.scale = scale if scale is not None else 1.5 / self.d ** 0.5
        self.q = [rnd(c + n, self.H, self.d).bfloat16() for c, n in portions]
        self.k = [rnd(c + n, self.G, self.d).bfloat16() for c, n in portions]
        self.v = [rnd(c + n, self.G, self.dv).bfloat16() for c, n in portions]
        self.r1 = 0.3 + rnd(self.H).abs() if bias else None
        self.r2 = 0.05 + 0.3 * rnd(self.H).abs() if bias else None
        self.sink = 2 * rnd(self.H) if sink else None
        self.gate = [rnd(c + n, self.H).bfloat16() for c, n in portions] if gate else None
        self.g = g

    def expected(self):
        f = lambda t: None if t is None else t.double()
        out = []
        for s, (c, n) in enumerate(self.portions):
            o = O.attend(f(self.q[s]), f(self.k[s]), f(self.v[s]), scale=self.scale, cap=self.cap, r1=f(self.r1), r2=f(self.r2),
                         sink=f(self.sink), size=self.window, keep=self.keep)
            if self.gate is not None:
                o = o * torch.sigmoid(f(self.gate[s]))[:, :, None]
            out.append(o[c:])
        return torch.cat(out)

    def run(self, device, dtype, impl=None, spare=3, bounded=None):
        dp, vp, bs = _up(self.d, 16), _up(self.dv, 16), self.block
        need = [(c + n + bs - 1) // bs for c, n in self.portions]
        total = sum(need) + spare
        perm = torch.randperm(total, generator=self.g).tolist()
        kc = torch.full((total, bs, self.G, dp), 7.0)           # stale contents that must never be read as keys
        vc = torch.full((total, bs, self.G, vp), 7.0)
        tables, rows_q, rows_g = [], [], []
        for s, (c, n) in enumerate(self.portions):
            pages = [perm.pop() for _ in range(need[s])]
            tables.append(pages)
            for t in range(c + n):
                kc[pages[t // bs], t % bs] = 0
                vc[pages[t // bs], t % bs] = 0
                kc[pages[t // bs], t % bs, :, :self.d] = self.k[s][t].float()
                vc[pages[t // bs], t % bs, :, :self.dv] = self.v[s][t].float()
            rows_q.append(self.q[s][c:])
            rows_g.append(self.gate[s][c:] if self.gate is not None else None)
        q = torch.cat(rows_q).float()
        T = q.shape[0]
        qp = torch.zeros(T, self.H, dp)
        qp[:, :, :self.d] = q
        seqs = SeqTable.build([n for _, n in self.portions], [c for c, _ in self.portions], tables, None, device)
        mv = lambda t: None if t is None else t.float().to(device)
        rule = ScoreRule(self.scale, self.cap, mv(self.r1), mv(self.r2), mv(self.sink), self.window, self.keep,
                         bounded=bounded_scores(self.cap, self.r1, self.r2) if bounded is None else bounded)
        out = torch.full((T, self.H * vp), float("nan"), dtype=dtype, device=device)
        gate = torch.cat(rows_g).to(device, dtype) if self.gate is not None else None
        window_attention(qp.to(device, dtype), kc.to(device, dtype), vc.to(device, dtype), seqs, rule, out, gate=gate, impl=impl)
        return out.float().cpu().view(T, self.H, vp)[:, :, :self.dv]


def _check(case, got, tol):
    want = case.expected()
    err = (got.double() - want).abs()
    lim = tol * (1.0 + want.abs())
    assert torch.isfinite(got).all()
    assert (err <= lim).all(), f"max error {err.max():.4g} at {(err - lim).argmax()}"


MIXED = [(0, 70), (130, 1), (40, 33), (0, 1), (300, 2), (17, 1)]
CASES = {
    "grouped": dict(shape=(12, 3, 80, 48), portions=MIXED, window=40, keep=7, cap=9.0),
    "odd_sizes": dict(shape=(6, 2, 40, 24), portions=MIXED, window=33, keep=5, cap=9.0),
    "one_head_per_group": dict(shape=(4, 4, 64, 32), portions=MIXED, window=20, keep=3, cap=4.0),
    "three_per_group": dict(shape=(3, 1, 16, 16), portions=[(5, 100), (200, 1)], window=50, keep=0, cap=5.0),
    "no_window": dict(shape=(4, 1, 32, 48), portions=MIXED, window=None, keep=0),
    "window_of_one": dict(shape=(4, 2, 32, 32), portions=MIXED, window=1, keep=2, cap=3.0),
    "window_of_one_alone": dict(shape=(4, 2, 32, 32), portions=MIXED, window=1, keep=0),
    "many_kept": dict(shape=(8, 2, 32, 32), portions=[(0, 400), (390, 1), (500, 40)], window=37, keep=150, cap=6.0),
    "plain": dict(shape=(8, 2, 64, 64), portions=MIXED, window=64, keep=4, bias=False, sink=False, gate=False),
    "bias_only": dict(shape=(8, 2, 64, 64), portions=MIXED, window=64, keep=4, sink=False, gate=False),
    "cap_only": dict(shape=(8, 2, 64, 64), portions=MIXED, window=64, keep=4, cap=2.0, bias=False, sink=False),
    "wide_group": dict(shape=(20, 1, 64, 80), portions=MIXED, window=45, keep=6, cap=9.0),
    "very_wide_group": dict(shape=(24, 1, 32, 16), portions=[(0, 50), (120, 1), (64, 1)], window=45, keep=6, cap=9.0),
    "page_of_8": dict(shape=(12, 3, 80, 48), portions=MIXED, window=40, keep=7, cap=9.0, block=8),
    "page_of_64": dict(shape=(12, 3, 80, 48), portions=MIXED, window=40, keep=7, cap=9.0, block=64),
}


@pytest.mark.parametrize("name", sorted(CASES))
def test_mixed_batch_cpu(name):
    c = Case(**CASES[name])
    _check(c, c.run("cpu", torch.float32), 2e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("name", sorted(CASES))
def test_mixed_batch_fp32_gpu(name):
    c = Case(**CASES[name])
    _check(c, c.run("cuda", torch.float32), 2e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("name", sorted(CASES))
def test_mixed_batch_bf16_gpu(name):
    c = Case(**CASES[name])
    _check(c, c.run("cuda", torch.bfloat16), 0.02)
    torch.cuda.synchronize()
    from vllm_omni_b200.ops import _native as nv
    nv.check_status()


LARGE = {
    "full_heads": dict(shape=(16, 2, 128, 128), portions=[(0, 300), (450, 1), (1000, 1), (700, 64)], window=256, keep=4, cap=20.0),
    "ungrouped_128": dict(shape=(2, 2, 128, 128), portions=[(100, 300), (450, 1)], window=200, keep=130, cap=20.0),
    "wide_keys": dict(shape=(4, 2, 256, 128), portions=[(60, 200), (330, 1)], window=150, keep=9, cap=20.0),
    "wide_keys_192": dict(shape=(4, 2, 192, 64), portions=[(60, 200), (330, 1)], window=150, keep=9, cap=20.0),
    "wide_values": dict(shape=(4, 2, 64, 256), portions=[(60, 40), (330, 1)], window=50, keep=9, cap=20.0),
    "huge_heads": dict(shape=(2, 1, 320, 272), portions=[(60, 40), (330, 1)], window=50, keep=9, cap=20.0),
    "long_decode": dict(shape=(8, 2, 128, 128), portions=[(3000, 1), (2047, 1), (15, 1)], window=None, keep=0, cap=15.0),
}


@pytest.mark.gpu
@pytest.mark.parametrize("name", sorted(LARGE))
def test_large_heads_bf16_gpu(name):
    c = Case(**LARGE[name])
    _check(c, c.run("cuda", torch.bfloat16), 0.02)


@pytest.mark.gpu
@pytest.mark.parametrize("name", [n for n in sorted(CASES) if CASES[n].get("cap")])
def test_bounded_and_running_maximum_agree(name):
    c = Case(**CASES[name])
    assert bounded_scores(c.cap, c.r1, c.r2)
    for bounded in (True, False):
        _check(c, c.run("cuda", torch.bfloat16, bounded=bounded), 0.02)


def test_when_the_cap_may_be_the_reference():
    one = torch.ones(3)
    assert bounded_scores(20.0) and not bounded_scores(None) and not bounded_scores(40.0)
    assert bounded_scores(20.0, one, one) and not bounded_scores(20.0, -one, one) and not bounded_scores(20.0, one, -one)


@pytest.mark.gpu
@pytest.mark.parametrize("cap", [31.0, 60.0])
def test_far_apart_scores(cap):
    """Rows whose visible scores all sit near -cap or near +cap, with large biases: both references give the rows."""
    for sign in (-1.0, 1.0):
        c = Case((4, 2, 64, 32), [(500, 90), (800, 1)], 300, 4, cap=cap, scale=1.0, seed=8)
        c.r1 = torch.full((4,), 6.0)
        for s in range(2):
            c.q[s] = c.q[s].abs()
            c.k[s] = (sign * c.k[s].float().abs()).bfloat16()
        c.sink = torch.full((4,), -200.0)
        _check(c, c.run("cuda", torch.bfloat16), 0.02)


@pytest.mark.gpu
def test_rows_kernel_agrees_in_bf16():
    c = Case(**CASES["grouped"])
    _check(c, c.run("cuda", torch.bfloat16, impl="rows"), 0.02)


DEVICES = [pytest.param("cpu", torch.float32, 1e-3), pytest.param("cuda", torch.float32, 1e-3, marks=pytest.mark.gpu),
           pytest.param("cuda", torch.bfloat16, 0.03, marks=pytest.mark.gpu)]


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("context,n", [(150, 1), (120, 31), (0, 151)])
def test_edges_stand_out(device, dtype, tol, context, n):
    """One key carries nearly all the weight if it is seen: placed just inside and just outside the window, at
    the last kept token and the first one that is not, and at page borders."""
    window, keep, i = 40, 5, 150
    for j in (0, keep - 1, keep, keep + 1, 15, 16, 31, 32, i - window - 1, i - window, i - window + 1, 127, 128, i - 1, i):
        c = Case((2, 1, 32, 16), [(context, n)], window, keep, bias=False, sink=False, gate=False, scale=1.0, seed=3)
        for h in range(2):
            c.q[0][i, h] = 0
            c.q[0][i, h, 0] = 6
        c.k[0] *= 0.05
        c.k[0][j, 0, 0] = 3
        c.v[0] *= 0.01
        c.v[0][j, 0, 0] = 1
        got = c.run(device, dtype)[i - context, 0, 0].item()
        seen = O.visible(i, j, window, keep)
        assert abs(got - (1.0 if seen else 0.0)) < max(tol, 0.02), (j, got, seen)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
@pytest.mark.parametrize("level", [-30.0, 0.0, 40.0])
def test_sink_takes_its_share(device, dtype, tol, level):
    c = Case((4, 2, 32, 16), [(0, 40), (60, 1)], 25, 3, cap=8.0, seed=5)
    c.sink = torch.full((4,), level)
    got = c.run(device, dtype)
    _check(c, got, tol)
    if level == 40.0:
        assert got.abs().max() < 1e-6
    c.sink = None
    free = c.run(device, dtype)
    if level == -30.0:
        assert (free - got).abs().max() < tol


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_bounded_scores_saturate(device, dtype, tol):
    c = Case((4, 2, 32, 16), [(10, 50), (80, 1)], 30, 4, cap=1.5, scale=30.0, seed=6)
    _check(c, c.run(device, dtype), tol)


@pytest.mark.parametrize("device,dtype,tol", DEVICES)
def test_distance_bias_far_key(device, dtype, tol):
    """A kept token hundreds of positions back competes with the window: its bias must use the true distance."""
    c = Case((2, 1, 32, 16), [(600, 1), (590, 12)], 20, 2, scale=1.0, sink=False, gate=False, seed=7)
    c.r1, c.r2 = torch.tensor([1.0, 2.2]), torch.tensor([0.5, 0.08])
    for s, at in ((0, 600), (1, 601)):
        c.q[s][at] = 0
        c.q[s][at, :, 0] = 4
        c.k[s] *= 0.1
        c.k[s][0, 0, 0] = 1.5
    _check(c, c.run(device, dtype), tol)


def test_decode_split_count():
    assert decode_splits(1, 1, 4, 10) == 1                       # few keys: one block
    assert decode_splits(1, 2, 4, 4096) == 32
    assert decode_splits(64, 8, 4, 4096) == 1                    # the batch fills the GPU by itself
    assert decode_splits(1, 8, 4, 100) == 2


def test_seq_table_layout():
    t = SeqTable.build([3, 1, 5], [10, 4, 0], [[7], [2, 9], [1]], [(0, 1), (5, 4), (2, 3)], "cpu")
    assert t.q_start.tolist() == [0, 3, 4, 9] and t.row_seq.tolist() == [0, 0, 0, 1, 2, 2, 2, 2, 2]
    assert t.block_tables.tolist() == [[7, 0], [2, 9], [1, 0]] and t.decode_list.tolist() == [1]
    assert t.state_in.tolist() == [0, 5, 2] and t.state_out.tolist() == [1, 4, 3] and t.max_context == 4
    items, n = t.prefill_items(2)
    assert n == 5 and sorted(map(tuple, items.tolist())) == [(0, 0), (0, 2), (2, 0), (2, 2), (2, 4)]
