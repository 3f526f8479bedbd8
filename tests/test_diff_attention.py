"""Attention with two maps per head over the same values (ops/window_attention.py, ``ScoreRule.diff``) against the plain
restatement: mixed batches over shuffled pages, sizes that take each of its kernels, maps that look at chosen keys."""
import pytest
import torch

import milivik_oracle as O
from vllm_omni_b200.models.seq_table import SeqTable
from vllm_omni_b200.ops.window_attention import DiffRule, ScoreRule, window_attention

GPU = pytest.mark.gpu
MODES = [pytest.param(("cpu", torch.float32, 2e-4), id="cpu"), pytest.param(("cuda", torch.float32, 2e-4), id="fp32", marks=GPU),
         pytest.param(("cuda", torch.bfloat16, 0.025), id="bf16", marks=GPU)]
EPS = 1e-3


def up16(n):
    return (n + 15) // 16 * 16


class Case:
    """``portions``: (tokens already in the cache, tokens of this step) per sequence."""

    def __init__(self, shape, portions, lam=0.7, diff=0.4, gate=True, window=None, scale=None, seed=0, block=16):
        self.H, self.G, self.d, self.dv = shape
        self.portions, self.lam, self.diff, self.window, self.block = portions, lam, diff, window, block
        self.g = g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g).bfloat16()
        self.scale = scale if scale is not None else 1.5 / self.d ** 0.5
        self.q = [rnd(c + n, self.H, 2, self.d) for c, n in portions]
        self.k = [rnd(c + n, self.G, 2, self.d) for c, n in portions]
        self.v = [rnd(c + n, self.G, self.dv) for c, n in portions]
        self.gate = [rnd(c + n, self.H) for c, n in portions] if gate else None

    def expected(self):
        out = []
        for s, (c, n) in enumerate(self.portions):
            a = O.attend_maps(self.q[s].double(), self.k[s].double(), self.v[s].double(), self.scale, O.visible(c + n, self.window))
            o = O.combine_maps(a, self.lam, self.diff, EPS)
            if self.gate is not None:
                o = o * torch.sigmoid(self.gate[s].double())[:, :, None]
            out.append(o[c:])
        return torch.cat(out)

    def run(self, device, dtype, impl=None):
        H, G, R, dp, vp, bs = self.H, self.G, self.H // self.G, up16(self.d), up16(self.dv), self.block
        need = [(c + n + bs - 1) // bs for c, n in self.portions]
        total = sum(need) + 3
        perm = torch.randperm(total, generator=self.g).tolist()
        kc = torch.full((total, bs, G, 2, dp), 7.0)             # stale contents that must never be read as keys
        vc = torch.full((total, bs, G, vp), 7.0)
        tables, rows_q, rows_g = [], [], []
        for s, (c, n) in enumerate(self.portions):
            pages = [perm.pop() for _ in range(need[s])]
            tables.append(pages)
            at = torch.tensor(pages)[torch.arange(c + n) // bs], torch.arange(c + n) % bs
            kc[at], vc[at] = 0.0, 0.0
            kc[(*at, slice(None), slice(None), slice(0, self.d))] = self.k[s].float()
            vc[(*at, slice(None), slice(0, self.dv))] = self.v[s].float()
            rows_q.append(self.q[s][c:])
            rows_g.append(self.gate[s][c:] if self.gate is not None else None)
        q = torch.cat(rows_q).float()
        T = q.shape[0]
        qp = torch.zeros(T, G, 2, R, dp)                        # heads in the order (KV head, map, head of the group)
        qp[..., :self.d] = q.view(T, G, R, 2, self.d).transpose(2, 3)
        seqs = SeqTable.build([n for _, n in self.portions], [c for c, _ in self.portions], tables, None, device)
        rule = ScoreRule(self.scale, window=self.window, diff=DiffRule(self.lam, 1 - self.diff, EPS, self.dv))
        out = torch.full((T, H * vp), float("nan"), dtype=dtype, device=device)
        gate = torch.cat(rows_g).to(device, dtype) if self.gate is not None else None
        window_attention(qp.view(T, 2 * H, dp).to(device, dtype), kc.view(total, bs, G, 2 * dp).to(device, dtype), vc.to(device, dtype),
                         seqs, rule, out, gate=gate, impl=impl)
        return out.float().cpu().view(T, H, vp)[:, :, :self.dv]


def compare(case, got, tol):
    want = case.expected()
    assert torch.isfinite(got).all()
    err = (got.double() - want).flatten(1).norm(dim=1) / want.flatten(1).norm(dim=1).mean()
    assert err.max() < tol, f"row {int(err.argmax())}: {float(err.max()):.4g}"


MIXED = [(0, 70), (130, 1), (40, 33), (0, 1), (300, 2), (17, 1)]
CASES = {
    "grouped": dict(shape=(12, 3, 80, 48), portions=MIXED),
    "odd_sizes": dict(shape=(6, 2, 40, 24), portions=MIXED),
    "one_head_per_group": dict(shape=(4, 4, 64, 32), portions=MIXED),
    "three_per_group": dict(shape=(3, 1, 16, 16), portions=[(5, 100), (200, 1)]),
    "nine_per_group": dict(shape=(9, 1, 32, 48), portions=MIXED),
    "wide_group": dict(shape=(20, 1, 48, 80), portions=MIXED),
    "full_heads": dict(shape=(8, 2, 64, 128), portions=[(0, 300), (450, 1), (1000, 1), (700, 64)]),
    "keys_of_128": dict(shape=(4, 2, 128, 128), portions=[(0, 200), (330, 1), (100, 40)]),
    "wide_values": dict(shape=(4, 2, 64, 256), portions=[(60, 40), (330, 1), (90, 1)]),
    "wide_values_decoded": dict(shape=(4, 2, 128, 200), portions=[(330, 1), (90, 1)]),
    "wide_keys": dict(shape=(2, 1, 160, 64), portions=[(60, 40), (330, 1)]),
    "long_decode": dict(shape=(8, 2, 64, 96), portions=[(1500, 1), (1023, 1), (15, 1)]),
    "window": dict(shape=(6, 3, 32, 48), portions=MIXED, window=37),
    "no_gate": dict(shape=(6, 3, 32, 48), portions=MIXED, gate=False),
    "page_of_8": dict(shape=(12, 3, 80, 48), portions=MIXED, block=8),
    "page_of_64": dict(shape=(12, 3, 80, 48), portions=MIXED, block=64),
    "first_map_only": dict(shape=(4, 2, 32, 32), portions=MIXED, lam=0.0, diff=0.0),
    "second_map_grows": dict(shape=(4, 2, 32, 32), portions=MIXED, lam=-1.3, diff=0.9),
}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", sorted(CASES))
def test_mixed_batch(mode, name):
    c = Case(**CASES[name])
    compare(c, c.run(mode[0], mode[1]), mode[2])


@pytest.mark.gpu
def test_rows_kernel_agrees_in_bf16():
    c = Case(**CASES["grouped"])
    compare(c, c.run("cuda", torch.bfloat16, impl="rows"), 0.02)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("context,n", [(270, 1), (140, 131), (0, 271)])
def test_each_map_finds_its_key(mode, context, n):
    """Far keys, page and tile borders: the first map's query looks at one key, the second map's at another; the next
    position, which stands out for both, is not seen."""
    dev, dtype, tol = mode
    i, places = 270, [0, 1, 15, 16, 31, 32, 127, 128, 129, 191, 255, 256, 269, 270]
    for a, b in zip(places, places[3:] + places[:3]):
        c = Case((4, 2, 32, 16), [(context, n + 5 if n > 1 else n)], lam=0.5, diff=0.2, gate=False, scale=1.0, seed=3)
        c.q[0][i] = 0
        c.q[0][i, :, 0, 0] = c.q[0][i, :, 1, 1] = 6
        c.k[0] *= 0.05
        c.k[0][a, :, 0, 0] = c.k[0][b, :, 1, 1] = 3
        if n > 1:
            c.k[0][i + 1, :, 0, 0] = c.k[0][i + 1, :, 1, 1] = 5
        got = c.run(dev, dtype)[i - context]
        u = c.v[0][a].double() - 0.5 * c.v[0][b].double()
        want = (u / torch.sqrt((u * u).mean(-1, keepdim=True) + EPS) * 0.8).repeat_interleave(2, 0)
        assert (got.double() - want).norm() / want.norm() < max(tol, 0.02), (a, b)


def test_refuses_what_does_not_fit():
    q, kc, vc = torch.zeros(1, 4, 16), torch.zeros(1, 16, 1, 16), torch.zeros(1, 16, 1, 16)
    seqs = SeqTable.build([1], [0], [[0]], None, "cpu")
    with pytest.raises(AssertionError):                    # a cached key must hold both maps
        window_attention(q, kc, vc, seqs, ScoreRule(1.0, diff=DiffRule(0.5, 0.5, EPS, 16)), torch.empty(1, 32))
