"""Latent attention op (ops/latent_attention.py) against the plain restatement: mixed batches over shuffled pages, sizes
that take each of its kernels, rows that look at one chosen key."""
import pytest
import torch

import nidilix_oracle as O
from vllm_omni_b200.models.seq_table import SeqTable
from vllm_omni_b200.ops import latent_attention as LA
from vllm_omni_b200.ops import stream

GPU = pytest.mark.gpu
MODES = [pytest.param(("cpu", torch.float32, 1e-4), id="cpu"), pytest.param(("cuda", torch.float32, 1e-4), id="fp32", marks=GPU),
         pytest.param(("cuda", torch.bfloat16, 0.02), id="bf16", marks=GPU)]
# heads, dim, rot, vdim, rank
SIZES = {"small": (3, 24, 12, 40, 48), "one_of_each": (1, 16, 2, 16, 16), "many_heads": (33, 40, 8, 20, 200),
         "real": (16, 128, 64, 128, 512), "twenty": (20, 64, 32, 64, 100), "one_query_tile": (5, 136, 40, 128, 80),
         "wide_keys": (4, 200, 72, 64, 64), "wide_values": (2, 32, 16, 144, 96), "wide_latent": (2, 16, 8, 16, 528)}
EPS = 1e-4


class Layer:
    """Random weights of one layer's attention and its packed forms."""

    def __init__(self, size, dtype, dev, seed=0):
        H, d, r, dv, rank = size
        g = torch.Generator().manual_seed(seed)
        self.s = s = LA.LatentShape(H, d, r, dv, rank)
        rnd = lambda *sh: torch.randn(*sh, generator=g).bfloat16().double()
        self.uk, self.uv = rnd(H, d, rank) * rank ** -0.5, rnd(H, dv, rank) * rank ** -0.5
        self.uk, self.uv = self.uk.bfloat16().double(), self.uv.bfloat16().double()
        self.norm = (0.5 + torch.rand(rank, generator=g)).double()
        self.uk_t = torch.zeros(H, s.rank_p, s.dim_p)
        self.uk_t[:, :rank, :d] = self.uk.transpose(1, 2)
        up_k, up_v = torch.zeros(H, s.dim_p, s.rank_p), torch.zeros(H, s.vdim_p, s.rank_p)
        up_k[:, :d, :rank], up_v[:, :dv, :rank] = self.uk, self.uv
        self.kv_up = torch.cat([up_k.flatten(0, 1), up_v.flatten(0, 1)]).to(dev, dtype)
        self.uk_t, self.norm_p = self.uk_t.to(dev, dtype), torch.zeros(s.rank_p, device=dev)
        self.norm_p[:rank] = self.norm

    def pack(self, q, z, gate):
        """Rows of the packed projection: q [T, H, d + r], z [T, rank + r], gate [T, H]."""
        s, T = self.s, q.shape[0]
        out = torch.zeros(T, s.q_cols + s.row + (s.heads + 7) // 8 * 8)
        qs = out[:, :s.q_cols].view(T, s.heads, s.head_cols)
        qs[:, :, :s.dim], qs[:, :, s.dim_p:s.dim_p + s.rot] = q[..., :s.dim], q[..., s.dim:]
        out[:, s.q_cols:s.q_cols + s.rank] = z[:, :s.rank]
        out[:, s.q_cols + s.rank_p:s.q_cols + s.rank_p + s.rot] = z[:, s.rank:]
        out[:, s.q_cols + s.row:s.q_cols + s.row + s.heads] = gate
        return out


def reference(layer, q, z, gate, scale, base):
    d, pos = layer.s.dim, torch.arange(q.shape[0], dtype=torch.float64)
    turn = lambda x: x if base is None else O.rotate_pairs(x, pos, base)
    c = O.rms_unit(z[:, :layer.s.rank], EPS) * layer.norm
    o = O.attend_latent(q[..., :d], turn(q[..., d:]), c, turn(z[:, layer.s.rank:]), layer.uk, layer.uv, scale)
    return o * torch.sigmoid(gate)[:, :, None]


def run(layer, data, rounds, mode, scale, base, bs=16, impl=None, seed=0):
    """``data``: per sequence (q, z, gate); ``rounds``: lists of {sequence: rows of this step}."""
    dev, dtype, _ = mode
    s = layer.s
    need = [(d[0].shape[0] + bs - 1) // bs for d in data]
    ids = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    tables = [[ids.pop() for _ in range(n)] for n in need]
    pages = torch.full((sum(need) + 3, bs, 1, s.row), 7.0, dtype=dtype, device=dev)       # stale contents
    at, got = [0] * len(data), [[] for _ in data]
    for step in rounds:
        seqs = sorted(step)
        rows = [layer.pack(*(t[at[i]:at[i] + step[i]] for t in data[i])) for i in seqs]
        proj = torch.cat(rows).to(dev, dtype)
        pos = torch.cat([torch.arange(at[i], at[i] + step[i]) for i in seqs])
        slots = torch.cat([torch.tensor(tables[i])[torch.arange(at[i], at[i] + step[i]) // bs] * bs
                           + torch.arange(at[i], at[i] + step[i]) % bs for i in seqs]).int().to(dev)
        tab = SeqTable.build([step[i] for i in seqs], [at[i] for i in seqs], [tables[i] for i in seqs], None, dev)
        LA.latent_rows(proj, s, stream.rotary_rows(pos.to(dev), base, s.rot), slots, pages, layer.norm_p, EPS)
        out = torch.empty(proj.shape[0], s.heads * s.vdim_p, dtype=dtype, device=dev)
        LA.latent_attention(proj, s, pages, tab, layer.uk_t, layer.kv_up, scale, out,
                            gate=proj[:, s.q_cols + s.row:s.q_cols + s.row + s.heads], impl=impl)
        o = 0
        for i in seqs:
            got[i].append(out[o:o + step[i]].view(-1, s.heads, s.vdim_p)[..., :s.vdim].cpu())
            at[i] += step[i]
            o += step[i]
    return [torch.cat(g) for g in got]


def compare(got, want, tol):
    got = got.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    err = (got - want).flatten(1).norm(dim=1) / want.flatten(1).norm(dim=1).mean()
    assert err.max() < tol, f"row {int(err.argmax())}: {float(err.max()):.4g}"


def random_rows(layer, T, seed):
    g = torch.Generator().manual_seed(seed)
    s = layer.s
    rnd = lambda *sh: torch.randn(*sh, generator=g).bfloat16().double()
    return rnd(T, s.heads, s.dim + s.rot), rnd(T, s.rank + s.rot), rnd(T, s.heads)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", sorted(SIZES))
def test_portions_beside_single_tokens(mode, name):
    layer = Layer(SIZES[name], mode[1], mode[0])
    data = [random_rows(layer, T, i) for i, T in enumerate((150, 41, 70, 1, 9))]
    rounds = [{0: 70, 1: 1, 3: 1, 4: 2}, {0: 1, 1: 33, 2: 5}, {0: 3, 1: 1, 2: 64, 4: 4}, {0: 75, 1: 1, 4: 3}, {0: 1, 1: 5, 2: 1}]
    got = run(layer, data, rounds, mode, 0.2, 1000.0)
    for g, d in zip(got, data):
        compare(g, reference(layer, *d, 0.2, 1000.0), mode[2])


@pytest.mark.gpu
@pytest.mark.parametrize("impl", ["latent", "rows"])
@pytest.mark.parametrize("name", ["small", "many_heads", "real"])
def test_forced_kernels(name, impl):
    mode = ("cuda", torch.bfloat16, 0.02)
    layer = Layer(SIZES[name], mode[1], mode[0])
    data = [random_rows(layer, T, i) for i, T in enumerate((90, 20))]
    got = run(layer, data, [{0: 60, 1: 19}, {0: 30, 1: 1}], mode, 0.2, 1000.0, impl=impl)
    for g, d in zip(got, data):
        compare(g, reference(layer, *d, 0.2, 1000.0), mode[2])


def pointed_rows(layer, targets, seed=0):
    """Rows whose rotated part picks one key each: row i of every head looks at key targets[i] (a key in the future
    must have no effect)."""
    q, z, gate = random_rows(layer, len(targets), seed)
    s = layer.s
    g = torch.Generator().manual_seed(seed + 1)
    code = (torch.randint(0, 2, (len(targets), s.rot), generator=g) * 2 - 1).double()
    z[:, s.rank:] = code
    q[..., s.dim:] = code[torch.tensor(targets)][:, None]
    return q * torch.cat([torch.full((s.dim,), 0.1), torch.ones(s.rot)]), z, gate


EDGES = [0, 1, 15, 16, 17, 31, 32, 33, 47, 48, 63, 64, 65, 95, 96, 127, 128, 129, 191, 192, 255, 256, 257, 299]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("cut", ["whole", "decoded", "pairs_and_more"])
def test_rows_that_look_at_one_key(mode, cut):
    """Far keys, keys at page and tile borders, the row itself, the one before, the next (not yet visible) one."""
    layer = Layer((3, 24, 48, 40, 64), mode[1], mode[0])
    T = 300
    pick = lambda i: [e for e in EDGES if e <= i]
    targets = [min(T - 1, i + 1) if i % 7 == 5 else (i if i % 7 == 3 else (max(0, i - 1) if i % 7 == 1 else
               pick(i)[(i * 5) % len(pick(i))])) for i in range(T)]
    d = pointed_rows(layer, targets)
    cuts = {"whole": [300], "decoded": [128] + [1] * 172, "pairs_and_more": [2, 3, 4, 5, 2, 17, 33, 64, 2, 2, 66, 100]}[cut]
    got = run(layer, [d], [{0: n} for n in cuts], mode, 0.35, None)[0]
    want = reference(layer, *d, 0.35, None)
    s = layer.s
    seen = (d[0][:, 0, s.dim:] @ d[1][:, s.rank:].T * 0.35).softmax(-1)
    assert seen.max(-1).values.median() > 0.95             # the construction does point at single keys
    compare(got, want, mode[2] * 2)


@pytest.mark.parametrize("mode", MODES)
def test_reused_pages(mode):
    """A sequence's pages hold another sequence's rows from before; only its own are visible."""
    dev, dtype, tol = mode
    layer = Layer(SIZES["small"], dtype, dev)
    a, b = random_rows(layer, 60, 5), random_rows(layer, 37, 6)
    for d in (a, b):
        got = run(layer, [d], [{0: 30}, {0: d[0].shape[0] - 31}, {0: 1}], mode, 0.3, 50.0, bs=8, seed=3)[0]
        compare(got, reference(layer, *d, 0.3, 50.0), tol)


@pytest.mark.gpu
def test_long_context_splits():
    """One decoded token after thousands of keys: the shares of several blocks are merged, the far key is found."""
    mode = ("cuda", torch.bfloat16, 0.03)
    layer = Layer((4, 32, 64, 32, 64), mode[1], mode[0])
    targets = list(range(3000))
    for i, t in zip(range(2990, 3000), (0, 1, 255, 256, 511, 1024, 1999, 2047, 2048, 2998)):
        targets[i] = t
    d = pointed_rows(layer, targets)
    got = run(layer, [d], [{0: 2990}] + [{0: 1}] * 6 + [{0: 4}], mode, 0.35, None)[0]
    compare(got, reference(layer, *d, 0.35, None), mode[2])


def test_split_choice():
    for blocks in (1, 7, 64, 148, 400):
        for keys in (1, 63, 64, 300, 4096, 100000):
            n = LA.decode_splits(blocks, keys)
            assert 1 <= n <= 64 and (n == 1 or (keys + n - 1) // n >= 128)


def test_groups_of_sequences():
    t = SeqTable.build([5, 1, 30, 7], [100, 4, 0, 50], [[0]] * 4, None, "cpu")
    g = t.long_groups(4, 120, 16)
    assert [x.keys for x in g] == [105, 87] and [x.n_members for x in g] == [1, 2]
    assert g[1].key_start.tolist() == [0, 0, 0, 30] and g[1].members.tolist() == [2, 0, 3, 30, -1, 87]
    assert sorted(map(tuple, g[1].items.tolist())) == [(2, 0), (2, 16), (3, 0)]
    rows, n, keys = t.short_rows(5)
    assert rows[:n].tolist() == [0, 1, 2, 3, 4, 5] and keys == 105
