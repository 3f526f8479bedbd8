"""Latent attention op (ops/latent_attention.py) against the plain restatements: mixed batches over shuffled pages, sizes
that take each of its kernels, rows that look at one chosen key, sliding windows, gates per head and per channel."""
import pytest
import torch

import milivik_oracle as M
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

    def gate_cols(self, gate):
        c = self.s.q_cols + self.s.row
        return slice(c, c + (self.s.heads if gate.dim() == 2 else self.s.heads * self.s.vdim_p))

    def pack(self, q, z, gate):
        """Rows of the packed projection: q [T, H, d + r], z [T, rank + r], gate [T, H] or [T, H, dv]."""
        s, T = self.s, q.shape[0]
        cols = self.gate_cols(gate)
        out = torch.zeros(T, (cols.stop + 7) // 8 * 8)
        qs = out[:, :s.q_cols].view(T, s.heads, s.head_cols)
        qs[:, :, :s.dim], qs[:, :, s.dim_p:s.dim_p + s.rot] = q[..., :s.dim], q[..., s.dim:]
        out[:, s.q_cols:s.q_cols + s.rank] = z[:, :s.rank]
        out[:, s.q_cols + s.rank_p:s.q_cols + s.rank_p + s.rot] = z[:, s.rank:]
        if gate.dim() == 2:
            out[:, cols] = gate
        else:
            out[:, cols].view(T, s.heads, s.vdim_p)[..., :s.vdim] = gate
        return out


def reference(layer, q, z, gate, scale, base, window=None):
    d, pos = layer.s.dim, torch.arange(q.shape[0], dtype=torch.float64)
    turn = lambda x: x if base is None else O.rotate_pairs(x, pos, base)
    c = O.rms_unit(z[:, :layer.s.rank], EPS) * layer.norm
    o = M.attend_latent(q[..., :d], turn(q[..., d:]), c, turn(z[:, layer.s.rank:]), layer.uk, layer.uv, scale, window)
    return o * torch.sigmoid(gate if gate.dim() == 3 else gate[:, :, None])


def run(layer, data, rounds, mode, scale, base, bs=16, impl=None, seed=0, window=None):
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
                            gate=proj[:, layer.gate_cols(data[0][2])], impl=impl, window=window)
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


def random_rows(layer, T, seed, per_channel=False):
    g = torch.Generator().manual_seed(seed)
    s = layer.s
    rnd = lambda *sh: torch.randn(*sh, generator=g).bfloat16().double()
    return rnd(T, s.heads, s.dim + s.rot), rnd(T, s.rank + s.rot), rnd(T, s.heads, *([s.vdim] if per_channel else []))


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


# ------------------------------------------------------------------------------ windows, gates per channel
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name,window", [("small", 21), ("small", 1), ("many_heads", 33), ("real", 64), ("one_query_tile", 40),
                                         ("wide_keys", 17), ("wide_values", 30), ("wide_latent", 16), ("one_of_each", 500)])
def test_windows_and_gates_per_channel(mode, name, window):
    layer = Layer(SIZES[name], mode[1], mode[0])
    data = [random_rows(layer, T, i, per_channel=True) for i, T in enumerate((130, 41, 70, 1))]
    rounds = [{0: 70, 1: 1, 3: 1}, {0: 1, 1: 33, 2: 5}, {0: 3, 1: 1, 2: 64}, {0: 55, 1: 1}, {0: 1, 1: 5, 2: 1}]
    got = run(layer, data, rounds, mode, 0.2, 1000.0, window=window)
    for g, d in zip(got, data):
        compare(g, reference(layer, *d, 0.2, 1000.0, window), mode[2])


@pytest.mark.gpu
@pytest.mark.parametrize("impl", ["latent", "rows"])
def test_forced_kernels_with_a_window(impl):
    mode = ("cuda", torch.bfloat16, 0.02)
    for name, per_channel in (("small", True), ("many_heads", False), ("real", True)):
        layer = Layer(SIZES[name], mode[1], mode[0])
        data = [random_rows(layer, T, i, per_channel) for i, T in enumerate((90, 20))]
        got = run(layer, data, [{0: 60, 1: 19}, {0: 30, 1: 1}], mode, 0.2, 1000.0, impl=impl, window=25)
        for g, d in zip(got, data):
            compare(g, reference(layer, *d, 0.2, 1000.0, 25), mode[2])


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("window", [1, 2, 16, 31, 33, 64, 100])
@pytest.mark.parametrize("cut", ["whole", "decoded", "pairs_and_more"])
def test_window_edges_stand_out(mode, window, cut):
    """Rows that look at the last key inside the window, at the first one outside, and at keys far outside."""
    T = 200
    layer = Layer((2, 24, 48, 16, 32), mode[1], mode[0])
    targets = [max(0, (i - window + 1, i - window, i - window + 2, i, i - window - 1, i - 2 * window, i + 1 if i + 1 < T else i)[i % 7])
               for i in range(T)]
    d = pointed_rows(layer, targets)
    cuts = {"whole": [200], "decoded": [90] + [1] * 110, "pairs_and_more": [2, 3, 4, 5, 2, 17, 33, 64, 2, 2, 66]}[cut]
    got = run(layer, [d], [{0: n} for n in cuts], mode, 0.35, None, window=window)[0]
    want = reference(layer, *d, 0.35, None, window)
    for wrong in (window - 1, window + 1):                  # the rows tell a window that is one token off
        if wrong:
            off = (reference(layer, *d, 0.35, None, wrong) - want).flatten(1).norm(dim=1) / want.flatten(1).norm(dim=1).mean()
            assert (off > 0.3).sum() >= 10
    compare(got, want, mode[2] * 2)


@pytest.mark.gpu
def test_window_far_into_a_long_context():
    """Shares of the window's keys go to several blocks; portions gather only the window from the pages."""
    mode = ("cuda", torch.bfloat16, 0.03)
    layer = Layer((4, 32, 64, 32, 64), mode[1], mode[0])
    window, T = 700, 2400
    targets = list(range(T))
    for i in range(1900, T):
        targets[i] = i - (0, window - 1, window, 350, 1)[i % 5]
    d = pointed_rows(layer, targets)
    got = run(layer, [d], [{0: 1890}, {0: 20}, {0: 1}, {0: 1}, {0: 3}, {0: 301}] + [{0: 1}] * 10 + [{0: 174}], mode, 0.35, None,
              window=window)[0]
    compare(got, reference(layer, *d, 0.35, None, window), mode[2])


@pytest.mark.parametrize("mode", MODES)
def test_rows_of_a_layer_with_a_query_latent(mode):
    """Norm of the query latent, page rows and query rotation as steps of their own; the rotated halves are handed over
    interleaved and meet again in the score."""
    dev, dtype, tol = mode
    s, T, qr = LA.LatentShape(3, 24, 12, 40, 44), 37, 20
    g = torch.Generator().manual_seed(3)
    rnd = lambda *sh: torch.randn(*sh, generator=g).bfloat16().double()
    qc, q, z = rnd(T, qr), rnd(T, s.heads, s.dim + s.rot), rnd(T, s.rank + s.rot)
    qn, cn = 0.5 + torch.rand(qr, generator=g), 0.5 + torch.rand(s.rank, generator=g)
    scaling = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
    pos = torch.arange(5, 5 + T)
    turns = stream.rotary_rows(pos.to(dev), 500.0, s.rot, stream.Yarn(4.0, 64, 8.0, 1.0))
    order = torch.arange(s.rot).view(2, -1).T.reshape(-1)   # stored channel -> channel of the halves
    proj = torch.zeros(T, 32 + s.row + 8)
    proj[:, :qr], proj[:, 32:32 + s.rank] = qc, z[:, :s.rank]
    proj[:, 32 + s.rank_p:32 + s.rank_p + s.rot] = z[:, s.rank:][:, order]
    proj = proj.to(dev, dtype)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.numel())).to(dev)
    pages = torch.full((5, 8, 1, s.row), 7.0, dtype=dtype, device=dev)
    slots = torch.randperm(40, generator=g)[:T].int()
    slots[4] = -1
    LA.cache_rows(proj[:, 32:], s, turns, slots.to(dev), pages, pad(cn, s.rank_p), EPS, query_latent=proj[:, :32], query_norm=pad(qn, 32),
                  query_rank=qr)
    compare(proj[:, :qr].cpu(), O.rms_unit(qc, EPS) * qn.double(), tol)
    assert not proj[:, qr:32].any()
    freq, mag = M.yarn_frequencies(s.rot, 500.0, scaling)
    kr = M.rotate_halves(z[:, s.rank:], pos, freq, mag)
    keep = slots >= 0
    rows = pages.view(-1, s.row)[slots[keep].long().to(dev)].cpu()
    compare(rows[:, :s.rank], (O.rms_unit(z[:, :s.rank], EPS) * cn.double())[keep], tol)
    compare(rows[:, s.rank_p:s.rank_p + s.rot], kr[:, order][keep], tol)
    assert (pages.view(-1, s.row).cpu() == 7).all(1).sum() == 40 - T + 1
    packed = torch.zeros(T, s.heads, s.head_cols)
    packed[..., :s.dim], packed[..., s.dim_p:s.dim_p + s.rot] = q[..., :s.dim], q[..., s.dim:][..., order]
    packed = packed.view(T, -1).to(dev, dtype)
    LA.rotate_queries(packed, s, turns)
    got = packed.view(T, s.heads, s.head_cols).double().cpu()
    want = M.rotate_halves(q[..., s.dim:], pos, freq, mag)
    compare(got[..., s.dim_p:s.dim_p + s.rot], want[..., order], tol)
    compare(got[..., :s.dim], q[..., :s.dim], 1e-9)
    stored = torch.einsum("thr,tr->th", got[:, :, s.dim_p:s.dim_p + s.rot][keep], rows[:, s.rank_p:s.rank_p + s.rot].double())
    compare(stored, torch.einsum("thr,tr->th", want, kr)[keep], tol * 2)


@pytest.mark.parametrize("mode", MODES)
def test_gate_by_itself(mode):
    dev, dtype, tol = mode
    x, g = torch.randn(9, 48).bfloat16().double(), 3 * torch.randn(9, 64).bfloat16().double()
    got = LA.gate_channels_(x.to(dev, dtype), g.to(dev, dtype)[:, 16:])
    compare(got.cpu(), x * torch.sigmoid(g[:, 16:]), tol)


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
    w = t.long_groups(4, 120, 16, window=40)                # positions 32.. of the first sequence, all of the others
    assert [x.keys for x in w] == [73 + 30, 57] and w[0].key_start.tolist() == [-32, 0, 73, 0]
    w = t.long_groups(4, 300, 16, window=10)
    assert [x.keys for x in w] == [5 + 100 - 64 + 30 + 7 + 50 - 32] and w[0].key_start.tolist() == [-64, 0, 41, 39]
    assert w[0].members.tolist() == [0, 0, 2, 41, 3, 71, -1, 96]
    rows, n, keys = t.short_rows(5)
    assert rows[:n].tolist() == [0, 1, 2, 3, 4, 5] and keys == 105
