"""Steps on the residual stream (ops/stream.py), experts and their routers (ops/moe.py) against the plain restatements."""
from types import SimpleNamespace

import pytest
import torch

import milivik_oracle as M
import nidilix_oracle as O
from vllm_omni_b200.ops import fused, gemm, moe, stream

GPU = pytest.mark.gpu
MODES = [pytest.param(("cpu", torch.float32, 1e-5), id="cpu"), pytest.param(("cuda", torch.float32, 1e-5), id="fp32", marks=GPU),
         pytest.param(("cuda", torch.bfloat16, 0.006), id="bf16", marks=GPU)]


def rnd(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed)).bfloat16().double()


def norm_of(D, dev, seed=9):
    n = SimpleNamespace(alpha=torch.tensor([0.8]), w=rnd(D, seed=seed).float(), b=rnd(D, seed=seed + 1).float())
    return n, SimpleNamespace(**{k: v.to(dev) for k, v in vars(n).items()})


def near(got, want, tol):
    got = got.detach().double().cpu()
    assert torch.isfinite(got).all()
    assert (got - want).norm() <= tol * want.norm(), float((got - want).norm() / want.norm())


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("D,n", [(104, 104), (104, 99), (312, 312), (2048, 2048), (9000, 9000), (20480, 20475)])
@pytest.mark.parametrize("kind", ["plain", "normed"])
def test_branch_and_next_rows(mode, D, n, kind):
    dev, dtype, tol = mode
    T, eps, mult = 5, 1e-3, 0.37
    x, y, gain = rnd(T, D, seed=1), 4 * rnd(T, D, seed=2), rnd(D, seed=3)
    for t in (x, y):
        t[:, n:] = 0
    gain[n:] = 0
    ref, dref = norm_of(D, dev)
    want = x + mult * (y if kind == "plain" else O.rms_unit(y[:, :n], eps).new_zeros(T, D).index_copy(
        1, torch.arange(n), O.rms_unit(y[:, :n], eps)) * gain)
    for rows in (None, stream.CAST, dref):
        xd = x.float().to(dev)
        out = torch.full((T, D), 5.0, dtype=dtype, device=dev)
        kw = {} if kind == "plain" else dict(gain=gain.float().to(dev), eps=eps, n=n)
        stream.add_branch_(xd, y.to(dev, dtype), mult, out, rows, **kw)
        near(xd, want, 1e-6 if kind == "plain" else 1e-5)
        if rows is None:
            assert (out == 5).all()
        else:
            near(out, want if rows is stream.CAST else O.tanh_norm(want, 0.8, ref.w.double(), ref.b.double()), tol)


@pytest.mark.parametrize("mode", MODES)
def test_embedding_and_overlay(mode):
    dev, dtype, tol = mode
    E, ids = rnd(50, 72), torch.tensor([3, 49, 0, 7])
    ref, dref = norm_of(72, dev)
    over, mask = rnd(4, 72, seed=4), torch.tensor([False, True, False, True])
    for o, m in ((None, None), (over, mask), (over, None)):
        x, xn = stream.embed_rows(ids.to(dev), E.to(dev, dtype), dref, overlay=None if o is None else o.to(dev, dtype),
                                  overlay_mask=None if m is None else m.to(dev))
        want = E[ids] if o is None else (o if m is None else torch.where(m[:, None], o, E[ids]))
        near(x, want, 1e-7)
        near(xn, O.tanh_norm(want, 0.8, ref.w.double(), ref.b.double()), tol)


@pytest.mark.parametrize("dev", ["cpu", pytest.param("cuda", marks=GPU)])
@pytest.mark.parametrize("base,dims", [(10000.0, 32), (250.0, 2), (500000.0, 64)])
def test_rotation_angles(dev, base, dims):
    pos = torch.tensor([0, 1, 77, 4095, 131071], device=dev)
    got = stream.rotary_rows(pos, base, dims).double().cpu()
    x = torch.zeros(5, dims, dtype=torch.float64)
    x[:, 0::2] = 1
    want = O.rotate_pairs(x, pos.cpu().double(), base)
    assert (got[..., 0] - want[:, 0::2]).abs().max() < 3e-7 and (got[..., 1] - want[:, 1::2]).abs().max() < 3e-7
    one = stream.rotary_rows(pos, None, dims)
    assert (one[..., 0] == 1).all() and (one[..., 1] == 0).all()


@pytest.mark.parametrize("mode", MODES)
def test_gelu_of_a_gate_times_a_table_row(mode):
    dev, dtype, tol = mode
    z, table, ids = 2 * rnd(6, 24), rnd(40, 66, seed=2), torch.tensor([0, 39, 5, 5, 17, 2])
    z[:, 22:] = 0
    got = stream.gelu_lookup_(z.to(dev, dtype), table.to(dev, dtype), ids.to(dev), 44, 22)
    near(got[:, :22], O.gelu_tanh(z[:, :22]) * table[ids][:, 44:], tol)
    assert not got[:, 22:].any()


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("T,D,ff,E,k", [(1, 104, 56, 6, 3), (5, 64, 24, 1, 1), (40, 344, 72, 10, 2), (300, 128, 40, 5, 5),
                                        (33, 96, 136, 70, 6), (17, 72, 16, 200, 16)])
def test_experts(mode, T, D, ff, E, k):
    dev, dtype, tol = mode
    x = rnd(T, D)
    router, rb = (rnd(E, D, seed=1) * D ** -0.5).bfloat16().double(), rnd(E, seed=2)
    up, down = ((rnd(E, a, b, seed=s) * b ** -0.5).bfloat16().double() for a, b, s in ((ff, D, 3), (D, ff, 4)))
    shared = rnd(T, D, seed=5)
    ids, w = O.route(x @ router.T + rb, k)
    want = torch.stack([sum(w[t, j] * O.expert(x[t], up[ids[t, j]], down[ids[t, j]]) for j in range(k)) for t in range(T)])
    Ep = (E + 7) // 8 * 8
    rw, rbp = torch.zeros(Ep, D), torch.zeros(Ep)
    rw[:E], rbp[:E] = router, rb
    er = moe.expert_rows(x.to(dev, dtype), rw.to(dev, dtype), rbp.to(dev), moe.Router(E, k), up.to(dev, dtype), down.to(dev, dtype), act="relu2")
    near(er.weights.sort(-1).values, w.sort(-1).values, 2e-5)
    for sh in (None, shared):
        s = torch.zeros(T, D, device=dev)
        out = torch.empty(T, D, dtype=dtype, device=dev)
        stream.add_expert_rows_(s, er, None if sh is None else sh.to(dev, dtype), 0.5, out, stream.CAST)
        near(s, 0.5 * (want if sh is None else want + sh), max(tol, 1e-5))
        near(out, s.double().cpu(), tol)


@pytest.mark.gpu
@pytest.mark.parametrize("T", [3, 70, 2500])
def test_router_keeps_fp32_logits(T):
    """Two experts whose logits differ by far less than a bf16 step of their size: the larger one is chosen."""
    D, E = 256, 40
    x = torch.zeros(T, D)
    x[:, 0], x[:, 1], x[:, 100] = 16.0, 0.01171875, 4.0
    w = torch.zeros(E, D)
    w[:, 0] = torch.linspace(-4, -1, E).bfloat16().float()
    w[7, 0] = w[21, 0] = 8.0
    b = torch.zeros(E)
    b[21] = 0.0009765625                                    # logits 128 and 128.00098
    er = moe.expert_rows(x.cuda().bfloat16(), w.cuda().bfloat16(), b.cuda(), moe.Router(E, 1), torch.ones(E, 8, D).cuda().bfloat16(),
                         (torch.arange(E).float()[:, None, None] * torch.ones(E, D, 8)).cuda().bfloat16(), act="relu2")
    s, out = torch.zeros(T, D, device="cuda"), torch.empty(T, D, dtype=torch.bfloat16, device="cuda")
    stream.add_expert_rows_(s, er, None, 1.0, out, stream.CAST)
    per_unit = s / 21.0
    assert (er.weights == 1).all() and torch.allclose(per_unit, per_unit[:1, :1].expand_as(per_unit))
    h = (x.bfloat16().double().sum(-1) ** 2 * 8)[0]
    assert abs(float(s[0, 0]) / float(h * 21) - 1) < 0.02


@pytest.mark.parametrize("mode", MODES)
def test_squared_relu_epilogue(mode):
    dev, dtype, tol = mode
    x, w, b = rnd(70, 96), rnd(136, 96, seed=1) * 0.1, rnd(136, seed=2)
    w = w.bfloat16().double()
    got = gemm.linear(x.to(dev, dtype), w.to(dev, dtype), b.to(dev, dtype), act="relu2")
    near(got, O.relu_squared(x @ w.T + b), tol)


@pytest.mark.gpu
def test_batched_fp32_products():
    a, w, b = rnd(37, 3 * 24, seed=1), rnd(3, 20, 24, seed=2), rnd(3, 20, seed=3)
    out = torch.empty(37, 60, device="cuda")
    gemm.batched_f32(a.float().cuda(), w.float().cuda()[0], out,
                     bias=b.float().cuda(), batch=3, a_stride=24, w_stride=480, c_stride=20, bias_stride=20)
    near(out, torch.cat([a[:, 24 * i:24 * i + 24] @ w[i].T + b[i] for i in range(3)], dim=1), 1e-6)


# ---------------------------------------------------------------- norms on branches, gated shared expert, scaled rows
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("D,n", [(104, 104), (104, 99), (2048, 2048), (9000, 9000)])
def test_branch_norm_then_rms_rows(mode, D, n):
    dev, dtype, tol = mode
    x, y, w, w2 = rnd(5, D, seed=1), 2 * rnd(5, D, seed=2), 0.3 * rnd(D, seed=3), 0.3 * rnd(D, seed=4)
    y[2] /= 1024                                            # eps counts
    for t in (x, y):
        t[:, n:] = 0
    gain, gain2 = ((1 + v).float() for v in (w, w2))
    gain[n:] = gain2[n:] = 0
    want = x.clone()
    want[:, :n] += M.branch_norm(y[:, :n], w[:n], 1e-3)
    rows = torch.zeros(5, D, dtype=torch.float64)
    rows[:, :n] = M.branch_norm(want[:, :n], w2[:n], 1e-4)
    xd, out = x.float().to(dev), torch.empty(5, D, dtype=dtype, device=dev)
    stream.add_branch_(xd, y.to(dev, dtype), 1.0, out, stream.RmsRows(gain2.to(dev), 1e-4, n), gain=gain.to(dev), eps=1e-3, n=n)
    near(xd, want, 1e-5)
    near(out, rows, tol)
    near(out[2], rows[2], tol)


@pytest.mark.parametrize("mode", MODES)
def test_scaled_embedding(mode):
    dev, dtype, tol = mode
    E, ids, w = rnd(50, 72), torch.tensor([3, 49, 0, 7]), 0.2 * rnd(72, seed=5)
    over, mask = rnd(4, 72, seed=4), torch.tensor([False, True, False, True])
    x, out = stream.embed_rows(ids.to(dev), E.to(dev, dtype), stream.CAST, mult=11.3)
    near(x, 11.3 * E[ids], 1e-6)
    near(out, 11.3 * E[ids], tol)
    x, out = stream.embed_rows(ids.to(dev), E.to(dev, dtype), stream.RmsRows((1 + w).float().to(dev), 1e-5, 72),
                               overlay=over.to(dev, dtype), overlay_mask=mask.to(dev), mult=11.3)
    want = torch.where(mask[:, None], over, 11.3 * E[ids])  # a replaced row comes as it is
    near(x, want, 1e-6)
    near(out, M.branch_norm(want, w, 1e-5), tol)


YARN = [(None, 10000.0, 32), ((2.5, 700, 24.0, 1.5), 30000.0, 64), ((8.0, 64, 4.0, 3.9), 300.0, 10), ((1.0, 4096, 32.0, 1.0), 10000.0, 64),
        ((16.0, 8, 32.0, 1.0), 10000.0, 16), ((3.0, 100000, 1.0, 1.0), 50.0, 6), ((4.0, 256, 16.0, 2.0), 10000.0, 2)]


@pytest.mark.parametrize("dev", ["cpu", pytest.param("cuda", marks=GPU)])
@pytest.mark.parametrize("yarn,base,dims", YARN)
def test_rotation_angles_with_slowed_pairs(dev, yarn, base, dims):
    pos = torch.tensor([0, 1, 77, 4095, 131071])
    scaling = None if yarn is None else dict(zip(("factor", "original", "fast", "slow"), yarn))
    freq, mag = M.yarn_frequencies(dims, base, scaling)
    x = torch.zeros(5, dims, dtype=torch.float64)
    x[:, :dims // 2] = 1
    want = M.rotate_halves(x, pos, freq, mag)
    got = stream.rotary_rows(pos.to(dev), base, dims, None if yarn is None else stream.Yarn(*yarn)).double().cpu()
    assert (got[..., 0] - want[:, :dims // 2]).abs().max() < 5e-7 and (got[..., 1] - want[:, dims // 2:]).abs().max() < 5e-7


ROUTERS = {"plain": (6, 3, 0, 0, 1.0), "scaled": (10, 2, 0, 0, 2.5), "groups": (12, 4, 3, 2, 1.7), "one_group": (8, 3, 1, 1, 1.0),
           "all_groups": (8, 3, 4, 4, 1.0), "groups_of_one": (9, 2, 9, 5, 0.5), "groups_of_two": (16, 6, 8, 3, 1.5), "all": (4, 4, 2, 2, 1.0),
           "many": (256, 16, 16, 4, 2.0), "odd": (105, 7, 15, 3, 1.0), "one": (1, 1, 1, 1, 3.0), "many_groups": (256, 8, 128, 20, 1.0)}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", sorted(ROUTERS))
@pytest.mark.parametrize("T", [1, 40])
def test_gated_experts_of_the_best_groups(mode, name, T):
    """Choice, weights and results of SwiGLU experts, a shared expert behind its own gate, the norm of the sum."""
    dev, dtype, tol = mode
    E, k, count, keep, scale = ROUTERS[name]
    D, ff = 72, 24
    x = rnd(T, D, seed=T)
    router = (2 * rnd(E, D, seed=1) * D ** -0.5).bfloat16().double()
    gate, up, down = ((rnd(E, a, b, seed=s) * b ** -0.5).bfloat16().double() for a, b, s in ((ff, D, 2), (ff, D, 3), (D, ff, 4)))
    shared, sg, w = rnd(T, D, seed=5), rnd(T, 3, seed=6), 0.2 * rnd(D, seed=7)
    want, weights, clear = torch.zeros(T, D, dtype=torch.float64), torch.zeros(T, E, dtype=torch.float64), torch.ones(T, dtype=torch.bool)
    for t in range(T):
        z = router @ x[t]
        args = (k, count or None, keep, scale)
        ids, wt = M.route(z, *args)
        clear[t] = M.steady(z, 1e-4, *args)                 # a choice that rounding could turn says nothing
        for e, v in zip(ids, wt):
            weights[t, e] = v
            want[t] += v * ((M.silu(gate[e] @ x[t]) * (up[e] @ x[t])) @ down[e].T)
    assert clear.sum() >= 0.9 * T
    Ep = (E + 7) // 8 * 8
    rw = torch.zeros(Ep, D)
    rw[:E] = router
    rule = moe.Router(E, k, True, count, keep, scale)
    er = moe.expert_rows(x.to(dev, dtype), rw.to(dev, dtype), None, rule, torch.cat([gate, up], 1).to(dev, dtype),
                         down.to(dev, dtype), act="swiglu")
    near(er.weights.cpu()[clear].sort(-1).values, weights[clear].sort(-1).values[:, E - k:], 2e-5)
    for sh, gl in ((None, None), (shared, None), (shared, sg[:, 1])):
        b = want if sh is None else want + sh * (1.0 if gl is None else torch.sigmoid(gl)[:, None])
        s, out = torch.zeros(T, D, device=dev), torch.empty(T, D, dtype=dtype, device=dev)
        kw = {} if gl is None else dict(shared_gate=sg.to(dev, dtype)[:, 1])
        sh_d = None if sh is None else sh.to(dev, dtype)
        stream.add_expert_rows_(s, er, sh_d, 0.5, out, stream.CAST, **kw)
        near(s.cpu()[clear], 0.5 * b[clear], max(tol, 2e-5))
        s.zero_()
        stream.add_expert_rows_(s, er, sh_d, 1.0, out, stream.CAST, gain=(1 + w).float().to(dev), eps=1e-4, n=D, **kw)
        near(s.cpu()[clear], M.branch_norm(b, w, 1e-4)[clear], max(tol, 2e-5))
        near(out.cpu()[clear], s.double().cpu()[clear], tol)


@pytest.mark.parametrize("mode", MODES)
def test_a_group_wins_by_its_two_best(mode):
    """The group with the best single score loses against two good ones; the third best of a group does not count."""
    dev, dtype, _ = mode
    z = torch.tensor([3.0, -3, -3, -3, 1.5, 1.4, -3, -3, 1.45, 1.3, 1.29, 1.28, 1.6, 1.35, -3, -3])
    x, rw = torch.zeros(1, 16), torch.eye(16)
    x[0] = z.bfloat16().float()
    up, down = torch.ones(16, 16, 16), torch.arange(16.0)[:, None, None] * torch.ones(16, 16, 8)
    for keep, k, ids in ((1, 2, {12, 13}), (2, 3, {12, 4, 5}), (2, 4, {12, 13, 4, 5}), (3, 2, {12, 4}), (4, 2, {0, 12})):
        er = moe.expert_rows(x.to(dev, dtype), rw.to(dev, dtype), None, moe.Router(16, k, True, 4, keep, 1.0), up.to(dev, dtype),
                             down.to(dev, dtype), act="swiglu")
        s, out = torch.zeros(1, 16, device=dev), torch.empty(1, 16, dtype=dtype, device=dev)
        stream.add_expert_rows_(s, er, None, 1.0, out, stream.CAST)
        sc = {e: 1 / (1 + float(torch.exp(-x[0, e]))) for e in ids}
        h = float(x[0].sum())
        unit = 8 * h * h / (1 + float(torch.exp(torch.tensor(-h))))
        want = sum(e * sc[e] for e in ids) / sum(sc.values()) * unit
        assert abs(float(s[0, 0]) / want - 1) < (1e-4 if dtype == torch.float32 else 0.02), (keep, k)


@pytest.mark.parametrize("bad", [(6, 7), (6, 0), (6, 2, True, 4, 1), (6, 2, True, 3, 4), (6, 3, True, 3, 1), (300, 2), (40, 17)])
def test_routers_that_cannot_choose(bad):
    with pytest.raises(ValueError, match="router"):
        moe.Router(*bad)


@pytest.mark.parametrize("mode", MODES)
def test_swiglu_of_a_wider_row(mode):
    dev, dtype, tol = mode
    z = 3 * rnd(7, 104)
    near(fused.silu_mul(z.to(dev, dtype)[:, :96]), M.silu(z[:, :48]) * z[:, 48:96], tol)
