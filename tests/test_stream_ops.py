"""Steps on the residual stream (ops/stream.py), squared-ReLU experts and their router (ops/moe.py) against the plain
restatement."""
from types import SimpleNamespace

import pytest
import torch

import nidilix_oracle as O
from vllm_omni_b200.ops import gemm, moe, stream

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
