"""Fikizen decoder through the framework: checkpoint folder, engine step, pages and state slots, decode graphs, sampling,
the public entry points — against the plain restatement (tests/fikizen_oracle.py)."""
import copy
import io
import json
import struct

import pytest
import torch

import fikizen_oracle as O
from lm_harness import Folder, check, folder_fixture, modes, replay, tokens
from vllm_omni_b200.entrypoints.omni_llm import OmniLLM
from vllm_omni_b200.entrypoints.trace import TraceReplay
from vllm_omni_b200.inputs.data import SamplingParams
from vllm_omni_b200.models.fikizen import FikizenConfig, FikizenDecoder, tiny_config_dict

MODES = modes(0.05)


def heads(n=4, kv=2, dim=24, vdim=20, window=21, rot=16, base=3000.0, scale=0.25):
    return {"heads": n, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}, "rot": {"base": base, "dims": rot}}


def mlp(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def attention(ff=88, **kw):
    return {"type": "attention", "mixer": heads(**kw), "mlp": mlp(ff)}


def delta(n=4, kv=2, dim=20, vdim=28, conv=3, ff=None):
    return {"type": "delta", "mixer": {"heads": n, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp(ff)}


def parallel(right=(3, 22), left_scale=0.8, right_scale=1.3, ff=56, **kw):
    return {"type": "parallel", "mlp": mlp(ff), "mixer": {"left": heads(**kw), "right": {"heads": right[0], "dim": right[1]}, "left_scale": left_scale,
                                                          "right_scale": right_scale}}


def shared(layer, j):
    return dict(copy.deepcopy(layer), weights_of=j)


def config(layers, width=72, vocab=211, eps=1e-4, cap=15.0):
    return {"architecture": "Fikizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


A, P, S = attention(), parallel(window=33), delta()
CONFIGS = {
    "base": config([P, A, S, shared(A, 1)]),
    "all_shared": config([S, A, P, shared(P, 2), shared(S, 0), shared(A, 1), shared(S, 0)], width=64),
    "layers_differ": config([delta(6, 3, 36, 16, 5, ff=40), attention(None, n=5, kv=1, dim=18, vdim=34, window=16, rot=18, base=50.0),
                             parallel((2, 40), 1.0, 1.0, None, n=6, kv=6, dim=10, vdim=12, window=1, rot=2), delta(2, 2, 64, 64, 2),
                             attention(24, n=2, kv=2, window=17, rot=0)], width=90, vocab=131, cap=4.0),
    "ones": config([attention(1, n=1, kv=1, dim=2, vdim=1, window=1, rot=2), delta(1, 1, 2, 3, 1), parallel((1, 2), ff=1, n=1, kv=1, dim=2, vdim=2, rot=2)],
                   width=8, vocab=40, cap=None),
    "wide_heads": config([attention(n=2, kv=1, dim=136, vdim=144, window=40, rot=64), delta(2, 1, 128, 128, 4), parallel((2, 96), n=8, kv=1, dim=64, vdim=64),
                          delta(1, 1, 200, 100, 3)], width=136),
    "only_recurrences": config([S, delta(3, 1, 64, 48, 4, ff=20)], cap=1.5),
    "only_attention": config([A, attention(n=3, kv=3, window=100, base=1e6)]),
    "later_owner": config([shared(A, 1), A, S]),
}
RANKS = {"base": 12, "all_shared": 16, "layers_differ": 5, "ones": 1, "wide_heads": 40, "later_owner": 8}


def weights(cfg, seed=0, rank=12):
    """Random bf16 weights whose every mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda s: torch.randn(s, generator=g)
    out = {}
    for name, shape in FikizenConfig.from_dict(cfg).tensor_shapes().items():
        shape = tuple(rank if n is None else n for n in shape)
        last = name.split(".")[-1]
        if last in ("norm1", "norm2", "norm"):
            w = 0.5 + torch.rand(shape, generator=g)
        elif last == "conv":
            w = 0.6 * rnd(shape)
        elif last == "A_log":
            w = rnd(shape) - 1
        elif len(shape) == 1:                                  # biases, act
            w = 0.5 * rnd(shape)
        elif last == "embed":
            w = rnd(shape)
        else:
            w = 1.3 * rnd(shape) * shape[-1] ** -0.5
        out[name] = w.bfloat16()
    return out


folder = folder_fixture(CONFIGS, lambda cfg: weights(cfg, rank=next((r for n, r in RANKS.items() if CONFIGS[n] is cfg), 12)), O.forward)


def tail(mode):
    return 0.1 if mode[1] == "bfloat16" else 0.0


def every_config(dtype):
    """Norms over one channel give its sign, which bf16 may turn: those sizes run in fp32 only."""
    return [n for n in sorted(CONFIGS) if n != "ones" or dtype != "bfloat16"]


CASES = [pytest.param(m.values[0], n, id=f"{n}-{m.id}", marks=m.marks) for m in MODES for n in every_config(m.values[0][1])]


# ----------------------------------------------------------------------------- prompts and portions
@pytest.mark.parametrize("mode,name", CASES)
def test_whole_prompt(folder, mode, name):
    f = folder(name)
    ids = tokens(f.cfg, 130)
    check(replay(f, mode, {"a": ids}, [{"a": 130}])["a"], f.expected(ids), mode[2], tail(mode))


@pytest.mark.parametrize("mode,name", CASES)
def test_token_by_token(folder, mode, name):
    f = folder(name)
    ids = tokens(f.cfg, 130)
    check(replay(f, mode, {"a": ids[:50]}, [{"a": 1}] * 50)["a"], f.expected(ids)[:50], mode[2], tail(mode))


CUTS = {"pairs": [2] * 65, "threes": [3] * 43 + [1], "page_and_more": [16, 17, 15, 1, 31, 33, 17], "growing": [2, 3, 5, 8, 13, 21, 34, 44],
        "tail_decoded": [90] + [1] * 40, "head_decoded": [1] * 20 + [110], "window_edges": [20, 1, 1, 11, 1, 1, 33, 2, 34, 26]}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("cut", sorted(CUTS))
def test_portions(folder, mode, cut):
    f = folder("base")
    ids = tokens(f.cfg, 130)
    assert sum(CUTS[cut]) == 130
    check(replay(f, mode, {"a": ids}, [{"a": n} for n in CUTS[cut]])["a"], f.expected(ids), mode[2], tail(mode))


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", ["base", "all_shared", "layers_differ"])
def test_mixed_batches_reuse_pages_and_slots(folder, mode, name):
    """Seven requests through four slots and a pool that holds only the live ones: portions beside decoded tokens,
    requests that sit out steps, pages and slots handed on with stale contents in them."""
    f = folder(name)
    # (first tokens whose query and key are nearly orthogonal are left out: the norm after the read-out gives the sign of their product)
    lens = {"a": 130, "b": 1, "c": 70, "d": 33, "e": 64, "f": 97, "g": 2}
    seqs = {r: tokens(f.cfg, n, seed=50 + i) for i, (r, n) in enumerate(lens.items())}
    rounds = [{"a": 40, "b": 1, "c": 2}, {"c": 17, "a": 1}, {"d": 2, "a": 1, "c": 1, "e": 30}, {"d": 3, "e": 1}, {"a": 50, "d": 28, "e": 1},
              {"c": 50, "e": 32}, {"f": 64, "a": 1, "g": 2}, {"a": 37, "f": 31}, {"f": 1}, {"f": 1}]
    got = replay(f, mode, seqs, rounds, max_tokens=192 + 128 + 64 + 64)
    for r, ids in seqs.items():
        check(got[r], f.expected(ids), mode[2], tail(mode))


@pytest.mark.parametrize("mode", MODES[1:])
def test_a_batch_gives_what_each_request_gives_alone(folder, mode):
    f = folder("base")
    seqs = {r: tokens(f.cfg, n, seed=30 + n) for r, n in (("a", 77), ("b", 19), ("c", 40), ("d", 5))}
    cuts = {"a": [50, 20, 7], "b": [1, 17, 1], "c": [3, 30, 7], "d": [2, 1, 2]}
    got = replay(f, mode, seqs, [{r: cuts[r][i] for r in seqs} for i in range(3)])
    for r, ids in seqs.items():
        alone = replay(f, mode, {r: ids}, [{r: n} for n in cuts[r]])[r]
        check(got[r], alone, 1e-6 if mode[1] == "float32" else 0.02)


@pytest.mark.parametrize("mode", MODES)
def test_long_decode(folder, mode):
    """Windows pass over decoded tokens many times."""
    f = folder("base")
    ids = tokens(f.cfg, 230, seed=4)
    check(replay(f, mode, {"a": ids}, [{"a": 3}] + [{"a": 1}] * 227)["a"], f.expected(ids), mode[2], tail(mode))


@pytest.mark.parametrize("mode", MODES)
def test_first_tokens(folder, mode):
    for name in ("base", "layers_differ"):
        f = folder(name)
        ids = tokens(f.cfg, 6, seed=5)
        for rounds in ([{"a": 6}], [{"a": 1}] * 6, [{"a": 2}] * 3, [{"a": 1}, {"a": 5}]):
            check(replay(f, mode, {"a": ids}, rounds)["a"], f.expected(ids), mode[2], tail(mode))


@pytest.mark.parametrize("mode", MODES)
def test_stream_after_every_layer(folder, mode):
    dev, dtype, tol = mode
    f = folder("all_shared")
    ids = tokens(f.cfg, 40)
    trace = []
    O.forward(f.cfg, f.weights, ids, trace=trace)
    rp = TraceReplay(f.path, dtype, 64, device=dev)
    dec, got = rp.llm.model.decoder, {}
    plain = dec.forward
    dec.forward = lambda b, kv, **kw: got.update(r=plain(b, kv, capture_layers=range(9))) or got["r"]
    rp.step([{"id": "a", "tokens": ids, "want": [0]}])
    for i, want in enumerate(trace):
        x = got["r"][1][i + 1][:, :f.cfg["width"]]
        assert x.dtype == torch.float32
        check(x.cpu(), want, tol, tail(mode))


EDGES = {"attention": 0, "parallel": 1}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("size", [1, 2, 16, 17, 33])
@pytest.mark.parametrize("kind", sorted(EDGES))
def test_window_edges(tmp_path, mode, size, kind):
    """One key outshines all others: the last token inside the window that ends at it sees it, the next one does not, in
    prompts, portions and decoding, at page borders too."""
    layer = attention(window=size, n=2, kv=1, dim=16, vdim=16, rot=0, scale=1.0) if kind == "attention" else \
        parallel(window=size, n=2, kv=1, dim=16, vdim=16, rot=0, scale=1.0, right_scale=0.01)
    cfg = config([layer], width=48, vocab=50, cap=None)
    W = weights(cfg, seed=3)
    p = "l0.mix." + ("left." if kind == "parallel" else "")
    # token 7's key and every token's query share a large channel
    mark = torch.zeros(48)
    mark[0] = 1
    W["embed"][:, 0] = 0
    W["embed"][7, 0] = 12
    W["embed"][:, 1] = 3
    for n in "qk":
        W[p + n].mul_(0.1)
        W[p + n][:, :2] = 0
    W[p + "q"][0::16, 1] = 4
    W[p + "k"][0, 0] = 4
    at, T = 31, 31 + size + 3
    ids = [t if t != 7 else 8 for t in tokens(cfg, T, seed=size)]
    plain = O.forward(cfg, W, ids)
    ids[at] = 7
    want = O.forward(cfg, W, ids)
    moved = (want - plain).norm(dim=1) / plain.norm(dim=1).mean()
    if size > 1:
        assert moved[at + size - 1] > 0.1
    assert moved[at + size] < 0.5 * moved[at + size - 1]
    f = Folder(tmp_path, cfg, W, O.forward)
    for rounds in ([T], [at + size - 1, 1, 1, 2], [at + size - 2, 2, 3] if size > 1 else [at, 2, 2], [at + size, 3]):
        if sum(rounds) != T:
            rounds = rounds + [T - sum(rounds)]
        check(replay(f, mode, {"a": ids}, [{"a": n} for n in rounds if n])["a"], want, mode[2], tail(mode))


CHANGES = {
    "window": lambda c, W: c["layers"][1]["mixer"]["mask"].update(size=20) or c["layers"][3]["mixer"]["mask"].update(size=20),
    "left window": lambda c, W: c["layers"][0]["mixer"]["left"]["mask"].update(size=34),
    "scale": lambda c, W: c["layers"][0]["mixer"]["left"].update(scale=0.3),
    "rotation base": lambda c, W: c["layers"][0]["mixer"]["left"]["rot"].update(base=300.0),
    "rotated channels": lambda c, W: [c["layers"][i]["mixer"]["rot"].update(dims=12) for i in (1, 3)],
    "left scale": lambda c, W: c["layers"][0]["mixer"].update(left_scale=0.6),
    "right scale": lambda c, W: c["layers"][0]["mixer"].update(right_scale=1.0),
    "eps": lambda c, W: c["norm"].update(eps=0.1),
    "cap": lambda c, W: c.update(logit_softcap=5.0),
    "no cap": lambda c, W: c.update(logit_softcap=None),
    "act above": lambda c, W: W["l1.mlp.act"][0].add_(0.5),
    "act below": lambda c, W: W["l1.mlp.act"][1].add_(0.5),
    "query bias": lambda c, W: W["l0.mix.left.q.b"].neg_(),
    "value bias": lambda c, W: W["l0.mix.left.v.b"].neg_(),
    "query row norm": lambda c, W: W["l0.mix.left.q.norm"].copy_(W["l0.mix.left.q.norm"].flip(0)),
    "key row norm": lambda c, W: W["l0.mix.left.k.norm"].copy_(W["l0.mix.left.k.norm"].flip(0)),
    "decay bias": lambda c, W: W["l0.mix.right.w0"].sub_(3),
    "removal bias": lambda c, W: W["l0.mix.right.a.b"].sub_(2),
    "low rank": lambda c, W: W["l0.mix.right.w2"].mul_(-2),
    "channel delta gain": lambda c, W: W["l0.mix.right.norm"].copy_(W["l0.mix.right.norm"].flip(0)),
    "head gates": lambda c, W: W["l1.mix.g"].neg_(),
    "decay rate": lambda c, W: W["l2.mix.A_log"].add_(2),
    "time step": lambda c, W: W["l2.mix.dt_bias"].add_(2),
    "step size": lambda c, W: W["l2.mix.b"].neg_(),
    "taps": lambda c, W: W["l2.mix.k.conv"].copy_(W["l2.mix.k.conv"].flip(1)),
    "delta gain": lambda c, W: W["l2.mix.norm"].copy_(W["l2.mix.norm"].flip(0)),
}


@pytest.mark.parametrize("change", sorted(CHANGES))
def test_every_constant_is_read(change, tmp_path):
    """A change of one constant or tensor moves the results, in the framework as in the restatement."""
    cfg, W = copy.deepcopy(CONFIGS["base"]), weights(CONFIGS["base"])
    ids = tokens(cfg, 60)
    before = O.forward(cfg, W, ids)
    CHANGES[change](cfg, W)
    after = O.forward(cfg, W, ids)
    assert ((after - before).pow(2).mean(-1).sqrt() / before.pow(2).mean().sqrt()).max() > 0.01
    f = Folder(tmp_path, cfg, W, O.forward)
    check(replay(f, ("cpu", "float32", 0), {"a": ids}, [{"a": 45}] + [{"a": 1}] * 15)["a"], after, 1e-4)


def test_shared_weights_are_loaded_once_and_caches_are_apart(folder):
    f = folder("all_shared")
    cfg = FikizenConfig.from_dict(f.cfg)
    assert {n.split(".")[0] for n in cfg.tensor_shapes()} == {"embed", "final", "head", "l0", "l1", "l2"}
    rp = TraceReplay(f.path, "float32", 64, device="cpu")
    assert len(rp.llm.model.decoder.owners) == 3
    rp.step([{"id": "a", "tokens": tokens(f.cfg, 21), "want": []}])
    kv = rp.engine.runner.extract_kv(rp.live["a"])
    assert not torch.equal(kv["layers"][1][0], kv["layers"][5][0]) and not torch.equal(kv["state"][0][0], kv["state"][4][0])


# --------------------------------------------------------------------------------- generation
@pytest.mark.parametrize("mode", MODES[:2])
def test_greedy_generation_matches(folder, mode):
    """Through the engine's own scheduler: a prompt longer than the step budget, short ones beside it."""
    f = folder("base")
    prompts = [tokens(f.cfg, n, seed=20 + n) for n in (45, 7, 1)]
    llm = OmniLLM(f.path, dtype=mode[1], device=mode[0], num_gpu_blocks=40, max_num_seqs=3, max_num_batched_tokens=16)
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts],
                        SamplingParams(temperature=0.0, max_tokens=16, ignore_eos=True, detokenize=False))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == f.greedy(p, 16)
    assert llm.engine.kv.state.num_free == 3


def test_preemption_recomputes_the_state(folder):
    """A pool that forces preemption, and fewer state slots than requests: the same tokens."""
    f = folder("base")
    prompts = [{"prompt_token_ids": tokens(f.cfg, n, seed=40 + n)} for n in (20, 9, 14, 5)]
    sp = SamplingParams(temperature=0.0, max_tokens=30, ignore_eos=True, detokenize=False)

    def run(blocks, seqs):
        llm = OmniLLM(f.path, dtype="float32", device="cpu", num_gpu_blocks=blocks, block_size=8, max_num_seqs=seqs)
        out = [list(o.outputs[0].token_ids) for o in llm.generate(prompts, sp)]
        assert llm.engine.kv.pool.num_free == blocks and llm.engine.kv.state.num_free == seqs
        return out
    free = run(64, 4)
    assert run(9, 4) == free and run(64, 2) == free


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_decode_graph_equals_eager(folder, dtype, monkeypatch):
    f = folder("base")
    prompts = [{"prompt_token_ids": tokens(f.cfg, n, seed=60 + n)} for n in (50, 3, 30)]
    sp = SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True, detokenize=False)

    def run(graph):
        monkeypatch.setenv("OMNI_AR_CUDA_GRAPH", graph)
        llm = OmniLLM(f.path, dtype=dtype, num_gpu_blocks=64, max_num_seqs=3)
        out = [list(o.outputs[0].token_ids) for o in llm.generate(prompts, sp)]
        if graph == "1":
            runner = llm.engine.runner.graph_runner
            assert runner.replays > 30 and runner.use_graph and any(b.graph is not None for b in runner._state.values())
        else:
            assert llm.engine.runner.graph_runner is None
        return out
    a, b = run("1"), run("0")
    if dtype == "float32":
        assert a == b
    else:           # the two differ in how many blocks share a sequence: a near tie may fall either way
        assert sum(x == y for s, t in zip(a, b) for x, y in zip(s, t)) > 60


def test_decode_buckets_on_cpu(folder, monkeypatch):
    """The static-buffer step a graph replays, with padding rows that write neither pages nor state."""
    f = folder("base")
    monkeypatch.setenv("OMNI_AR_CUDA_GRAPH", "1")
    ids = {r: tokens(f.cfg, 30, seed=i) for i, r in enumerate("abc")}
    got = replay(f, ("cpu", "float32", 0), ids, [{"a": 10, "b": 12, "c": 11}] + [{"a": 1, "b": 1, "c": 1}] * 18 + [{"a": 2, "c": 1}])
    for r in "ac":
        check(got[r], f.expected(ids[r]), 1e-4)


def test_runs_without_a_checkpoint():
    llm = OmniLLM(None, model_arch="Fikizen", device="cpu", num_gpu_blocks=16)
    out = llm.generate({"prompt_token_ids": list(range(30))}, SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))[0]
    assert len(out.outputs[0].token_ids) == 5 and llm.model.decoder_config.vocab_size == tiny_config_dict()["vocab"]


def test_omni_serves_the_folder(folder):
    """The public entry point picks the model by its config.json and runs it as one text stage."""
    from vllm_omni_b200.entrypoints.omni import Omni
    f = folder("base")
    p = tokens(f.cfg, 12, seed=3)
    with Omni(f.path, dtype="float32", device="cpu", num_gpu_blocks=32) as omni:
        out = omni.generate({"prompt_token_ids": p}, SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True, detokenize=False))[0]
    assert list(out.request_output[0].outputs[0].token_ids if isinstance(out.request_output, list)
                else out.request_output.outputs[0].token_ids) == f.greedy(p, 8)


# ------------------------------------------------------------------------------------- replay
def test_replay_program(folder, tmp_path):
    from vllm_omni_b200.entrypoints import trace
    f = folder("base")
    ids = tokens(f.cfg, 20)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:9], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[9:], "want": [0, 10]}, {"id": "b", "tokens": ids[:1], "want": [0]}],
              "end": ["a"]},
             {"step": 2, "entries": [], "end": ["b"]}]
    args = trace.make_parser().parse_args(["--model", f.path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128"])
    out = io.StringIO()
    assert trace.run(args, io.StringIO("\n".join(map(json.dumps, steps)) + "\n"), out) == 0
    assert out.getvalue().split("\n")[:3] == ["done 0", "done 1", "done 2"]
    raw = (tmp_path / "1.f32").read_bytes()
    got = torch.tensor(struct.unpack(f"<{len(raw) // 4}f", raw)).view(3, -1)
    check(got, f.expected(ids)[[9, 19, 0]], 1e-4)


def test_state_and_pages_of_a_request(folder):
    """What a hand-off of a request carries: keys and values of the attention layers, state and history of the others."""
    f = folder("base")
    rp = TraceReplay(f.path, "float32", 64, device="cpu")
    rp.step([{"id": "a", "tokens": tokens(f.cfg, 21), "want": []}])
    kv = rp.engine.runner.extract_kv(rp.live["a"])
    assert [tuple(k.shape) for k, _ in kv["layers"]] == [(21, 2, 32), (21, 2, 32), (21, 0, 0), (21, 2, 32)]
    assert [[tuple(t.shape) for t in s] for s in kv["state"]] == [[(3, 32, 32)], [], [(4, 32, 32), (2, 256)], []]
    assert kv["layers"][0][0].abs().sum() > 0 and kv["state"][2][0].dtype == torch.float32


# ------------------------------------------------------------------------------ configuration
@pytest.mark.parametrize("change", [
    lambda l: l[0].update(type="something"),
    lambda l: l[1]["mixer"]["rot"].update(dims=7),
    lambda l: l[1]["mixer"]["rot"].update(dims=26),
    lambda l: l[1]["mixer"].update(kv_heads=3),
    lambda l: l[1]["mixer"]["mask"].update(size=0),
    lambda l: l[2]["mixer"].update(kv_heads=3),
    lambda l: l[2]["mixer"].update(conv=0),
    lambda l: l[3].update(weights_of=2),
    lambda l: l[3].update(weights_of=7),
    lambda l: l[3]["mixer"].update(scale=0.1),
    lambda l: l[1].update(weights_of=3),
    lambda l: l[1]["mlp"].update(kind="moe")])
def test_configuration_errors(change):
    bad = copy.deepcopy(CONFIGS["base"])
    FikizenConfig.from_dict(bad)
    change(bad["layers"])
    with pytest.raises(ValueError):
        FikizenConfig.from_dict(bad)


def test_checkpoint_errors():
    cfg = CONFIGS["base"]
    W = weights(cfg)
    dec = FikizenDecoder(FikizenConfig.from_dict(cfg), torch.float32, "cpu")
    assert dec.load_weights(W.items()) == set(W)
    with pytest.raises(ValueError, match="lacks"):
        dec.load_weights((n, w) for n, w in W.items() if n != "l2.mix.A_log")
    for name, bad in (("l1.mix.q", W["l1.mix.q"].t()), ("l0.mix.right.w1", W["l0.mix.right.w1"][:, :5]), ("l0.mix.right.w2", W["l0.mix.right.w2"][0])):
        with pytest.raises(ValueError, match="shape"):
            dec.load_weights([(name, bad)])
    with pytest.raises(ValueError, match="rank"):
        dec.load_weights(dict(W, **{"l0.mix.right.w2": W["l0.mix.right.w2"][:, :7]}).items())


@pytest.mark.parametrize("first", [0, 1])
def test_the_checkpoint_tells_the_rank(first):
    """In either order of its two tensors, and again when another checkpoint follows."""
    cfg = CONFIGS["base"]
    dec = FikizenDecoder(FikizenConfig.from_dict(cfg), torch.float32, "cpu")
    for rank in (9, 33, 3):
        W = weights(cfg, rank=rank)
        dec.load_weights(sorted(W.items(), reverse=bool(first)))
        mix = dec.layer(0).mix
        assert mix.rank == rank and torch.equal(mix.proj.weight[mix.low_col:mix.low_col + rank, :72], W["l0.mix.right.w1"].float())
        assert torch.equal(mix.w2.weight[32:54, :rank], W["l0.mix.right.w2"][22:44].float())
