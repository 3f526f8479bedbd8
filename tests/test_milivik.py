"""Milivik decoder through the framework: checkpoint folder, engine step, pages, decode graphs, sampling, the public entry
points — against the plain restatement (tests/milivik_oracle.py)."""
import copy
import io
import json
import struct

import pytest
import torch

import milivik_oracle as O
from lm_harness import check, folder_fixture, modes, replay, tokens
from vllm_omni_b200.entrypoints.omni_llm import OmniLLM
from vllm_omni_b200.entrypoints.trace import TraceReplay
from vllm_omni_b200.inputs.data import SamplingParams
from vllm_omni_b200.models.milivik import MilivikConfig, MilivikDecoder, tiny_config_dict

MODES = modes(0.1)
EMBED = 7.0


def near(f, got, ids, mode):
    """``got``: logits of ``ids`` (its first rows).  In bf16 the rows whose router choice rounding may turn say nothing, and
    one row in ten may be off because such a row lies among its keys."""
    want = f.expected(ids)[:got.shape[0]]
    if mode[1] != "bfloat16":
        return check(got, want, mode[2])
    key = ("clear", *ids)
    if key not in f._memo:
        f._memo[key] = torch.ones(len(ids), dtype=torch.bool)
        O.forward(f.cfg, f.weights, ids, clear=f._memo[key])
    clear = f._memo[key][:got.shape[0]]
    assert clear.float().mean() > 0.8 or len(ids) < 20
    if clear.any():
        check(got[clear], want[clear], mode[2], 0.5)


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(ff=40, experts=6, top=2, shared=24, groups=(3, 2), scale=1.6):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r, "shared": None if shared is None else {"ff": shared}}


def latent(heads=3, dim=24, rot=12, vdim=20, rank=40, q_rank=28, scale=0.15, window=21, base=5000.0, yarn=(3.0, 64, 8.0, 1.0), mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale,
         "rot": {"base": base, "dims": rot}}
    if yarn is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def diff(heads=6, kv=2, dim=20, vdim=36, scale=0.2, lam=0.4, temp=(0.25, 9), mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": lam}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(layers, width=72, vocab=211, eps=1e-4, logit=0.3):
    return {"architecture": "Milivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": EMBED},
            "logit_scale": logit, "layers": layers}


CONFIGS = {
    "base": config([latent(mlp=dense()), diff(mlp=moe()), latent(window=34, heads=5, mlp=moe()), diff(heads=3, kv=3, mlp=dense())]),
    "layers_differ": config([diff(heads=4, kv=1, dim=12, vdim=8, lam=0.8, temp=(0.2, 1), mlp=moe(24, 5, 1, None, None, 1.0)),
                             latent(heads=2, rank=24, window=1, mlp=None), latent(heads=4, rot=8, rank=72, base=100.0, yarn=None, window=None,
                                                                                  mlp=moe(136, 12, 4, 16, (4, 3))),
                             diff(temp=None, lam=0.1, mlp=None), latent(heads=1, q_rank=90, window=2, mlp=dense(16))], width=90, vocab=131,
                            logit=1.7),
    "small_values": config([latent(1, 2, 2, 3, 4, 4, window=3, mlp=dense(3)), diff(1, 1, 2, 4, mlp=moe(3, 1, 1, 2, (1, 1)))], width=8, vocab=40),
    "ones": config([latent(1, 1, 2, 1, 1, 1, window=2, mlp=dense(1)), diff(1, 1, 1, 1, mlp=moe(1, 1, 1, 1, (1, 1)))], width=8, vocab=40),
    "wide_heads": config([latent(heads=2, dim=136, rot=40, vdim=128, rank=96, q_rank=130, scale=0.05, mlp=dense(200)),
                          latent(heads=18, dim=40, rot=64, vdim=24, rank=200, scale=0.07, window=70),
                          diff(18, 2, 64, 128, scale=0.1), diff(2, 1, 136, 40, scale=0.07)]),
    "wide_values": config([latent(vdim=144, window=16), diff(vdim=144, mlp=moe(top=3, groups=(2, 1)))]),
    "only_latent": config([latent(mlp=dense()), latent(window=64, mlp=moe())]),
    "only_differential": config([diff(mlp=moe(groups=(6, 4))), diff(8, 2, 64, 64, scale=0.15, mlp=dense())]),
}


def weights(cfg, seed=0):
    """Random bf16 weights whose every mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda s: torch.randn(s, generator=g)
    out = {}
    for name, shape in MilivikConfig.from_dict(cfg).tensor_shapes().items():
        last = name.split(".")[-1]
        if last in ("norm1", "norm2") or name == "final.norm":
            w = 0.4 * rnd(shape)
        elif last == "norm":
            w = 0.5 + torch.rand(shape, generator=g)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            w = 0.3 * rnd(shape)
        elif name == "embed":
            w = 1.3 / EMBED * rnd(shape)
        else:
            w = 1.5 * rnd(shape) * shape[-1] ** -0.5
        out[name] = w.bfloat16()
    return out


folder = folder_fixture(CONFIGS, weights, O.forward)


def every_config(mode):
    """Norms over one channel give its sign, which bf16 may turn: those sizes run in fp32 only."""
    return [n for n in sorted(CONFIGS) if n != "ones" or mode != "bfloat16"]


CASES = [pytest.param(m.values[0], n, id=f"{n}-{m.id}", marks=m.marks) for m in MODES for n in every_config(m.values[0][1])]


# ----------------------------------------------------------------------------- prompts and portions
@pytest.mark.parametrize("mode,name", CASES)
def test_whole_prompt(folder, mode, name):
    f = folder(name)
    ids = tokens(f.cfg, 130)
    near(f, replay(f, mode, {"a": ids}, [{"a": 130}])["a"], ids, mode)


@pytest.mark.parametrize("mode,name", CASES)
def test_token_by_token(folder, mode, name):
    f = folder(name)
    ids = tokens(f.cfg, 130)[:50]
    near(f, replay(f, mode, {"a": ids}, [{"a": 1}] * 50)["a"], tokens(f.cfg, 130), mode)


CUTS = {"pairs": [2] * 65, "threes": [3] * 43 + [1], "page_and_more": [16, 17, 15, 1, 31, 33, 17], "growing": [2, 3, 5, 8, 13, 21, 34, 44],
        "tail_decoded": [90] + [1] * 40, "head_decoded": [1] * 20 + [110], "window_edges": [20, 1, 1, 11, 1, 1, 33, 2, 34, 26]}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("cut", sorted(CUTS))
def test_portions(folder, mode, cut):
    f = folder("base")
    ids = tokens(f.cfg, 130)
    assert sum(CUTS[cut]) == 130
    near(f, replay(f, mode, {"a": ids}, [{"a": n} for n in CUTS[cut]])["a"], ids, mode)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", ["base", "layers_differ"])
def test_mixed_batches_reuse_pages(folder, mode, name):
    """Seven requests, four at a time, over a pool that holds only the live ones: portions beside decoded tokens, requests
    that sit out steps, pages handed on with stale contents in them."""
    f = folder(name)
    lens = {"a": 130, "b": 1, "c": 70, "d": 33, "e": 64, "f": 97, "g": 2}
    seqs = {r: tokens(f.cfg, n, seed=10 + i) for i, (r, n) in enumerate(lens.items())}
    rounds = [{"a": 40, "b": 1, "c": 2}, {"c": 17, "a": 1}, {"d": 2, "a": 1, "c": 1, "e": 30}, {"d": 3, "e": 1}, {"a": 50, "d": 28, "e": 1},
              {"c": 50, "e": 32}, {"f": 64, "a": 1, "g": 2}, {"a": 37, "f": 31}, {"f": 1}, {"f": 1}]
    got = replay(f, mode, seqs, rounds, max_tokens=192 + 128 + 64 + 64)
    for r, ids in seqs.items():
        near(f, got[r], ids, mode)


@pytest.mark.parametrize("mode", MODES[1:])
def test_a_batch_gives_what_each_request_gives_alone(folder, mode):
    """Beyond rounding (fp32: to the last bit where the same kernels run)."""
    f = folder("base")
    seqs = {r: tokens(f.cfg, n, seed=30 + n) for r, n in (("a", 77), ("b", 19), ("c", 40), ("d", 5))}
    cuts = {"a": [50, 20, 7], "b": [1, 17, 1], "c": [3, 30, 7], "d": [2, 1, 2]}
    got = replay(f, mode, seqs, [{r: cuts[r][i] for r in seqs} for i in range(3)])
    for r, ids in seqs.items():
        alone = replay(f, mode, {r: ids}, [{r: n} for n in cuts[r]])[r]
        check(got[r], alone, 1e-6 if mode[1] == "float32" else 0.1, 0 if mode[1] == "float32" else 0.8)


@pytest.mark.parametrize("mode", MODES)
def test_long_decode(folder, mode):
    """Windows pass over decoded tokens many times; queries grow with every period."""
    f = folder("base")
    ids = tokens(f.cfg, 230, seed=4)
    near(f, replay(f, mode, {"a": ids}, [{"a": 3}] + [{"a": 1}] * 227)["a"], ids, mode)


@pytest.mark.parametrize("mode", MODES)
def test_first_tokens(folder, mode):
    for name in ("base", "layers_differ"):
        f = folder(name)
        ids = tokens(f.cfg, 6, seed=5)
        for rounds in ([{"a": 6}], [{"a": 1}] * 6, [{"a": 2}] * 3, [{"a": 1}, {"a": 5}]):
            near(f, replay(f, mode, {"a": ids}, rounds)["a"], ids, mode)


@pytest.mark.parametrize("mode", MODES)
def test_stream_after_every_layer(folder, mode):
    dev, dtype, tol = mode
    f = folder("layers_differ")
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
        check(x.cpu(), want, tol, 0.8 if dtype == "bfloat16" else 0)


CHANGES = {
    "window": lambda c, W: c["layers"][0]["mixer"]["mask"].update(size=22),
    "second window": lambda c, W: c["layers"][2]["mixer"]["mask"].update(size=33),
    "yarn factor": lambda c, W: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=2.0),
    "yarn range": lambda c, W: c["layers"][0]["mixer"]["rot"]["scaling"].update(fast=2.0),
    "query latent norm": lambda c, W: W["l0.mix.dq.norm"].mul_(W["l0.mix.uk"][:28, 0].abs() + 0.5),
    "channel gates": lambda c, W: W["l0.mix.g"].copy_(W["l0.mix.g"].flip(0)),
    "growth": lambda c, W: c["layers"][1]["mixer"]["q_temp"].update(every=10),
    "lambda": lambda c, W: W["l1.mix.lq2"].mul_(2),
    "diff": lambda c, W: c["layers"][1]["mixer"].update(diff=0.3),
    "maps": lambda c, W: W["l1.mix.k"].copy_(W["l1.mix.k"].view(2, 2, 20, 72).flip(1).reshape(80, 72)),
    "groups": lambda c, W: c["layers"][1]["mlp"]["router"]["groups"].update(keep=3),
    "router scale": lambda c, W: c["layers"][1]["mlp"]["router"].update(scale=1.0),
    "shared gate": lambda c, W: W["l1.mlp.shared.sg"].neg_(),
    "embedding scale": lambda c, W: c["embedding"].update(scale=6.0),
    "logit scale": lambda c, W: c.update(logit_scale=0.31),
    "norm gain": lambda c, W: W["l3.norm2"].add_(0.5),
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
    from lm_harness import Folder
    f = Folder(tmp_path, cfg, W, O.forward)
    check(replay(f, ("cpu", "float32", 0), {"a": ids}, [{"a": 45}] + [{"a": 1}] * 15)["a"], after, 1e-4)


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


def test_preemption_recomputes(folder):
    """A pool that forces preemption: the same tokens."""
    f = folder("base")
    prompts = [{"prompt_token_ids": tokens(f.cfg, n, seed=40 + n)} for n in (20, 9, 14, 5)]
    sp = SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True, detokenize=False)

    def run(blocks, seqs):
        llm = OmniLLM(f.path, dtype="float32", device="cpu", num_gpu_blocks=blocks, block_size=8, max_num_seqs=seqs)
        out = [list(o.outputs[0].token_ids) for o in llm.generate(prompts, sp)]
        assert llm.engine.kv.pool.num_free == blocks
        return out
    free = run(64, 4)
    assert run(8, 4) == free and run(64, 2) == free


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
    """The static-buffer step a graph replays, with padding rows that write no pages."""
    f = folder("base")
    monkeypatch.setenv("OMNI_AR_CUDA_GRAPH", "1")
    ids = {r: tokens(f.cfg, 30, seed=i) for i, r in enumerate("abc")}
    got = replay(f, ("cpu", "float32", 0), ids, [{"a": 10, "b": 12, "c": 11}] + [{"a": 1, "b": 1, "c": 1}] * 18 + [{"a": 2, "c": 1}])
    for r in "ac":
        check(got[r], f.expected(ids[r]), 1e-4)


def test_runs_without_a_checkpoint():
    llm = OmniLLM(None, model_arch="Milivik", device="cpu", num_gpu_blocks=16)
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


@pytest.mark.parametrize("mode", MODES)
def test_rows_of_a_request(folder, mode):
    """What a hand-off of a request carries: latent rows, keys of both maps side by side with the values they share."""
    f = folder("base")
    rp = TraceReplay(f.path, mode[1], 128, device=mode[0])
    rp.step([{"id": "b", "tokens": tokens(f.cfg, 17), "want": []}, {"id": "a", "tokens": tokens(f.cfg, 21), "want": []}])
    runner, req = rp.engine.runner, rp.live["a"]
    kv = runner.extract_kv(req)
    assert kv["num_tokens"] == 21
    for got, pages in zip(kv["layers"], runner.kv_caches):
        for g, c in zip(got, pages):
            assert torch.equal(g, torch.cat([c[b] for b in req.block_ids])[:21])
    assert [(tuple(k.shape), tuple(v.shape)) for k, v in kv["layers"]] == [
        ((21, 1, 64), (21, 1, 0)), ((21, 2, 64), (21, 2, 48)), ((21, 1, 64), (21, 1, 0)), ((21, 3, 64), (21, 3, 48))]
    assert all(k.abs().sum() > 0 for k, _ in kv["layers"])


# ------------------------------------------------------------------------------ configuration
@pytest.mark.parametrize("change", [
    lambda l: l[0].update(type="something"),
    lambda l: l[0]["mixer"].update(rot_dim=7, rot={"base": 10.0, "dims": 7}),
    lambda l: l[0]["mixer"].update(rot={"base": 10.0, "dims": 8}),
    lambda l: l[0]["mixer"]["mask"].update(size=0),
    lambda l: l[1]["mixer"].update(kv_heads=4),
    lambda l: l[1]["mixer"]["q_temp"].update(every=0),
    lambda l: l[0]["mlp"].update(kind="other"),
    lambda l: l[1]["mlp"]["router"].update(top=7),
    lambda l: l[1]["mlp"]["router"]["groups"].update(count=4),
    lambda l: l[1]["mlp"]["router"].update(top=5)])
def test_configuration_errors(change):
    bad = copy.deepcopy(CONFIGS["base"])
    MilivikConfig.from_dict(bad)
    change(bad["layers"])
    with pytest.raises(ValueError, match="layer"):
        MilivikConfig.from_dict(bad)


def test_checkpoint_errors():
    cfg = CONFIGS["base"]
    W = weights(cfg)
    dec = MilivikDecoder(MilivikConfig.from_dict(cfg), torch.float32, "cpu")
    assert dec.load_weights(W.items()) == set(W)
    with pytest.raises(ValueError, match="lacks"):
        dec.load_weights((n, w) for n, w in W.items() if n != "l1.mix.lq1")
    with pytest.raises(ValueError, match="shape"):
        dec.load_weights([("l0.mix.uq", W["l0.mix.uq"].t())])
