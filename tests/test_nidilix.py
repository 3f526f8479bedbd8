"""Nidilix decoder through the framework: checkpoint folder, engine step, pages and state slots, decode graphs, sampling,
the public entry points — against the plain restatement (tests/nidilix_oracle.py)."""
import copy
import io
import json
import struct

import pytest
import torch

import nidilix_oracle as O
from lm_harness import check, folder_fixture, modes, replay, tokens
from vllm_omni_b200.entrypoints.omni_llm import OmniLLM
from vllm_omni_b200.entrypoints.trace import TraceReplay
from vllm_omni_b200.inputs.data import SamplingParams
from vllm_omni_b200.models.nidilix import NidilixConfig, NidilixDecoder, tiny_config_dict

MODES = modes(0.06)


def tail(mode):
    return 0.25 if mode[1] == "bfloat16" else 0.0


def moe(ff=56, experts=6, top=2, shared=40):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top},
            "shared": None if shared is None else {"ff": shared}}


def attention(heads=3, dim=24, rot=12, vdim=20, rank=40, scale=0.25, base=5000.0, kv_from=None, mlp=moe()):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def scan(width=96, blocks=3, conv=4, mlp=moe()):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def config(layers, width=72, vocab=211, eps=1e-4, mult=0.4, side=20):
    return {"architecture": "Nidilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "token_side": None if side is None else {"dim": side}, "layers": layers}


CONFIGS = {
    "base": config([attention(), scan(), attention(kv_from=0, heads=5, dim=16, vdim=36, scale=0.3), scan()]),
    "layers_differ": config([scan(width=60, blocks=2, conv=2, mlp=moe(24, 5, 5, None)), attention(heads=2, rank=24, mlp=None),
                             attention(heads=4, rot=8, rank=72, base=100.0), scan(mlp=None), scan(width=40, blocks=1, conv=1),
                             attention(heads=1, rot=8, rank=72, base=100.0, kv_from=2, mlp=moe(136, 9, 4, 16))], width=90, vocab=131),
    "smallest_values": config([attention(1, 2, 2, 1, 1, mlp=moe(1, 1, 1, 1)), scan(1, 1, 1, mlp=moe(1, 2, 1, 1))], width=8, vocab=40, side=1),
    "no_side": config([scan(), attention(), scan(mlp=None)], side=None, mult=1.0),
    "wide_heads": config([attention(heads=2, dim=136, rot=40, vdim=128, rank=96), attention(heads=18, dim=40, rot=64, vdim=24, rank=200)]),
    "only_scans": config([scan(conv=3), scan(width=544, blocks=2, conv=6)]),
    "only_attention": config([attention(), attention(kv_from=0), attention(kv_from=0, vdim=144)], side=7),
}


def weights(cfg, seed=0):
    """Random bf16 weights whose every mechanism moves the logits.  Router logits lie far apart, so that rounding decides
    no choice that matters."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda s: torch.randn(s, generator=g)
    out = {}
    for name, shape in NidilixConfig.from_dict(cfg).tensor_shapes().items():
        last = name.split(".")[-1]
        if last.startswith("norm"):
            w = 0.4 + torch.rand(shape, generator=g)
        elif last == "alpha":
            w = 0.5 + 0.5 * torch.rand(shape, generator=g)
        elif last == "b":
            w = 0.3 * rnd(shape)
        elif last == "lam":
            w = rnd(shape) - 3
        elif last == "conv":
            w = 0.6 * rnd(shape)
        elif last == "router":
            w = 12 * rnd(shape) * shape[-1] ** -0.5
        else:
            w = rnd(shape) * (1.0 if name in ("embed", "side.embed") else 1.5 * shape[-1] ** -0.5)
        out[name] = w.bfloat16()
    return out


folder = folder_fixture(CONFIGS, weights, O.forward)


# ----------------------------------------------------------------------------- prompts and portions
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt(folder, mode, name):
    f = folder(name)
    ids = tokens(f.cfg, 150)
    check(replay(f, mode, {"a": ids}, [{"a": 150}])["a"], f.expected(ids), mode[2], tail(mode))


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_token_by_token(folder, mode, name):
    f = folder(name)
    ids = tokens(f.cfg, 150)[:60]
    check(replay(f, mode, {"a": ids}, [{"a": 1}] * 60)["a"], f.expected(tokens(f.cfg, 150))[:60], mode[2], tail(mode))


CUTS = {"pairs": [2] * 75, "threes": [3] * 50, "page_and_more": [16, 17, 15, 1, 31, 33, 37], "growing": [2, 3, 5, 8, 13, 21, 34, 64],
        "tail_decoded": [100] + [1] * 50, "head_decoded": [1] * 20 + [130], "borders": [127, 1, 1, 1, 2, 4, 5, 9]}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("cut", sorted(CUTS))
def test_portions(folder, mode, cut):
    f = folder("base")
    ids = tokens(f.cfg, 150)
    assert sum(CUTS[cut]) == 150
    check(replay(f, mode, {"a": ids}, [{"a": n} for n in CUTS[cut]])["a"], f.expected(ids), mode[2], tail(mode))


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", ["base", "layers_differ"])
def test_mixed_batches_reuse_pages_and_slots(folder, mode, name):
    """Seven requests through four slots and a pool that holds only the live ones: portions beside decoded tokens,
    requests that sit out steps, pages and slots handed on with stale contents in them."""
    f = folder(name)
    lens = {"a": 130, "b": 1, "c": 70, "d": 33, "e": 64, "f": 97, "g": 2}
    seqs = {r: tokens(f.cfg, n, seed=10 + i) for i, (r, n) in enumerate(lens.items())}
    rounds = [{"a": 40, "b": 1, "c": 2}, {"c": 17, "a": 1}, {"d": 2, "a": 1, "c": 1, "e": 30}, {"d": 3, "e": 1}, {"a": 50, "d": 28, "e": 1},
              {"c": 50, "e": 32}, {"f": 64, "a": 1, "g": 2}, {"a": 37, "f": 31}, {"f": 1}, {"f": 1}]
    got = replay(f, mode, seqs, rounds, max_tokens=192 + 128 + 64 + 64)
    for r, ids in seqs.items():
        check(got[r], f.expected(ids), mode[2], tail(mode))


@pytest.mark.parametrize("mode", MODES)
def test_long_decode(folder, mode):
    f = folder("base")
    ids = tokens(f.cfg, 260, seed=4)
    check(replay(f, mode, {"a": ids}, [{"a": 3}] + [{"a": 1}] * 257)["a"], f.expected(ids), mode[2], tail(mode))


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
        check(x.cpu(), want, tol, tail(mode))


def test_a_layer_reads_the_latents_of_another(folder):
    """Changing the source layer's latents changes a reader's logits through its pages alone: the reader has none."""
    f = folder("only_attention")
    cfg = NidilixConfig.from_dict(f.cfg)
    assert [s[0] for s in cfg.kv_layer_shapes()] == [1, 0, 0]
    assert "l1.mix.dkv" not in cfg.tensor_shapes() and "l0.mix.dkv" in cfg.tensor_shapes()
    own = copy.deepcopy(f.cfg)
    del own["layers"][1]["mixer"]["kv_from"]
    W = dict(f.weights, **{"l1.mix.dkv": f.weights["l0.mix.dkv"].flip(0).contiguous(), "l1.mix.dkv.norm": f.weights["l0.mix.dkv.norm"]})
    ids = tokens(f.cfg, 30)
    assert (O.forward(own, W, ids) - f.expected(ids)).abs().max() > 0.05


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
    llm = OmniLLM(None, model_arch="Nidilix", device="cpu", num_gpu_blocks=16)
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


def test_state_and_rows_of_a_request(folder):
    """What a hand-off of a request carries: latent rows of the layers that have pages, both state tensors of a scan."""
    f = folder("base")
    rp = TraceReplay(f.path, "float32", 64, device="cpu")
    rp.step([{"id": "a", "tokens": tokens(f.cfg, 21), "want": []}])
    kv = rp.engine.runner.extract_kv(rp.live["a"])
    assert kv["num_tokens"] == 21 and [tuple(k.shape) for k, _ in kv["layers"]] == [(21, 1, 64), (21, 0, 0), (21, 0, 0), (21, 0, 0)]
    assert [[tuple(t.shape) for t in s] for s in kv["state"]] == [[], [(3, 96), (96,)], [], [(3, 96), (96,)]]
    assert kv["layers"][0][0].abs().sum() > 0 and kv["state"][1][1].dtype == torch.float32


# ------------------------------------------------------------------------------ configuration
@pytest.mark.parametrize("change", [
    lambda l: l[0].update(type="something"),
    lambda l: l[0]["mixer"].update(rot_dim=7, rot={"base": 10.0, "dims": 7}),
    lambda l: l[0]["mixer"].update(rot={"base": 10.0, "dims": 8}),
    lambda l: l[1]["mixer"].update(blocks=5),
    lambda l: l[2]["mixer"].update(kv_from=1),
    lambda l: l[2]["mixer"].update(kv_from=2),
    lambda l: l[2]["mixer"].update(kv_rank=48),
    lambda l: l[2]["mixer"]["rot"].update(base=1.0),
    lambda l: l[0]["mlp"].update(kind="dense"),
    lambda l: l[0]["mlp"]["router"].update(top=7)])
def test_configuration_errors(change):
    bad = copy.deepcopy(CONFIGS["base"])
    NidilixConfig.from_dict(bad)
    change(bad["layers"])
    with pytest.raises(ValueError):
        NidilixConfig.from_dict(bad)


def test_checkpoint_errors():
    cfg = CONFIGS["base"]
    W = weights(cfg)
    dec = NidilixDecoder(NidilixConfig.from_dict(cfg), torch.float32, "cpu")
    assert dec.load_weights(W.items()) == set(W)
    with pytest.raises(ValueError, match="lacks"):
        dec.load_weights((n, w) for n, w in W.items() if n != "l1.mix.lam")
    with pytest.raises(ValueError, match="shape"):
        dec.load_weights([("l0.mix.q", W["l0.mix.q"].t())])


def test_pages_hold_only_what_they_must():
    """Latent layers cost one row per token for all heads; scans and readers cost no pages."""
    cfg = NidilixConfig.from_dict(CONFIGS["layers_differ"])
    assert cfg.kv_layer_shapes() == [(0, 0, 0), (1, 32 + 16, 0), (1, 80 + 16, 0), (0, 0, 0), (0, 0, 0), (0, 0, 0)]
    assert [len(s) for s in cfg.state_shapes()] == [2, 0, 0, 2, 2, 0]
