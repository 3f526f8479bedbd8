"""Tavulix decoder through the framework: checkpoint folder, engine step, pages and state slots, decode graphs, sampling,
the public entry points — against the plain restatement (tests/tavulix_oracle.py)."""
import io
import json
import struct

import pytest
import torch

import tavulix_oracle as O
from lm_harness import check, folder_fixture, modes, replay, tokens
from vllm_omni_b200.entrypoints.omni_llm import OmniLLM
from vllm_omni_b200.entrypoints.trace import TraceReplay
from vllm_omni_b200.inputs.data import SamplingParams
from vllm_omni_b200.models.tavulix import TavulixConfig, tiny_config_dict

MODES = modes(0.04)


def mixer(heads=6, kv=2, dim=40, vdim=24, conv=3, size=30, keep=4, cap=9.0, mix=True, scale=0.3):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "softcap": cap,
            "v_mix": mix, "mask": {"size": size, "keep_first": keep}}


def config(mixers, ffs, width=72, vocab=211, positions=512, cap=21.0, eps=1e-4):
    return {"architecture": "Tavulix", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
            "logit_softcap": cap,
            "layers": [{"type": "attention", "mixer": m, "mlp": None if f is None else {"kind": "dense", "ff": f}}
                       for m, f in zip(mixers, ffs)]}


CONFIGS = {
    "base": config([mixer(), mixer(size=50, keep=7), mixer(size=17, keep=0)], [96, 40, 136]),
    "layers_differ": config([mixer(heads=4, kv=4, dim=16, vdim=24, conv=2, mix=False), mixer(heads=8, kv=1, dim=72, vdim=20),
                             mixer(heads=2, kv=1, dim=24, vdim=20, conv=5, size=300, keep=0),
                             mixer(heads=3, kv=3, dim=20, vdim=33, conv=4, mix=False)], [None, 52, None, 100], width=90, vocab=131),
    "smallest_values": config([mixer(heads=1, kv=1, dim=16, vdim=16, conv=1, size=1, keep=1)] * 2, [8, 8], width=8, vocab=40),
    "without_options": config([mixer(conv=0, cap=None, mix=False), mixer(conv=0, cap=None, mix=False, size=64, keep=64)],
                              [48, None], cap=None),
    "wide_window": config([mixer(size=4096, keep=3), mixer(size=2, keep=100)], [64, 72]),
}
CONFIGS["no_mask"] = config([mixer(), mixer()], [40, 40])
CONFIGS["no_mask"]["layers"][1]["mixer"]["mask"] = None


def weights(cfg, seed=0):
    """Random bf16 weights whose every mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda s: torch.randn(s, generator=g)
    out = {}
    for name, shape in TavulixConfig.from_dict(cfg).tensor_shapes().items():
        last = name.split(".")[-1]
        if last in ("r1", "r2"):
            w = 0.05 + rnd(shape).abs() * (0.8 if last == "r1" else 0.2)
        elif last == "vmix":
            w = 0.3 + 0.3 * torch.rand(shape, generator=g)
        elif last.startswith("norm") or last == "act":
            w = 0.4 + torch.rand(shape, generator=g)
        elif last == "sink":
            w = 2 * rnd(shape)
        elif last == "conv":
            w = 0.7 * rnd(shape)
        else:
            w = rnd(shape) * (1.0 if name in ("embed", "pos") else 1.5 * shape[-1] ** -0.5)
        out[name] = w.bfloat16()
    return out


folder = folder_fixture(CONFIGS, weights, O.forward)


# ----------------------------------------------------------------------------- prompts and portions
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt(folder, mode, name):
    f = folder(name)
    ids = tokens(f.cfg, 150)
    check(replay(f, mode, {"a": ids}, [{"a": 150}])["a"], f.expected(ids), mode[2])


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_token_by_token(folder, mode, name):
    f = folder(name)
    ids = tokens(f.cfg, 90)
    check(replay(f, mode, {"a": ids}, [{"a": 1}] * 90)["a"], f.expected(ids), mode[2])


CUTS = {"pairs": [2] * 75, "threes": [3] * 50, "page_and_more": [16, 17, 15, 1, 31, 33, 37], "growing": [2, 3, 5, 8, 13, 21, 34, 64],
        "tail_decoded": [100] + [1] * 50, "head_decoded": [1] * 20 + [130], "window_edges": [29, 1, 1, 18, 1, 1, 49, 2, 48]}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("cut", sorted(CUTS))
def test_portions(folder, mode, cut):
    f = folder("base")
    ids = tokens(f.cfg, 150)
    assert sum(CUTS[cut]) == 150
    check(replay(f, mode, {"a": ids}, [{"a": n} for n in CUTS[cut]])["a"], f.expected(ids), mode[2])


@pytest.mark.parametrize("mode", MODES)
def test_mixed_batches_reuse_pages_and_slots(folder, mode):
    """Seven requests through four slots and a pool that holds only the live ones: portions beside decoded tokens,
    requests that sit out steps, pages and slots handed on with stale contents in them."""
    f = folder("base")
    lens = {"a": 130, "b": 1, "c": 70, "d": 33, "e": 64, "f": 97, "g": 2}
    seqs = {r: tokens(f.cfg, n, seed=10 + i) for i, (r, n) in enumerate(lens.items())}
    rounds = [{"a": 40, "b": 1, "c": 2}, {"c": 17, "a": 1}, {"d": 2, "a": 1, "c": 1, "e": 30}, {"d": 3, "e": 1}, {"a": 50, "d": 28, "e": 1},
              {"c": 50, "e": 32}, {"f": 64, "a": 1, "g": 2}, {"a": 37, "f": 31}, {"f": 1}, {"f": 1}]
    got = replay(f, mode, seqs, rounds, max_tokens=192 + 128 + 64 + 64)
    for r, ids in seqs.items():
        check(got[r], f.expected(ids), mode[2])


@pytest.mark.parametrize("mode", MODES)
def test_long_decode(folder, mode):
    """Windows of 30, 50 and 17 tokens pass several times over decoded tokens."""
    f = folder("base")
    ids = tokens(f.cfg, 260, seed=4)
    check(replay(f, mode, {"a": ids}, [{"a": 3}] + [{"a": 1}] * 257)["a"], f.expected(ids), mode[2])


@pytest.mark.parametrize("mode", MODES)
def test_first_tokens(folder, mode):
    f = folder("base")
    ids = tokens(f.cfg, 6, seed=5)
    for rounds in ([{"a": 6}], [{"a": 1}] * 6, [{"a": 2}] * 3, [{"a": 1}, {"a": 5}]):
        check(replay(f, mode, {"a": ids}, rounds)["a"], f.expected(ids), mode[2])


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
        check(x.cpu(), want, tol)


# --------------------------------------------------------------------------------- generation
@pytest.mark.parametrize("mode", MODES[:2])
def test_greedy_generation_matches(folder, mode):
    """Through the engine's own scheduler: a prompt longer than the step budget, short ones beside it."""
    f = folder("base")
    prompts = [tokens(f.cfg, n, seed=20 + n) for n in (45, 7, 1)]
    llm = OmniLLM(f.path, dtype=mode[1], device=mode[0], num_gpu_blocks=40, max_num_seqs=3, max_num_batched_tokens=16)
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts],
                        SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True, detokenize=False))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == f.greedy(p, 24)
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
        assert (llm.engine.runner.graph_runner.replays > 30) if graph == "1" else llm.engine.runner.graph_runner is None
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


def test_length_limit(folder):
    """Generation ends at the last learned position; longer prompts are refused."""
    cfg = tiny_config_dict(max_positions=40)
    llm = OmniLLM(None, model_arch="Tavulix", device="cpu", num_gpu_blocks=16, model_overrides={"config": {"max_positions": 40}})
    assert llm.model.decoder_config.max_positions == cfg["max_positions"]
    out = llm.generate({"prompt_token_ids": list(range(30))}, SamplingParams(temperature=0.0, max_tokens=100, ignore_eos=True))[0]
    assert len(out.outputs[0].token_ids) == 10 and out.outputs[0].finish_reason == "length"
    with pytest.raises(ValueError):
        llm.add_request("long", {"prompt_token_ids": list(range(41))})


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
    assert sorted(p.name for p in tmp_path.iterdir()) == ["1.f32"]
    raw = (tmp_path / "1.f32").read_bytes()
    got = torch.tensor(struct.unpack(f"<{len(raw) // 4}f", raw)).view(3, -1)
    want = f.expected(ids)
    check(got, want[[9, 19, 0]], 1e-4)


def test_replay_refuses_what_does_not_fit(folder):
    f = folder("base")
    rp = TraceReplay(f.path, "float32", 64, device="cpu")
    with pytest.raises(RuntimeError):
        rp.step([{"id": "a", "tokens": tokens(f.cfg, 65), "want": []}])
    rp = TraceReplay(f.path, "float32", 1024, device="cpu")
    with pytest.raises(ValueError):
        rp.step([{"id": "a", "tokens": tokens(f.cfg, 513), "want": []}])
    with pytest.raises(ValueError):
        rp.step([{"id": "b", "tokens": [1, 2], "want": [2]}])
    with pytest.raises(RuntimeError):
        rp.step([{"id": str(i), "tokens": [1], "want": []} for i in range(5)])


# ------------------------------------------------------------------------------ configuration
def test_configuration_errors():
    for change in ({"heads": 5}, {"mask": {"size": 0}}):
        bad = config([dict(mixer(), **change)], [8])
        with pytest.raises(ValueError):
            TavulixConfig.from_dict(bad)
    bad = config([mixer()], [8])
    bad["layers"][0]["type"] = "something"
    with pytest.raises(ValueError):
        TavulixConfig.from_dict(bad)
    with pytest.raises(ValueError):
        TavulixConfig.from_dict(config([mixer(), mixer(vdim=32)], [8, 8]))


def test_checkpoint_errors():
    from vllm_omni_b200.models.tavulix import TavulixDecoder
    cfg = CONFIGS["base"]
    W = weights(cfg)
    dec = TavulixDecoder(TavulixConfig.from_dict(cfg), torch.float32, "cpu")
    assert dec.load_weights(W.items()) == set(W)
    with pytest.raises(ValueError, match="lacks"):
        dec.load_weights((n, w) for n, w in W.items() if n != "l1.mix.sink")
    with pytest.raises(ValueError, match="shape"):
        dec.load_weights([("l0.mix.q", W["l0.mix.q"].t())])


def test_state_slots():
    from vllm_omni_b200.engine.kv_cache_manager import KVCacheManager
    from vllm_omni_b200.engine.request import Request
    kv = KVCacheManager(4, 16, num_state_slots=2)
    a, b, c = (Request(x, [0] * 40, SamplingParams()) for x in "abc")
    assert kv.allocate_slots(a, 16) and kv.allocate_slots(b, 16) and not kv.allocate_slots(c, 16)
    assert c.block_ids == [] and kv.pool.num_free == 2
    seen = {kv.state.rows(a), kv.state.rows(b)}
    assert len({r for p in seen for r in p}) == 4
    r, w = kv.state.rows(a)
    kv.state.advance(a)
    assert kv.state.rows(a) == (w, r)
    kv.free(a)
    assert a.state_slot is None and not kv.allocate_slots(c, 64)      # too few pages: the slot goes back
    assert c.state_slot is None and kv.state.num_free == 1
    assert kv.allocate_slots(c, 16) and kv.state.rows(c)[0] % 2 == 0
