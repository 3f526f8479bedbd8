"""Shared by the tests of decoder-only language models: checkpoint folders with random weights, replay of schedules
through the engine, comparison of logits with a model's plain restatement."""
import json

import pytest
import torch

from vllm_omni_b200.entrypoints.trace import TraceReplay
from vllm_omni_b200.utils.safetensors_reader import save_safetensors


def modes(bf16_tol: float):
    return [pytest.param(("cpu", "float32", 1e-4), id="cpu"),
            pytest.param(("cuda", "float32", 1e-4), id="fp32", marks=pytest.mark.gpu),
            pytest.param(("cuda", "bfloat16", bf16_tol), id="bf16", marks=pytest.mark.gpu)]


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


class Folder:
    """A checkpoint folder on disk and the model's restatement with memoised results."""

    def __init__(self, path, cfg, weights, oracle):
        self.path, self.cfg, self.weights, self.oracle, self._memo = str(path), cfg, weights, oracle, {}
        (path / "config.json").write_text(json.dumps(cfg))
        save_safetensors(weights, str(path / "model.safetensors"))

    def expected(self, ids):
        key = tuple(ids)
        if key not in self._memo:
            self._memo[key] = self.oracle(self.cfg, self.weights, ids)
        return self._memo[key]

    def greedy(self, prompt, n):
        ids = list(prompt)
        for _ in range(n):
            ids.append(int(self.oracle(self.cfg, self.weights, ids)[-1].argmax()))
        return ids[len(prompt):]


def folder_fixture(configs, weights, oracle):
    @pytest.fixture(scope="module")
    def folder(tmp_path_factory):
        made = {}

        def make(name):
            if name not in made:
                made[name] = Folder(tmp_path_factory.mktemp(name), configs[name], weights(configs[name]), oracle)
            return made[name]
        yield make
    return folder


def check(got, want, tol, tail: float = 0.0):
    """Every row's error (relative to the size of all logits) is below ``tol``; with ``tail``, one row in ten (or one) may
    reach that instead: where a near tie of a router is decided by rounding."""
    got, want = got.double(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert torch.isfinite(got).all() and got.shape == want.shape
    assert err.max() < (tail or tol), f"row {int(err.argmax())}: {float(err.max()):.4g}"
    assert not tail or (err > tol).sum() <= max(1, 0.1 * err.numel()), f"{int((err > tol).sum())} of {err.numel()} rows over {tol}"


def replay(f, mode, seqs, rounds, max_tokens=None):
    """Runs ``rounds`` (lists of {request: tokens of this step}); returns every row's logits per request."""
    dev, dtype, _ = mode
    room = max_tokens or sum((len(s) + 63) // 64 * 64 for s in seqs.values())
    rp = TraceReplay(f.path, dtype, room, device=dev)
    at, out = {r: 0 for r in seqs}, {r: [] for r in seqs}
    for step in rounds:
        entries = [{"id": r, "tokens": seqs[r][at[r]:at[r] + n], "want": list(range(n))} for r, n in step.items()]
        for r, n in step.items():
            at[r] += n
        end = [r for r in step if at[r] == len(seqs[r])]
        lg, o = rp.step(entries, end), 0
        for r, n in step.items():
            out[r].append(lg[o:o + n])
            o += n
    kv = rp.engine.kv
    assert kv.pool.num_free == kv.pool.num_blocks and not rp.engine.scheduler.running
    assert kv.state is None or kv.state.num_free == kv.state.num_slots
    return {r: torch.cat(v) for r, v in out.items()}
