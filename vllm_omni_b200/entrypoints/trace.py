"""Replay of a recorded schedule: token ids in, logits out, step by step through the engine.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps arrive on standard input, one JSON object per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}], "end": []}

``entries``: the next tokens of each request (all of a step's entries are one batch) and the places among
them whose logits are wanted; ``end``: requests that are finished after the step.  A step in which something
is wanted writes ``OUT/<step>.f32`` (little-endian fp32 [wanted, vocab]); every step prints ``done <step>``."""
from __future__ import annotations

import argparse
import json
import os
import sys

BLOCK = 16            # tokens per page
LIVE = 4              # requests that may be live at any time


def make_parser(sub=None) -> argparse.ArgumentParser:
    text = "replay a schedule of token ids from standard input and write logits"
    p = sub.add_parser("trace", help=text) if sub is not None else argparse.ArgumentParser("trace_run", description=text)
    p.add_argument("--model", required=True, help="folder with config.json and the weights")
    p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    p.add_argument("--out", required=True, help="folder for the logits")
    p.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    return p


def prepare(model: str) -> None:
    """Compile what serving the model's architecture loads, if it is not built yet."""
    from ..build import build_set
    from ..models.registry import arch_from_config, native_libs, supported_archs
    with open(os.path.join(model, "config.json")) as f:
        arch = arch_from_config(json.load(f))
    if arch not in supported_archs():
        raise ValueError(f"unknown architecture {arch!r}; supported: {supported_archs()}")
    libs = native_libs(arch)
    if libs is None:
        from ..build import build_all
        build_all(verbose=False)
    else:
        build_set(libs)


class TraceReplay:
    def __init__(self, model: str, dtype: str, max_tokens: int, device: str | None = None):
        from ..engine.portion_scheduler import PortionScheduler
        from .omni_llm import OmniLLM
        self.llm = OmniLLM(model, dtype=dtype, device=device, block_size=BLOCK, num_gpu_blocks=max(1, -(-max_tokens // BLOCK)),
                           max_num_seqs=LIVE, scheduler_cls=PortionScheduler)
        self.engine = self.llm.engine
        self.live: dict = {}

    def _admit(self, rid: str):
        from ..inputs.data import SamplingParams
        req = self.engine.add_request(rid, {"prompt_token_ids": [], "additional_information": {"__expects_chunks__": True}},
                                      SamplingParams(max_tokens=None, ignore_eos=True, detokenize=False))
        self.live[rid] = req
        return req

    def step(self, entries, end=()):
        """Runs one step; returns the wanted logits (a CPU tensor [wanted, vocab]) or None."""
        sch = self.engine.scheduler
        for e in entries:
            rid = str(e["id"])
            sch.plan(self.live.get(rid) or self._admit(rid), [int(t) for t in e["tokens"]], e.get("want") or ())
        logits = None
        if entries:
            self.engine.step()
            logits = sch.last_output.logits
        for rid in end:
            req = self.live.pop(str(rid))
            sch.finish(req)
            self.engine.abort_request(req.request_id)
        return None if logits is None else logits.float().cpu()


def run(args, stdin=None, stdout=None) -> int:
    stdin, stdout = stdin or sys.stdin, stdout or sys.stdout
    import torch
    from ..ops import _native as nv
    if torch.cuda.is_available():
        prepare(args.model)
        torch.backends.cuda.matmul.allow_tf32 = False
    rp = TraceReplay(args.model, args.dtype, args.max_tokens)
    for line in stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = rp.step(s.get("entries") or [], s.get("end") or [])
        if logits is not None:
            with open(os.path.join(args.out, f"{s['step']}.f32"), "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4").tobytes())
        if torch.cuda.is_available():
            nv.check_status()
        stdout.write(f"done {s['step']}\n")
        stdout.flush()
    return 0


def main(argv=None) -> int:
    return run(make_parser().parse_args(argv))
