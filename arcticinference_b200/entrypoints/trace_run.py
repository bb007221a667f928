"""Trace runner: feed given token ids through a model step by step and write logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [0, 1]}], "end": []}

All entries of a step run as one batch; ``want`` names the places among an entry's tokens whose
logits go to ``OUT/<step>.f32`` (little-endian fp32, in the order of the entries); requests in
``end`` are finished and give back what they hold. After each step ``done <step>`` is printed.

Nothing is sampled, and the schedule is the caller's; everything else is the engine's: its model,
batch preparation, captured decode steps, cache manager and pool. Exit code 3: the model is not
served in the requested element type.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64


class TraceSession:
    """Drives an engine's runner and cache manager with a given schedule."""

    def __init__(self, engine):
        self.engine = engine
        self.live: dict = {}

    def step(self, entries: list, end: list):
        """Runs the entries as one batch; returns the wanted logits [wanted, vocab] (None when
        nothing is wanted)."""
        from ..engine.request import Request, RequestStatus
        from ..engine.sampling_params import SamplingParams
        from ..engine.scheduler import ScheduledRequest, SchedulerOutput
        kv, runner = self.engine.kv_manager, self.engine.runner
        out = SchedulerOutput()
        vocab = self.engine.config.model.vocab_size
        for e in entries:
            tokens = e["tokens"]
            if not tokens:
                continue
            if min(tokens) < 0 or max(tokens) >= vocab:
                raise ValueError("token id outside the vocabulary")
            req = self.live.get(e["id"])
            if req is None:
                req = self.live[e["id"]] = Request(e["id"], [], SamplingParams(
                    temperature=0.0, ignore_eos=True))
                req.status = RequestStatus.RUNNING
            n, start = len(tokens), req.num_computed_tokens
            kv.allocate(req, n)
            req.prompt_token_ids.extend(int(t) for t in tokens)
            out.scheduled.append(ScheduledRequest(req, start, n, 0, True, want=list(e["want"])))
            out.total_tokens += n
        logits = None
        if out.scheduled:
            logits = runner.score(out)
            for s in out.scheduled:
                s.request.num_computed_tokens += s.num_tokens
        for rid in end:
            req = self.live.pop(rid, None)
            if req is not None:
                kv.free(req)
        return logits


def build_engine(model: str, dtype: str, max_tokens: int, device=None):
    from ..config import EngineArgs
    from ..engine.llm_engine import LLMEngine
    args = EngineArgs(
        model=model, dtype=dtype, block_size=PAGE, max_model_len=max(max_tokens, PAGE),
        # (block 0 is the pool's null block)
        num_gpu_blocks_override=-(-max_tokens // PAGE) + 1, max_num_seqs=4,
        enable_prefix_caching=False)
    return LLMEngine(args.create_engine_config(), device=device)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens live requests hold at any time, each rounded up to 64")
    ap.add_argument("--device", default="cuda", help="cuda (default), or cpu to use the PyTorch "
                                                     "restatements of the kernels")
    ns = ap.parse_args(argv)
    from ..config import ModelConfig
    cfg = ModelConfig.from_pretrained(ns.model)
    if ns.dtype == "float32" and not cfg.supports_float32:
        print("%s is not served in float32" % cfg.architecture, file=sys.stderr)
        return 3
    import numpy as np
    import torch
    from .. import build, ops
    if ns.device == "cuda" and not torch.cuda.is_available():
        print("no CUDA device", file=sys.stderr)
        return 2
    build.select_kernel_set(cfg.architecture)
    session = TraceSession(build_engine(ns.model, ns.dtype, ns.max_tokens, ns.device))
    os.makedirs(ns.out, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        d = json.loads(line)
        logits = session.step(d["entries"], d.get("end", []))
        if logits is not None and logits.shape[0]:
            data = logits.float().cpu().numpy().astype("<f4")
            if ns.device == "cuda":
                ops.check_status()
            path = os.path.join(ns.out, "%d.f32" % d["step"])
            np.ascontiguousarray(data).tofile(path)
        print("done %d" % d["step"], flush=True)
    return 0
