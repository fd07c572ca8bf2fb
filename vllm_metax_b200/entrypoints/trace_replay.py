"""Replays a recorded trace of requests through the engine, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Standard input holds one step per line,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``tokens`` are a request's next token ids, ``want`` the places among them whose logits are asked for, ``end`` the requests
that are finished after the step.  All entries of a step run as one batch through the engine's own scheduler, block pool,
state slots, model and captured decode graphs; nothing is sampled.  Wanted logits go to ``OUT/<step>.f32`` (little-endian
fp32 ``[wanted, vocab]``, in the order of the entries and of ``want``), and ``done <step>`` is printed after every step.

The cache pool holds N tokens (in blocks of 64) and there are state slots for four requests.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

from ..config import CacheConfig, EngineConfig, ModelConfig, SchedulerConfig
from ..engine.llm import LLMEngine
from ..engine.sampling_params import Request, SamplingParams

BLOCK = 64
MAX_LIVE = 4


class TraceReplay:
    """Feeds dictated steps to an engine; ``step`` returns the wanted logits (fp32, host) or None."""

    def __init__(self, engine: LLMEngine):
        self.engine = engine
        self.live: dict[str, Request] = {}

    @classmethod
    def open(cls, model: str, dtype: str, max_tokens: int, device: str = "cuda", max_live: int = MAX_LIVE,
             block_size: int = BLOCK, enforce_eager: bool = False) -> "TraceReplay":
        blocks = -(-max_tokens // block_size)
        n = blocks * block_size
        return cls(LLMEngine(EngineConfig(
            model=ModelConfig.from_pretrained(model, dtype=dtype),
            cache=CacheConfig(block_size=block_size, num_gpu_blocks=blocks),
            scheduler=SchedulerConfig(max_num_seqs=max_live, max_num_batched_tokens=n, max_model_len=n),
            device=device, enforce_eager=enforce_eager)))

    def step(self, entries: list[dict], end: list[str]):
        sch, runner = self.engine.scheduler, self.engine.runner
        places, portions = {}, []
        for e in entries:
            rid, toks = str(e["id"]), [int(t) for t in e["tokens"]]
            req = self.live.get(rid)
            if req is None:
                req = self.live[rid] = Request(rid, [], SamplingParams(max_tokens=1, ignore_eos=True), None, None, None)
            req.prompt_token_ids.extend(toks)
            portions.append((req, len(toks)))
            places[rid] = [int(p) for p in e.get("want") or []]
        logits = None
        if portions:
            so = sch.schedule_portions(portions)
            order = [s.request.request_id for s in so.scheduled]
            logits = runner.execute_logits(so, [places[r] for r in order])
            sch.advance_portions(so)
            if logits is not None:               # from the batch's order back to the entries'
                at, n = {}, 0
                for r in order:
                    at[r] = (n, n + len(places[r]))
                    n += len(places[r])
                logits = torch.cat([logits[slice(*at[str(e["id"])])] for e in entries])
        for rid in end:
            req = self.live.pop(str(rid), None)
            if req is not None:
                sch.retire(req)
        return logits


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of requests and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    replay = TraceReplay.open(a.model, a.dtype, a.max_tokens, a.device)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"], step.get("end") or [])
        if logits is not None:
            path = os.path.join(a.out, f"{int(step['step'])}.f32")
            with open(path, "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4").tobytes())
        if a.device == "cuda":
            torch.cuda.synchronize()
            from .. import _custom_ops as ops

            ops.check_kernel_status(0)
        print(f"done {int(step['step'])}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
