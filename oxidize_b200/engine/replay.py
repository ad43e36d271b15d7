"""Trace replay: feed given token ids through an engine step by step and write the logits that are asked for.

The steps come as JSON lines on standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

every entry being the next tokens of a request and the places among them whose logits are wanted; ``end`` names the
requests that are finished after the step.  The logits of a step go to ``OUT/<step>.f32`` (little-endian float32,
[wanted, vocab], in the order of the entries), and ``done <step>`` is printed after every step.  All entries of a step are
one batch through the engine's scheduler, paged cache, runner and model; nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < trace.jsonl
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Any, Dict, List, Optional

import torch

from .llm import LLM, EngineConfig
from .sampler import SamplingParams
from .scheduler import Sequence

LIVE_REQUESTS = 4  # requests that hold cache pages at the same time
TOKEN_UNIT = 64  # a request's share of --max-tokens is rounded up to this many tokens


class TraceReplay:
    """Requests whose tokens the caller supplies portion by portion, on one engine."""

    def __init__(self, llm: LLM):
        self.llm = llm
        self.live: Dict[str, Sequence] = {}

    def step(self, entries: List[Dict[str, Any]], end: List[str]) -> torch.Tensor:
        """Run one batch; returns the wanted logits [n, vocab] (float32, on the engine's device)."""
        llm = self.llm
        portions = []
        for e in entries:
            toks = [int(t) for t in e["tokens"]]
            bad = [t for t in toks if not 0 <= t < llm.cfg.vocab_size]
            if bad:
                raise ValueError(f"token id {bad[0]} outside vocabulary of {llm.cfg.vocab_size}")
            seq = self.live.get(e["id"])
            if seq is None:
                seq = self.live[e["id"]] = Sequence([], SamplingParams(temperature=0.0), request_id=str(e["id"]))
            seq.prompt.extend(toks)
            want = [int(w) for w in e.get("want", ())]
            if any(not 0 <= w < len(toks) for w in want):
                raise ValueError(f"request {e['id']}: a wanted place lies outside its {len(toks)} tokens")
            portions.append((seq, len(toks), want))
        logits = torch.empty(0, llm.cfg.vocab_size, device=llm.device)
        if portions:
            out = llm.scheduler.schedule_portions(portions)
            logits = llm.runner.score(out)
            llm.scheduler.finish_portions(out)
        for rid in end:
            llm.scheduler.abort(str(rid))
            self.live.pop(rid, None)
        return logits


def replay_config(max_tokens: int, dtype: str, page: int = 16) -> EngineConfig:
    """An engine whose cache pool holds ``max_tokens`` tokens of live requests."""
    tokens = (max_tokens + TOKEN_UNIT - 1) // TOKEN_UNIT * TOKEN_UNIT
    return EngineConfig(kv_page_size=page, num_kv_blocks=tokens // page, max_model_len=tokens, max_num_seqs=LIVE_REQUESTS,
                        max_num_batched_tokens=tokens, enable_prefix_cache=False,
                        compute_dtype="f32" if dtype == "float32" else "bf16")


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write the logits asked for")
    ap.add_argument("--model", required=True, help="checkpoint: a directory with config.json and model.safetensors, or a GGUF file")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most")
    a = ap.parse_args(argv)
    if not torch.cuda.is_available():
        raise SystemExit("trace_run: no CUDA device")
    torch.backends.cuda.matmul.allow_tf32 = False
    llm = LLM.from_checkpoint(a.model, replay_config(a.max_tokens, a.dtype), device="cuda:0")
    os.makedirs(a.out, exist_ok=True)
    rep = TraceReplay(llm)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = rep.step(s.get("entries", []), s.get("end", []))
        if logits.shape[0]:
            part = os.path.join(a.out, f".{s['step']}.part")
            logits.float().cpu().numpy().astype("<f4").tofile(part)
            os.replace(part, os.path.join(a.out, f"{s['step']}.f32"))
        elif llm.device.type == "cuda":
            torch.cuda.synchronize()
        print(f"done {s['step']}", flush=True)
    from ..ops import cuda as opcuda

    code, detail, count = opcuda.status()
    if code != 0:
        raise RuntimeError(f"device status {code} (detail {detail}, {count} reports)")
    return 0


if __name__ == "__main__":
    sys.exit(main())
