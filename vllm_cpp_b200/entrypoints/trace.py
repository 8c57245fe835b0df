"""Replays a trace of given token ids through the engine, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Reads one JSON object a line from standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every entry's tokens are appended to its request (a request with open input, see
``LLM.extend_request``) and the entries run as one engine step. ``want`` lists places among the
entry's tokens whose logits are written to ``<out>/<step>.f32`` (little-endian fp32, entries in
order); ``end`` names the requests that are finished after the step. ``done <step>`` is printed after
each step. Nothing is sampled. The cache holds ``--max-tokens`` tokens, each request's count rounded
up to whole pages."""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64
MAX_REQUESTS = 4


class TraceReplay:
    def __init__(self, model: str, dtype: str, max_tokens: int, device: str = "cuda", max_requests: int = MAX_REQUESTS,
                 page: int = PAGE):
        from ..config import EngineArgs
        from ..engine import LLM
        pages = (max_tokens + page - 1) // page
        # one page beyond the pool is the block pool's null page
        self.llm = LLM(EngineArgs(model=model, dtype=dtype, device=device, block_size=page, num_blocks=pages + 1,
                                  max_model_len=pages * page + 2, max_num_seqs=max_requests,
                                  max_num_batched_tokens=pages * page, max_score_rows=pages * page,
                                  enable_prefix_caching=False))
        self.length: dict[str, int] = {}
        self.name: dict[str, str] = {}       # of a live request in the engine (a trace may use an id again)
        self.count = 0

    def step(self, entries: list, end: list):
        """-> the wanted logits rows, in the order of the entries and their ``want``."""
        from ..engine import SamplingParams
        llm, order, total = self.llm, [], 0
        for e in entries:
            if e["id"] not in self.name:
                self.count += 1
                self.name[e["id"]] = f"{e['id']}.{self.count}"
            rid, toks = self.name[e["id"]], e["tokens"]
            at = self.length.get(rid, 0)
            want = [at + w for w in e.get("want", [])]
            if want:
                llm.score_positions(rid, sorted(set(want)))
            if rid in self.length:
                llm.extend_request(rid, toks)
            else:
                llm.add_request(toks, SamplingParams(temperature=0.0, prompt_logprobs=0), request_id=rid, input_open=True)
            self.length[rid] = at + len(toks)
            total += len(toks)
            order += [(rid, p) for p in want]
        if total:
            llm.step()
            ran = llm.step_stats()["scheduled_tokens"]
            if ran != total:
                raise RuntimeError(f"the engine ran {ran} of the step's {total} tokens")
        rows = {(rid, p): row for rid, items in llm.take_scores().items() for p, row in items}
        for rid in (self.name.pop(i) for i in end if i in self.name):
            llm.abort_request(rid)
            self.length.pop(rid, None)
        return [rows[k] for k in order]


def main(argv=None) -> int:
    ap = argparse.ArgumentParser("trace_run", description="replay a token trace and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    replay = TraceReplay(a.model, a.dtype, a.max_tokens, a.device)
    import torch
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        rows = replay.step(s.get("entries", []), s.get("end", []))
        if rows:
            torch.stack(rows).contiguous().numpy().astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0
