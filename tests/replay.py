"""What the engine tests of the families with listed layers share: random token ids, steps of (request,
count) pairs through the trace replay, small engines."""
import random

import torch


def tokens(n, vocab, seed):
    return [random.Random(seed).randrange(vocab) for _ in range(n)] if n < 2 else \
        [random.Random(seed * 1000003 + i).randrange(vocab) for i in range(n)]


def rel(got, want):
    """Row-wise error of the logits with their mean taken off."""
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return (d.norm(dim=-1) / w.norm(dim=-1)).max().item()


def random_steps(left, seed, sizes=(1, 1, 1, 2, 5, 16)):
    """Portions of the requests ``left`` {id: tokens} beside single tokens; requests pause now and then."""
    left, rnd, steps = dict(left), random.Random(seed), []
    while left:
        step = []
        for r in list(left):
            if rnd.random() < 0.25:
                continue
            n = min(left[r], rnd.choice(sizes))
            step.append((r, n))
            left[r] -= n
            if not left[r]:
                del left[r]
        if step:
            steps.append(step)
    return steps


class Replay:
    """Steps of (request, count) pairs through the engine; collects the logits of every position."""

    def __init__(self, model, dtype, dev, max_tokens, page=8, max_requests=4):
        from vllm_cpp_b200.entrypoints.trace import TraceReplay
        self.r = TraceReplay(model, dtype, max_tokens, dev, max_requests=max_requests, page=page)

    def run(self, prompts, steps):
        at, got = {}, {}
        for step in steps:
            entries, end = [], []
            for rid, n in step:
                lo = at.get(rid, 0)
                entries.append({"id": rid, "tokens": prompts[rid][lo:lo + n], "want": list(range(n))})
                at[rid] = lo + n
                if at[rid] == len(prompts[rid]):
                    end.append(rid)
            rows = self.r.step(entries, end)
            for e in entries:
                got.setdefault(e["id"], []).extend(rows[:len(e["tokens"])])
                rows = rows[len(e["tokens"]):]
        assert all(len(v) == at[k] for k, v in got.items())
        return {k: torch.stack(v) for k, v in got.items()}

    def free_pages(self):
        return self.r.llm.core.scheduler().num_free_blocks()


def engine(model, dtype, dev, **kw):
    from vllm_cpp_b200.config import EngineArgs
    from vllm_cpp_b200.engine import LLM
    args = dict(model=model, dtype=dtype, device=dev, block_size=8, num_blocks=80, max_model_len=256, max_num_seqs=4,
                max_num_batched_tokens=64)
    return LLM(EngineArgs(**{**args, **kw}))


def greedy(n, **kw):
    from vllm_cpp_b200.engine import SamplingParams
    return SamplingParams(temperature=0.0, max_tokens=n, ignore_eos=True, **kw)
