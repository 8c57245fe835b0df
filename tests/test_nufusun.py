"""Nufusun through the engine (registry, loader, scheduler, paged cache, batches) against the plain
implementation in ``nufusun_reference.py``; every test runs on the CPU back end and, on a GPU box,
on the kernels."""
import json
import os
import subprocess
import sys

import pytest
import torch

import nufusun_case as C
import nufusun_reference as R
from replay import Replay, engine, greedy, random_steps, rel, tokens

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
TOL = {"float32": 2e-5, "bfloat16": 4e-2}
both = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
device = pytest.mark.parametrize("dev", DEVICES)
CLOSE_CALL = 0.05       # router margin below which rounding to bf16 may change the chosen experts
_logits: dict = {}


def oracle(name, toks, seed=0):
    key = (name, tuple(toks), seed)
    if key not in _logits:
        cfg, w = C.case(name, seed)
        margins = []
        lg = R.forward(cfg, w, toks, dtype=torch.float64, margins=margins)
        _logits[key] = lg, torch.stack(margins).min(0).values
    return _logits[key][0]


def agrees(got, name, toks, dtype):
    """The logits of every position agree; in bf16, of every position whose experts are no close call
    (there are few of those)."""
    want, margin = oracle(name, toks), _logits[name, tuple(toks), 0][1]
    if dtype == "bfloat16":
        clear = margin > CLOSE_CALL
        assert clear.float().mean() > 0.8 or len(toks) < 20
        got, want = got[clear], want[clear]
        if not len(want):
            return
    assert rel(got, want) < TOL[dtype]


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    base = tmp_path_factory.mktemp("nufusun")
    done = {}

    def get(name, seed=0):
        if (name, seed) not in done:
            done[name, seed] = C.write(base / f"{name}{seed}", *C.case(name, seed))
        return done[name, seed]
    return get


# ------------------------------------------------------------------------------ one sequence
@device
@both
@pytest.mark.parametrize("name", list(C.CASES))
def test_whole_prompt(folder, name, dtype, dev):
    toks = tokens(150, C.CASES[name][0]["vocab"], 1)
    got = Replay(folder(name), dtype, dev, 160).run({"a": toks}, [[("a", len(toks))]])["a"]
    agrees(got, name, toks, dtype)


@device
@both
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_token_by_token(folder, name, dtype, dev):
    toks = tokens(70, C.CASES[name][0]["vocab"], 2)
    got = Replay(folder(name), dtype, dev, 80).run({"a": toks}, [[("a", 1)]] * len(toks))["a"]
    agrees(got, name, toks, dtype)


@device
@both
def test_first_tokens(folder, dtype, dev):
    for n in (1, 2, 3):
        toks = tokens(n, 96, 3 + n)
        for steps in ([[("a", n)]], [[("a", 1)]] * n):
            got = Replay(folder("aligned"), dtype, dev, 8).run({"a": toks}, steps)["a"]
            agrees(got, "aligned", toks, dtype)


@device
@both
@pytest.mark.parametrize("sizes", [[2], [3, 1], [7, 2, 64], [8], [65, 63, 1, 2]])
def test_portions(folder, sizes, dtype, dev):
    toks = tokens(150, 96, 4)
    steps, left, i = [], len(toks), 0
    while left:
        n = min(left, sizes[i % len(sizes)])
        steps.append([("a", n)])
        left, i = left - n, i + 1
    got = Replay(folder("aligned"), dtype, dev, 160).run({"a": toks}, steps)["a"]
    agrees(got, "aligned", toks, dtype)


@device
@pytest.mark.parametrize("name", ["wide_bias", "aligned"])
def test_every_distance_counts(folder, name, dev):
    """Large bias steps: a bucket that is one token off, at any distance up to the last bucket, in a
    prompt or decoded, shows in the logits far above the tolerance."""
    cfg, w = C.case(name)
    toks = tokens(170, cfg["vocab"], 5)
    want = oracle(name, toks)
    steps = [[("a", 100)]] + [[("a", 1)]] * 70
    got = Replay(folder(name), "float32", dev, 176).run({"a": toks}, steps)["a"]
    assert rel(got, want) < TOL["float32"]
    # the oracle with one edge moved differs: the test can see what it claims to
    shifted = {k: v for k, v in w.items()}
    moved = json.loads(json.dumps(cfg))
    for l in moved["layers"]:
        l["mixer"]["bias_max"] += 8
    assert rel(R.forward(moved, shifted, toks)[120:], want[120:]) > 100 * TOL["float32"]


@device
def test_null_entry_and_head_mix_show(folder, dev):
    """Without the null entry, or with the heads unmixed, the logits are far away."""
    cfg, w = C.case("aligned")
    toks = tokens(40, 96, 6)
    got = Replay(folder("aligned"), "float32", dev, 48).run({"a": toks}, [[("a", 40)]])["a"]
    assert rel(got, oracle("aligned", toks)) < TOL["float32"]
    plain = R.softmax_with_null
    try:
        R.softmax_with_null = lambda s: torch.softmax(s, -1)
        assert rel(got, R.forward(cfg, w, toks)) > 1e-2
    finally:
        R.softmax_with_null = plain
    unmixed = dict(w)
    for l, c in enumerate(cfg["layers"]):
        unmixed[f"l{l}.mix.talk"] = torch.eye(c["mixer"]["heads"])
    assert rel(got, R.forward(cfg, unmixed, toks)) > 1e-2


@device
@both
def test_far_key_stands_out(tmp_path, dtype, dev):
    """One query-key pair far apart carries almost the whole weight."""
    cfg = C.config([((2, 2, 64, 16, 0.5, 24), None)], width=64, vocab=24)
    w = C.weights(cfg, seed=9, sharp=0.2, bias=0.2)
    w["l0.mix.talk"] = torch.eye(2).to(torch.bfloat16)
    h = R.rms_norm(w["embed"].double() * 2.0, w["l0.norm1"].double(), 1e-5)
    keys = (h @ w["l0.mix.k"].double().T + w["l0.mix.k.b"].double()).view(24, 2, 64)
    # a direction per head that meets the key of token 7 and no other key; queries of token 11 take it
    d = torch.cat([torch.linalg.pinv(keys[:, g])[:, 7] for g in range(2)])
    w["l0.mix.q"] = (w["l0.mix.q"].double() + 40.0 * torch.outer(d, h[11]) / (h[11] @ h[11])).to(torch.bfloat16)
    toks = [t if t != 7 else 8 for t in tokens(300, 24, 10)]
    toks[3] = 7
    for p in (280, 299):
        toks[p] = 11
    want = R.forward(cfg, w, toks)
    without = list(toks)
    without[3] = 8
    assert rel(R.forward(cfg, w, without)[[280, 299]], want[[280, 299]]) > 0.2
    model = C.write(tmp_path / "far", cfg, w)
    for steps in ([[("a", 300)]], [[("a", 270)]] + [[("a", 1)]] * 30, [[("a", 150)], [("a", 150)]]):
        got = Replay(model, dtype, dev, 304).run({"a": toks}, steps)["a"]
        assert rel(got, want) < TOL[dtype]


@device
def test_long_decoding(folder, dev):
    toks = tokens(330, 96, 11)
    got = Replay(folder("aligned"), "float32", dev, 336).run({"a": toks}, [[("a", 4)]] + [[("a", 1)]] * 326)["a"]
    assert rel(got, oracle("aligned", toks)) < TOL["float32"]


# ------------------------------------------------------------------------------ batches and pages
@device
@both
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_mixed_batches(folder, name, dtype, dev):
    """Portions beside single tokens, requests that pause, unequal lengths."""
    vocab = C.CASES[name][0]["vocab"]
    prompts = {r: tokens(n, vocab, 20 + i) for i, (r, n) in enumerate([("a", 90), ("b", 17), ("c", 41), ("d", 3)])}
    steps = random_steps({r: len(p) for r, p in prompts.items()}, 5)
    got = Replay(folder(name), dtype, dev, 176).run(prompts, steps)
    for r, p in prompts.items():
        agrees(got[r], name, p, dtype)


@device
def test_batch_does_not_change_a_request(folder, dev):
    prompts = {r: tokens(n, 96, 30 + i) for i, (r, n) in enumerate([("a", 60), ("b", 33), ("c", 20)])}
    steps = [[("a", 30), ("b", 33)], [("a", 1), ("c", 12)], [("a", 29), ("c", 1)], [("c", 7)]]
    alone = [[("a", 30)], [("a", 1)], [("a", 29)]]
    together = Replay(folder("aligned"), "float32", dev, 128).run(prompts, steps)["a"]
    single = Replay(folder("aligned"), "float32", dev, 128).run({"a": prompts["a"]}, alone)["a"]
    assert (together - single).abs().max() < 1e-4


@device
@both
def test_pages_and_slots_are_used_again(folder, dtype, dev):
    """A pool for two requests serves twelve, two alive at a time."""
    r = Replay(folder("aligned"), dtype, dev, 96, page=8, max_requests=2)
    total = r.free_pages()
    for i in range(6):
        prompts = {f"x{i}": tokens(40, 96, 40 + i), f"y{i}": tokens(33 - i, 96, 50 + i)}
        x, y = prompts
        ny = len(prompts[y])
        steps = [[(x, 9), (y, ny - 5)], [(x, 1), (y, 1)], [(y, 2), (x, 25)], [(x, 5), (y, 2)]]
        got = r.run(prompts, steps)
        for k, p in prompts.items():
            agrees(got[k], "aligned", p, dtype)
    r.r.step([], [])
    assert r.free_pages() == total


# ------------------------------------------------------------------------------ generation
def check_greedy(name, prompt, out, margin):
    """Every generated token is the oracle's choice, or within ``margin`` of it (with a bf16-sized
    margin: except where the choice of experts is a close call)."""
    lg = oracle(name, prompt + out)
    clear = _logits[name, tuple(prompt + out), 0][1] > (CLOSE_CALL if margin > 1e-3 else 0.0)
    for i, t in enumerate(out):
        if not clear[len(prompt) - 1 + i]:
            continue
        row = lg[len(prompt) - 1 + i]
        assert row.max() - row[t] <= margin, (i, t, int(row.argmax()))


@device
@both
@pytest.mark.parametrize("name", ["aligned", "odd"])
def test_greedy_generation(folder, name, dtype, dev):
    """Six requests over four seats, prompts longer than the step budget, prefix caching on."""
    vocab = C.CASES[name][0]["vocab"]
    prompts = [tokens(n, vocab, 60 + i) for i, n in enumerate([1, 100, 8, 23, 64, 5])]
    prompts.append(prompts[1][:80] + tokens(9, vocab, 70))
    llm = engine(folder(name), dtype, dev)
    outs = llm.generate(prompts, greedy(24))
    for p, o in zip(prompts, outs):
        assert len(o.outputs[0].token_ids) == 24
        check_greedy(name, p, list(o.outputs[0].token_ids), 1e-4 if dtype == "float32" else 0.25)
    again = llm.generate(prompts[1:2], greedy(24))[0]
    assert again.num_cached_tokens > 0
    check_greedy(name, prompts[1], list(again.outputs[0].token_ids), 1e-4 if dtype == "float32" else 0.25)


@device
def test_preemption(folder, dev):
    """The pool runs out: requests are preempted and computed again."""
    prompts = [tokens(30, 96, 80 + i) for i in range(4)]
    llm = engine(folder("aligned"), "float32", dev, num_blocks=22, enable_prefix_caching=False)
    outs = llm.generate(prompts, greedy(30))
    for p, o in zip(prompts, outs):
        check_greedy("aligned", p, list(o.outputs[0].token_ids), 1e-4)


@device
def test_speculative_drafts_are_verified(folder, dev):
    from vllm_cpp_b200.spec_decode import SpeculativeConfig
    spec = SpeculativeConfig(method="ngram", num_speculative_tokens=3, prompt_lookup_min=1, prompt_lookup_max=3)
    prompt = tokens(20, 96, 90) * 2
    out = engine(folder("aligned"), "float32", dev, speculative_config=spec).generate([prompt], greedy(30))[0]
    check_greedy("aligned", prompt, list(out.outputs[0].token_ids), 1e-4)


@pytest.mark.gpu
def test_async_scheduling(folder):
    prompts = [tokens(n, 96, 95 + n) for n in (12, 40)]
    outs = engine(folder("aligned"), "bfloat16", "cuda", async_scheduling=True).generate(prompts, greedy(20))
    for p, o in zip(prompts, outs):
        check_greedy("aligned", p, list(o.outputs[0].token_ids), 0.25)


@pytest.mark.gpu
@both
def test_captured_decode_equals_launched_decode(folder, dtype):
    prompts = [tokens(n, 96, 97 + n) for n in (3, 30, 65)]
    a = engine(folder("aligned"), dtype, "cuda").generate(prompts, greedy(16))
    b = engine(folder("aligned"), dtype, "cuda", enable_cuda_graphs=False).generate(prompts, greedy(16))
    assert [list(x.outputs[0].token_ids) for x in a] == [list(x.outputs[0].token_ids) for x in b]


@device
def test_sampling_with_penalties(folder, dev):
    from vllm_cpp_b200.engine import SamplingParams
    llm = engine(folder("aligned"), "float32", dev)
    sp = SamplingParams(temperature=0.8, top_k=20, seed=3, max_tokens=12, ignore_eos=True, presence_penalty=0.5)
    outs = [list(llm.generate([tokens(10, 96, 99)], sp)[0].outputs[0].token_ids) for _ in range(2)]
    assert outs[0] == outs[1] and len(outs[0]) == 12 and max(outs[0]) < 96


# ------------------------------------------------------------------------------ requests with open input
@device
def test_open_input_then_generation(folder, dev):
    """A prompt in portions, closed with the last, generates what the whole prompt generates; another
    open request and a plain one share its steps."""
    prompt, other = tokens(50, 96, 100), tokens(20, 96, 101)
    llm = engine(folder("aligned"), "float32", dev)
    rid = llm.add_request(prompt[:13], greedy(10), input_open=True)
    idle = llm.add_request(other, greedy(1), input_open=True)
    assert llm.step() == []
    plain = llm.generate([other], greedy(10))[0]             # returns although open requests remain
    llm.extend_request(rid, prompt[13:14])
    llm.step()
    llm.extend_request(rid, prompt[14:], close=True)
    done = []
    while not done:
        done = [s for s in llm.step() if s.finished]
    check_greedy("aligned", prompt, list(done[0].outputs[0].token_ids), 1e-4)
    assert done[0].prompt_token_ids == prompt and len(done[0].outputs[0].token_ids) == 10
    check_greedy("aligned", other, list(plain.outputs[0].token_ids), 1e-4)
    with pytest.raises(ValueError):
        llm.extend_request(rid, [1])
    llm.abort_request(idle)
    llm.step()
    assert not llm.has_unfinished_requests()


@device
def test_closing_portion_longer_than_the_step_budget(folder, dev):
    prompt = tokens(150, 96, 102)
    llm = engine(folder("aligned"), "float32", dev)
    rid = llm.add_request(prompt[:5], greedy(6), input_open=True)
    llm.step()
    llm.extend_request(rid, prompt[5:], close=True)
    out = []
    while llm.has_unfinished_requests():
        out += [s for s in llm.step() if s.finished]
    check_greedy("aligned", prompt, list(out[0].outputs[0].token_ids), 1e-4)


def test_open_input_limits(folder):
    llm = engine(folder("aligned"), "float32", "cpu")
    rid = llm.add_request([1, 2], greedy(4), input_open=True)
    with pytest.raises(ValueError):
        llm.extend_request(rid, [], close=True)
    with pytest.raises(ValueError):
        llm.extend_request(rid, [1] * 300)
    with pytest.raises(ValueError):
        llm.extend_request("nobody", [1])
    with pytest.raises(ValueError):
        llm.score_positions(rid, [0])                        # no rows reserved


@device
def test_scores_beside_sampled_tokens(folder, dev):
    """Scored prompt positions of a request that also generates, in one batch with another."""
    llm = engine(folder("aligned"), "float32", dev, max_score_rows=64)
    p, q = tokens(30, 96, 103), tokens(9, 96, 104)
    rid = llm.add_request(p, greedy(5, prompt_logprobs=0))
    other = llm.add_request(q, greedy(5))
    llm.score_positions(rid, [0, 7, 29, 31])
    got, outs = {}, {}
    while llm.has_unfinished_requests():
        for s in llm.step():
            outs[s.request_id] = list(s.outputs[0].token_ids)
        for k, v in llm.take_scores().items():
            got.setdefault(k, []).extend(v)
    assert list(got) == [rid] and [x for x, _ in got[rid]] == [0, 7, 29, 31]
    want = oracle("aligned", p + outs[rid])
    assert rel(torch.stack([r for _, r in got[rid]]), want[[0, 7, 29, 31]]) < TOL["float32"]
    check_greedy("aligned", p, outs[rid], 1e-4)
    check_greedy("aligned", q, outs[other], 1e-4)


# ------------------------------------------------------------------------------ configuration and tools
def test_registry_and_configuration(folder):
    from vllm_cpp_b200.config import block_config_dict, load_model_config
    from vllm_cpp_b200.models import registry
    cfg = load_model_config(folder("aligned"))
    assert "Nufusun" in registry.supported_architectures()
    assert registry.resolve(cfg.architecture)[1].__name__ == "NufusunModel"
    assert block_config_dict(cfg) == C.CASES["aligned"][0]
    assert cfg.num_layers == 3 and cfg.blocks[1].mlp is None and cfg.blocks[2].attention.vdim == 32
    assert cfg.is_moe and not cfg.is_hybrid


@pytest.mark.parametrize("edit", ["mixer", "feed", "groups", "top", "arch"])
def test_unknown_branches_are_refused(edit):
    from vllm_cpp_b200.config import model_config_from_blocks
    cfg = json.loads(json.dumps(C.CASES["aligned"][0]))
    l = cfg["layers"][0]
    if edit == "mixer":
        l["type"] = "other"
    elif edit == "feed":
        l["mlp"]["kind"] = "other"
    elif edit == "groups":
        l["mixer"]["kv_heads"] = 3
    elif edit == "top":
        l["mlp"]["router"]["top"] = 9
    else:
        cfg["architecture"] = "Other"
    with pytest.raises(ValueError):
        model_config_from_blocks(cfg)


def test_incomplete_checkpoint_is_refused(tmp_path):
    cfg, w = C.case("one_of_each")
    del w["l0.mix.talk"]
    with pytest.raises(ValueError, match="talk"):
        engine(C.write(tmp_path / "m", cfg, w), "float32", "cpu")


def test_other_families_refuse_float32():
    from vllm_cpp_b200.config import EngineArgs, synthetic_config
    from vllm_cpp_b200.engine import LLM
    with pytest.raises(ValueError, match="float32"):
        LLM(EngineArgs(model_config=synthetic_config("tiny-dense"), device="cpu", dtype="float32"))


@pytest.mark.parametrize("buckets,reach", [(4, 9), (8, 128), (10, 17), (12, 40), (32, 130), (32, 256), (7, 50), (16, 8)])
def test_distance_buckets(buckets, reach):
    from vllm_cpp_b200.ops.bias_attn import bucket_of_distance, distance_bias_table
    rel_ = torch.arange(buckets * 3, dtype=torch.float32).view(buckets, 3)
    table = distance_bias_table(rel_, reach)
    for n in range(3 * reach):
        want = R.distance_bucket(n, buckets, reach) if reach > buckets // 2 else min(n, buckets - 1) if n < buckets // 2 else buckets - 1
        assert bucket_of_distance(n, buckets, reach) == want
        assert torch.equal(table[:, min(n, table.shape[1] - 1)], rel_[want])
    assert bucket_of_distance(0, buckets, reach) == 0 and bucket_of_distance(buckets // 2 - 1, buckets, reach) == buckets // 2 - 1


def test_exact_bucket_boundaries():
    """Distances that lie exactly on a boundary open the next bucket."""
    from vllm_cpp_b200.ops.bias_attn import bucket_of_distance
    assert [bucket_of_distance(n, 32, 256) for n in (31, 32, 63, 64, 127, 128)] == [19, 20, 23, 24, 27, 28]
    assert [bucket_of_distance(n, 16, 128) for n in (15, 16, 31, 32, 63, 64)] == [9, 10, 11, 12, 13, 14]


@device
def test_trace_runner(folder, tmp_path, dev):
    name, V = "odd", C.CASES["odd"][0]["vocab"]
    a, b = tokens(20, V, 110), tokens(70, V, 111)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [6, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:64], "want": []}, {"id": "a", "tokens": a[7:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[64:], "want": [5]}, {"id": "a", "tokens": a[8:], "want": [11, 0]}],
              "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b[:3], "want": [2]}], "end": ["c"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder(name), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "192", "--device", dev],
                       input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=280)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "2.f32", "3.f32"]

    def read(n):
        return torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, V)
    wa, wb = oracle(name, a), oracle(name, b)
    assert rel(read(0), wa[[6, 0]]) < 2e-5
    assert rel(read(2), torch.stack([wb[69], wa[19], wa[8]])) < 2e-5
    assert rel(read(3), wb[[2]]) < 2e-5


@device
def test_synthetic_checkpoint_and_command_line(tmp_path, dev, capsys):
    from vllm_cpp_b200.config import synthetic_config
    from vllm_cpp_b200.entrypoints import cli
    from vllm_cpp_b200.loader import write_synthetic_checkpoint
    out = write_synthetic_checkpoint(str(tmp_path / "ckpt"), synthetic_config("tiny-nufusun"), seed=1)
    assert cli.main(["--model", out, "--prompt-ids", "5,6,7", "--max-tokens", "4", "--device", dev, "--dtype", "float32",
                     "--max-model-len", "64"]) == 0
    ids = capsys.readouterr().out.strip().splitlines()[-1]
    assert all(0 <= int(x) < 500 for x in ids.split(",")) and len(ids.split(",")) <= 4
    assert cli.main(["--model", out, "--prompt", "the thing", "--max-tokens", "3", "--device", dev,
                     "--max-model-len", "64"]) == 0
