"""Diforax through the engine (registry, loader, scheduler, paged cache, state slots, batches) against the
plain implementation in ``diforax_reference.py``; every test runs on the CPU back end and, on a GPU box, on
the kernels."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import diforax_case as C                                                       # noqa: E402
import diforax_reference as R                                                  # noqa: E402
from replay import Replay, engine, greedy, random_steps, rel, tokens           # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
TOL = {"float32": 4e-5, "bfloat16": 0.06}   # (three times that where single values are normed)
both = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
device = pytest.mark.parametrize("dev", DEVICES)
_logits: dict = {}


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """(the models are so small that threads only wait for one another)"""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def oracle(name, toks, dtype="float32"):
    key = (name, tuple(toks), dtype)
    if key not in _logits:
        margins = []
        _logits[key] = R.forward(*C.case(name, dtype), toks, dtype=torch.float64, margins=margins)
        assert all(float(m.min()) > (0.3 if dtype == "bfloat16" else 5e-7) for m in margins)
    return _logits[key]


def agrees(got, name, toks, dtype):
    assert rel(got, oracle(name, toks, dtype)) < TOL[dtype] * (3 if name in ("odd", "ones") else 1)


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    base = tmp_path_factory.mktemp("diforax")
    done = {}

    def get(name, dtype="float32"):
        if (name, dtype) not in done:
            done[name, dtype] = C.write(base / f"{name}_{dtype}", *C.case(name, dtype))
        return done[name, dtype]
    return get


# ------------------------------------------------------------------------------ one sequence
@device
@both
@pytest.mark.parametrize("page", [8, 16])
@pytest.mark.parametrize("name", list(C.CASES))
def test_whole_prompt(folder, name, page, dtype, dev):
    toks = tokens(150, C.CASES[name][0]["vocab"], 1)
    got = Replay(folder(name, dtype), dtype, dev, 160, page=page).run({"a": toks}, [[("a", len(toks))]])["a"]
    agrees(got, name, toks, dtype)


@device
@both
@pytest.mark.parametrize("name", ["mixed", "odd", "delta_only", "ones"])
def test_token_by_token(folder, name, dtype, dev):
    toks = tokens(70, C.CASES[name][0]["vocab"], 2)
    got = Replay(folder(name, dtype), dtype, dev, 80, page=16).run({"a": toks}, [[("a", 1)]] * len(toks))["a"]
    agrees(got, name, toks, dtype)


@device
@both
def test_first_tokens(folder, dtype, dev):
    """One-token prompts included: nothing of the slot's last user may be seen."""
    r = Replay(folder("mixed", dtype), dtype, dev, 48, page=16, max_requests=1)
    for i, n in enumerate((5, 1, 2, 3, 1)):
        toks = tokens(n, 96, 3 + n)
        for a, cuts in ((f"a{i}", [n]), (f"b{i}", [1] * n)):
            agrees(r.run({a: toks}, [[(a, c)] for c in cuts])[a], "mixed", toks, dtype)


@device
@both
@pytest.mark.parametrize("name", ["mixed", "odd", "attention_only"])
@pytest.mark.parametrize("sizes", [[2], [3, 1], [7, 2, 64], [8], [65, 63, 1, 2]])
def test_portions(folder, name, sizes, dtype, dev):
    V = C.CASES[name][0]["vocab"]
    toks = tokens(150, V, 4)
    steps, left, i = [], len(toks), 0
    while left:
        n = min(left, sizes[i % len(sizes)])
        steps.append([("a", n)])
        left, i = left - n, i + 1
    got = Replay(folder(name, dtype), dtype, dev, 160).run({"a": toks}, steps)["a"]
    agrees(got, name, toks, dtype)


def edited(cfg, f):
    out = json.loads(json.dumps(cfg))
    for l in out["layers"]:
        f(l)
    return out


@device
def test_every_mechanism_shows(folder, dev):
    """The engine agrees with the oracle, and the oracle with one mechanism changed is far away."""
    cfg, w = C.case("mixed")
    toks = tokens(140, 96, 6)
    got = Replay(folder("mixed"), "float32", dev, 144).run({"a": toks}, [[("a", 90)]] + [[("a", 1)]] * 50)["a"]
    assert rel(got, oracle("mixed", toks)) < TOL["float32"]

    def differs(cfg2, w2, rows=slice(None), least=1e-2):
        d = rel(R.forward(cfg2, w2, toks)[rows], oracle("mixed", toks)[rows])
        assert d > least, d

    def att(l, **kw):
        if l["type"] == "attention":
            l["mixer"].update(kw)
    for l, c in enumerate(cfg["layers"]):                             # a chunk's edge one token off
        if c["type"] == "attention":
            moved = json.loads(json.dumps(cfg))
            moved["layers"][l]["mixer"]["mask"]["size"] -= 1
            differs(moved, w)
    differs(edited(cfg, lambda l: att(l, scale=l["mixer"].get("scale", 1) * 1.5)), w)
    differs(edited(cfg, lambda l: att(l, rot={"base": 4e4, "dims": 30})), w)
    differs(edited(cfg, lambda l: att(l, rot={"base": 2e4, "dims": 32})), w)
    own = json.loads(json.dumps(cfg))                                 # keys of its own instead of layer 1's
    del own["layers"][3]["mixer"]["kv_from"]
    differs(own, {**w, "l3.mix.k": w["l1.mix.k"], "l3.mix.v": w["l1.mix.v"]})
    for name in ("l0.mix.A_log", "l0.mix.dt_bias", "l0.mix.norm", "l1.norm1b", "l3.norm2b", "l1.mlp.correction", "l4.mix.v.conv"):
        differs(cfg, {**w, name: w[name] + 0.5 * torch.randn(w[name].shape, generator=torch.Generator().manual_seed(1)).to(w[name])})
    differs(edited(cfg, lambda l: l["mlp"]["router"]["groups"].update(keep=l["mlp"]["router"]["groups"]["count"])
                   if l["mlp"] and l["mlp"]["kind"] == "moe" else None), w)
    last = {**w, "l0.mix.q.conv": w["l0.mix.q.conv"].flip(1)}         # the order of the taps
    differs(cfg, last)


@device
@both
@pytest.mark.parametrize("chunk", [50, 64])
def test_far_key_stands_out(tmp_path, chunk, dtype, dev):
    """One query-key pair carries almost the whole weight, at the far end of a chunk; one chunk further
    it is not seen."""
    cfg = C.config([C.attention(2, 2, 64, 16, 0.3, chunk, 1e9, 2)], width=64, vocab=24)
    w = C.weights(cfg, seed=9)
    h = R.rms(w["embed"].double(), 1e-5) * w["l0.norm1"].double()
    d = torch.linalg.pinv(h)                                          # column t answers to token t alone
    dirs = torch.randn(2, 64, generator=torch.Generator().manual_seed(2)).double()
    dirs[:, :2] = 0.0                                                 # (not where positions turn it)
    for n, t in (("k", 7), ("q", 11)):
        x = w[f"l0.mix.{n}"].double() + 6.0 * torch.cat([torch.outer(dirs[g], d[:, t]) for g in range(2)])
        w[f"l0.mix.{n}"] = x.to(torch.bfloat16)
    toks = [t if t != 7 else 8 for t in tokens(4 * chunk, 24, 10)]
    toks[2 * chunk] = 7
    for p in (3 * chunk - 1, 3 * chunk):
        toks[p] = 11
    want = R.forward(cfg, w, toks)
    without = list(toks)
    without[2 * chunk] = 8
    moved = R.forward(cfg, w, without)
    assert rel(moved[[3 * chunk - 1]], want[[3 * chunk - 1]]) > 0.2 and rel(moved[[3 * chunk]], want[[3 * chunk]]) < 1e-12
    model = C.write(tmp_path / "far", cfg, w)
    n, k = len(toks), 3 * chunk - 10
    for steps in ([[("a", n)]], [[("a", k)]] + [[("a", 1)]] * (n - k), [[("a", n // 2 + 3)], [("a", n - n // 2 - 3)]]):
        got = Replay(model, dtype, dev, n + 16, page=16).run({"a": toks}, steps)["a"]
        assert rel(got, want) < TOL[dtype]


@device
@both
def test_state_reaches_far_back(folder, dtype, dev):
    """Slow decays: a token hundreds of positions back still shows."""
    toks = tokens(420, 50, 12)
    want = oracle("delta_only", toks, dtype)
    other = list(toks)
    other[20] = (toks[20] + 1) % 50
    assert rel(oracle("delta_only", other, dtype)[[419]], want[[419]]) > 1e-3
    for steps in ([[("a", 420)]], [[("a", 400)]] + [[("a", 1)]] * 20, [[("a", 70)]] * 6):
        got = Replay(folder("delta_only", dtype), dtype, dev, 424).run({"a": toks}, steps)["a"]
        agrees(got, "delta_only", toks, dtype)


@device
def test_long_decoding(folder, dev):
    toks = tokens(330, 96, 11)
    got = Replay(folder("mixed"), "float32", dev, 336).run({"a": toks}, [[("a", 4)]] + [[("a", 1)]] * 326)["a"]
    assert rel(got, oracle("mixed", toks)) < TOL["float32"]


# ------------------------------------------------------------------------------ batches, pages and slots
@device
@both
@pytest.mark.parametrize("name", ["mixed", "odd", "attention_only"])
def test_mixed_batches(folder, name, dtype, dev):
    """Portions beside single tokens, requests that pause, unequal lengths."""
    vocab = C.CASES[name][0]["vocab"]
    prompts = {r: tokens(n, vocab, 20 + i) for i, (r, n) in enumerate([("a", 90), ("b", 17), ("c", 41), ("d", 3)])}
    got = Replay(folder(name, dtype), dtype, dev, 176).run(prompts, random_steps({r: len(p) for r, p in prompts.items()}, 5))
    for r, p in prompts.items():
        agrees(got[r], name, p, dtype)


@device
@both
def test_batch_does_not_change_a_request(folder, dtype, dev):
    prompts = {r: tokens(n, 96, 30 + i) for i, (r, n) in enumerate([("a", 60), ("b", 33), ("c", 20)])}
    steps = [[("a", 30), ("b", 33)], [("a", 1), ("c", 12)], [("a", 29), ("c", 1)], [("c", 7)]]
    alone = [[("a", 30)], [("a", 1)], [("a", 29)]]
    together = Replay(folder("mixed", dtype), dtype, dev, 128).run(prompts, steps)["a"]
    single = Replay(folder("mixed", dtype), dtype, dev, 128).run({"a": prompts["a"]}, alone)["a"]
    assert (together - single).abs().max() < (1e-4 if dtype == "float32" else 5e-2)


@device
@both
@pytest.mark.parametrize("name", ["mixed", "attention_only"])
def test_pages_and_slots_are_used_again(folder, name, dtype, dev):
    """A pool and slots for two requests serve twelve, two alive at a time."""
    V = C.CASES[name][0]["vocab"]
    r = Replay(folder(name, dtype), dtype, dev, 96, page=8, max_requests=2)
    total = r.free_pages()
    for i in range(6):
        prompts = {f"x{i}": tokens(40, V, 40 + i), f"y{i}": tokens(33 - i, V, 50 + i)}
        x, y = prompts
        ny = len(prompts[y])
        steps = [[(x, 9), (y, ny - 5)], [(x, 1), (y, 1)], [(y, 2), (x, 25)], [(x, 5), (y, 2)]]
        got = r.run(prompts, steps)
        for k, p in prompts.items():
            agrees(got[k], name, p, dtype)
    r.r.step([], [])
    assert r.free_pages() == total


@device
def test_pages_behind_the_chunk_are_given_back(folder, dev):
    """Blocks that all see chunks of 24: a prompt of 150 tokens runs in a pool of 64."""
    toks = tokens(150, 72, 13)
    r = Replay(folder("attention_only"), "float32", dev, 160, page=8, max_requests=1)
    free, at, got = r.free_pages(), 0, []
    while at < 150:
        n = min(10, 150 - at)
        rows = r.r.step([{"id": "a", "tokens": toks[at:at + n], "want": list(range(n))}], [])
        got += rows
        at += n
        assert free - r.free_pages() <= (24 + 10 + 7) // 8 + 2
    assert rel(torch.stack(got), oracle("attention_only", toks)) < TOL["float32"]


# ------------------------------------------------------------------------------ generation
def check_greedy(name, prompt, out, dtype="float32"):
    """Every generated token is the oracle's choice, or (rounding) next to it."""
    lg = oracle(name, prompt + out, dtype)
    for i, t in enumerate(out):
        row = lg[len(prompt) - 1 + i]
        assert row.max() - row[t] <= {"float32": 2e-4, "bfloat16": 0.25}[dtype], (i, t, int(row.argmax()))


@device
@both
@pytest.mark.parametrize("name", ["mixed", "odd", "attention_only"])
def test_greedy_generation(folder, name, dtype, dev):
    """Seven requests over four seats, prompts longer than the step budget; prefix caching where no state
    is kept."""
    vocab = C.CASES[name][0]["vocab"]
    prompts = [tokens(n, vocab, 60 + i) for i, n in enumerate([1, 100, 8, 23, 64, 5])]
    prompts.append(prompts[1][:80] + tokens(9, vocab, 70))
    llm = engine(folder(name, dtype), dtype, dev)
    outs = llm.generate(prompts, greedy(24))
    for p, o in zip(prompts, outs):
        assert len(o.outputs[0].token_ids) == 24
        check_greedy(name, p, list(o.outputs[0].token_ids), dtype)
    again = llm.generate(prompts[1:2], greedy(24))[0]
    assert (again.num_cached_tokens > 0) == (name == "attention_only")
    check_greedy(name, prompts[1], list(again.outputs[0].token_ids), dtype)


@device
def test_preemption(folder, dev):
    """The pool runs out: requests are preempted and computed again, state and all."""
    prompts = [tokens(30, 96, 80 + i) for i in range(4)]
    llm = engine(folder("mixed"), "float32", dev, num_blocks=22)
    outs = llm.generate(prompts, greedy(30))
    for p, o in zip(prompts, outs):
        check_greedy("mixed", p, list(o.outputs[0].token_ids))


@device
def test_speculative_drafts_are_verified(folder, dev):
    """Rejected drafts: the state goes back to before the step and the kept tokens run again."""
    from vllm_cpp_b200.spec_decode import SpeculativeConfig
    spec = SpeculativeConfig(method="ngram", num_speculative_tokens=3, prompt_lookup_min=1, prompt_lookup_max=3)
    prompt = tokens(20, 96, 90) * 2
    llm = engine(folder("mixed"), "float32", dev, speculative_config=spec)
    out = llm.generate([prompt], greedy(30))[0]
    check_greedy("mixed", prompt, list(out.outputs[0].token_ids))
    assert llm.runner.spec_stats["drafted"] > llm.runner.spec_stats["accepted"]


@pytest.mark.gpu
def test_async_scheduling(folder):
    prompts = [tokens(n, 96, 95 + n) for n in (12, 40)]
    outs = engine(folder("mixed", "bfloat16"), "bfloat16", "cuda", async_scheduling=True).generate(prompts, greedy(20))
    for p, o in zip(prompts, outs):
        check_greedy("mixed", p, list(o.outputs[0].token_ids), "bfloat16")


@pytest.mark.gpu
@both
def test_captured_decode_equals_launched_decode(folder, dtype):
    prompts = [tokens(n, 96, 97 + n) for n in (3, 30, 65)]
    a = engine(folder("mixed", dtype), dtype, "cuda", block_size=16).generate(prompts, greedy(16))
    b = engine(folder("mixed", dtype), dtype, "cuda", block_size=16, enable_cuda_graphs=False).generate(prompts, greedy(16))
    assert [list(x.outputs[0].token_ids) for x in a] == [list(x.outputs[0].token_ids) for x in b]


@device
def test_open_input_then_generation(folder, dev):
    """A prompt in portions, closed with the last, generates what the whole prompt generates."""
    prompt = tokens(50, 96, 100)
    llm = engine(folder("mixed"), "float32", dev)
    rid = llm.add_request(prompt[:13], greedy(10), input_open=True)
    assert llm.step() == []
    llm.extend_request(rid, prompt[13:14])
    llm.step()
    llm.extend_request(rid, prompt[14:], close=True)
    done = []
    while not done:
        done = [s for s in llm.step() if s.finished]
    check_greedy("mixed", prompt, list(done[0].outputs[0].token_ids))


@device
def test_sampling(folder, dev):
    from vllm_cpp_b200.engine import SamplingParams
    llm = engine(folder("mixed"), "float32", dev)
    sp = SamplingParams(temperature=0.8, top_k=20, seed=3, max_tokens=12, ignore_eos=True, presence_penalty=0.5)
    outs = [list(llm.generate([tokens(10, 96, 99)], sp)[0].outputs[0].token_ids) for _ in range(2)]
    assert outs[0] == outs[1] and len(outs[0]) == 12 and max(outs[0]) < 96


# ------------------------------------------------------------------------------ configuration and tools
def test_registry_and_configuration(folder):
    from vllm_cpp_b200.config import block_config_dict, load_model_config
    from vllm_cpp_b200.models import registry
    for name in C.CASES:
        cfg = load_model_config(folder(name))
        assert registry.resolve(cfg.architecture)[1].__name__ == "DiforaxModel"
        assert block_config_dict(cfg) == C.CASES[name][0]
        assert cfg.is_hybrid == (name != "attention_only")
    assert "Diforax" in registry.supported_architectures()


def test_absent_parts_of_the_configuration():
    from vllm_cpp_b200.config import model_config_from_blocks
    cfg = json.loads(json.dumps(C.CASES["mixed"][0]))
    del cfg["layers"][1]["mixer"]["mask"], cfg["layers"][1]["mixer"]["rot"]
    del cfg["layers"][1]["mlp"]["router"]["groups"], cfg["layers"][1]["mlp"]["router"]["identity"]
    b = model_config_from_blocks(cfg).blocks[1]
    assert (b.attention.chunk, b.attention.rot_dims, b.mlp.groups, b.mlp.identity) == (0, 0, 1, 0)


@pytest.mark.parametrize("edit", ["mixer", "feed", "heads", "top", "groups", "kv_from", "kv_sizes", "rot", "conv", "arch"])
def test_unknown_or_impossible_parts_are_refused(edit):
    from vllm_cpp_b200.config import model_config_from_blocks
    cfg = json.loads(json.dumps(C.CASES["mixed"][0]))
    l = cfg["layers"]
    if edit == "mixer":
        l[0]["type"] = "other"
    elif edit == "feed":
        l[0]["mlp"]["kind"] = "other"
    elif edit == "heads":
        l[0]["mixer"]["kv_heads"] = 3
    elif edit == "top":
        l[1]["mlp"]["router"]["top"] = 5               # two groups of two are kept
    elif edit == "groups":
        l[1]["mlp"]["router"]["groups"]["count"] = 3
    elif edit == "kv_from":
        l[3]["mixer"]["kv_from"] = 2
    elif edit == "kv_sizes":
        l[3]["mixer"]["vdim"] = 64
    elif edit == "rot":
        l[1]["mixer"]["rot"]["dims"] = 50
    elif edit == "conv":
        l[0]["mixer"]["conv"] = 0
    else:
        cfg["architecture"] = "Other"
    with pytest.raises(ValueError):
        model_config_from_blocks(cfg)


@pytest.mark.parametrize("name", ["l0.mix.a", "l1.norm2b", "l3.mix.q", "l1.mlp.e3.up", "l4.mlp.correction", "final.norm", "head"])
def test_incomplete_checkpoint_is_refused(tmp_path, name):
    cfg, w = C.case("mixed")
    del w[name]
    with pytest.raises(ValueError, match=name.split(".", 1)[-1] if name != "head" else "lm_head"):
        engine(C.write(tmp_path / "m", cfg, w), "float32", "cpu")


@device
def test_trace_runner(folder, tmp_path, dev):
    name, V = "odd", C.CASES["odd"][0]["vocab"]
    a, b = tokens(20, V, 110), tokens(70, V, 111)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [6, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:64], "want": []}, {"id": "a", "tokens": a[7:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[64:], "want": [5]}, {"id": "a", "tokens": a[8:], "want": [11, 0]}],
              "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b[:1], "want": [0]}], "end": ["c"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder(name), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "192", "--device", dev],
                       input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=280)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]

    def read(n):
        return torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, V)
    wa, wb = oracle(name, a), oracle(name, b)
    assert rel(read(0), wa[[6, 0]]) < 4e-5
    assert rel(read(2), torch.stack([wb[69], wa[19], wa[8]])) < 4e-5
    assert rel(read(3), wb[[0]]) < 4e-5


@device
def test_synthetic_checkpoint_and_command_line(tmp_path, dev, capsys):
    from vllm_cpp_b200.config import synthetic_config
    from vllm_cpp_b200.entrypoints import cli
    from vllm_cpp_b200.loader import write_synthetic_checkpoint
    out = write_synthetic_checkpoint(str(tmp_path / "ckpt"), synthetic_config("tiny-diforax"), seed=1)
    assert cli.main(["--model", out, "--prompt-ids", "5,6,7", "--max-tokens", "4", "--device", dev, "--dtype", "float32",
                     "--max-model-len", "64"]) == 0
    ids = capsys.readouterr().out.strip().splitlines()[-1]
    assert all(0 <= int(x) < 500 for x in ids.split(",")) and len(ids.split(",")) <= 4
    assert cli.main(["--model", out, "--prompt", "the thing", "--max-tokens", "3", "--device", dev,
                     "--max-model-len", "64"]) == 0
