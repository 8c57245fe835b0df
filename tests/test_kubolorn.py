"""Kubolorn through the engine (registry, loader, scheduler, paged cache, state slots, batches) against the
plain implementation in ``kubolorn_reference.py``; every test runs on the CPU back end and, on a GPU box, on
the kernels."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import kubolorn_case as C                                                      # noqa: E402
import kubolorn_reference as R                                                 # noqa: E402
from replay import Replay, engine, greedy, random_steps, rel, tokens           # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
TOL = {"float32": 4e-5, "bfloat16": 0.06}   # (three times that where a few values are normed)
both = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
device = pytest.mark.parametrize("dev", DEVICES)
NAMES = ["mixed", "odd", "attention", "recurrent", "fading", "ones"]
_logits: dict = {}


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """(the models are so small that threads only wait for one another)"""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def of(name, dtype):
    """Where rounding could change the choice of experts, the case whose choice is fixed."""
    return "steady" if name == "mixed" and dtype == "bfloat16" else name


def vocab(name):
    return C.CASES[name][0]["vocab"]


def oracle(name, toks):
    key = (name, tuple(toks))
    if key not in _logits:
        _logits[key] = R.forward(*C.case(name), toks)
    return _logits[key]


def agrees(got, name, toks, dtype):
    """In bf16 a row in twenty (or one) may be further off: a head's output is divided by its size, and where query and
    key are almost orthogonal, as they may be for a first token, rounding turns its sign."""
    e = sorted(rel(g[None], w[None]) for g, w in zip(got, oracle(name, toks)))
    tol = TOL[dtype] * (3 if name in ("odd", "ones") else 1)
    if dtype == "bfloat16":
        assert e[-1] < 0.7
        e = e[: len(e) - max(1, len(e) // 20)] or [0.0]
    assert e[-1] < tol, e[-5:]


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    base = tmp_path_factory.mktemp("kubolorn")
    done = {}

    def get(name):
        if name not in done:
            done[name] = C.write(base / name, *C.case(name))
        return done[name]
    return get


# ------------------------------------------------------------------------------ one sequence
@device
@both
@pytest.mark.parametrize("page", [8, 16])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt(folder, name, page, dtype, dev):
    name = of(name, dtype)
    toks = tokens(150, vocab(name), 1)
    got = Replay(folder(name), dtype, dev, 160, page=page).run({"a": toks}, [[("a", len(toks))]])["a"]
    agrees(got, name, toks, dtype)


@device
@both
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token(folder, name, dtype, dev):
    name = of(name, dtype)
    toks = tokens(70, vocab(name), 2)
    got = Replay(folder(name), dtype, dev, 80, page=16).run({"a": toks}, [[("a", 1)]] * len(toks))["a"]
    agrees(got, name, toks, dtype)


@device
@both
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_first_tokens(folder, name, dtype, dev):
    """One-token prompts included: nothing of the slot's last user may be seen, neither its last token."""
    name = of(name, dtype)
    r = Replay(folder(name), dtype, dev, 48, page=16, max_requests=1)
    for i, n in enumerate((5, 1, 2, 3, 1)):
        toks = tokens(n, vocab(name), 3 + n)
        for a, cuts in ((f"a{i}", [n]), (f"b{i}", [1] * n)):
            agrees(r.run({a: toks}, [[(a, c)] for c in cuts])[a], name, toks, dtype)


@device
@both
@pytest.mark.parametrize("name", ["mixed", "odd", "attention", "recurrent", "fading"])
@pytest.mark.parametrize("sizes", [[2], [3, 1], [7, 2, 64], [8], [65, 63, 1, 2], [17, 15, 18]])
def test_portions(folder, name, sizes, dtype, dev):
    name = of(name, dtype)
    toks = tokens(150, vocab(name), 4)
    steps, left, i = [], len(toks), 0
    while left:
        n = min(left, sizes[i % len(sizes)])
        steps.append([("a", n)])
        left, i = left - n, i + 1
    got = Replay(folder(name), dtype, dev, 160).run({"a": toks}, steps)["a"]
    agrees(got, name, toks, dtype)


def edited(cfg, f):
    out = json.loads(json.dumps(cfg))
    f(out)
    return out


@device
def test_every_mechanism_shows(folder, dev):
    """The engine agrees with the oracle, and the oracle with one mechanism changed is far away."""
    cfg, w = C.case("mixed")
    toks = tokens(48, 96, 6)
    got = Replay(folder("mixed"), "float32", dev, 72).run({"a": toks}, [[("a", 30)]] + [[("a", 1)]] * 18)["a"]
    want = oracle("mixed", toks)
    assert rel(got, want) < TOL["float32"]

    def differs(cfg2, w2=w, least=2e-3):
        d = rel(R.forward(cfg2, w2, toks), want)
        assert d > least, d

    def change(*path, by):
        def f(c):
            for k in path[:-1]:
                c = c[k]
            c[path[-1]] = by(c[path[-1]])
        differs(edited(cfg, f))
    change("embedding", "scale", by=lambda v: v * 1.2)
    for k in ("mul_prev", "mul_cur"):
        change("embedding", "bigram", k, by=lambda v: v + 1)
    change("norm", "groups", by=lambda v: v // 2)
    change("norm", "eps", by=lambda v: 0.05)
    change("loop", "times", by=lambda v: 1)
    change("loop", "stop", by=lambda v: v - 1)
    for l in (0, 2):
        change("layers", l, "mixer", "tau", by=lambda v: v * 1.5)
    left = ("layers", 1, "mixer", "left")
    change(*left, "scale", by=lambda v: v * 1.5)
    change(*left, "rot", "base", by=lambda v: v * 3)
    change(*left, "rot", "dims", by=lambda v: v - 2)
    for k, v in (("factor", 6.0), ("original", 40), ("fast", 4.0), ("slow", 6.0)):
        change(*left, "rot", "scaling", k, by=lambda _: v)
    for k in ("left_scale", "right_scale"):
        change("layers", 1, "mixer", k, by=lambda v: v + 0.2)
    change("layers", 1, "mixer", "right", "norm_groups", by=lambda v: 6)
    change("layers", 1, "mlp", "router", "top", by=lambda v: v + 1)
    g = torch.Generator().manual_seed(1)
    used = {f"l{l}.mlp.e{e}.{n}" for l, E in ((1, 5), (2, 6)) for e in range(E) for n in ("up", "down")}
    for n in w:                                                                       # every tensor
        if n not in used or n.startswith("l1.mlp.e0"):
            differs(cfg, {**w, n: w[n] + (0.5 * w[n].float().std().nan_to_num(0.2).clamp_min(0.1) *
                                          torch.randn(w[n].shape, generator=g)).to(w[n])}, least=1e-3)
    for n in ("l0.canon1", "l1.canon2", "l1.mix.right.conv"):
        differs(cfg, {**w, n: w[n].flip(1)})                                          # the order of the taps


@device
@both
def test_far_key_stands_out(tmp_path, dtype, dev):
    """One query-key pair far apart carries almost the whole weight, across many pages; its value is the key before the
    rotation, and positions turn the rotated part only. Without the key the sink takes the weight."""
    cfg = C.config([C.parallel((2, 2, 64, 1.0, 1e9, 32, (1e6, 1e-3, 2.0, 1.0)), (1, 1, 16, 16, 2, 1), (1.0, 0.05))], width=64, vocab=24,
                   groups=1, taps=1, bigram=(5, 1, 1))
    w = C.weights(cfg, seed=9)
    w["bigram"] *= 0
    w["l0.canon1"] *= 0
    w["l0.mix.left.q"], w["l0.mix.left.k"] = w["l0.mix.left.q"] * 0.1, w["l0.mix.left.k"] * 0.1
    x = R.rms(w["embed"].double() * 3.0, 1e-5) * w["embed.norm"].double()
    h = R.rms(x, 1e-5) * w["l0.norm1"].double()
    d = torch.linalg.pinv(h)                                          # column t answers to token t alone
    dirs = torch.randn(2, 64, generator=torch.Generator().manual_seed(2)).double()
    for n, t in (("k", 7), ("q", 11)):
        y = w[f"l0.mix.left.{n}"].double() + torch.cat([torch.outer(dirs[i], d[:, t]) for i in range(2)]) * 0.6
        w[f"l0.mix.left.{n}"] = y.to(torch.bfloat16)
    w["l0.mix.left.sink"] = torch.full((2,), 6.0, dtype=torch.bfloat16)
    toks = [t if t not in (7, 11) else 8 for t in tokens(300, 24, 10)]
    toks[13] = 7
    for p in (14, 140, 299):
        toks[p] = 11
    want = R.forward(cfg, w, toks)
    without = list(toks)
    without[13] = 8
    for p in (140, 299):
        assert rel(R.forward(cfg, w, without)[[p]], want[[p]]) > 0.2
    assert rel(R.forward(cfg, {**w, "l0.mix.left.sink": w["l0.mix.left.sink"] * 0 - 9}, without)[[299]], R.forward(cfg, w, without)[[299]]) > 5e-3
    model = C.write(tmp_path / "far", cfg, w)
    for seq, ref in ((toks, want), (without, R.forward(cfg, w, without))):
        for steps in ([[("a", 300)]], [[("a", 129)], [("a", 2)], [("a", 150)]] + [[("a", 1)]] * 19):
            got = Replay(model, dtype, dev, 320, page=16).run({"a": seq}, steps)["a"]
            assert rel(got, ref) < TOL[dtype]


@device
@both
def test_state_reaches_far_back(folder, dtype, dev):
    """Slow decays: a token hundreds of positions back still shows."""
    toks = tokens(420, 50, 12)
    want = oracle("recurrent", toks)
    other = list(toks)
    other[20] = (toks[20] + 1) % 50
    assert rel(oracle("recurrent", other)[[419]], want[[419]]) > 5e-4
    for steps in ([[("a", 420)]], [[("a", 400)]] + [[("a", 1)]] * 20, [[("a", 70)]] * 6):
        got = Replay(folder("recurrent"), dtype, dev, 424).run({"a": toks}, steps)["a"]
        agrees(got, "recurrent", toks, dtype)


@device
def test_long_decoding(folder, dev):
    toks = tokens(330, 96, 11)
    got = Replay(folder("mixed"), "float32", dev, 336).run({"a": toks}, [[("a", 4)]] + [[("a", 1)]] * 326)["a"]
    assert rel(got, oracle("mixed", toks)) < TOL["float32"]


# ------------------------------------------------------------------------------ batches, pages and slots
@device
@both
@pytest.mark.parametrize("name", ["mixed", "odd", "attention", "fading"])
def test_mixed_batches(folder, name, dtype, dev):
    """Portions beside single tokens, requests that pause, unequal lengths."""
    name = of(name, dtype)
    prompts = {r: tokens(n, vocab(name), 20 + i) for i, (r, n) in enumerate([("a", 90), ("b", 17), ("c", 41), ("d", 3)])}
    got = Replay(folder(name), dtype, dev, 176).run(prompts, random_steps({r: len(p) for r, p in prompts.items()}, 5))
    for r, p in prompts.items():
        agrees(got[r], name, p, dtype)


@device
@both
def test_batch_does_not_change_a_request(folder, dtype, dev):
    prompts = {r: tokens(n, 96, 30 + i) for i, (r, n) in enumerate([("a", 60), ("b", 33), ("c", 20)])}
    steps = [[("a", 30), ("b", 33)], [("a", 1), ("c", 12)], [("a", 29), ("c", 1)], [("c", 7)]]
    alone = [[("a", 30)], [("a", 1)], [("a", 29)]]
    name = of("mixed", dtype)
    together = Replay(folder(name), dtype, dev, 128).run(prompts, steps)["a"]
    single = Replay(folder(name), dtype, dev, 128).run({"a": prompts["a"]}, alone)["a"]
    assert rel(together, single.double()) < (1e-5 if dtype == "float32" else 2e-2)


@device
@both
@pytest.mark.parametrize("name", ["mixed", "attention"])
def test_pages_and_slots_are_used_again(folder, name, dtype, dev):
    """A pool and slots for two requests serve twelve, two alive at a time."""
    name = of(name, dtype)
    r = Replay(folder(name), dtype, dev, 96, page=8, max_requests=2)
    total = r.free_pages()
    for i in range(6):
        prompts = {f"x{i}": tokens(40, vocab(name), 140 + i), f"y{i}": tokens(33 - i, vocab(name), 150 + i)}
        x, y = prompts
        ny = len(prompts[y])
        steps = [[(x, 9), (y, ny - 5)], [(x, 1), (y, 1)], [(y, 2), (x, 25)], [(x, 5), (y, 2)]]
        got = r.run(prompts, steps)
        for k, p in prompts.items():
            agrees(got[k], name, p, dtype)
    r.r.step([], [])
    assert r.free_pages() == total


@device
def test_an_id_is_used_again(folder, dev):
    """A finished request's id at once for another one."""
    r = Replay(folder("mixed"), "float32", dev, 64, max_requests=2)
    for i in range(3):
        toks = tokens(30 + i, 96, 160 + i)
        agrees(r.run({"a": toks}, [[("a", 29)], [("a", 1 + i)]])["a"], "mixed", toks, "float32")


# ------------------------------------------------------------------------------ generation
def check_greedy(name, prompt, out, dtype="float32"):
    """Every generated token is the oracle's choice, or (rounding) next to it."""
    lg = oracle(name, prompt + out)
    for i, t in enumerate(out):
        row = lg[len(prompt) - 1 + i]
        assert row.max() - row[t] <= {"float32": 1e-3, "bfloat16": 0.15}[dtype] * row.std() * 4, (i, t, int(row.argmax()))


@device
@both
@pytest.mark.parametrize("name", ["mixed", "odd", "attention", "recurrent"])
def test_greedy_generation(folder, name, dtype, dev):
    """Seven requests over four seats, prompts longer than the step budget."""
    name = of(name, dtype)
    prompts = [tokens(n, vocab(name), 60 + i) for i, n in enumerate([1, 100, 8, 23, 64, 5])]
    prompts.append(prompts[1][:80] + tokens(9, vocab(name), 70))
    llm = engine(folder(name), dtype, dev)
    outs = llm.generate(prompts, greedy(24))
    for p, o in zip(prompts, outs):
        assert len(o.outputs[0].token_ids) == 24
        check_greedy(name, p, list(o.outputs[0].token_ids), dtype)
    again = llm.generate(prompts[1:2], greedy(24))[0]
    assert again.num_cached_tokens == 0                # (state is kept for whole requests only)
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
    outs = engine(folder("steady"), "bfloat16", "cuda", async_scheduling=True).generate(prompts, greedy(20))
    for p, o in zip(prompts, outs):
        check_greedy("steady", p, list(o.outputs[0].token_ids), "bfloat16")


@pytest.mark.gpu
@both
def test_captured_decode_equals_launched_decode(folder, dtype):
    prompts = [tokens(n, 96, 97 + n) for n in (3, 30, 65)]
    a = engine(folder("mixed"), dtype, "cuda", block_size=16).generate(prompts, greedy(16))
    b = engine(folder("mixed"), dtype, "cuda", block_size=16, enable_cuda_graphs=False).generate(prompts, greedy(16))
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
@pytest.mark.parametrize("dims,base,yarn", [(16, 3e3, (3.0, 90, 24.0, 1.5)), (64, 1e4, (40.0, 4096, 32.0, 1.0)), (6, 700.0, (2.5, 30, 8.0, 0.5)),
                                            (8, 3.0, (2.0, 100000, 32.0, 1.0)), (4, 1e6, (3.0, 10, 9.0, 8.0)), (48, 1e4, (1.0, 64, 4.0, 1.0))])
def test_rotation_frequencies(dims, base, yarn):
    from vllm_cpp_b200.config import RotaryScaling
    from vllm_cpp_b200.models.rope import rope_parameters
    want, mag = R.yarn_frequencies(base, dims, *yarn)
    inv, m, _ = rope_parameters(RotaryScaling(*yarn).rope(base, dims), dims, 64)
    assert torch.allclose(inv, torch.tensor(want, dtype=torch.float64), rtol=1e-12) and math.isclose(m, mag)


def test_registry_and_configuration(folder):
    from vllm_cpp_b200.config import block_config_dict, load_model_config
    from vllm_cpp_b200.models import registry
    for name in C.CASES:
        cfg = load_model_config(folder(name))
        assert registry.resolve(cfg.architecture)[1].__name__ == "KubolornModel"
        assert block_config_dict(cfg) == C.CASES[name][0]
        assert cfg.is_hybrid
    assert "Kubolorn" in registry.supported_architectures()
    cfg = load_model_config(folder("mixed"))
    assert [b.layer for b in cfg.blocks] == R.layer_order(5, C.MIXED["loop"])
    assert [b.weights_of for b in cfg.blocks] == [None, None, None, None, 1, 2, 3, None]


@device
def test_absent_parts_of_the_configuration(tmp_path, dev):
    """No loop, no token pairs, no input convolution, no rotation, one normed part."""
    cfg, w = C.case("mixed")
    cfg = json.loads(json.dumps(cfg))
    del cfg["loop"], cfg["embedding"]["bigram"], cfg["layers"][1]["mixer"]["left"]["rot"], cfg["layers"][4]["mixer"]["left"]["rot"]["scaling"]
    plain = json.loads(json.dumps(cfg))
    del cfg["canon"], cfg["norm"]["groups"]
    plain["norm"]["groups"] = 1
    w = {n: t for n, t in w.items() if "canon" not in n and n != "bigram"}
    toks = tokens(40, 96, 14)
    still = {f"l{l}.canon{i}": torch.zeros(64, 1) for l in range(5) for i in (1, 2)}
    want = R.forward(plain, {**w, **still}, toks)
    got = Replay(C.write(tmp_path / "m", cfg, w), "float32", dev, 48).run({"a": toks}, [[("a", 20)], [("a", 17)]] + [[("a", 1)]] * 3)["a"]
    assert rel(got, want) < TOL["float32"]


@pytest.mark.parametrize("edit", ["mixer", "feed", "heads", "rot", "vdim", "conv", "groups", "norm_groups", "parts", "top", "loop", "times"])
def test_unknown_or_impossible_parts_are_refused(edit):
    from vllm_cpp_b200.config import model_config_from_blocks
    cfg = json.loads(json.dumps(C.MIXED))
    l, left, right = cfg["layers"], cfg["layers"][1]["mixer"]["left"], cfg["layers"][1]["mixer"]["right"]
    if edit == "mixer":
        l[0]["type"] = "other"
    elif edit == "feed":
        l[0]["mlp"]["kind"] = "other"
    elif edit == "heads":
        left["kv_heads"] = 4
    elif edit == "rot":
        left["rot"]["dims"] = 34
    elif edit == "vdim":
        left["vdim"] = 16
    elif edit == "conv":
        right["conv"] = 0
    elif edit == "groups":
        right["groups"] = 4
    elif edit == "norm_groups":
        right["norm_groups"] = 5
    elif edit == "parts":
        cfg["norm"]["groups"] = 5
    elif edit == "top":
        l[1]["mlp"]["router"]["top"] = 6
    elif edit == "loop":
        cfg["loop"]["stop"] = 6
    else:
        cfg["loop"]["times"] = 0
    with pytest.raises(ValueError):
        model_config_from_blocks(cfg)


@pytest.mark.parametrize("name", ["l0.mix.a2.b", "l1.canon2", "l1.mix.left.sink", "l1.mix.right.D", "l2.mlp.e3.up", "l1.mlp.router", "l3.norm1",
                                  "bigram", "embed.norm", "final.norm"])
def test_incomplete_checkpoint_is_refused(tmp_path, name):
    cfg, w = C.case("mixed")
    del w[name]
    with pytest.raises(ValueError, match=name.split(".", 1)[-1] if name[0] == "l" else name.replace(".", "_")):
        engine(C.write(tmp_path / "m", cfg, w), "float32", "cpu")


@pytest.mark.parametrize("name", ["l5.norm1", "l0.mix.left.q", "head"])
def test_unknown_tensors_are_refused(tmp_path, name):
    cfg, w = C.case("mixed")
    w[name] = w["l0.norm1"].clone()
    with pytest.raises(ValueError):
        engine(C.write(tmp_path / "m", cfg, w), "float32", "cpu")


@device
def test_trace_runner(folder, tmp_path, dev):
    name, V = "odd", vocab("odd")
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
    assert rel(read(0), wa[[6, 0]]) < 1e-4
    assert rel(read(2), torch.stack([wb[69], wa[19], wa[8]])) < 1e-4
    assert rel(read(3), wb[[0]]) < 1e-4


@device
def test_synthetic_checkpoint_and_command_line(tmp_path, dev, capsys):
    from vllm_cpp_b200.config import synthetic_config
    from vllm_cpp_b200.entrypoints import cli
    from vllm_cpp_b200.loader import write_synthetic_checkpoint
    out = write_synthetic_checkpoint(str(tmp_path / "ckpt"), synthetic_config("tiny-kubolorn"), seed=1)
    assert cli.main(["--model", out, "--prompt-ids", "5,6,7", "--max-tokens", "4", "--device", dev, "--dtype", "float32",
                     "--max-model-len", "64"]) == 0
    ids = capsys.readouterr().out.strip().splitlines()[-1]
    assert all(0 <= int(x) < 500 for x in ids.split(",")) and len(ids.split(",")) <= 4
    assert cli.main(["--model", out, "--prompt", "the thing", "--max-tokens", "3", "--device", dev,
                     "--max-model-len", "64"]) == 0
