"""Tabupel through the engine (registry, loader, scheduler, paged cache, state slots, batches) against the
plain implementation in ``tabupel_reference.py``; every test runs on the CPU back end and, on a GPU box, on
the kernels."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import tabupel_case as C                                                       # noqa: E402
import tabupel_reference as R                                                  # noqa: E402
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


def oracle(name, toks):
    key = (name, tuple(toks))
    if key not in _logits:
        _logits[key] = R.forward(*C.case(name), toks)
    return _logits[key]


def agrees(got, name, toks, dtype):
    e = rel(got, oracle(name, toks))
    assert e < TOL[dtype] * (3 if name in ("odd", "ones") else 1), e


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    base = tmp_path_factory.mktemp("tabupel")
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
@pytest.mark.parametrize("name", list(C.CASES))
def test_whole_prompt(folder, name, page, dtype, dev):
    toks = tokens(150, C.CASES[name][0]["vocab"], 1)
    got = Replay(folder(name), dtype, dev, 160, page=page).run({"a": toks}, [[("a", len(toks))]])["a"]
    agrees(got, name, toks, dtype)


@device
@both
@pytest.mark.parametrize("name", list(C.CASES))
def test_token_by_token(folder, name, dtype, dev):
    toks = tokens(70, C.CASES[name][0]["vocab"], 2)
    got = Replay(folder(name), dtype, dev, 80, page=16).run({"a": toks}, [[("a", 1)]] * len(toks))["a"]
    agrees(got, name, toks, dtype)


@device
@both
def test_first_tokens(folder, dtype, dev):
    """One-token prompts included: nothing of the slot's last user may be seen."""
    r = Replay(folder("mixed"), dtype, dev, 48, page=16, max_requests=1)
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
    got = Replay(folder(name), dtype, dev, 160).run({"a": toks}, steps)["a"]
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
    toks = tokens(64, 96, 6)
    got = Replay(folder("mixed"), "float32", dev, 72).run({"a": toks}, [[("a", 44)]] + [[("a", 1)]] * 20)["a"]
    assert rel(got, oracle("mixed", toks)) < TOL["float32"]

    def differs(cfg2, w2=w, least=2e-3):
        d = rel(R.forward(cfg2, w2, toks), oracle("mixed", toks))
        assert d > least, d

    def of(kind, f):
        return edited(cfg, lambda l: f(l["mixer"]) if l["type"] == kind else None)
    for kind in ("attention", "latent_attention"):
        differs(of(kind, lambda m: m["mask"].update(size=m["mask"]["size"] - 1)))     # a window's edge one token off
        differs(of(kind, lambda m: m.update(scale=m["scale"] * 1.5)))
        differs(of(kind, lambda m: m["rot"].update(base=m["rot"]["base"] * 3)))
        differs(of(kind, lambda m: m["rot"]["scaling"].update(factor=m["rot"]["scaling"]["factor"] * 2)))
    differs(of("attention", lambda m: m["rot"].update(dims=m["rot"]["dims"] - 2)))
    differs(of("attention", lambda m: m.update(diff=m["diff"] + 0.1)))
    for k, v in (("original", 40), ("fast", 4.0), ("slow", 6.0)):
        differs(of("latent_attention", lambda m: m["rot"]["scaling"].update({k: v})))
    differs({**cfg, "residual_mult": 0.5})
    differs({**cfg, "logit_softcap": 20.0})
    g = torch.Generator().manual_seed(1)
    for n in w:                                                                       # every tensor
        differs(cfg, {**w, n: w[n] + (0.5 * w[n].float().std().clamp_min(0.1) * torch.randn(w[n].shape, generator=g)).to(w[n])})
    differs(cfg, {**w, "l0.mix.conv": w["l0.mix.conv"].flip(1)})                      # the order of the taps
    differs(cfg, {**w, "l0.mix.ra": w["l0.mix.ri"], "l0.mix.ri": w["l0.mix.ra"]})


@device
@both
@pytest.mark.parametrize("kind", ["attention", "latent"])
@pytest.mark.parametrize("window", [50, 64])
def test_far_key_stands_out(tmp_path, kind, window, dtype, dev):
    """One query-key pair carries almost the whole weight, at the far end of a window; one token further it is
    not seen. Positions hardly turn anything."""
    l = C.attention(2, 2, 64, 16, 0.3, window, 1e9, 2, 1e6, 0.3) if kind == "attention" else \
        C.latent(2, 16, 64, 16, 64, 64, 0.3, window, 1e9, (1e6, 1e-3, 2.0, 1.0))
    cfg = C.config([l], width=64, vocab=24)
    w = C.weights(cfg, seed=9)
    h = R.rms(w["embed"].double(), 1e-5) * w["l0.norm1"].double()
    d = torch.linalg.pinv(h)                                          # column t answers to token t alone
    dirs = torch.randn(4, 64, generator=torch.Generator().manual_seed(2)).double()
    dirs[:, :2] = 0.0                                                 # (not where positions turn it)
    if kind == "attention":
        for n, t in (("k", 7), ("q", 11)):
            x = w[f"l0.mix.{n}"].double() + 6.0 * torch.cat([torch.outer(dirs[i], d[:, t]) for i in range(4)])
            w[f"l0.mix.{n}"] = x.to(torch.bfloat16)
        w["l0.mix.q.norm"], w["l0.mix.k.norm"] = (w[n] * 2 for n in ("l0.mix.q.norm", "l0.mix.k.norm"))
    else:
        # the shared key part of one token, and the query latent of the other; only the rotated part scores
        x = w["l0.mix.dkv"].double()
        x[64:] = 0.1 * x[64:] + 5.0 * torch.outer(dirs[0], d[:, 7])
        w["l0.mix.dkv"] = x.to(torch.bfloat16)
        w["l0.mix.dq"] = (0.3 * w["l0.mix.dq"].double() + 8.0 * torch.outer(dirs[1], d[:, 11])).to(torch.bfloat16)
        uq = w["l0.mix.uq"].double().view(2, 80, 64) * 0.3
        uq[:, 16:] += torch.outer(dirs[0], dirs[1] / dirs[1].norm()) * 0.4
        w["l0.mix.uq"] = uq.view(160, 64).to(torch.bfloat16)
    toks = [t if t not in (7, 11) else 8 for t in tokens(4 * window, 24, 10)]
    at = 2 * window - 14
    toks[at] = 7
    for p in (at + window - 1, at + window):
        toks[p] = 11
    want = R.forward(cfg, w, toks)
    without = list(toks)
    without[at] = 8
    moved = R.forward(cfg, w, without)
    assert rel(moved[[at + window - 1]], want[[at + window - 1]]) > 0.2 and rel(moved[[at + window]], want[[at + window]]) < 1e-12
    model = C.write(tmp_path / "far", cfg, w)
    n, k = len(toks), at + window - 10
    for steps in ([[("a", n)]], [[("a", k)]] + [[("a", 1)]] * (n - k), [[("a", n // 2 + 3)], [("a", n - n // 2 - 3)]]):
        got = Replay(model, dtype, dev, n + 16, page=16).run({"a": toks}, steps)["a"]
        assert rel(got, want) < TOL[dtype]


@device
@both
def test_state_reaches_far_back(folder, dtype, dev):
    """Slow decays: a token hundreds of positions back still shows."""
    toks = tokens(420, 50, 12)
    want = oracle("recurrent_only", toks)
    other = list(toks)
    other[20] = (toks[20] + 1) % 50
    assert rel(oracle("recurrent_only", other)[[419]], want[[419]]) > 5e-4
    for steps in ([[("a", 420)]], [[("a", 400)]] + [[("a", 1)]] * 20, [[("a", 70)]] * 6):
        got = Replay(folder("recurrent_only"), dtype, dev, 424).run({"a": toks}, steps)["a"]
        agrees(got, "recurrent_only", toks, dtype)


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
    got = Replay(folder(name), dtype, dev, 176).run(prompts, random_steps({r: len(p) for r, p in prompts.items()}, 5))
    for r, p in prompts.items():
        agrees(got[r], name, p, dtype)


@device
@both
def test_batch_does_not_change_a_request(folder, dtype, dev):
    prompts = {r: tokens(n, 96, 30 + i) for i, (r, n) in enumerate([("a", 60), ("b", 33), ("c", 20)])}
    steps = [[("a", 30), ("b", 33)], [("a", 1), ("c", 12)], [("a", 29), ("c", 1)], [("c", 7)]]
    alone = [[("a", 30)], [("a", 1)], [("a", 29)]]
    together = Replay(folder("mixed"), dtype, dev, 128).run(prompts, steps)["a"]
    single = Replay(folder("mixed"), dtype, dev, 128).run({"a": prompts["a"]}, alone)["a"]
    assert rel(together, single.double()) < (1e-5 if dtype == "float32" else 2e-2)


@device
@both
@pytest.mark.parametrize("name", ["mixed", "attention_only"])
def test_pages_and_slots_are_used_again(folder, name, dtype, dev):
    """A pool and slots for two requests serve twelve, two alive at a time."""
    V = C.CASES[name][0]["vocab"]
    r = Replay(folder(name), dtype, dev, 96, page=8, max_requests=2)
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
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_behind_the_window_are_given_back(folder, dtype, dev):
    """The widest window is 24: a prompt of 150 tokens holds few pages at a time, and others overwrite the rest."""
    toks, V = tokens(150, 72, 13), 72
    r = Replay(folder("attention_only"), dtype, dev, 160, page=8, max_requests=2)
    free, at, got = r.free_pages(), 0, []
    while at < 150:
        n = min(10, 150 - at)
        rows = r.r.step([{"id": "a", "tokens": toks[at:at + n], "want": list(range(n))}], [])
        got += rows
        at += n
        assert free - r.free_pages() <= (24 + 10 + 7) // 8 + 2
        if at % 30 == 0:                                      # (somebody else fills the pages given back)
            b = tokens(60, V, at)
            agrees(torch.stack(r.r.step([{"id": f"b{at}", "tokens": b, "want": list(range(60))}], [f"b{at}"])), "attention_only", b, dtype)
    agrees(torch.stack(got), "attention_only", toks, dtype)


# ------------------------------------------------------------------------------ generation
def check_greedy(name, prompt, out, dtype="float32"):
    """Every generated token is the oracle's choice, or (rounding) next to it."""
    lg = oracle(name, prompt + out)
    for i, t in enumerate(out):
        row = lg[len(prompt) - 1 + i]
        assert row.max() - row[t] <= {"float32": 1e-3, "bfloat16": 0.6}[dtype], (i, t, int(row.argmax()))


@device
@both
@pytest.mark.parametrize("name", ["mixed", "odd", "attention_only"])
def test_greedy_generation(folder, name, dtype, dev):
    """Seven requests over four seats, prompts longer than the step budget; prefix caching where no state
    is kept."""
    vocab = C.CASES[name][0]["vocab"]
    prompts = [tokens(n, vocab, 60 + i) for i, n in enumerate([1, 100, 8, 23, 64, 5])]
    prompts.append(prompts[1][:80] + tokens(9, vocab, 70))
    llm = engine(folder(name), dtype, dev)
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
    outs = engine(folder("mixed"), "bfloat16", "cuda", async_scheduling=True).generate(prompts, greedy(20))
    for p, o in zip(prompts, outs):
        check_greedy("mixed", p, list(o.outputs[0].token_ids), "bfloat16")


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
@pytest.mark.parametrize("dims,base,yarn", [(16, 4e3, (6.0, 100, 24.0, 1.5)), (64, 1e4, (40.0, 4096, 32.0, 1.0)), (6, 50.0, (2.5, 30, 8.0, 0.5)),
                                            (8, 3.0, (2.0, 100000, 32.0, 1.0)), (4, 1e6, (3.0, 10, 9.0, 8.0)), (32, 1e4, (1.0, 64, 4.0, 1.0))])
def test_rotation_frequencies(dims, base, yarn):
    """YaRN and linear scaling, also where the ramp is empty, clamped or past the last dimension."""
    from vllm_cpp_b200.config import RotaryScaling
    from vllm_cpp_b200.models.rope import rope_parameters
    want, mag = R.yarn_frequencies(base, dims, *yarn)
    inv, m, _ = rope_parameters(RotaryScaling(*yarn).rope(base, dims), dims, 64)
    assert torch.allclose(inv, torch.tensor(want, dtype=torch.float64), rtol=1e-12) and math.isclose(m, mag)
    inv, m, _ = rope_parameters(RotaryScaling(yarn[0]).rope(base, dims), dims, 64)
    assert torch.allclose(inv, torch.tensor(R.linear_frequencies(base, dims, yarn[0]), dtype=torch.float64), rtol=1e-12) and m == 1.0


def test_registry_and_configuration(folder):
    from vllm_cpp_b200.config import block_config_dict, load_model_config
    from vllm_cpp_b200.models import registry
    for name in C.CASES:
        cfg = load_model_config(folder(name))
        assert registry.resolve(cfg.architecture)[1].__name__ == "TabupelModel"
        assert block_config_dict(cfg) == C.CASES[name][0]
        assert cfg.is_hybrid == (name != "attention_only")
    assert "Tabupel" in registry.supported_architectures()


def test_absent_parts_of_the_configuration():
    from vllm_cpp_b200.config import model_config_from_blocks
    cfg = json.loads(json.dumps(C.CASES["attention_only"][0]))
    del cfg["layers"][0]["mixer"]["mask"], cfg["layers"][0]["mixer"]["rot"]["scaling"]
    m = model_config_from_blocks(cfg)
    assert m.blocks[0].attention.window == 0 and m.blocks[0].attention.rot_scaling is None
    assert m.layer_types == ["full_attention", "sliding_attention", "sliding_attention"]


@device
def test_blocks_without_a_window(tmp_path, dev):
    """One block sees everything: no page is given back."""
    cfg, w = C.case("attention_only")
    cfg = json.loads(json.dumps(cfg))
    del cfg["layers"][1]["mixer"]["mask"]
    far = json.loads(json.dumps(cfg))
    far["layers"][1]["mixer"]["mask"] = {"size": 1000}
    toks = tokens(150, 72, 14)
    got = Replay(C.write(tmp_path / "m", cfg, w), "float32", dev, 160).run({"a": toks}, [[("a", 100)], [("a", 47)]] + [[("a", 1)]] * 3)["a"]
    assert rel(got, R.forward(far, w, toks)) < TOL["float32"]


@pytest.mark.parametrize("edit", ["mixer", "feed", "heads", "rot", "rot_dim", "conv", "blocks", "shared", "shared_chain", "shared_sizes", "arch"])
def test_unknown_or_impossible_parts_are_refused(edit):
    from vllm_cpp_b200.config import model_config_from_blocks
    cfg = json.loads(json.dumps(C.CASES["mixed"][0]))
    l = cfg["layers"]
    if edit == "mixer":
        l[0]["type"] = "other"
    elif edit == "feed":
        l[0]["mlp"]["kind"] = "other"
    elif edit == "heads":
        l[2]["mixer"]["kv_heads"] = 3
    elif edit == "rot":
        l[2]["mixer"]["rot"]["dims"] = 50
    elif edit == "rot_dim":
        l[1]["mixer"]["rot"]["dims"] = 8
    elif edit == "conv":
        l[0]["mixer"]["conv"] = 0
    elif edit == "blocks":
        l[0]["mixer"]["blocks"] = 5
    elif edit == "shared":
        l[4]["weights_of"] = 11
    elif edit == "shared_chain":
        l[5]["weights_of"] = 5
    elif edit == "shared_sizes":
        l[5]["weights_of"] = 2
    else:
        cfg["architecture"] = "Other"
    with pytest.raises(ValueError):
        model_config_from_blocks(cfg)


@pytest.mark.parametrize("name", ["l0.mix.lam", "l1.norm2", "l2.mix.lq2", "l1.mix.dkv.norm", "l3.mix.conv.b", "l2.mlp.up", "final.norm", "head"])
def test_incomplete_checkpoint_is_refused(tmp_path, name):
    cfg, w = C.case("mixed")
    del w[name]
    with pytest.raises(ValueError, match=name.split(".", 1)[-1] if name != "head" else "lm_head"):
        engine(C.write(tmp_path / "m", cfg, w), "float32", "cpu")


def test_tensors_of_a_block_with_shared_weights_are_refused(tmp_path):
    cfg, w = C.case("mixed")
    w["l4.norm1"] = w["l0.norm1"]
    with pytest.raises(ValueError, match="norm1"):
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
    assert rel(read(0), wa[[6, 0]]) < 1e-4
    assert rel(read(2), torch.stack([wb[69], wa[19], wa[8]])) < 1e-4
    assert rel(read(3), wb[[0]]) < 1e-4


@device
def test_synthetic_checkpoint_and_command_line(tmp_path, dev, capsys):
    from vllm_cpp_b200.config import synthetic_config
    from vllm_cpp_b200.entrypoints import cli
    from vllm_cpp_b200.loader import write_synthetic_checkpoint
    out = write_synthetic_checkpoint(str(tmp_path / "ckpt"), synthetic_config("tiny-tabupel"), seed=1)
    assert cli.main(["--model", out, "--prompt-ids", "5,6,7", "--max-tokens", "4", "--device", dev, "--dtype", "float32",
                     "--max-model-len", "64"]) == 0
    ids = capsys.readouterr().out.strip().splitlines()[-1]
    assert all(0 <= int(x) < 500 for x in ids.split(",")) and len(ids.split(",")) <= 4
    assert cli.main(["--model", out, "--prompt", "the thing", "--max-tokens", "3", "--device", dev,
                     "--max-model-len", "64"]) == 0
