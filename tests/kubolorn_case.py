"""Small Kubolorn models with random weights, written as checkpoints for the tests."""
import json
import os

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def gla(heads, dim, vdim, tau, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def parallel(left, right, scales, mlp=None):
    """left: heads, kv heads, size, scale, base, rotated dimensions, (factor, original, fast, slow); right: heads, groups,
    state, size, taps, normed parts."""
    H, G, D, scale, base, dims, yarn = left
    rot = {"base": base, "dims": dims, "scaling": dict(zip(("factor", "original", "fast", "slow"), yarn))}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": scale, "rot": rot},
                      "right": dict(zip(("heads", "groups", "state", "vdim", "conv", "norm_groups"), right)),
                      "left_scale": scales[0], "right_scale": scales[1]}}


def config(layers, vocab=90, width=48, eps=1e-5, groups=3, taps=4, scale=3.0, bigram=(23, 5, 3), loop=None):
    c = {"architecture": "Kubolorn", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "canon": {"taps": taps},
         "embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def weights(cfg, seed=0, rank=7, decay=0.0, steady=False):
    """``decay``: mean of the decay's logits (large: the state reaches far back). ``steady``: the first channel of the
    stream is about the same for every token and fixes the choice of experts (rounding cannot change it)."""
    g = torch.Generator().manual_seed(seed)
    W, taps = cfg["width"], cfg["canon"]["taps"]

    def r(*shape, s=1.0, m=0.0):
        return (torch.randn(*shape, generator=g) * s + m).to(torch.bfloat16)

    def lin(rows, cols, s=1.0):
        return r(rows, cols, s=s * cols ** -0.5)
    t = {"embed": r(cfg["vocab"], W, s=0.4), "embed.norm": r(W, s=0.2, m=1.0), "final.norm": r(W, s=0.2, m=1.0),
         "bigram": r(cfg["embedding"]["bigram"]["buckets"] + 1, W)}
    if steady:
        t["embed"][:, 0] = 3.0
        t["bigram"][:, 0] = 0.0
    for l, c in enumerate(cfg["layers"]):
        m, f, p = c["mixer"], c["mlp"], f"l{l}.mix."
        for i in (1, 2) if f else (1,):
            t[f"l{l}.norm{i}"], t[f"l{l}.canon{i}"] = r(W, s=0.2, m=1.0), r(W, taps, s=0.35)
        if c["type"] == "gla":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * V), ("g", H * V)):
                t[p + n] = lin(rows, W)
            t[p + "a1"], t[p + "a2"], t[p + "a2.b"] = lin(rank, W), lin(H * D, rank, 1.5), r(H * D, s=0.7, m=decay)
            t[p + "norm"], t[p + "o"] = r(V, s=0.3, m=1.0), lin(W, H * V, 1.5)
        else:
            a, b = m["left"], m["right"]
            H, G, D = a["heads"], a["kv_heads"], a["dim"]
            t[p + "left.q"], t[p + "left.k"] = lin(H * D, W, 1.5), lin(G * D, W, 1.2)
            t[p + "left.sink"], t[p + "left.o"] = r(H, s=1.0, m=0.5), lin(W, H * D, 2.0)
            p += "right."
            inner, gn = b["heads"] * b["vdim"], b["groups"] * b["state"]
            t[p + "in"] = lin(2 * inner + 2 * gn + b["heads"], W)
            t[p + "conv"], t[p + "conv.b"] = r(inner + 2 * gn, b["conv"], s=0.6), r(inner + 2 * gn, s=0.2)
            t[p + "dt_bias"], t[p + "A_log"] = r(b["heads"], s=0.7, m=-1.0 - decay / 2), r(b["heads"], s=0.6)
            t[p + "D"], t[p + "norm"], t[p + "o"] = r(b["heads"], s=0.6, m=0.8), r(inner, s=0.2, m=1.0), lin(W, inner, 1.5)
        units = [""] if f and f["kind"] == "dense" else [f"e{e}." for e in range(f["router"]["experts"])] if f else []
        ff = 0 if not f else f["ff"] if f["kind"] == "dense" else f["expert"]["ff"]
        for u in units:
            t[f"l{l}.mlp.{u}up"], t[f"l{l}.mlp.{u}down"] = lin(ff, W), lin(W, ff, 1.5)
        if f and f["kind"] == "moe":
            E = f["router"]["experts"]
            x = lin(E, W, 1.5)
            if steady:
                x = (x * 0.3).to(torch.bfloat16)
                x[:, 0] = (torch.randperm(E, generator=g) * 4.0).to(torch.bfloat16)
                t[f"l{l}.canon2"][0] = 0.1
            t[f"l{l}.mlp.router"] = x
    if steady:
        for n in t:                              # (nothing is added to that channel)
            if n.endswith((".o", ".down")):
                t[n][0] = 0.0
    return t


def write(path, cfg, tensors):
    from vllm_cpp_b200.loader import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(tensors, os.path.join(path, "model.safetensors"))
    return str(path)


P1 = parallel((6, 2, 32, 0.3, 3e3, 16, (3.0, 90, 24.0, 1.5)), (6, 3, 32, 16, 3, 2), (0.8, 1.3))
MIXED = config([gla(3, 32, 64, 8.0, dense(72)), {**P1, "mlp": moe(5, 2, 40)}, gla(2, 64, 16, 4.0, moe(6, 3, 24)), gla(3, 32, 64, 8.0),
                parallel((4, 1, 64, 0.2, 2e4, 64, (1.5, 400, 16.0, 2.0)), (2, 1, 64, 48, 5, 1), (1.1, 0.7), dense(56))],
               width=64, vocab=96, groups=4, loop=(1, 4, 2))
# name -> (config, weight options). Some sizes take the tensor-core kernels, some the any-size kernels.
CASES = {
    "mixed": (MIXED, {"rank": 12}),
    "steady": (MIXED, {"rank": 12, "steady": True}),
    "odd": (config([gla(2, 10, 7, 2.5, dense(11)), parallel((3, 3, 10, 0.5, 700.0, 6, (2.5, 30, 8.0, 0.5)), (3, 1, 5, 6, 2, 9), (1.7, -0.6), dense(9)),
                    gla(3, 5, 21, 11.0)], width=35, vocab=61, eps=1e-3, groups=5, taps=2, scale=0.7, bigram=(7, 13, 11), loop=(0, 2, 3)), {"rank": 3}),
    "attention": (config([parallel((8, 4, 16, 0.4, 900.0, 8, (4.0, 64, 16.0, 1.0)), (4, 4, 16, 32, 4, 8), (0.9, 1.4), dense(50)),
                          parallel((20, 1, 48, 0.2, 1e4, 48, (1.0, 64, 4.0, 1.0)), (3, 1, 80, 32, 1, 3), (1.0, 1.0), dense(30))],
                         width=56, vocab=72, groups=1, taps=1, bigram=(11, 2, 7)), {}),
    "recurrent": (config([gla(2, 48, 80, 16.0, dense(40)), gla(1, 144, 32, 16.0)], width=40, vocab=50, groups=2, taps=5, loop=(0, 1, 2)),
                  {"decay": 4.0, "rank": 20}),
    "fading": (config([gla(2, 32, 32, 0.05, dense(40)), gla(2, 16, 48, 0.4)], width=48, vocab=50, groups=3, taps=3),
               {"decay": 1.0, "rank": 6}),
    "ones": (config([gla(1, 1, 1, 1.0, dense(1)), parallel((1, 1, 2, 1.0, 10.0, 2, (1.0, 8, 2.0, 1.0)), (1, 1, 1, 1, 1, 1), (1.0, 1.0), moe(1, 1, 1))],
                    width=8, vocab=16, groups=1, taps=1, scale=1.0, bigram=(1, 1, 1), loop=(0, 2, 1)), {"rank": 1}),
}


def case(name):
    cfg, opt = CASES[name]
    return cfg, weights(cfg, **opt)
