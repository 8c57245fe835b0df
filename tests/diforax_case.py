"""Small Diforax models with random weights, written as checkpoints for the tests."""
import json
import os

import torch


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, scale, chunk, base, dims, mlp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk},
         "rot": {"base": base, "dims": dims}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, count, keep, ff):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top,
                                      "groups": {"count": count, "keep": keep}}, "expert": {"ff": ff}}


def config(layers, vocab=90, width=48, eps=1e-5):
    return {"architecture": "Diforax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def weights(cfg, seed=0, slow=False, steady=False):
    """``slow``: decays near one, so that the state reaches back over hundreds of tokens. ``steady``: the
    corrections outweigh the scores, so that rounding changes no choice of experts (a choice changed at one
    token would reach all later ones through the states)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def r(*shape, s=1.0, m=0.0):
        return (torch.randn(*shape, generator=g) * s + m).to(torch.bfloat16)

    t = {"embed": r(cfg["vocab"], W), "head": r(cfg["vocab"], W, s=W ** -0.5), "final.norm": r(W, s=0.2, m=1.0)}
    for l, c in enumerate(cfg["layers"]):
        m, p = c["mixer"], f"l{l}.mix."
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if c["mlp"] else ()):
            t[f"l{l}.{n}"] = r(W, s=0.2, m=1.0)
        t[p + "o"] = r(W, H * V, s=(H * V) ** -0.5)
        if c["type"] == "delta":
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                t[p + n] = r(rows, W, s=W ** -0.5)
                t[p + n + ".conv"] = r(rows, m["conv"], s=0.7)
            t[p + "g"] = r(H * V, W, s=W ** -0.5)
            t[p + "a"], t[p + "b"] = r(H, W, s=W ** -0.5), r(H, W, s=W ** -0.5)
            t[p + "A_log"], t[p + "dt_bias"] = r(H, s=0.5), r(H, s=0.5, m=-7.0 if slow else -2.0)
            t[p + "norm"] = r(V, s=0.2, m=1.0)
        else:
            t[p + "q"] = r(H * D, W, s=W ** -0.5)
            if m.get("kv_from") is None:
                t[p + "k"], t[p + "v"] = r(G * D, W, s=W ** -0.5), r(G * V, W, s=W ** -0.5)
        f, p = c["mlp"], f"l{l}.mlp."
        if f is None:
            continue
        ff = f["ff"] if f["kind"] == "dense" else f["expert"]["ff"]
        for u in [""] if f["kind"] == "dense" else [f"e{e}." for e in range(f["router"]["experts"])]:
            t[p + u + "gate"], t[p + u + "up"] = r(ff, W, s=W ** -0.5), r(ff, W, s=W ** -0.5)
            t[p + u + "down"] = r(W, ff, s=ff ** -0.5)
        if f["kind"] == "moe":
            n = f["router"]["experts"] + f["router"]["identity"]
            t[p + "router"] = r(n, W, s=1.5 * W ** -0.5)
            t[p + "correction"] = (1.5 * (torch.randperm(n, generator=g) - n / 2)).to(torch.bfloat16) if steady else r(n, s=0.1, m=-0.05)
    return t


def write(path, cfg, tensors):
    from vllm_cpp_b200.loader import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(tensors, os.path.join(path, "model.safetensors"))
    return str(path)


# name -> (config, weight options). Sizes differ from layer to layer; some take the tensor-core kernels,
# some the any-size kernels.
CASES = {
    "mixed": (config([delta(4, 2, 32, 48, 4, dense(72)), attention(4, 2, 48, 32, 0.2, 40, 4e4, 32, moe(6, 2, 3, 4, 2, 40)),
                      delta(2, 2, 64, 16, 3), attention(6, 2, 48, 32, 0.3, 64, 4e4, 32, dense(130), kv_from=1),
                      delta(3, 1, 16, 80, 2, moe(5, 3, 2, 2, 1, 24))], width=64, vocab=96), {}),
    "odd": (config([attention(3, 1, 10, 7, 0.5, 13, 700.0, 6, dense(11)), delta(4, 2, 5, 9, 5, moe(5, 1, 4, 3, 2, 13)),
                    attention(2, 1, 10, 7, 0.4, 21, 700.0, 6, moe(3, 0, 1, 1, 1, 9), kv_from=0), delta(1, 1, 33, 18, 1, None)],
                   width=37, vocab=61, eps=1e-3), {}),
    "attention_only": (config([attention(4, 4, 16, 16, 0.4, 24, 1e4, 16), attention(8, 2, 32, 64, 0.3, 24, 300.0, 8, dense(64)),
                               attention(8, 2, 32, 64, 0.5, 24, 300.0, 8, moe(4, 4, 2, 2, 2, 32), kv_from=1)], width=56, vocab=72), {}),
    "delta_only": (config([delta(2, 1, 24, 40, 4, dense(50)), delta(6, 3, 16, 16, 4)], width=40, vocab=50), {"slow": True}),
    "ones": (config([delta(1, 1, 1, 1, 1), attention(1, 1, 2, 1, 1.0, 1, 10.0, 2, moe(1, 0, 1, 1, 1, 1))], width=8, vocab=16), {}),
}


def case(name, dtype="float32"):
    cfg, opt = CASES[name]
    return cfg, weights(cfg, steady=dtype == "bfloat16", **opt)
