"""Small Nufusun models with random weights, written as checkpoints for the tests."""
import json
import os

import torch


def config(layers, vocab=90, width=48, eps=1e-5, scale=2.0):
    """``layers``: (heads, kv_heads, dim, vdim, scale, bias_max) and (experts, top, ff, limit) or None."""
    out = []
    for (h, g, d, v, s, bm), mlp in layers:
        out.append({"type": "attention",
                    "mixer": {"heads": h, "kv_heads": g, "dim": d, "vdim": v, "scale": s, "bias_max": bm},
                    "mlp": None if mlp is None else {"kind": "moe", "router": {"experts": mlp[0], "top": mlp[1]},
                                                     "expert": {"ff": mlp[2], "limit": mlp[3]}}})
    return {"architecture": "Nufusun", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "layers": out}


def weights(cfg, seed=0, buckets=12, sharp=3.0, bias=1.0):
    """``sharp`` scales the queries (a few keys stand out), ``bias`` the distance bias."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def r(*shape, s=1.0, m=0.0):
        return (torch.randn(*shape, generator=g) * s + m).to(torch.bfloat16)

    t = {"embed": r(cfg["vocab"], W), "head": r(cfg["vocab"], W, s=W ** -0.5), "final.norm": r(W, s=0.2)}
    for l, c in enumerate(cfg["layers"]):
        m, p = c["mixer"], f"l{l}.mix."
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        t[f"l{l}.norm1"] = r(W, s=0.2)
        t[p + "q"] = r(H * D, W, s=sharp * W ** -0.5)
        t[p + "k"] = r(G * D, W, s=W ** -0.5)
        t[p + "v"] = r(G * V, W, s=W ** -0.5)
        t[p + "o"] = r(W, H * V, s=(H * V) ** -0.5)
        for n, rows in (("q", H * D), ("k", G * D), ("v", G * V), ("o", W)):
            t[p + n + ".b"] = r(rows, s=0.3)
        t[p + "rel"] = r(buckets, H, s=bias)
        t[p + "talk"] = (torch.eye(H) + torch.randn(H, H, generator=g) * 0.3).to(torch.bfloat16)
        t[p + "temp"] = r(H, s=0.3, m=1.0)
        if c["mlp"] is None:
            continue
        E, F, p = c["mlp"]["router"]["experts"], c["mlp"]["expert"]["ff"], f"l{l}.mlp."
        t[p + "router"] = r(E, W, s=W ** -0.5)
        for e in range(E):
            t[p + f"e{e}.gate"] = r(F, W, s=W ** -0.5)
            t[p + f"e{e}.up"] = r(F, W, s=W ** -0.5)
            t[p + f"e{e}.down"] = r(W, F, s=F ** -0.5)
    return t


def write(path, cfg, tensors):
    from vllm_cpp_b200.loader import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(tensors, os.path.join(path, "model.safetensors"))
    return str(path)


# name -> (config, weight options). Sizes differ from layer to layer; some take the tensor-core
# kernels, some the any-size kernels (odd widths, head sizes that are no multiple of 8).
CASES = {
    "aligned": (config([((4, 2, 16, 24, 0.25, 40), (4, 2, 32, 1.2)), ((8, 2, 32, 16, 0.2, 20), None),
                        ((6, 6, 8, 32, 0.4, 64), (3, 1, 24, 0.5))], width=64, vocab=96), {}),
    "odd": (config([((3, 1, 5, 7, 0.5, 33), (5, 3, 11, 0.8)), ((10, 5, 9, 3, 0.3, 17), (1, 1, 13, 2.0))],
                   width=37, vocab=61, eps=1e-3, scale=0.7), {"buckets": 10}),
    "one_of_each": (config([((1, 1, 8, 8, 1.0, 9), (1, 1, 8, 1.0))], width=8, vocab=16, scale=1.0), {"buckets": 4}),
    "wide_bias": (config([((4, 4, 16, 16, 0.3, 130), (2, 2, 16, 1.5)), ((4, 1, 64, 40, 0.1, 130), (6, 2, 40, 0.9))],
                         width=56, vocab=72), {"buckets": 32, "bias": 4.0, "sharp": 1.0}),
}


def case(name, seed=0):
    cfg, opt = CASES[name]
    return cfg, weights(cfg, seed=seed, **opt)
