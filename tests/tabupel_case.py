"""Small Tabupel models with random weights, written as checkpoints for the tests."""
import json
import os

import torch


def attention(heads, kv_heads, dim, vdim, scale, size, base, dims, factor, diff, ff=None, weights_of=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "mask": {"size": size},
         "rot": {"base": base, "dims": dims, "scaling": {"factor": factor}}}
    return layer("attention", m, ff, weights_of)


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, size, base, yarn, ff=None, weights_of=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "mask": {"size": size}, "rot": {"base": base, "dims": rot_dim,
                                         "scaling": dict(zip(("factor", "original", "fast", "slow"), yarn))}}
    return layer("latent_attention", m, ff, weights_of)


def rglru(width, blocks, conv, ff=None, weights_of=None):
    return layer("rglru", {"width": width, "blocks": blocks, "conv": conv}, ff, weights_of)


def layer(kind, mixer, ff, weights_of):
    l = {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    if weights_of is not None:
        l["weights_of"] = weights_of
    return l


def config(layers, vocab=90, width=48, eps=1e-5, mult=0.6, cap=25.0):
    return {"architecture": "Tabupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "logit_softcap": cap, "layers": layers}


def weights(cfg, seed=0, slow=False):
    """``slow``: decays near one, so that the state reaches back over hundreds of tokens."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def r(*shape, s=1.0, m=0.0):
        return (torch.randn(*shape, generator=g) * s + m).to(torch.bfloat16)

    def lin(rows, cols, s=1.0):
        return r(rows, cols, s=s * cols ** -0.5)
    t = {"embed": r(cfg["vocab"], W), "head": lin(cfg["vocab"], W, 8.0), "final.norm": r(W, s=0.2, m=1.0)}
    for l, c in enumerate(cfg["layers"]):
        if c.get("weights_of") is not None:
            continue
        m, p = c["mixer"], f"l{l}.mix."
        t[f"l{l}.norm1"] = r(W, s=0.2, m=1.0)
        if c["type"] == "attention":
            H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            t[p + "q"], t[p + "k"], t[p + "v"] = lin(H * 2 * D, W), lin(G * 2 * D, W), lin(G * V, W)
            for n in ("q.norm", "k.norm"):
                t[p + n] = r(D, s=0.3, m=1.2)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                t[p + n] = r(D, s=0.8 * D ** -0.25)
            t[p + "o"] = lin(W, H * V, 1.5)
        elif c["type"] == "latent_attention":
            H, D, R, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
            t[p + "dq"], t[p + "dq.norm"] = lin(m["q_rank"], W), r(m["q_rank"], s=0.2, m=1.0)
            t[p + "uq"] = lin(H * (D + R), m["q_rank"], 1.5)
            t[p + "dkv"], t[p + "dkv.norm"] = lin(m["kv_rank"] + R, W, 1.5), r(m["kv_rank"], s=0.2, m=1.0)
            t[p + "uk"], t[p + "uv"] = lin(H * D, m["kv_rank"]), lin(H * V, m["kv_rank"], 2.0)
            t[p + "g"], t[p + "o"] = lin(H, W, 1.5), lin(W, H * V, 2.0)
        else:
            C, N, n = m["width"], m["blocks"], m["width"] // m["blocks"]
            for k in ("y", "x"):
                t[p + k], t[p + k + ".b"] = lin(C, W), r(C, s=0.3)
            t[p + "conv"], t[p + "conv.b"] = r(C, m["conv"], s=0.6), r(C, s=0.2)
            for k in ("ra", "ri"):
                t[p + k], t[p + k + ".b"] = r(N, n, n, s=1.5 * n ** -0.5), r(N, n, s=0.5)
            t[p + "lam"] = r(C, s=0.7, m=-9.0 if slow else -3.0)
            t[p + "o"] = lin(W, C, 2.0)
        if c["mlp"] is not None:
            ff = c["mlp"]["ff"]
            t[f"l{l}.norm2"] = r(W, s=0.2, m=1.0)
            t[f"l{l}.mlp.gate"], t[f"l{l}.mlp.up"], t[f"l{l}.mlp.down"] = lin(ff, W), lin(ff, W), lin(W, ff, 2.0)
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
    "mixed": (config([rglru(96, 3, 4, 72), latent(3, 48, 16, 32, 40, 56, 0.2, 43, 4e3, (6.0, 100, 24.0, 1.5), 130),
                      attention(4, 2, 32, 48, 0.25, 24, 7e3, 20, 3.0, 0.45, 64), rglru(64, 1, 2), rglru(96, 3, 4, 72, weights_of=0),
                      latent(3, 48, 16, 32, 40, 56, 0.2, 43, 4e3, (6.0, 100, 24.0, 1.5), 130, weights_of=1),
                      attention(6, 1, 16, 64, 0.4, 33, 900.0, 16, 1.5, 0.2), rglru(64, 1, 2, weights_of=3)], width=64, vocab=96), {}),
    "odd": (config([latent(2, 10, 6, 7, 9, 11, 0.4, 13, 50.0, (2.5, 30, 8.0, 0.5), 11), rglru(21, 3, 3),
                    attention(3, 1, 10, 7, 0.5, 17, 700.0, 6, 2.0, 0.7, 9), rglru(10, 10, 5, 13),
                    attention(3, 1, 10, 7, 0.5, 17, 700.0, 6, 2.0, 0.7, 9, weights_of=2)], width=37, vocab=61, eps=1e-3, mult=0.8, cap=9.0), {}),
    "attention_only": (config([attention(2, 2, 48, 32, 0.2, 24, 1e4, 48, 4.0, 0.3, 50),
                               latent(2, 16, 32, 16, 24, 130, 0.2, 20, 1e4, (4.0, 64, 16.0, 1.0)),
                               attention(8, 2, 16, 128, 0.3, 24, 300.0, 8, 1.0, 0.0)], width=56, vocab=72), {}),
    "recurrent_only": (config([rglru(80, 5, 4, 50), rglru(48, 2, 3)], width=40, vocab=50), {"slow": True}),
    "ones": (config([rglru(1, 1, 1, 1), latent(1, 1, 2, 1, 1, 1, 1.0, 1, 10.0, (1.0, 8, 2.0, 1.0), 1),
                     attention(1, 1, 2, 1, 1.0, 1, 10.0, 2, 1.0, 0.5, 1)], width=8, vocab=16, mult=1.0), {}),
}


def case(name, dtype="float32"):
    cfg, opt = CASES[name]
    return cfg, weights(cfg, **opt)
