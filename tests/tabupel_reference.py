"""Plain, slow restatement of the Tabupel decoder in float64 / float32 on the CPU: one function per
mechanism, whole sequences only (no cache, no state, no batch). It is the oracle of the tests and
shares no code with the package."""
import math

import torch


def rms(x, eps):
    """x over the root mean square of its last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def linear(x, w):
    return x @ w.T


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------ positions
def plain_frequencies(base, dims):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def linear_frequencies(base, dims, factor):
    return [f / factor for f in plain_frequencies(base, dims)]


def yarn_frequencies(base, dims, factor, original, fast, slow):
    """(frequencies, magnitude): fast dimensions keep their frequency, slow ones are divided by the factor."""
    def dim(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim(fast)), 0), min(math.ceil(dim(slow)), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(base, dims)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1 - r))
    return out, 0.1 * math.log(factor) + 1


def rotate(x, pos, freqs, magnitude=1.0):
    """x [T, heads, D]: dimensions 2i and 2i + 1 turn together; those past the frequencies stay."""
    n = 2 * len(freqs)
    a = pos.double()[:, None] * torch.tensor(freqs, dtype=torch.float64)
    cos, sin = ((magnitude * f(a)).to(x.dtype)[:, None] for f in (torch.cos, torch.sin))
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2], out[..., 1:n:2] = u * cos - v * sin, v * cos + u * sin
    return out


# ------------------------------------------------------------------------------ differential attention
def in_window(i, j, size):
    return 0 <= i - j < size


def softmax_attention(q, k, v, scale, size):
    """One head: q, k [T, D], v [T, V], each query over the keys of its window."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=v.dtype)
    for i in range(T):
        seen = [j for j in range(T) if in_window(i, j, size)]
        out[i] = torch.softmax(k[seen] @ q[i] * scale, -1) @ v[seen]
    return out


def difference_weight(w, diff):
    """lambda: what of the second map is taken off."""
    return torch.exp((w("lq1") * w("lk1")).sum()) - torch.exp((w("lq2") * w("lk2")).sum()) + diff


def attention(h, w, c, eps):
    T, H, G, D = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    pos, rot = torch.arange(T), c["rot"]
    freqs = linear_frequencies(rot["base"], rot["dims"], rot["scaling"]["factor"])

    def maps(n, heads):
        x = linear(h, w(n)).view(T, heads * 2, D)
        return rotate(rms(x, eps) * w(n + ".norm"), pos, freqs).view(T, heads, 2, D)
    q, k, v = maps("q", H), maps("k", G), linear(h, w("v")).view(T, G, c["vdim"])
    lam, out = difference_weight(w, c["diff"]), []
    for x in range(H):
        g = x // (H // G)
        a1, a2 = (softmax_attention(q[:, x, m], k[:, g, m], v[:, g], c["scale"], c["mask"]["size"]) for m in (0, 1))
        out.append(rms(a1 - lam * a2, eps) * (1 - c["diff"]))
    return linear(torch.cat(out, -1), w("o"))


# ------------------------------------------------------------------------------ latent attention
def latent_attention(h, w, c, eps):
    T, H, D, V, R = h.shape[0], c["heads"], c["dim"], c["vdim"], c["kv_rank"]
    pos, s = torch.arange(T), c["rot"]["scaling"]
    freqs, mag = yarn_frequencies(c["rot"]["base"], c["rot"]["dims"], s["factor"], s["original"], s["fast"], s["slow"])
    q = linear(rms(linear(h, w("dq")), eps) * w("dq.norm"), w("uq")).view(T, H, D + c["rot_dim"])
    down = linear(h, w("dkv"))
    latent = rms(down[:, :R], eps) * w("dkv.norm")
    shared = rotate(down[:, R:].view(T, 1, -1), pos, freqs, mag)[:, 0]
    turned = rotate(q[..., D:], pos, freqs, mag)
    k, v = linear(latent, w("uk")).view(T, H, D), linear(latent, w("uv")).view(T, H, V)
    gate = torch.sigmoid(linear(h, w("g")))
    out = []
    for x in range(H):
        qx, kx = torch.cat([q[:, x, :D], turned[:, x]], -1), torch.cat([k[:, x], shared], -1)
        out.append(softmax_attention(qx, kx, v[:, x], c["scale"], c["mask"]["size"]) * gate[:, x, None])
    return linear(torch.cat(out, -1), w("o"))


# ------------------------------------------------------------------------------ gated linear recurrence
def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K]: y[t] = sum_j taps[:, K - 1 - j] x[t - j] + bias, zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x) + bias
    for j in range(min(K, T)):
        y[j:] += x[: T - j] * taps[:, K - 1 - j]
    return y


def block_gate(u, w, b):
    """sigmoid(w[n] u_n + b[n]) for each of the equal parts u_n of a row; w [blocks, out, in]."""
    parts = u.view(u.shape[0], w.shape[0], -1)
    return torch.sigmoid(torch.einsum("tni,noi->tno", parts, w) + b).reshape(u.shape)


def linear_recurrence(u, r, i, lam):
    S, out = torch.zeros_like(u[0]), []
    rate = -8 * torch.log1p(torch.exp(lam))
    for t in range(u.shape[0]):
        log_a = rate * r[t]
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def rglru(h, w, c):
    y = gelu_tanh(linear(h, w("y")) + w("y.b"))
    u = causal_conv(linear(h, w("x")) + w("x.b"), w("conv"), w("conv.b"))
    r, i = (block_gate(u, w(n), w(n + ".b")) for n in ("ra", "ri"))
    return linear(linear_recurrence(u, r, i, w("lam")) * y, w("o"))


# ------------------------------------------------------------------------------ model
def gated_unit(x, w):
    return linear(silu(linear(x, w("gate"))) * linear(x, w("up")), w("down"))


def softcap(x, cap):
    return cap * torch.tanh(x / cap)


def forward(config, tensors, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence. ``trace``: a list that receives the stream after every layer."""
    t = lambda n: tensors[n].to(dtype)                               # noqa: E731
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = t("embed")[torch.tensor(tokens)]
    for l, c in enumerate(config["layers"]):
        src = c.get("weights_of")
        p = f"l{l if src is None else src}."
        norm = lambda n, y: rms(y, eps) * t(p + n)                   # noqa: E731
        w = lambda n: t(p + "mix." + n)                              # noqa: E731
        h, f = norm("norm1", x), c["mixer"]
        y = {"attention": lambda: attention(h, w, f, eps), "latent_attention": lambda: latent_attention(h, w, f, eps),
             "rglru": lambda: rglru(h, w, f)}[c["type"]]()
        x = x + m * y
        if c.get("mlp"):
            x = x + m * gated_unit(norm("norm2", x), lambda n: t(p + "mlp." + n))
        if trace is not None:
            trace.append(x)
    return softcap(linear(rms(x, eps) * t("final.norm"), t("head")), config["logit_softcap"])
