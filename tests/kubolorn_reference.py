"""Plain, slow restatement of the Kubolorn decoder in float64 / float32 on the CPU: one function per
mechanism, whole sequences only (no cache, no state, no batch). It is the oracle of the tests and
shares no code with the package."""
import math

import torch


def linear(x, w):
    return x @ w.T


def rms(x, eps):
    """x over the root mean square of its last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def part_rms(x, parts, eps):
    """Each of the equal consecutive parts of the last dimension over its own root mean square."""
    return rms(x.reshape(*x.shape[:-1], parts, -1), eps).reshape(x.shape)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def log_sigmoid(x):
    return -softplus(-x)


def causal_conv(x, taps, bias=None):
    """x [T, C], taps [C, K]: y[t] = sum_j taps[:, K - 1 - j] x[t - j] (+ bias), zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(min(K, T)):
        y[j:] += x[: T - j] * taps[:, K - 1 - j]
    return y if bias is None else y + bias


# ------------------------------------------------------------------------------ embedding
def bigram_rows(tokens, c):
    """Row of the pair (token before, token) of every place; the last row where there is none before."""
    rows = [c["buckets"]]
    for before, cur in zip(tokens, tokens[1:]):
        rows.append((before * c["mul_prev"] + cur * c["mul_cur"]) % c["buckets"])
    return rows[: len(tokens)]


# ------------------------------------------------------------------------------ positions
def frequencies(base, dims):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(base, dims, factor, original, fast, slow):
    """(frequencies, magnitude): fast dimensions keep their frequency, slow ones are divided by the factor."""
    def dim(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim(fast)), 0), min(math.ceil(dim(slow)), dims - 1)
    out = []
    for i, f in enumerate(frequencies(base, dims)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1 - r))
    return out, 0.1 * math.log(factor) + 1


def rotate(x, pos, freqs, magnitude=1.0):
    """x [T, heads, D]: dimensions i and i + len(freqs) turn together; those past them stay."""
    n = len(freqs)
    a = pos.double()[:, None] * torch.tensor(freqs, dtype=torch.float64)
    cos, sin = ((magnitude * f(a)).to(x.dtype)[:, None] for f in (torch.cos, torch.sin))
    u, v = x[..., :n], x[..., n: 2 * n]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * n:]], -1)


# ------------------------------------------------------------------------------ attention
def sink_attention(q, k, v, scale, sink):
    """One head, causal: q, k [T, D], v [T, V]; exp(sink) joins the softmax's denominator."""
    out = torch.zeros(q.shape[0], v.shape[1], dtype=v.dtype)
    for i in range(q.shape[0]):
        s = torch.cat([k[: i + 1] @ q[i] * scale, sink.reshape(1)])
        out[i] = torch.softmax(s, 0)[:-1] @ v[: i + 1]
    return out


def attention(h, w, c):
    """Values are the keys before their rotation."""
    T, H, G, D, rot = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c.get("rot") or {"dims": 0}
    q, k = linear(h, w("q")).view(T, H, D), linear(h, w("k")).view(T, G, D)
    v, pos = k, torch.arange(T)
    if rot["dims"]:
        s = rot.get("scaling")
        freqs, mag = (frequencies(rot["base"], rot["dims"]), 1.0) if s is None else \
            yarn_frequencies(rot["base"], rot["dims"], s["factor"], s["original"], s["fast"], s["slow"])
        q, k = rotate(q, pos, freqs, mag), rotate(k, pos, freqs, mag)
    out = [sink_attention(q[:, x], k[:, x // (H // G)], v[:, x // (H // G)], c["scale"], w("sink")[x]) for x in range(H)]
    return linear(torch.cat(out, -1), w("o"))


# ------------------------------------------------------------------------------ recurrences
def outer_recurrence(q, k, v, log_decay):
    """S_t = e^g_t S_{t-1} + k_t v_t^T (g per key channel), o_t = S_t^T q_t; one head, [T, D] and [T, V]."""
    S, out = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype), []
    for t in range(k.shape[0]):
        S = torch.exp(log_decay[t])[:, None] * S + k[t][:, None] * v[t][None]
        out.append(q[t] @ S)
    return torch.stack(out)


def gated_linear_attention(h, w, c, eps):
    T, H, D, V = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q, k = (linear(h, w(n)).view(T, H, D) for n in "qk")
    v, gate = linear(h, w("v")).view(T, H, V), linear(h, w("g"))
    g = (log_sigmoid(linear(linear(h, w("a1")), w("a2")) + w("a2.b")) / c["tau"]).view(T, H, D)
    o = [rms(outer_recurrence(q[:, x] * D ** -0.5, k[:, x], v[:, x], g[:, x]), eps) * w("norm") for x in range(H)]
    return linear(torch.cat(o, -1) * silu(gate), w("o"))


def state_space(h, w, c, eps):
    T, H, V, N, G = h.shape[0], c["heads"], c["vdim"], c["state"], c["groups"]
    inner = H * V
    z, u, dt = torch.split(linear(h, w("in")), [inner, inner + 2 * G * N, H], -1)
    u = silu(causal_conv(u, w("conv"), w("conv.b")))
    x, B, C = u[:, :inner].view(T, H, V), u[:, inner: inner + G * N].view(T, G, N), u[:, inner + G * N:].view(T, G, N)
    dt = softplus(dt + w("dt_bias"))
    y = []
    for i in range(H):
        g, d = i // (H // G), dt[:, i, None]
        decay = (-torch.exp(w("A_log")[i]) * d).expand(T, N)
        y.append(outer_recurrence(C[:, g], B[:, g], d * x[:, i], decay) + w("D")[i] * x[:, i])
    return linear(part_rms(torch.cat(y, -1) * silu(z), c["norm_groups"], eps) * w("norm"), w("o"))


def side_by_side(h, w, c, eps):
    left, right = attention(h, lambda n: w("left." + n), c["left"]), state_space(h, lambda n: w("right." + n), c["right"], eps)
    return c["left_scale"] * left + c["right_scale"] * right


# ------------------------------------------------------------------------------ feed-forward
def dense(x, w):
    return linear(gelu_tanh(linear(x, w("up"))), w("down"))


def experts(x, w, c):
    z, top = linear(x, w("router")), c["router"]["top"]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        best = torch.argsort(z[t], descending=True, stable=True)[:top]
        for e, p in zip(best.tolist(), torch.softmax(z[t][best], 0)):
            a = torch.relu(linear(x[t], w(f"e{e}.up"))) ** 2
            out[t] += p * linear(a, w(f"e{e}.down"))
    return out


# ------------------------------------------------------------------------------ model
def layer_order(n, loop):
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(config, tensors, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence. ``trace``: a list that receives the stream after every layer run."""
    t = lambda n: tensors[n].to(dtype)                               # noqa: E731
    eps, parts, e = config["norm"]["eps"], config["norm"]["groups"], config["embedding"]
    norm = lambda x, n: part_rms(x, parts, eps) * t(n)               # noqa: E731
    x = t("embed")[torch.tensor(tokens)] * e["scale"]
    if e.get("bigram"):
        x = x + t("bigram")[torch.tensor(bigram_rows(tokens, e["bigram"]))]
    x = norm(x, "embed.norm")
    for l in layer_order(len(config["layers"]), config.get("loop")):
        c, p = config["layers"][l], f"l{l}."
        w = lambda n: t(p + "mix." + n)                              # noqa: E731

        def read(i):
            h = norm(x, f"{p}norm{i}")
            return h + causal_conv(h, t(f"{p}canon{i}"))
        h = read(1)
        y = gated_linear_attention(h, w, c["mixer"], eps) if c["type"] == "gla" else side_by_side(h, w, c["mixer"], eps)
        if c.get("mlp"):
            f = lambda n: t(p + "mlp." + n)                          # noqa: E731
            y = y + (dense(read(2), f) if c["mlp"]["kind"] == "dense" else experts(read(2), f, c["mlp"]))
        x = x + y
        if trace is not None:
            trace.append(x)
    return linear(norm(x, "final.norm"), t("embed"))
