"""Plain, slow restatement of the Diforax decoder in float64 / float32 on the CPU: one function per
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


# ------------------------------------------------------------------------------ delta mixer
def causal_conv(x, taps):
    """x [T, C], taps [C, K]: y[t] = sum_j taps[:, K - 1 - j] x[t - j], zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(K):
        y[j:] += x[: T - j] * taps[:, K - 1 - j] if j < T else 0
    return y


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def decay(a, A_log, dt_bias):
    return torch.exp(-torch.exp(A_log) * torch.log1p(torch.exp(a + dt_bias)))


def delta_step(S, q, k, v, g, beta):
    """One head, one token: S [D, V] -> (S, o)."""
    S = g * S
    u = beta * (v - k @ S)
    S = S + torch.outer(k, u)
    return S, q @ S


def delta(h, w, c, eps):
    T, H, G, D, V = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(causal_conv(linear(h, w(n)), w(n + ".conv"))) for n in ("q", "k", "v"))
    q = unit(q.view(T, G, D)) / math.sqrt(D)
    k, v = unit(k.view(T, G, D)), v.view(T, H, V)
    beta = torch.sigmoid(linear(h, w("b")))
    g = decay(linear(h, w("a")), w("A_log"), w("dt_bias"))
    o = torch.zeros(T, H, V, dtype=h.dtype)
    for x in range(H):
        S = torch.zeros(D, V, dtype=h.dtype)
        kv = x // (H // G)
        for t in range(T):
            S, o[t, x] = delta_step(S, q[t, kv], k[t, kv], v[t, x], g[t, x], beta[t, x])
    y = rms(o, eps) * w("norm") * silu(linear(h, w("g"))).view(T, H, V)
    return linear(y.reshape(T, H * V), w("o"))


# ------------------------------------------------------------------------------ attention mixer
def rotate(x, pos, base, dims):
    """x [T, heads, D]; dimension i < dims / 2 is paired with dimension i + dims / 2."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = pos.double()[:, None] * f
    cos, sin = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def same_chunk(i, j, size):
    return i // size == j // size


def keys_values(h, w, c, eps):
    T, G = h.shape[0], c["kv_heads"]
    k = linear(h, w("k")).view(T, G, c["dim"])
    k = rms(rotate(k, torch.arange(T), c["rot"]["base"], c["rot"]["dims"]), eps)
    return k, linear(h, w("v")).view(T, G, c["vdim"])


def attention(h, w, c, eps, kv):
    """``kv``: the keys (rotated, normalised) and values of this layer or of the one it reads."""
    T, H, G = h.shape[0], c["heads"], c["kv_heads"]
    q = rms(rotate(linear(h, w("q")).view(T, H, c["dim"]), torch.arange(T), c["rot"]["base"], c["rot"]["dims"]), eps)
    k, v = kv
    out = torch.zeros(T, H, c["vdim"], dtype=h.dtype)
    for i in range(T):
        seen = [j for j in range(i + 1) if same_chunk(i, j, c["mask"]["size"])]
        for x in range(H):
            g = x // (H // G)
            p = torch.softmax(k[seen, g] @ q[i, x] * c["scale"], -1)
            out[i, x] = p @ v[seen, g]
    return linear(out.reshape(T, -1), w("o"))


# ------------------------------------------------------------------------------ feed-forwards
def gated_unit(x, w, prefix, act):
    return linear(act(linear(x, w(prefix + "gate"))) * linear(x, w(prefix + "up")), w(prefix + "down"))


def choice_scores(h, w):
    """(scores s, scores of the choice) [T, all experts]."""
    s = torch.softmax(linear(h, w("router")), -1)
    return s, s + w("correction")


def keep_groups(choice, count, keep):
    """Minus infinity outside the ``keep`` groups whose largest entry is largest."""
    T, n = choice.shape
    best = choice.view(T, count, n // count).max(-1).values
    out = torch.full_like(choice, -math.inf)
    for t in range(T):
        for g in best[t].topk(keep).indices.tolist():
            lo = g * (n // count)
            out[t, lo: lo + n // count] = choice[t, lo: lo + n // count]
    return out


def experts(h, w, c, margins=None):
    r = c["router"]
    s, choice = choice_scores(h, w)
    eligible = keep_groups(choice, r["groups"]["count"], r["groups"]["keep"])
    if margins is not None:
        margins.append(choice_margin(choice, eligible, r))
    out = torch.zeros_like(h)
    for t, ids in enumerate(eligible.topk(r["top"], -1).indices.tolist()):
        for e in ids:
            y = h[t] if e >= r["experts"] else gated_unit(h[t], w, f"e{e}.", silu)
            out[t] += s[t, e] * y
    return out


def choice_margin(choice, eligible, r):
    """[T]: how far the choice is from another one (the lesser of the groups' and the experts' gap)."""
    T, n = choice.shape
    count, keep = r["groups"]["count"], r["groups"]["keep"]
    e = eligible.sort(-1, descending=True).values
    m = e[:, r["top"] - 1] - e[:, r["top"]] if n > r["top"] else torch.full((T,), math.inf, dtype=choice.dtype)
    if keep < count:
        b = choice.view(T, count, n // count).max(-1).values.sort(-1, descending=True).values
        m = torch.minimum(m, b[:, keep - 1] - b[:, keep])
    return m


# ------------------------------------------------------------------------------ model
def forward(config, tensors, tokens, dtype=torch.float64, trace=None, margins=None):
    """Logits [T, vocab] of one sequence. ``trace``: a list that receives the stream after every
    layer; ``margins``: one that receives every layer's router margins."""
    t = lambda n: tensors[n].to(dtype)                               # noqa: E731
    eps = config["norm"]["eps"]
    x = t("embed")[torch.tensor(tokens)]
    kept = {}
    for l, c in enumerate(config["layers"]):
        mixer, w = c["mixer"], lambda n: t(f"l{l}.mix.{n}")          # noqa: E731
        norm = lambda n, y: rms(y, eps) * t(f"l{l}.{n}")             # noqa: E731
        h = norm("norm1", x)
        if c["type"] == "delta":
            y = delta(h, w, mixer, eps)
        else:
            j = mixer.get("kv_from")
            kept[l] = keys_values(h, w, mixer, eps) if j is None else kept[j]
            y = attention(h, w, mixer, eps, kept[l])
        x = x + norm("norm1b", y)
        if c.get("mlp"):
            h, w = norm("norm2", x), lambda n: t(f"l{l}.mlp.{n}")    # noqa: E731
            y = gated_unit(h, w, "", gelu_tanh) if c["mlp"]["kind"] == "dense" else experts(h, w, c["mlp"], margins)
            x = x + norm("norm2b", y)
        if trace is not None:
            trace.append(x)
    return linear(rms(x, eps) * t("final.norm"), t("head"))
