"""Plain, slow restatement of the Nufusun decoder in float64 / float32 on the CPU: one function per
mechanism, whole sequences only (no cache, no batch). It is the oracle of the tests and shares no
code with the package."""
import math

import torch


def rms_norm(x, w, eps):
    """The stored weight is an offset from one."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * (1 + w)


def linear(x, w, b=None):
    y = x @ w.T
    return y if b is None else y + b


def distance_bucket(n, num_buckets, max_distance):
    """One bucket per distance up to half the table, logarithmically spaced buckets beyond."""
    half = num_buckets // 2
    if n < half:
        return n
    steps = math.log(n / half) / math.log(max_distance / half) * (num_buckets - half)
    return min(num_buckets - 1, half + math.floor(steps + 1e-9))


def distance_bias(i, rel, max_distance):
    """[H, i + 1]: the bias of query position ``i`` towards keys 0 .. i; ``rel`` is [buckets, H]."""
    idx = [distance_bucket(i - j, rel.shape[0], max_distance) for j in range(i + 1)]
    return rel[idx].T


def head_scores(q, keys, i, rel, temp, scale, max_distance):
    """q [H, D], keys [i + 1, G, D] -> [H, i + 1] before the heads are mixed."""
    H, G = q.shape[0], keys.shape[1]
    k = keys[:, [h // (H // G) for h in range(H)]]                   # [i + 1, H, D]
    s = (q[None] * k).sum(-1).T * scale
    return s * temp[:, None] + distance_bias(i, rel, max_distance)


def mix_heads(s, talk):
    return talk @ s


def softmax_with_null(s):
    """exp(s_j) / (1 + sum exp(s_j)) over the last dimension, evaluated around max(s, 0)."""
    m = s.max(-1, keepdim=True).values.clamp(min=0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def attention(h, w, c):
    """h [T, width]; ``w(name)`` gives the mixer's tensors, ``c`` its sizes."""
    T, H, G, D, V = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = linear(h, w("q"), w("q.b")).view(T, H, D)
    k = linear(h, w("k"), w("k.b")).view(T, G, D)
    v = linear(h, w("v"), w("v.b")).view(T, G, V)
    vh = v[:, [x // (H // G) for x in range(H)]]                     # [T, H, V]
    out = []
    for i in range(T):
        s = head_scores(q[i], k[: i + 1], i, w("rel"), w("temp"), c["scale"], c["bias_max"])
        p = softmax_with_null(mix_heads(s, w("talk")))
        out.append(torch.einsum("hj,jhv->hv", p, vh[: i + 1]).reshape(-1))
    return linear(torch.stack(out), w("o"), w("o.b"))


def clamped_gated_unit(gate, up, limit):
    g = gate.clamp(max=limit)
    u = up.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def expert(x, w, e, limit):
    y = clamped_gated_unit(linear(x, w(f"e{e}.gate")), linear(x, w(f"e{e}.up")), limit)
    return linear(y, w(f"e{e}.down"))


def route(h, w_router, top):
    """-> (ids [T, top], weights [T, top]): sigmoid scores, not renormalised."""
    s = torch.sigmoid(linear(h, w_router))
    return s.topk(top, -1).indices, s.topk(top, -1).values


def router_margin(h, w_router, top):
    """[T]: distance of the router logits on the two sides of the choice (inf: all are chosen)."""
    z = linear(h, w_router).sort(-1, descending=True).values
    return z[:, top - 1] - z[:, top] if z.shape[1] > top else torch.full_like(z[:, 0], math.inf)


def experts(h, w, c):
    """The routing weight scales what goes into an expert."""
    ids, wt = route(h, w("router"), c["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(c["router"]["experts"]):
        for j in range(ids.shape[1]):
            rows = (ids[:, j] == e).nonzero().flatten()
            if rows.numel():
                out[rows] += expert(wt[rows, j, None] * h[rows], w, e, c["expert"]["limit"])
    return out


def forward(config, tensors, tokens, dtype=torch.float64, trace=None, margins=None):
    """Logits [T, vocab] of one sequence. ``trace``: a list that receives the stream after every
    layer; ``margins``: one that receives every layer's router margins."""
    t = lambda n: tensors[n].to(dtype)                               # noqa: E731
    eps = config["norm"]["eps"]
    x = t("embed")[torch.tensor(tokens)] * config["embedding"]["scale"]
    for l, c in enumerate(config["layers"]):
        h = rms_norm(x, t(f"l{l}.norm1"), eps)
        d = attention(h, lambda n: t(f"l{l}.mix.{n}"), c["mixer"])
        if c.get("mlp"):
            d = d + experts(h, lambda n: t(f"l{l}.mlp.{n}"), c["mlp"])
            if margins is not None:
                margins.append(router_margin(h, t(f"l{l}.mlp.router"), c["mlp"]["router"]["top"]))
        x = x + d
        if trace is not None:
            trace.append(x)
    return linear(rms_norm(x, t("final.norm"), eps), t("head"))
