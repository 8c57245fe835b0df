"""Recurrences over outer products (chunks on the tensor cores, segments side by side, token by token) against the plain
implementation, over portions, decode rows and unequal requests with reused slots."""
from types import SimpleNamespace

import pytest
import torch

import kubolorn_reference as R
from vllm_cpp_b200.ops import outer as O
from vllm_cpp_b200.ops.reference import build_prefill_tiles

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
# kind, states, key heads, key size, value size, rank or normed parts
CHANNEL = [("channel", 3, 3, 32, 64, 12), ("channel", 2, 2, 128, 128, 16), ("channel", 1, 1, 10, 7, 3), ("channel", 2, 2, 80, 96, 40),
           ("channel", 1, 1, 256, 80, 16), ("channel", 1, 1, 300, 48, 20)]
HEAD = [("head", 4, 2, 128, 64, 2), ("head", 6, 3, 32, 16, 4), ("head", 3, 1, 5, 6, 9), ("head", 2, 1, 256, 96, 1), ("head", 2, 2, 72, 128, 8),
        ("head", 1, 1, 290, 20, 1)]
TOL = {BF: 1e-2, F32: 3e-5}
EPS = 1e-5


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """(the plain implementations work on small tensors)"""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def make(shape, T, seed=0, dtype=F32, fade=0.0):
    """Random inputs and weights, fp32 on the CPU. ``fade``: mean of the decay's logits."""
    kind, H, G, D, V, x = shape
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, m=1.0, a=0.0: (torch.randn(*s, generator=g) * m + a).to(dtype).float()      # noqa: E731
    d = {"q": r(T, G * D), "k": r(T, G * D), "v": r(T, H * V), "gate": r(T, H * V)}
    if kind == "channel":
        d["a1"], w = r(T, x), {"a2": r(H * D, x, m=1.5 * x ** -0.5), "bias": r(H * D, m=0.7, a=fade), "norm": r(V, m=0.3, a=1.0)}
    else:
        d["dt"], w = r(T, H), {"bias": r(H, m=0.5, a=-1.0 - fade), "A": torch.exp(r(H, m=0.6)), "D": r(H), "norm": r(H * V, m=0.2, a=1.0)}
    return d, w


TAU = 4.0


def plain(shape, d, w, tau=TAU):
    """Whole sequence in float64 -> (o before norm and gate [T, H * V], out)."""
    kind, H, G, D, V, x = shape
    f = {n: t.double() for n, t in d.items()}
    w = {n: t.double() for n, t in w.items()}
    T = f["q"].shape[0]
    q, k, v = f["q"].view(T, G, D), f["k"].view(T, G, D), f["v"].view(T, H, V)
    if kind == "channel":
        lg = (R.log_sigmoid(f["a1"] @ w["a2"].T + w["bias"]) / tau).view(T, H, D)
        o = torch.stack([R.outer_recurrence(q[:, h] * D ** -0.5, k[:, h], v[:, h], lg[:, h]) for h in range(H)], 1)
        return o.flatten(1), (R.rms(o, EPS) * w["norm"]).flatten(1) * R.silu(f["gate"])
    dt = R.softplus(f["dt"] + w["bias"])
    o = torch.stack([R.outer_recurrence(q[:, h // (H // G)], k[:, h // (H // G)], dt[:, h, None] * v[:, h],
                                        (-w["A"][h] * dt[:, h, None]).expand(T, D)) for h in range(H)], 1)
    y = (o + w["D"][:, None] * v).flatten(1) * R.silu(f["gate"])
    return o.flatten(1), 1.3 * R.part_rms(y, x, EPS) * w["norm"]


class Engine:
    """Steps of (slot, rows already seen, inputs) items over shared state, as the model runner lays them out."""

    def __init__(self, shape, w, dtype, slots, tau=TAU, **how):
        kind, H, G, D, V, x = shape
        self.shape, self.dtype, self.how, self.tau = shape, dtype, how, tau
        self.s = s = O.OuterShape(H=H, G=G, dim=D, vdim=V, rank=(x + 15) // 16 * 16 if kind == "channel" else 0)
        f32 = lambda t: t.to(F32).to(DEV).contiguous()                             # noqa: E731
        if kind == "channel":
            a2 = torch.zeros(H, s.D, s.rank)
            a2[:, :D, :x] = w["a2"].view(H, D, x)
            self.w = {"a2": a2.view(H * s.D, s.rank).to(dtype).to(DEV), "a2_bias": f32(self.spread(w["bias"], H, D, s.D)),
                      "norm": f32(self.spread(w["norm"], 1, V, s.V))}
        else:
            self.w = {"dt_bias": f32(w["bias"]), "A": f32(w["A"]), "D": f32(w["D"]), "norm": f32(self.spread(w["norm"], H, V, s.V))}
        # what a freed slot leaves behind must not be seen
        self.state = torch.full((slots, H, s.D, s.V), 3.0, device=DEV)

    @staticmethod
    def spread(t, heads, size, padded):
        out = torch.zeros(*t.shape[:-1], heads, padded, dtype=t.dtype)
        out[..., :size] = t.reshape(*t.shape[:-1], heads, size)
        return out.flatten(-2)

    def step(self, items):
        """-> (items in the order they ran, their (o, out) [n, H * V])."""
        (kind, H, G, D, V, x), s, dtype = self.shape, self.s, self.dtype
        size = lambda i: i[2]["q"].shape[0]                                        # noqa: E731
        items = [i for i in items if size(i) == 1] + [i for i in items if size(i) > 1]
        n = [size(i) for i in items]
        nd, pre = sum(m == 1 for m in n), [m for m in n if m > 1]
        T = sum(n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)             # noqa: E731
        tr, tq = build_prefill_tiles(pre) if pre else ([], [])
        ctx = SimpleNamespace(num_decodes=nd, num_prefills=len(pre), num_tiles=len(tr), seq_lens=i32([i[1] + m for i, m in zip(items, n)]),
                              state_slots=i32([i[0] for i in items]), prefill_q_start=i32([sum(pre[:i]) for i in range(len(pre) + 1)]),
                              tile_req=i32(tr or [0]), tile_q0=i32(tq or [0]))
        cat = lambda name: torch.cat([i[2][name] for i in items])                  # noqa: E731
        q, k, v, gate = (self.spread(cat(a), h, z, p) for a, h, z, p in (("q", G, D, s.D), ("k", G, D, s.D), ("v", H, V, s.V),
                                                                         ("gate", H, V, s.V)))
        nan = float("nan")
        out = torch.full((T, s.inner), nan, dtype=dtype, device=DEV)
        work = O.Workspace(DEV, T, len(items))
        work.segments = 2 * (len(tr) + 2)                                          # (tests cut portions finer than the model does)
        work.reserve(s, O.CHANNEL if kind == "channel" else O.HEAD)
        bufs = {"o": torch.full((T, s.inner), nan, device=DEV), **{k: t.fill_(nan) for k, t in work.allocate().items()}}
        if kind == "channel":
            a1 = self.spread(cat("a1"), 1, x, s.rank)
            row = torch.cat([q, k, v, gate, a1], 1).to(dtype).to(DEV)
            parts = torch.split(row, [s.H * s.D, s.H * s.D, s.inner, s.inner, s.rank], 1)
            O.gated_linear_attention(*parts, self.w, s, self.state, ctx, bufs, out, tau=self.tau, eps=EPS, **self.how)
        else:
            u, z, dt = (t.to(dtype).to(DEV) for t in (torch.cat([v, k, q], 1), gate, cat("dt")))
            O.state_space(u, z, dt, self.w, s, self.state, ctx, bufs, out, parts=x, eps=EPS, scale=1.3, **self.how)
        got = []
        assert not out.view(T, H, s.V)[..., V:].any()                              # (padding)
        for t in (bufs["o"], out):
            t = t.float().cpu().view(T, H, s.V)
            got.append(t[..., :V].reshape(T, -1).split(n))
        return items, list(zip(*got))


def rows(d, a, b):
    return {n: t[a:b] for n, t in d.items()}


def run(shape, d, w, dtype, cuts, **kw):
    e, at, got = Engine(shape, w, dtype, 3, **kw), 0, []
    for n in cuts:
        got.append(e.step([(1, at, rows(d, at, at + n))])[1][0])
        at += n
    assert at == d["q"].shape[0]
    return [torch.cat(x) for x in zip(*got)]


def worst(got, want):
    """Largest error of a row against its size (or the rows' typical size, if that is larger)."""
    size = want.norm(dim=-1)
    return ((got.double() - want).norm(dim=-1) / size.clamp_min(size.mean())).max().item()


def check(got, want, dtype, shape, chunks=True, note=None):
    n, H = want[0].shape[0], shape[1]
    size = want[0].view(n, H, -1).norm(dim=-1)
    # (a head whose query and key are almost orthogonal is divided by next to nothing)
    firm = (size > 0.03 * size.mean()).all(1) if shape[0] == "channel" else torch.ones(n, dtype=torch.bool)
    assert firm.sum() >= 0.8 * n - 1
    if firm.any():
        assert worst(got[1][firm], want[1][firm]) < TOL[dtype], note
    if chunks and (shape[0] == "head" or dtype == BF and shape[3] <= 256):         # o in fp32, before it is normed
        assert worst(got[0], want[0]) < 3e-5, note


@pytest.mark.parametrize("shape", CHANNEL + HEAD)
@pytest.mark.parametrize("dtype", [F32, BF])
def test_whole_and_portions(shape, dtype):
    T = 300
    d, w = make(shape, T, seed=1, dtype=dtype, fade=1.0)
    want = plain(shape, d, w)
    for cuts in ([T], [1] * 5 + [T - 5], [2, 3, 60, T - 65], [64, 1, 1, T - 66], [129, T - 130, 1], [2] * 150):
        check(run(shape, d, w, dtype, cuts), want, dtype, shape, chunks=1 not in cuts, note=cuts)


@pytest.mark.parametrize("shape", CHANNEL + HEAD)
def test_chunks_equal_token_by_token(shape):
    d, w = make(shape, 200, seed=2, dtype=BF, fade=2.0)
    a = run(shape, d, w, BF, [70, 130])
    b = run(shape, d, w, BF, [70, 130], token_by_token=True)
    want = plain(shape, d, w)
    check(a, want, BF, shape)
    check(b, want, BF, shape, chunks=False)


@pytest.mark.parametrize("shape", [CHANNEL[0], CHANNEL[1], CHANNEL[4], HEAD[0], HEAD[3]])
@pytest.mark.parametrize("seg_tiles", [1, 2])
def test_segments_side_by_side(shape, seg_tiles):
    """A long portion cut into segments, with a state from before and one to go on from, beside short ones."""
    d, w = make(shape, 1100, seed=3, dtype=BF, fade=4.0)
    want = plain(shape, d, w)
    check(run(shape, d, w, BF, [1100], seg_tiles=seg_tiles), want, BF, shape)
    check(run(shape, d, w, BF, [100, 700, 300], seg_tiles=seg_tiles), want, BF, shape)
    e = Engine(shape, w, BF, 4, seg_tiles=seg_tiles)
    first = {}
    for lens in ({0: 130, 1: 513, 2: 64, 3: 1}, {0: 700, 1: 2, 2: 1, 3: 800}):
        items, got = e.step([(s, first.get(s, 0), rows(d, first.get(s, 0), first.get(s, 0) + n)) for s, n in lens.items()])
        for (s, at, x), g in zip(items, got):
            n = x["q"].shape[0]
            check(g, [y[at:at + n] for y in want], BF, shape, chunks=n > 1, note=(s, at))
            first[s] = at + n


@pytest.mark.parametrize("tau,fade", [(0.02, 1.0), (0.2, 1.0), (1.0, -12.0), (0.01, 5.0)])
@pytest.mark.parametrize("shape", CHANNEL[:2] + CHANNEL[4:5])
def test_channels_that_fade_fast(shape, tau, fade):
    """Decays beyond what a chunk, or 16 tokens, or one token can hold as factors."""
    d, w = make(shape, 150, seed=4, dtype=BF, fade=fade)
    d["a1"][::7] *= 0.05                               # (some tokens fade little beside others that fade much)
    d["a1"] = d["a1"].to(BF).float()
    want = plain(shape, d, w, tau)
    got = run(shape, d, w, BF, [150], tau=tau)
    assert torch.isfinite(got[1]).all()
    check(got, want, BF, shape, note=(tau, fade))


@pytest.mark.parametrize("shape", [CHANNEL[1], HEAD[0]])
def test_slow_decays_over_many_tokens(shape):
    """A state that hardly fades: the first tokens are still there after two thousand."""
    d, w = make(shape, 2000, seed=5, dtype=BF, fade=8.0)
    want = plain(shape, d, w)
    for cuts in ([2000], [700, 1, 1299]):
        got = run(shape, d, w, BF, cuts)
        check(got, want, BF, shape, chunks=cuts == [2000], note=cuts)


@pytest.mark.parametrize("shape", CHANNEL[:3] + HEAD[:3])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_batches_and_slots(shape, dtype):
    """Portions beside decode rows, slots freed and used again; each request as if it were alone."""
    e = Engine(shape, make(shape, 1, seed=6, dtype=dtype)[1], dtype, 3)
    w = make(shape, 1, seed=6, dtype=dtype)[1]
    for turn in range(3):
        lens = {0: 90 - turn, 1: 70, 2: 33}
        data = {s: make(shape, n, seed=10 * turn + s, dtype=dtype)[0] for s, n in lens.items()}
        want = {s: plain(shape, x, w) for s, x in data.items()}
        at = dict.fromkeys(lens, 0)
        for sizes in ({0: 1, 1: 65, 2: 2}, {0: 64, 2: 1}, {0: 1, 1: 1, 2: 30}, {0: 24 - turn, 1: 4}):
            items, got = e.step([(s, at[s], rows(data[s], at[s], at[s] + n)) for s, n in sizes.items()])
            for (s, a, x), g in zip(items, got):
                n = x["q"].shape[0]
                check(g, [y[a:a + n] for y in want[s]], dtype, shape, chunks=False, note=(turn, s, a))
                at[s] = a + n


def test_padding_rows_are_finite():
    shape = HEAD[0]
    d, w = make(shape, 1, dtype=BF)
    e = Engine(shape, w, BF, 2)
    before = e.state.clone()
    _, got = e.step([(-1, 0, d)])
    assert torch.isfinite(got[0][1]).all() and torch.equal(e.state, before)


def test_wrong_sizes_are_refused():
    s = O.OuterShape(H=2, G=2, dim=32, vdim=32, rank=8)                # (a rank that is no multiple of 16)
    x = torch.zeros(1, 64, dtype=BF, device=DEV)
    i = torch.zeros(2, dtype=torch.int32, device=DEV)
    ctx = SimpleNamespace(num_decodes=1, num_prefills=0, num_tiles=0, seq_lens=i + 1, state_slots=i, prefill_q_start=i, tile_req=i, tile_q0=i)
    w = {"a2": torch.zeros(64, 8, dtype=BF, device=DEV), "a2_bias": torch.zeros(64, device=DEV), "norm": torch.zeros(32, device=DEV)}
    with pytest.raises(Exception):
        O.gated_linear_attention(x, x, x, x, x[:, :8], w, s, torch.zeros(1, 2, 32, 32, device=DEV), ctx,
                                 {"o": torch.zeros(1, 64, device=DEV)}, torch.zeros_like(x), tau=1.0, eps=EPS)
