"""The short convolution and the gated linear recurrence (tensor-core and any-size forms) against the plain
implementation, over portions, decode rows and unequal requests with reused slots."""
from types import SimpleNamespace

import pytest
import torch

import tabupel_reference as R
from vllm_cpp_b200.ops import rglru as G
from vllm_cpp_b200.ops.reference import build_prefill_tiles

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
# blocks, channels of one, taps: blocks below, at and above one 128-row product, and beyond the tensor-core form
SHAPES = [(3, 64, 4), (5, 16, 3), (3, 21, 2), (1, 130, 1), (2, 256, 4), (1, 1, 6), (4, 128, 4), (1, 300, 4)]
TOL = {BF: 1.5e-2, F32: 2e-5}


def make(blocks, size, taps, T, seed=0, dtype=F32, rate=-4.0):
    """Random inputs x (of the convolution), y and weights, fp32 on the CPU."""
    g = torch.Generator().manual_seed(seed)
    C = blocks * size
    r = lambda *s, m=1.0, a=0.0: (torch.randn(*s, generator=g) * m + a).to(dtype).float()      # noqa: E731
    w = {"conv": r(C, taps, m=0.6), "conv.b": r(C, m=0.3), "ra": r(blocks, size, size, m=1.5 * size ** -0.5), "ra.b": r(C, m=0.5),
         "ri": r(blocks, size, size, m=1.5 * size ** -0.5), "ri.b": r(C, m=0.5), "lam": r(C, m=0.7, a=rate)}
    return G.RglruShape(blocks=blocks, size=size, taps=taps), r(T, C), r(T, C), w


def plain(s, x, y, w, dtype):
    """Whole sequence in float64 -> out [T, C] (the convolution's result rounded as the kernels store it)."""
    f = torch.float64
    u = R.causal_conv(x.to(f), w["conv"].to(f), w["conv.b"].to(f)).to(dtype).to(f)
    r, i = (R.block_gate(u, w[n].to(f), w[n + ".b"].to(f).view(s.blocks, s.size)) for n in ("ra", "ri"))
    return R.linear_recurrence(u, r, i, w["lam"].to(f)) * R.gelu_tanh(y.to(f))


class Engine:
    """Steps of (slot, rows already seen, x, y) items over shared state, as the model runner lays them out."""

    def __init__(self, s, w, dtype, slots, any_size=False):
        self.s, self.dtype, self.any = s, dtype, any_size
        f32 = lambda t: t.to(F32).to(DEV).contiguous()                             # noqa: E731
        self.w = {"conv": f32(self.spread(w["conv"].t())), "bias": f32(self.spread(w["conv.b"])),
                  "gate_bias": f32(torch.stack([self.spread(w[n + ".b"]) for n in ("ra", "ri")])),
                  "rate": f32(self.spread(-8 * torch.nn.functional.softplus(w["lam"].double(), threshold=1e9)))}
        gates = torch.zeros(s.blocks, 2, s.M, s.B)
        gates[:, 0, : s.size, : s.size], gates[:, 1, : s.size, : s.size] = w["ra"], w["ri"]
        self.w["gates"] = gates.to(dtype).to(DEV)
        # what a freed slot leaves behind must not be seen
        self.conv = torch.full((slots, s.taps - 1, s.C), 7.0, dtype=dtype, device=DEV)
        self.state = torch.full((slots, s.C), 3.0, device=DEV)

    def spread(self, t):
        """Channels (last dimension) to padded blocks."""
        out = torch.zeros(*t.shape[:-1], self.s.blocks, self.s.B, dtype=t.dtype)
        out[..., : self.s.size] = t.reshape(*t.shape[:-1], self.s.blocks, self.s.size)
        return out.flatten(-2)

    def step(self, items):
        """-> (items in the order they ran, their outputs [n, C])."""
        s, dtype = self.s, self.dtype
        items = [i for i in items if i[2].shape[0] == 1] + [i for i in items if i[2].shape[0] > 1]
        n = [i[2].shape[0] for i in items]
        nd, pre = sum(x == 1 for x in n), [x for x in n if x > 1]
        T = sum(n)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)             # noqa: E731
        tr, tq = build_prefill_tiles(pre) if pre else ([], [])
        ctx = SimpleNamespace(num_decodes=nd, num_prefills=len(pre), num_tiles=len(tr), seq_lens=i32([i[1] + m for i, m in zip(items, n)]),
                              state_slots=i32([i[0] for i in items]), prefill_q_start=i32([sum(pre[:i]) for i in range(len(pre) + 1)]),
                              tile_req=i32(tr or [0]), tile_q0=i32(tq or [0]))
        proj = torch.cat([self.spread(torch.cat([i[j] for i in items])) for j in (3, 2)], 1).to(dtype).to(DEV)     # [y | x]
        nan = float("nan")
        u, out = (torch.full((T, s.C), nan, dtype=dtype, device=DEV) for _ in range(2))
        bufs = {"summary": torch.full((G.summary_values(s),), nan, device=DEV)} if not self.any and G.tensor_core_size(s) and dtype == BF \
            else {k: torch.full((T, s.C), nan, device=DEV) for k in "ab"}
        G.short_conv(proj[:, s.C:], self.w["conv"], self.w["bias"], self.conv, ctx, u)
        G.rglru(u, proj[:, : s.C], self.w, s, self.state, ctx, bufs, out, any_size=self.any)
        o = out.float().cpu().view(T, s.blocks, s.B)
        assert not o[..., s.size:].any()
        return items, o[..., : s.size].reshape(T, -1).split(n)


def run(s, x, y, w, dtype, cuts, **kw):
    e, at, got = Engine(s, w, dtype, 3, **kw), 0, []
    for n in cuts:
        got.append(e.step([(1, at, x[at:at + n], y[at:at + n])])[1][0])
        at += n
    assert at == x.shape[0]
    return torch.cat(got)


def err(got, want):
    return ((got.double() - want).norm() / want.norm()).item()


def worst(got, want):
    """Largest error of a row against its size (or the rows' typical size, if that is larger)."""
    size = want.norm(dim=-1)
    return ((got.double() - want).norm(dim=-1) / size.clamp_min(size.mean())).max().item()


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF])
def test_whole_and_portions(shape, dtype):
    T = 300
    s, x, y, w = make(*shape, T, seed=1, dtype=dtype)
    want = plain(s, x, y, w, dtype)
    for cuts in ([T], [1] * 5 + [T - 5], [2, 3, 60, T - 65], [64, 1, 1, T - 66], [129, T - 130, 1], [2] * 150):
        assert worst(run(s, x, y, w, dtype, cuts), want) < TOL[dtype], cuts


@pytest.mark.parametrize("shape", [(3, 64, 4), (2, 256, 4), (3, 100, 4)])
@pytest.mark.parametrize("T", [3000, 64, 65, 128, 129])
def test_long_prompts_run_in_slices(shape, T):
    """A portion over many slices of rows and one that follows it in the same step."""
    s, x, y, w = make(*shape, T + 200, seed=2, dtype=BF, rate=-6.0)
    a, b = (Engine(s, w, BF, 3, any_size=v) for v in (False, True))
    for parts in ([(0, 0, 0, T), (2, 0, T, T + 200)], [(0, T, T, T + 130), (2, 200, 0, 40), (1, 0, 50, 200)]):
        items = [(slot, at, x[lo:hi], y[lo:hi]) for slot, at, lo, hi in parts]
        for o, o2 in zip(a.step(items)[1], b.step(items)[1]):
            assert worst(o, o2.double()) < 6e-3             # (two roundings of the output)
        assert ((a.state - b.state).norm(dim=-1) / b.state.norm(dim=-1)).max() < 1e-4
        assert torch.equal(a.conv, b.conv)


@pytest.mark.parametrize("rate", [-9.0, 1.5])
def test_slow_and_fast_decays(rate):
    """States that keep almost everything for the whole prompt, and ones that forget within a token."""
    s, x, y, w = make(2, 48, 4, 700, seed=3, rate=rate)
    assert worst(run(s, x, y, w, F32, [699, 1]), plain(s, x, y, w, F32)) < 3e-5
    s, x, y, w = make(2, 48, 4, 700, seed=3, dtype=BF, rate=rate)
    assert worst(run(s, x, y, w, BF, [130, 570]), plain(s, x, y, w, BF)) < TOL[BF]


def test_an_early_token_is_read_far_away():
    """Decays near one: what one token wrote shows hundreds of positions later, in prompts and in decoding."""
    s, x, y, w = make(1, 32, 4, 600, seed=4, rate=-11.0)
    x, w["conv.b"] = x * 0.05, torch.zeros(32)
    x[7] = 20.0
    want, other = plain(s, x, y, w, F32), x.clone()
    other[7] = 0.0
    assert err(plain(s, other, y, w, F32)[[599]], want[[599]]) > 0.3
    for cuts in ([600], [590] + [1] * 10, [100] * 6):
        assert err(run(s, x, y, w, F32, cuts)[[599]], want[[599]]) < 3e-5


@pytest.mark.parametrize("shape", [(3, 64, 4), (3, 21, 3), (1, 256, 2)])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_unequal_requests_and_reused_slots(shape, dtype):
    """Decode rows beside portions of unequal requests, in slots that others have used; a step's other
    rows change nothing."""
    s, _, _, w = make(*shape, 1, seed=5, dtype=dtype)
    data = {r: make(*shape, n, seed=10 + r, dtype=dtype)[1:3] for r, n in enumerate([190, 7, 66, 2, 131, 1])}
    want = {r: plain(s, x, y, w, dtype) for r, (x, y) in data.items()}
    e, at, got = Engine(s, w, dtype, 3), {}, {r: [] for r in data}
    # (request, slot, rows)
    steps = [[(0, 2, 129), (1, 0, 6), (3, 1, 1)], [(0, 2, 1), (1, 0, 1), (3, 1, 1)], [(2, 0, 64), (0, 2, 58)],
             [(0, 2, 2), (2, 0, 1), (5, 1, 1)], [(2, 0, 1), (4, 1, 130)], [(4, 1, 1)]]
    for st in steps:
        items = []
        for r, slot, n in st:
            lo = at.get(r, 0)
            items.append((slot, lo, data[r][0][lo:lo + n], data[r][1][lo:lo + n], r))
            at[r] = lo + n
        ordered, outs = e.step(items)
        for it, o in zip(ordered, outs):
            got[it[4]].append(o)
    for r in data:
        assert worst(torch.cat(got[r]), want[r][: at[r]]) < TOL[dtype], r


def test_many_decode_rows():
    """More decode rows than one product takes, beside a portion."""
    s, x, y, w = make(3, 64, 4, 200, seed=6, dtype=BF)
    a, b = (Engine(s, w, BF, 151, any_size=v) for v in (False, True))
    for at in (0, 1, 2):
        items = [(i, at, x[[(i + at) % 200]], y[[(i + at) % 200]]) for i in range(150)] + [(150, 200 * at, x, y)]
        for o, o2 in zip(a.step(items)[1], b.step(items)[1]):
            assert (o - o2).abs().max() < 0.02 * o2.abs().max().clamp_min(0.5)
    assert ((a.state - b.state).norm() / b.state.norm()) < 1e-5 and torch.equal(a.conv, b.conv)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_padding_rows_leave_the_state_alone(dtype):
    s, x, y, w = make(1, 16, 4, 4, seed=7, dtype=dtype)
    e = Engine(s, w, dtype, 2)
    before = e.state.clone(), e.conv.clone()
    _, out = e.step([(-1, 3, x[:1], y[:1]), (-1, 3, x[1:2], y[1:2])])
    assert all(torch.isfinite(o).all() for o in out)
    assert torch.equal(e.state, before[0]) and torch.equal(e.conv, before[1])


@pytest.mark.parametrize("dtype", [F32, BF])
def test_convolution_with_activation(dtype):
    g = torch.Generator().manual_seed(8)
    x, w, T, C = torch.randn(50, 40, generator=g).to(dtype), torch.randn(4, 40, generator=g), 50, 40
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)                 # noqa: E731
    ctx = SimpleNamespace(num_decodes=0, num_prefills=1, num_tiles=1, seq_lens=i32([T]), state_slots=i32([0]),
                          prefill_q_start=i32([0, T]), tile_req=i32([0]), tile_q0=i32([0]))
    out = torch.empty(T, C, dtype=dtype, device=DEV)
    G.short_conv(x.to(DEV), w.to(DEV), None, torch.zeros(1, 3, C, dtype=dtype, device=DEV), ctx, out, act="silu")
    want = R.silu(R.causal_conv(x.double(), w.double().t(), torch.zeros(C, dtype=torch.float64)))
    assert (out.double().cpu() - want).abs().max() < (1e-5 if dtype == F32 else 8e-3) * want.abs().max()
