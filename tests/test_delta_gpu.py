"""The delta-rule kernels (preparation, token by token, in chunks) against the plain implementation, over
portions, decode rows and unequal requests with reused slots."""
from types import SimpleNamespace

import pytest
import torch

import diforax_reference as R
from vllm_cpp_b200.ops import delta as D

pytestmark = pytest.mark.gpu
DEV = "cuda"


def make(G, H, dim, vdim, taps, T, seed=0, dtype=torch.float32, decay=1.0):
    """Random inputs: padded projection rows, a | b, weights (on the CPU, fp32)."""
    g = torch.Generator().manual_seed(seed)
    pad = lambda n: (n + 15) // 16 * 16                                 # noqa: E731
    s = D.DeltaShape(G=G, H=H, D=pad(dim), V=pad(vdim), dim=dim, vdim=vdim, taps=taps)
    heads = [(s.D, dim)] * (2 * G) + [(s.V, vdim)] * (2 * H)
    real = torch.cat([torch.arange(p) < n for p, n in heads])
    proj = (torch.randn(T, s.columns, generator=g) * real).to(dtype)
    ab = torch.cat([torch.randn(T, H, generator=g) * 2, torch.randn(T, H, generator=g) * 2], 1)
    w = {"conv_w": torch.randn(taps, s.channels, generator=g) * 0.6 * real[: s.channels],
         "A": torch.rand(H, generator=g) * decay + 0.01, "dt": torch.randn(H, generator=g) - 2.0,
         "norm": torch.cat([torch.rand(vdim, generator=g) + 0.5, torch.zeros(s.V - vdim)])}
    return s, proj, ab, w


def plain(s, proj, ab, w, eps=1e-5):
    """Whole sequence in float64 -> out [T, H, vdim]."""
    f = torch.float64
    x, T, H = proj.to(f), proj.shape[0], s.H
    y = R.silu(R.causal_conv(x[:, : s.channels], w["conv_w"].to(f).t()))
    gd = s.G * s.D
    q, k = (y[:, i * gd: (i + 1) * gd].view(T, s.G, s.D)[..., : s.dim] for i in (0, 1))
    v = y[:, 2 * gd:].view(T, H, s.V)[..., : s.vdim]
    if proj.dtype == torch.bfloat16:
        v = v.to(torch.bfloat16).to(f)
    q, k = R.unit(q) / s.dim ** 0.5, R.unit(k)
    g = R.decay(ab[:, :H].to(f), torch.log(w["A"].to(f)), w["dt"].to(f))
    beta = torch.sigmoid(ab[:, H:].to(f))
    o = torch.zeros(T, H, s.vdim, dtype=f)
    for h in range(H):
        S, kv = torch.zeros(s.dim, s.vdim, dtype=f), h // (H // s.G)
        for t in range(T):
            S, o[t, h] = R.delta_step(S, q[t, kv], k[t, kv], v[t, h], g[t, h], beta[t, h])
    z = x[:, s.channels:].view(T, H, s.V)[..., : s.vdim]
    return R.rms(o, eps) * w["norm"][: s.vdim].to(f) * R.silu(z)


class Engine:
    """Steps of (request, count) pairs over shared state, as the model runner lays them out."""

    def __init__(self, s, w, dtype, slots, token_by_token=False):
        self.s, self.dtype, self.tbt = s, dtype, token_by_token
        self.w = {k: v.to(DEV).contiguous() for k, v in w.items()}
        # what a freed slot leaves behind must not be seen
        self.conv = torch.full((slots, s.taps - 1, s.channels), 7.0, dtype=dtype, device=DEV)
        self.state = torch.full((slots, s.H, s.D, s.V), 3.0, dtype=torch.float32, device=DEV)

    def step(self, items):
        """items: (slot, position of the first row, proj rows, ab rows), decode rows first."""
        s = self.s
        items = sorted(items, key=lambda x: x[2].shape[0] > 1)
        n = [x[2].shape[0] for x in items]
        nd, T = sum(c == 1 for c in n), sum(n)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)   # noqa: E731
        pq, tr, tq = [0], [], []
        for i, c in enumerate(n[nd:]):
            pq.append(pq[-1] + c)
            for q0 in range(0, c, 128):
                tr.append(i)
                tq.append(q0)
        rows = SimpleNamespace(seq_lens=i32([x[1] + c for x, c in zip(items, n)]), state_slots=i32([x[0] for x in items]),
                               prefill_q_start=i32(pq), tile_req=i32(tr or [0]), tile_q0=i32(tq or [0]), num_decodes=nd,
                               num_prefills=len(n) - nd, num_tiles=len(tr))
        f = dict(dtype=torch.float32, device=DEV)
        nan = float("nan")
        bufs = {"q": torch.full((T, s.G, s.D), nan, **f), "k": torch.full((T, s.G, s.D), nan, **f),
                "v": torch.full((T, s.H, s.V), nan, dtype=self.dtype, device=DEV), "g": torch.full((T, s.H), nan, **f),
                "beta": torch.full((T, s.H), nan, **f), "o": torch.full((T, s.H, s.V), nan, **f),
                "chunks": D.chunk_workspace(DEV, len(tr) + 1, s.H)}
        bufs["chunks"][0].fill_(nan)
        out = torch.full((T, s.H * s.V), nan, dtype=self.dtype, device=DEV)
        D.delta_mixer(torch.cat([x[2] for x in items]).to(DEV), torch.cat([x[3] for x in items]).to(DEV), self.w, s,
                      self.conv, self.state, rows, bufs, out, 1e-5, token_by_token=self.tbt)
        return items, out.float().cpu().view(T, s.H, s.V).split(n)


def run(s, proj, ab, w, cuts, **kw):
    e, at, got = Engine(s, w, proj.dtype, 3, **kw), 0, []
    for n in cuts:
        got.append(e.step([(1, at, proj[at:at + n], ab[at:at + n])])[1][0])
        at += n
    assert at == proj.shape[0]
    return torch.cat(got)


def err(got, want, vdim):
    assert not got[..., vdim:].abs().max() > 0 if got.shape[-1] > vdim else True
    d = (got[..., :vdim].double() - want).norm(dim=-1)
    return (d / want.norm(dim=-1).clamp_min(1e-3 * want.norm(dim=-1).mean())).max().item()


# sizes below, at and above the chunk kernels' pieces; values that differ in every place
SHAPES = [(2, 4, 32, 48, 4), (1, 3, 128, 128, 4), (2, 2, 20, 37, 3), (3, 6, 64, 80, 2), (1, 1, 112, 16, 1), (1, 5, 96, 136, 6)]
TOL = {torch.float32: 3e-5, torch.bfloat16: 1.2e-2}


@pytest.mark.parametrize("shape", SHAPES + [(1, 2, 144, 64, 4), (1, 2, 256, 256, 4), (1, 1, 300, 40, 4)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_whole_and_portions(shape, dtype):
    T = 150 if shape[2] <= 128 else 70
    s, proj, ab, w = make(*shape, T, seed=1, dtype=dtype)
    want = plain(s, proj, ab, w)
    for cuts in ([T], [1] * 5 + [T - 5], [2, 3, 60, T - 65], [64, 1, 1, T - 66], [T - 1, 1]):
        assert err(run(s, proj, ab, w, cuts), want, s.vdim) < TOL[dtype], cuts


@pytest.mark.parametrize("shape", SHAPES)
def test_chunks_have_fp32_accuracy(shape):
    """Chunked and token-by-token prompts of the bf16 mode agree far below bf16 rounding (state and all)."""
    s, proj, ab, w = make(*shape, 300, seed=2, dtype=torch.bfloat16)
    a, b = (Engine(s, w, torch.bfloat16, 2, token_by_token=x) for x in (False, True))
    for lo, hi in ((0, 200), (200, 300)):
        for e in (a, b):
            e.step([(0, lo, proj[lo:hi], ab[lo:hi])])
    rel = ((a.state[0] - b.state[0]).norm() / b.state[0].norm()).item()
    assert rel < 3e-5 and torch.equal(a.conv[0], b.conv[0])


@pytest.mark.parametrize("decay", [0.0, 30.0])
def test_slow_and_fast_decays(decay):
    """States that keep everything for the whole prompt, and heads that forget within a token."""
    s, proj, ab, w = make(2, 4, 48, 32, 4, 400, seed=3, decay=decay)
    want = plain(s, proj, ab, w)
    # (a head that forgets reads one q . k, which can be small beside its terms, and the norm scales it up)
    assert err(run(s, proj, ab, w, [399, 1]), want, s.vdim) < (3e-5 if decay == 0 else 2e-4)
    pb = proj.to(torch.bfloat16)
    assert err(run(s, pb, ab, w, [130, 270]), plain(s, pb, ab, w), s.vdim) < TOL[torch.bfloat16]


def test_a_written_value_is_read_far_away():
    """One token writes along a key of its own, the others keep off it: the last token reads it back."""
    s, proj, ab, w = make(1, 1, 64, 16, 1, 700, seed=4, decay=0.0)
    w["A"], w["conv_w"] = torch.tensor([1e-4]), torch.ones_like(w["conv_w"])
    proj[:, 0] = proj[:, 64] = -40.0            # (silu: nothing of this direction)
    proj[5, 64:128], proj[5, 64] = -40.0, 30.0
    proj[699, :64], proj[699, 0] = -40.0, 30.0
    want = plain(s, proj, ab, w)
    other = proj.clone()
    other[5, 64] = -40.0
    assert err(plain(s, other, ab, w)[[699]].float(), want[[699]], 16) > 0.3
    for cuts in ([700], [690] + [1] * 10, [100] * 7):
        assert err(run(s, proj, ab, w, cuts)[[699]], want[[699]], 16) < 3e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_unequal_requests_and_reused_slots(dtype):
    """Decode rows beside portions of unequal requests, in slots that others have used; a step's other
    rows change nothing."""
    s, *_ , w = make(2, 4, 32, 48, 4, 1, seed=5)
    data = {r: make(2, 4, 32, 48, 4, n, seed=10 + r, dtype=dtype)[1:3] for r, n in enumerate([190, 7, 66, 2, 131, 1])}
    want = {r: plain(s, p, a, w) for r, (p, a) in data.items()}
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
        if at[r] == len(data[r][0]):
            assert err(torch.cat(got[r]), want[r], 48) < TOL[dtype], r
        else:
            assert err(torch.cat(got[r]), want[r][: at[r]], 48) < TOL[dtype], r


def test_padding_rows_leave_the_state_alone():
    s, proj, ab, w = make(1, 2, 16, 16, 4, 4, seed=6)
    e = Engine(s, w, torch.float32, 2)
    before = e.state.clone(), e.conv.clone()
    _, out = e.step([(-1, 3, proj[:1], ab[:1]), (-1, 3, proj[1:2], ab[1:2])])
    assert all(float(o.abs().max()) == 0 for o in out)
    assert torch.equal(e.state, before[0]) and torch.equal(e.conv, before[1])
