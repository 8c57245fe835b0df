"""Embeddings of token pairs and the pass between layers (stream update, norm in parts, input convolutions) against the
plain implementation, over portions, decode rows and unequal requests with reused slots."""
from types import SimpleNamespace

import pytest
import torch

import kubolorn_reference as R
from vllm_cpp_b200.config import BigramSpec
from vllm_cpp_b200.ops import conv_norm as N
from vllm_cpp_b200.ops.reference import build_prefill_tiles

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
EPS = 1e-4
# width, parts, taps: parts of one to many threads, of odd sizes, with tails
SHAPES = [(64, 4, 4), (256, 1, 3), (36, 3, 2), (35, 5, 4), (2048, 4, 3), (4096, 1, 4), (24, 1, 9), (1200, 1, 1), (40, 20, 2), (602, 1, 3), (8, 2, 17)]
TOL = {BF: 5e-3, F32: 1e-5}


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """(the plain implementations work on small tensors)"""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def context(items):
    """(items, decode rows first), their sizes and the step's rows; an item: (slot, rows already seen, rows)."""
    items = [i for i in items if i[2] == 1] + [i for i in items if i[2] > 1]
    n = [i[2] for i in items]
    pre = [m for m in n if m > 1]
    tr, tq = build_prefill_tiles(pre) if pre else ([], [])
    return items, SimpleNamespace(num_decodes=len(n) - len(pre), num_prefills=len(pre), num_tiles=len(tr),
                                  seq_lens=i32([i[1] + i[2] for i in items]), state_slots=i32([i[0] for i in items]),
                                  prefill_q_start=i32([sum(pre[:i]) for i in range(len(pre) + 1)]), tile_req=i32(tr or [0]), tile_q0=i32(tq or [0]))


def padded(t, cols):
    out = torch.zeros(t.shape[0], cols, dtype=t.dtype)
    out[:, : t.shape[1]] = t
    return out


class Layer:
    def __init__(self, shape, dtype, slots=3, seed=0, sublayers=2):
        self.W, self.groups, self.taps = shape
        self.cols, self.dtype = (self.W + 7) // 8 * 8, dtype
        g = torch.Generator().manual_seed(seed)
        self.norms = [torch.randn(self.W, generator=g) * 0.2 + 1 for _ in range(sublayers)]
        self.canon = [torch.randn(self.W, self.taps, generator=g) * 0.4 for _ in range(sublayers)]
        self.weights = [N.conv_weights(padded(n[None], self.cols)[0], padded(c.t(), self.cols).t()).to(DEV)
                        for n, c in zip(self.norms, self.canon)]
        self.state = torch.full((slots, max(1, self.taps - 1), self.cols), 9.0, device=DEV)     # (of somebody before)

    def plain(self, x):
        out = []
        for n, c in zip(self.norms, self.canon):
            h = R.part_rms(x.double(), self.groups, EPS) * n.double()
            out.append(h + R.causal_conv(h, c.double()))
        return out

    def step(self, items, add):
        """items: (slot, rows already seen, x [n, W]); x = what src, a and pairs add up to (``add``: which of these)."""
        order, ctx = context([(s, at, x.shape[0]) for s, at, x in items])
        by = {i[0]: i[2] for i in items}
        x = padded(torch.cat([by[s] for s, _, _ in order]), self.cols)
        T, kw, g = x.shape[0], {}, torch.Generator().manual_seed(T_SEED)
        src = x.clone()
        if "a" in add:
            a = torch.randn(T, self.cols, generator=g)
            src -= a
            kw["a"] = a.to(DEV)
        if "pairs" in add:
            k = 3
            y = torch.randn(T * k + 5, self.cols, generator=g).to(self.dtype)
            pos = torch.randperm(T * k + 5, generator=g)[: T * k].view(T, k).to(torch.int32)
            w = torch.rand(T, k, generator=g)
            w[:, -1] = 0.5
            pos[::2, -1] = -1                                              # (no output)
            live = (pos >= 0)[..., None]
            src -= (y[pos.long().clamp(min=0)].float() * live * w[..., None]).sum(1)
            kw.update(y=y.to(DEV), pair_pos=pos.to(DEV), pair_w=w.to(DEV))
        dst = torch.full_like(src, float("nan")).to(DEV)
        outs = [torch.full((T, self.cols), float("nan"), dtype=self.dtype, device=DEV) for _ in self.weights]
        N.norm_conv(src.to(DEV), ctx, self.weights, outs, width=self.W, groups=self.groups, eps=EPS,
                    state=self.state if self.taps > 1 else None, dst=dst, **kw)
        assert torch.allclose(dst[:, : self.W].cpu(), x[:, : self.W], atol=1e-5)
        for o in outs:
            assert not o[:, self.W:].any()
        n = [i[2] for i in order]
        return order, list(zip(*[o[:, : self.W].float().cpu().split(n) for o in outs]))


T_SEED = 5


def close(got, want, dtype, note=None):
    for g, w in zip(got, want):
        assert ((g.double() - w).norm(dim=-1) / w.norm(dim=-1)).max() < TOL[dtype], note


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("add", [(), ("a",), ("a", "pairs")])
def test_whole_and_portions(shape, dtype, add):
    L, T = Layer(shape, dtype, seed=1), 150
    x = torch.randn(T, shape[0], generator=torch.Generator().manual_seed(2)) * 2
    want = L.plain(x)
    for cuts in ([T], [1] * 5 + [T - 5], [2, 3, 60, T - 65], [15, 1, 17, T - 33], [129, T - 130, 1], [2] * 75):
        at = 0
        for n in cuts:
            got = L.step([(1, at, x[at:at + n])], add)[1][0]
            close(got, [w[at:at + n] for w in want], dtype, (cuts, at))
            at += n


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("shape", SHAPES[:4])
def test_batches_and_slots(shape, dtype):
    L = Layer(shape, dtype, seed=3)
    for turn in range(3):
        x = {s: torch.randn(n, shape[0], generator=torch.Generator().manual_seed(10 * turn + s)) for s, n in ((0, 40), (1, 70), (2, 3))}
        want = {s: L.plain(v) for s, v in x.items()}
        at = dict.fromkeys(x, 0)
        for sizes in ({0: 1, 1: 65, 2: 2}, {0: 1, 2: 1}, {0: 37, 1: 1}, {0: 1, 1: 4}):
            order, got = L.step([(s, at[s], x[s][at[s]:at[s] + n]) for s, n in sizes.items()], ("a",))
            for (s, a, n), g in zip(order, got):
                close(g, [w[a:a + n] for w in want[s]], dtype, (turn, s, a))
                at[s] = a + n


def test_norm_alone():
    """One output, one tap: the norm before the head."""
    x = torch.randn(33, 96, generator=torch.Generator().manual_seed(4))
    L = Layer((96, 3, 1), BF, sublayers=1)
    _, ctx = context([(0, 0, 33)])
    out = torch.empty(33, 96, dtype=BF, device=DEV)
    N.norm_conv(x.to(DEV), ctx, [L.norms[0][None].to(DEV)], [out], width=96, groups=3, eps=EPS)
    close([out.float().cpu()], [R.part_rms(x.double(), 3, EPS) * L.norms[0].double()], BF)


@pytest.mark.parametrize("shape", [(64, 4), (35, 5), (2048, 1), (24, 24)])
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("pairs", [True, False])
def test_embeddings(shape, dtype, pairs):
    W, groups = shape
    cols, V = (W + 7) // 8 * 8, 50
    g = torch.Generator().manual_seed(5)
    table, bigram = (padded(torch.randn(n, W, generator=g), cols).to(dtype) for n in (V, 14))
    nw = torch.randn(W, generator=g) * 0.2 + 1
    c = {"buckets": 13, "mul_prev": 31, "mul_cur": 1000003}
    prev = torch.full((3,), 44, dtype=torch.int64, device=DEV)          # (of somebody before)
    toks = {s: torch.randint(0, V, (60,), generator=g) for s in range(3)}

    def plain(t):
        x = table[t, :W].double() * 1.7
        if pairs:
            x = x + bigram[torch.tensor(R.bigram_rows(t.tolist(), c)), :W].double()
        return R.part_rms(x, groups, EPS) * nw.double()
    for turn in range(2):
        at = dict.fromkeys(toks, 0)
        for sizes in ({0: 1, 1: 40, 2: 2}, {0: 1, 2: 1}, {0: 30, 1: 1}, {0: 1, 1: 4, 2: 20}):
            order, ctx = context([(s, at[s], n) for s, n in sizes.items()])
            ids = torch.cat([toks[s][a:a + n] for s, a, n in order])
            stream = torch.full((len(ids), cols), float("nan"), device=DEV)
            N.embed_pairs(stream, ids.to(DEV), table.to(DEV), ctx, width=W, scale=1.7, norm_w=padded(nw[None], cols)[0].to(DEV), groups=groups,
                          eps=EPS, **(dict(bigram=bigram.to(DEV), prev=prev, spec=BigramSpec(**c)) if pairs else {}))
            assert not stream[:, W:].any()
            for (s, a, n), got in zip(order, stream[:, :W].cpu().split([i[2] for i in order])):
                w = plain(toks[s])[a:a + n]
                assert ((got.double() - w).norm(dim=-1) / w.norm(dim=-1)).max() < 3e-6, (turn, s, a)
                at[s] = a + n
