"""Attention whose values are the unrotated keys (rotation and cache rows, prompts, decode, sinks; tensor-core and
any-size forms) and plain expert and dense units, each against the plain implementation."""
import pytest
import torch

import kubolorn_reference as R
from vllm_cpp_b200.ops import bias_attn as A
from vllm_cpp_b200.ops.reference import build_prefill_tiles

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
TOL = {BF: 9e-3, F32: 1e-5}
# heads, groups, size, rotated dimensions
SHAPES = [(8, 2, 64, 32), (6, 2, 32, 32), (32, 4, 128, 64), (20, 1, 48, 16), (3, 3, 10, 6), (4, 2, 80, 24), (2, 1, 256, 64), (8, 1, 64, 0),
          (4, 1, 128, 128), (2, 2, 16, 2)]


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """(the plain implementations work on small tensors)"""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


class Case:
    """Random q and k of requests of ``lens`` tokens, written to pages in random order by the rotation kernel."""

    def __init__(self, shape, lens, bs, dtype, seed=0, base=300.0, mag=1.2):
        H, G, D, rot = shape
        self.s, self.lens, self.bs, self.dtype, self.shape = A.TiedShape(H, G, D, rot), lens, bs, dtype, shape
        g = torch.Generator().manual_seed(seed)
        r = lambda *z: torch.randn(*z, generator=g).to(dtype).float()      # noqa: E731
        self.qk = [(r(n, H, D), r(n, G, D)) for n in lens]
        self.sink = torch.randn(H, generator=g) * 2
        self.scale = 1.5 * D ** -0.5
        self.freqs, self.mag = R.frequencies(base, rot), mag
        nb = [-(-n // bs) for n in lens]
        order = torch.randperm(sum(nb) + 3, generator=g)
        s = self.s
        self.pages = torch.full((len(order), bs * G * s.pitch), 60.0, dtype=dtype, device=DEV)      # (others' rows)
        table, at = torch.zeros(len(lens), max(nb), dtype=torch.int32), 0
        for i, n in enumerate(nb):
            table[i, :n] = order[at: at + n]
            at += n
        self.table = table.to(DEV)
        pos = torch.arange(max(lens))
        a = pos.double()[:, None] * torch.tensor(self.freqs, dtype=torch.float64)
        cs = torch.cat([mag * torch.cos(a), mag * torch.sin(a)], 1).float().to(DEV) if rot else None
        rows = torch.cat([torch.cat([s.spread(q.reshape(n, -1), H, 1), s.spread(k.reshape(n, -1), G, 1)], 1)
                          for n, (q, k) in zip(lens, self.qk)]).to(dtype).to(DEV)
        p = torch.cat([pos[:n] for n in lens])
        slots = torch.cat([table[i, pos[:n] // bs].long() * bs + pos[:n] % bs for i, n in enumerate(lens)])
        self.q = torch.full((len(p), H * s.D), float("nan"), dtype=dtype, device=DEV)
        A.rotate_tied(rows, p.to(DEV), cs, self.q, slots.to(DEV), self.pages, s, block_size=bs)
        self.first = [sum(lens[:i]) for i in range(len(lens))]
        self.args = dict(H=H, G=G, kw=G * s.pitch, vdim=s.D, block_size=bs, grouped=True, values_in_keys=True, key_at=s.r8)

    def plain(self, i, rows):
        """Outputs of ``rows`` of request i, [n, H, D]; in bf16 the rotated halves are rounded as they are stored."""
        (q, k), (H, G, D, rot), f = self.qk[i], self.shape, torch.float64
        pos = torch.arange(q.shape[0])
        qr, kr = (R.rotate(x.to(f), pos, self.freqs, self.mag).to(self.dtype).to(f) if rot else x.to(f) for x in (q, k))
        out = []
        for h in range(H):
            g = h // (H // G)
            sc = torch.full((len(rows), q.shape[0] + 1), -float("inf"), dtype=f)
            sc[:, :-1] = (qr[rows, h] @ kr[:, g].T * self.scale).masked_fill(pos[None] > torch.tensor(rows)[:, None], -float("inf"))
            sc[:, -1] = self.sink[h].to(f)
            out.append(torch.softmax(sc, -1)[:, :-1] @ k[:, g].to(f))
        return 0.7 * torch.stack(out, 1)

    def heads(self, out):
        """[rows, H * padded] in the kernel's order -> [rows, H, D]."""
        s = self.s
        x = out.double().cpu().view(-1, s.H, s.D)
        assert not x[..., s.rot: s.r8].any() and not x[..., s.r8 + s.dim - s.rot:].any()
        return torch.cat([x[..., : s.rot], x[..., s.r8: s.r8 + s.dim - s.rot]], -1)

    def close(self, got, want, note=None):
        e = (got - want).flatten(1).norm(dim=-1) / want.flatten(1).norm(dim=-1).clamp_min(0.05)
        assert e.max() < TOL[self.dtype], (note, int(e.argmax()), e.max().item())


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("bs", [16, 64])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_decode(shape, bs, dtype):
    lens = [1, 2, 15, 16, 17, 64, 65, 100, 257]
    c = Case(shape, lens, bs, dtype, seed=1)
    q = torch.stack([c.q[f + n - 1] for f, n in zip(c.first, lens)])
    want = torch.cat([c.plain(i, [n - 1]) for i, n in enumerate(lens)])
    for splits, any_size in ((1, False), (3, False), (1, True)):
        out = torch.full_like(q, float("nan"))
        A.decode(q, c.pages, out, block_table=c.table, seq_lens=i32(lens), scale=c.scale, splits=splits, any_size=any_size,
                 sink=c.sink.to(DEV), out_scale=0.7, **c.args)
        c.close(c.heads(out), want, (splits, any_size))
    kind = A.kernel_kind("decode", q, c.pages, scale=c.scale, **c.args)
    assert kind == ("tensor-core" if dtype == BF else "any-size")


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("bs", [8, 64, 256])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_prompt_portions(shape, bs, dtype):
    """Portions that start anywhere: (rows already there, rows of the portion)."""
    portions = [(0, 2), (0, 130), (99, 3), (61, 200), (127, 5)]
    lens = [a + n for a, n in portions]
    c = Case(shape, lens, bs, dtype, seed=2)
    q = torch.cat([c.q[f + a: f + a + n] for f, (a, n) in zip(c.first, portions)]).contiguous()
    n = [x[1] for x in portions]
    tr, tq = build_prefill_tiles(n)
    for any_size in (False, True):
        out = torch.full_like(q, float("nan"))
        A.prefill(q, c.pages, out, block_table=c.table, seq_lens=i32(lens), q_start=i32([sum(n[:i]) for i in range(len(n) + 1)]),
                  num_reqs=len(n), tile_req=i32(tr), tile_q0=i32(tq), scale=c.scale, any_size=any_size, sink=c.sink.to(DEV),
                  out_scale=0.7, **c.args)
        for i, (g, (a, m)) in enumerate(zip(c.heads(out).split(n), portions)):
            c.close(g, c.plain(i, list(range(a, a + m))), (any_size, i))
    kind = A.kernel_kind("prefill", q, c.pages, scale=c.scale, **c.args)
    assert kind == ("tensor-core" if dtype == BF else "any-size")


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("sink", [-40.0, 0.0, 9.0, 60.0])
def test_sinks(dtype, sink):
    """From no weight at all to almost all of it."""
    c = Case((4, 2, 64, 32), [200], 16, dtype, seed=3)
    c.sink = torch.full((4,), sink)
    c.scale = 0.1
    want = c.plain(0, list(range(200)))
    size = want.norm(dim=(1, 2)).clamp_min(1e-20)
    for kernel in ("decode", "prefill"):
        for any_size in (False, True):
            out = torch.full_like(c.q, float("nan"))
            kw = dict(scale=c.scale, any_size=any_size, sink=c.sink.to(DEV), out_scale=0.7, **c.args)
            if kernel == "decode":
                A.decode(c.q, c.pages, out, block_table=c.table.expand(200, -1).contiguous(), seq_lens=i32(list(range(1, 201))), splits=2, **kw)
            else:
                tr, tq = build_prefill_tiles([200])
                A.prefill(c.q, c.pages, out, block_table=c.table, seq_lens=i32([200]), q_start=i32([0, 200]), num_reqs=1, tile_req=i32(tr),
                          tile_q0=i32(tq), **kw)
            assert ((c.heads(out) - want).norm(dim=(1, 2)) / size).max() < 2 * TOL[dtype], (kernel, any_size)


# ------------------------------------------------------------------------------ ungated units
ACTS = {"gelu_tanh": R.gelu_tanh, "relu2": lambda x: torch.relu(x) ** 2}


@pytest.mark.parametrize("act", list(ACTS))
@pytest.mark.parametrize("T,N,K", [(1, 40, 24), (7, 1000, 512), (64, 2048, 8192), (130, 512, 64), (200, 20000, 128), (300, 640, 256), (1024, 4096, 512)])
def test_product_with_activation(act, T, N, K):
    from vllm_cpp_b200.models.backend import GpuBackend
    g = torch.Generator().manual_seed(7)
    x, w = torch.randn(T, K, generator=g), torch.randn(N, K, generator=g) * K ** -0.5
    for dtype in (BF, F32):
        if dtype == F32 and N * K * T > 1 << 30:
            continue
        a, b = x.to(dtype), w.to(dtype)
        want = ACTS[act](a.double() @ b.double().T)
        wide = torch.full((T, N + 16), float("nan"), dtype=dtype, device=DEV)
        GpuBackend().plain_unit(a.to(DEV), b.to(DEV), act, wide[:, 16:])
        e = (wide[:, 16:].double().cpu() - want).norm() / want.norm()
        assert e < {BF: 4e-3, F32: 5e-6}[dtype] and wide[:, :16].isnan().all()


@pytest.mark.parametrize("act", list(ACTS))
@pytest.mark.parametrize("T,E,top,W,ff", [(1, 4, 2, 32, 24), (9, 6, 3, 48, 40), (700, 16, 4, 256, 128), (40, 1, 1, 64, 16)])
def test_experts(act, T, E, top, W, ff):
    from vllm_cpp_b200.models.backend import GpuBackend
    from vllm_cpp_b200.ops.moe import MoeWorkspace
    g = torch.Generator().manual_seed(8)
    x, up, down = torch.randn(T, W, generator=g), torch.randn(E, ff, W, generator=g) * W ** -0.5, torch.randn(E, W, ff, generator=g) * ff ** -0.5
    logits = torch.randn(T, E, generator=g) * 2
    for dtype in (BF, F32):
        a, u, d = x.to(dtype), up.to(dtype), down.to(dtype)
        y, pos, w = GpuBackend().plain_experts(a.to(DEV), logits.to(DEV), u.to(DEV), d.to(DEV), MoeWorkspace(torch.device(DEV), T, top, E, W, ff, dtype),
                                               top=top, act=act)
        got = (y[pos.long()].double() * w.double()[..., None]).sum(1).cpu()
        want = torch.zeros(T, W, dtype=torch.float64)
        for t in range(T):
            best = logits[t].argsort(descending=True)[:top]
            for e, p in zip(best.tolist(), torch.softmax(logits[t][best].double(), 0)):
                h = ACTS[act](u[e].double() @ a[t].double()).to(dtype).double()
                want[t] += p * (d[e].double() @ h)
        assert ((got - want).norm() / want.norm()) < {BF: 6e-3, F32: 2e-6}[dtype]
