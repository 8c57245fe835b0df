"""Kernels of the grouped, chunk-limited attention over split pages (rotation and unit norm, prompts, decode;
tensor-core and any-size forms), the sandwich norm of the fp32 stream and the grouped router, each against
the plain implementation."""
import pytest
import torch

import diforax_reference as R
from vllm_cpp_b200.ops import bias_attn as A
from vllm_cpp_b200.ops.reference import build_prefill_tiles

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


class Pages:
    """Keys [n, G, D] and values [n, G, V] of requests, scattered over pages in random order."""

    def __init__(self, kv, bs, dtype, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.bs, self.G, self.D, self.V = bs, kv[0][0].shape[1], kv[0][0].shape[2], kv[0][1].shape[2]
        nb = [max(1, -(-k.shape[0] // bs)) for k, _ in kv]
        order = torch.randperm(sum(nb) + 3, generator=g)
        self.table = torch.zeros(len(kv), max(nb), dtype=torch.int32)
        kw, vw = self.G * self.D, self.G * self.V
        # pages others have used hold large finite values
        pages = torch.full((len(order), bs * (kw + vw)), 50.0)
        at = 0
        for r, (k, v) in enumerate(kv):
            for b in range(nb[r]):
                page = int(order[at])
                at += 1
                self.table[r, b] = page
                kk, vv = k[b * bs:(b + 1) * bs], v[b * bs:(b + 1) * bs]
                pages[page, : kk.numel()] = kk.reshape(-1)
                pages[page, bs * kw: bs * kw + vv.numel()] = vv.reshape(-1)
        self.pages, self.table = pages.to(dtype).to(DEV), self.table.to(DEV)

    def args(self, H):
        return dict(H=H, G=self.G, kw=self.G * self.D, vdim=self.V, block_size=self.bs, grouped=True)


def plain(q, k, v, at, scale, chunk):
    """q [n, H, D] at positions ``at`` over keys 0 .. at -> [n, H, V] in float64."""
    f, H, G = torch.float64, q.shape[1], k.shape[1]
    at, j = torch.tensor(at)[:, None], torch.arange(k.shape[0])[None]
    seen = (j <= at) & (R.same_chunk(at, j, chunk) if chunk else True)
    out = []
    for h in range(H):
        s = (q[:, h].to(f) @ k[:, h // (H // G)].to(f).T * scale).masked_fill(~seen, float("-inf"))
        out.append(torch.softmax(s, -1) @ v[:, h // (H // G)].to(f))
    return torch.stack(out, 1)


def data(H, G, D, V, lens, dtype, seed=0, sharp=1.0):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()      # noqa: E731
    kv = [(r(n, G, D), r(n, G, V)) for n in lens]
    return kv, [(r(n, H, D) * sharp).to(dtype).float() for n in lens]


# the last of each group: values that no tensor-core form takes
SHAPES = [(4, 2, 64, 48), (6, 2, 112, 96), (16, 1, 128, 128), (3, 3, 32, 16), (4, 1, 256, 192), (8, 4, 80, 256), (6, 3, 20, 36)]
TOL = {BF: 8e-3, F32: 1e-5}


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("bs", [8, 16, 64])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_decode(shape, bs, dtype):
    H, G, D, V = shape
    lens = [1, 2, 15, 16, 17, 63, 64, 65, 100, 199, 200, 201, 257, 400]
    kv, qs = data(H, G, D, V, lens, dtype, seed=1)
    p, scale = Pages(kv, bs, dtype), 1.7 * D ** -0.5
    q = torch.stack([x[-1] for x in qs]).reshape(len(lens), -1).to(dtype).to(DEV)
    for chunk in (0, 100, 64, 37, 1000, 1):
        want = torch.cat([plain(x[-1:], k, v, [n - 1], scale, chunk) for x, (k, v), n in zip(qs, kv, lens)])
        for splits, any_size in ((1, False), (3, False), (1, True)):
            out = torch.full((len(lens), H * V), float("nan"), dtype=dtype, device=DEV)
            A.decode(q, p.pages, out, block_table=p.table, seq_lens=i32(lens), scale=scale, chunk=chunk, splits=splits,
                     any_size=any_size, **p.args(H))
            d = (out.double().cpu().view_as(want) - want).norm(dim=-1) / want.norm(dim=-1)
            assert d.max() < TOL[dtype], (chunk, splits, any_size, int(d.max(-1).values.argmax()))
    kind = A.kernel_kind("decode", q, p.pages, scale=scale, chunk=64, **p.args(H))
    assert kind == ("tensor-core" if dtype == BF and bs % 16 == 0 and D % 16 == 0 and V % 16 == 0 else "any-size")


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("bs", [8, 64, 256])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_prompt_portions(shape, bs, dtype):
    """Portions that start anywhere: (rows already there, rows of the portion)."""
    H, G, D, V = shape
    portions = [(0, 2), (0, 130), (99, 3), (100, 2), (61, 200), (250, 131), (127, 5)]
    lens = [a + n for a, n in portions]
    kv, qs = data(H, G, D, V, lens, dtype, seed=2)
    p, scale = Pages(kv, bs, dtype), 1.7 * D ** -0.5
    rows = torch.cat([x[a:] for x, (a, _) in zip(qs, portions)])
    q = rows.reshape(rows.shape[0], -1).to(dtype).to(DEV)
    n = [x for _, x in portions]
    tr, tq = build_prefill_tiles(n)
    start = [sum(n[:i]) for i in range(len(n) + 1)]
    for chunk in (0, 100, 128, 37, 300):
        want = torch.cat([plain(x[a:], k, v, list(range(a, a + m)), scale, chunk)
                          for x, (k, v), (a, m) in zip(qs, kv, portions)])
        for any_size in (False, True):
            out = torch.full((rows.shape[0], H * V), float("nan"), dtype=dtype, device=DEV)
            A.prefill(q, p.pages, out, block_table=p.table, seq_lens=i32(lens), q_start=i32(start), num_reqs=len(n),
                      tile_req=i32(tr), tile_q0=i32(tq), scale=scale, chunk=chunk, any_size=any_size, **p.args(H))
            d = (out.double().cpu().view_as(want) - want).norm(dim=-1) / want.norm(dim=-1)
            assert d.max() < TOL[dtype], (chunk, any_size, int(d.max(-1).values.argmax()))
        if dtype == F32:
            break
    kind = A.kernel_kind("prefill", q, p.pages, scale=scale, chunk=37, **p.args(H))
    assert kind == ("tensor-core" if dtype == BF and D % 16 == 0 and V % 8 == 0 else "any-size")


@pytest.mark.parametrize("dtype", [BF, F32])
def test_edges_of_chunks_and_pages(dtype):
    """One key carries the whole weight: the first and the last of a chunk, of a page, and the neighbours
    just outside, in decode and in prompts."""
    H, G, D, V, n, chunk, bs = 2, 1, 64, 16, 150, 48, 16
    for key in (0, 15, 16, 47, 48, 95, 96, 143, 144):
        kv, qs = data(H, G, D, V, [n], dtype, seed=3)
        k, v = kv[0]
        k[key] = 8.0
        v[key] = 5.0
        q = torch.full((n, H, D), 0.5)
        p = Pages([(k, v)], bs, dtype)
        want = plain(q, k, v, list(range(n)), 0.3, chunk)
        seen = [i for i in range(n) if i >= key and i // chunk == key // chunk]
        assert all((want[i].mean() > 4.9) == (i in seen) for i in range(n))
        qd = q.reshape(n, -1).to(dtype).to(DEV)
        out = torch.empty(n, H * V, dtype=dtype, device=DEV)
        tr, tq = build_prefill_tiles([n])
        A.prefill(qd, p.pages, out, block_table=p.table, seq_lens=i32([n]), q_start=i32([0, n]), num_reqs=1,
                  tile_req=i32(tr), tile_q0=i32(tq), scale=0.3, chunk=chunk, **p.args(H))
        assert (out.double().cpu().view_as(want) - want).abs().max() < 0.05
        A.decode(qd, p.pages, out, block_table=p.table.expand(n, -1).contiguous(), seq_lens=i32(list(range(1, n + 1))),
                 scale=0.3, chunk=chunk, splits=2, **p.args(H))
        assert (out.double().cpu().view_as(want) - want).abs().max() < 0.05


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("shape", [(4, 2, 64, 48, 64), (3, 3, 24, 16, 10), (2, 1, 100, 36, 48), (5, 1, 128, 128, 128), (2, 2, 16, 8, 0)])
def test_rotation_unit_norm_and_cache(dtype, shape):
    H, G, dim, V, rot = shape
    D, T, bs, base, eps = (dim + 15) // 16 * 16, 77, 16, 5e4, 1e-5
    g = torch.Generator().manual_seed(4)
    real = torch.cat([torch.arange(D) < dim] * (H + G) + [torch.ones(V, dtype=torch.bool)] * G)
    qkv = (torch.randn(T, (H + G) * D + G * V, generator=g) * real).to(dtype)
    pos = torch.randint(0, 3000, (T,), generator=g)
    slots = torch.randperm(200, generator=g)[:T]
    slots[5] = -1
    x = qkv[:, : (H + G) * D].double().view(T, H + G, D)[..., :dim]
    want = R.rms(R.rotate(x, pos, base, rot) if rot else x, eps)
    table = None
    if rot:
        from vllm_cpp_b200 import ops
        table = ops.rope_table((base ** (-torch.arange(0, rot, 2, dtype=torch.float64) / rot)).to(DEV), 3000)
    cache = torch.full((13, bs * G * (D + V)), 9.0, dtype=dtype, device=DEV)
    q = torch.full((T, H * D), float("nan"), dtype=dtype, device=DEV)
    A.rotate_kv(qkv.to(DEV), pos.to(DEV), table, rot, eps, q, slots.to(DEV), cache, H=H, G=G, D=D, V=V, dim=dim, block_size=bs)
    tol = 3e-6 if dtype == F32 else 8e-3
    got = q.double().cpu().view(T, H, D)
    assert (got[..., :dim] - want[:, :H]).abs().max() < tol * 4 and not bool((got[..., dim:] != 0).any())
    keys, vals = A.page_views(cache.cpu(), bs, G * D)
    for t in range(T):
        if slots[t] >= 0:
            b, o = divmod(int(slots[t]), bs)
            assert (keys[b, o].double().view(G, D)[:, :dim] - want[t, H:]).abs().max() < tol * 4
            assert torch.equal(vals[b, o], qkv[t, (H + G) * D:])
    assert int((keys.reshape(-1, G * D) == 9.0).all(-1).sum()) == 13 * bs - (T - 1)
    only_q = torch.empty_like(q)
    A.rotate_kv(qkv[:, : H * D].contiguous().to(DEV), pos.to(DEV), table, rot, eps, only_q, slots.to(DEV), cache, H=H, G=0, D=D,
                V=V, dim=dim, block_size=bs)
    assert (only_q.double() - q.double()).abs().max() < tol


@pytest.mark.parametrize("width", [40, 37, 1024, 5000])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_sandwich_norm_with_identity_experts(width, dtype):
    from vllm_cpp_b200.ops.stream import stream_norm
    T, k, cols = 9, 3, (width + 7) // 8 * 8
    g = torch.Generator().manual_seed(5)

    def r(*s):
        x = torch.zeros(*s[:-1], cols)
        x[..., :width] = torch.randn(*s, generator=g)
        return x
    stream, y, h = r(T, width), r(20, width).to(dtype), r(T, width).to(dtype)
    pos = torch.randint(-1, 20, (T, k), generator=g).to(torch.int32)
    pos[0], pos[1] = -1, torch.tensor([3, -1, -1])
    w, post, nxt = torch.rand(T, k, generator=g), r(width), r(width)
    add = torch.zeros(T, cols, dtype=torch.float64)
    for t in range(T):
        for j in range(k):
            add[t] += w[t, j].double() * (h[t] if pos[t, j] < 0 else y[pos[t, j]]).double()
    eps = 1e-5
    want = stream.double()
    want[:, :width] += R.rms(add[:, :width], eps) * post[:width].double()
    norm = R.rms(want[:, :width], eps) * nxt[:width].double()
    sd, out = stream.to(DEV), h.clone().to(DEV)          # (the norm's output takes the place of the experts' input)
    stream_norm(sd, nxt.to(DEV), eps, out, width=width, y=y.to(DEV), pair_pos=pos.to(DEV), pair_w=w.to(DEV), post_w=post.to(DEV),
                ident=out, norm_offset=0.0)
    assert (sd.double().cpu() - want).abs().max() < 2e-5
    assert (out.double().cpu()[:, :width] - norm).abs().max() < (2e-5 if dtype == F32 else 2e-2) * norm.abs().max().clamp_min(1)
    a = r(T, width)
    want[:, :width] += R.rms(a[:, :width].double(), eps) * post[:width].double()
    stream_norm(sd, nxt.to(DEV), eps, out, width=width, a=a.to(DEV), post_w=post.to(DEV), norm_offset=0.0)
    assert (sd.double().cpu() - want).abs().max() < 3e-5


@pytest.mark.parametrize("n,identity,count,keep,top", [(16, 4, 4, 2, 3), (15, 0, 5, 1, 3), (8, 8, 1, 1, 5), (160, 32, 8, 3, 8), (6, 2, 2, 2, 6)])
def test_grouped_choice(n, identity, count, keep, top):
    """Groups by their best corrected score, weights without the correction; negative choice scores."""
    from vllm_cpp_b200.ops import moe as M
    g = torch.Generator().manual_seed(6)
    z = torch.randn(200, n + 3, generator=g) * 2
    corr = torch.randn(n, generator=g) * 0.2 - 0.3
    s = torch.softmax(z[:, :n].double(), -1)
    eligible = R.keep_groups(s + corr.double(), count, keep)
    want = eligible.topk(top, -1).indices.sort(-1).values
    zd = z.to(DEV)
    ids, w = M.router_topk(zd[:, :n], top, renorm=False, e_bias=corr.to(DEV), n_group=count, topk_group=keep, group_best=1)
    got, order = ids.cpu().long().sort(-1)
    assert torch.equal(got, want)
    assert (w.cpu().gather(1, order).double() - s.gather(1, want)).abs().max() < 1e-6
    rid, rw = M.ref_router_topk(z[:, :n], top, renorm=False, e_bias=corr, n_group=count, topk_group=keep, group_best=1)
    assert torch.equal(rid.long().sort(-1).values, want)
