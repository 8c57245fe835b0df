"""Kernels of the windowed attention with two maps a head (weighted norm and rotation, prompts, decode;
tensor-core and any-size forms) and of the maps' difference, each against the plain implementation."""
import pytest
import torch

import tabupel_reference as R
from vllm_cpp_b200.ops import bias_attn as A
from vllm_cpp_b200.ops.reference import build_prefill_tiles

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def scatter(rows, bs, dtype, seed=0):
    """Requests' page parts [(part [n, w], ...)] over pages in random order -> (pages, table). Positions nobody
    wrote and pages of others hold large finite values."""
    g = torch.Generator().manual_seed(seed)
    nb = [max(1, -(-r[0].shape[0] // bs)) for r in rows]
    order = torch.randperm(sum(nb) + 3, generator=g)
    widths = [p.shape[1] for p in rows[0]]
    pages = torch.full((len(order), bs * sum(widths)), 50.0)
    table, at = torch.zeros(len(rows), max(nb), dtype=torch.int32), 0
    for r, parts in enumerate(rows):
        for b in range(nb[r]):
            page = table[r, b] = int(order[at])
            at, off = at + 1, 0
            for part, w in zip(parts, widths):
                x = part[b * bs:(b + 1) * bs]
                pages[page, off: off + x.numel()] = x.reshape(-1)
                off += bs * w
    return pages.to(dtype).to(DEV), table.to(DEV)


def plain(q, k, v, at, scale, window, maps):
    """q [n, H, D], k [N, G, maps, D], v [N, G, V] -> [n, H, V] in float64; head h reads map h % maps."""
    f, H, G = torch.float64, q.shape[1], k.shape[1]
    i, j = torch.tensor(at)[:, None], torch.arange(k.shape[0])[None]
    seen = (j <= i) & (i - j < window) if window else j <= i
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h].to(f) @ k[:, g, h % maps].to(f).T * scale).masked_fill(~seen, float("-inf"))
        out.append(torch.softmax(s, -1) @ v[:, g].to(f))
    return torch.stack(out, 1)


def data(H, G, D, V, maps, lens, dtype, seed=0):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).to(dtype).float()      # noqa: E731
    return [(r(n, G, maps, D), r(n, G, V)) for n in lens], [r(n, H, D) for n in lens]


def setup(kv, bs, dtype):
    return scatter([(k.flatten(1), v.flatten(1)) for k, v in kv], bs, dtype)


# heads counted with their maps; the last: values that no tensor-core form takes
SHAPES = [(4, 2, 64, 48, 2), (12, 2, 48, 80, 2), (16, 1, 32, 128, 2), (36, 1, 64, 64, 2), (2, 1, 128, 256, 2), (8, 4, 16, 16, 1),
          (6, 3, 64, 96, 1), (20, 1, 112, 32, 1), (8, 2, 20, 36, 2)]
TOL = {BF: 8e-3, F32: 1e-5}


def shape_args(shape, bs):
    H, G, D, V, maps = shape
    return dict(H=H, G=G, kw=G * maps * D, vdim=V, block_size=bs, grouped=True, maps=maps)


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("bs", [16, 64])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_decode(shape, bs, dtype):
    H, G, D, V, maps = shape
    lens = [1, 2, 15, 16, 17, 44, 45, 64, 65, 100, 199, 200, 201, 257]
    kv, qs = data(H, G, D, V, maps, lens, dtype, seed=1)
    (pages, table), scale = setup(kv, bs, dtype), 1.7 * D ** -0.5
    q = torch.stack([x[-1] for x in qs]).reshape(len(lens), -1).to(dtype).to(DEV)
    for window in (0, 44, 64, 1, 17, 1000):
        want = torch.cat([plain(x[-1:], k, v, [n - 1], scale, window, maps) for x, (k, v), n in zip(qs, kv, lens)])
        for splits, any_size in ((1, False), (3, False), (1, True)):
            out = torch.full((len(lens), H * V), float("nan"), dtype=dtype, device=DEV)
            A.decode(q, pages, out, block_table=table, seq_lens=i32(lens), scale=scale, window=window, splits=splits,
                     any_size=any_size, **shape_args(shape, bs))
            d = (out.double().cpu().view_as(want) - want).norm(dim=-1) / want.norm(dim=-1)
            assert d.max() < TOL[dtype], (window, splits, any_size, int(d.max(-1).values.argmax()))
    kind = A.kernel_kind("decode", q, pages, scale=scale, window=64, **shape_args(shape, bs))
    assert kind == ("tensor-core" if dtype == BF and D % 16 == 0 else "any-size")


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("bs", [8, 64, 256])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_prompt_portions(shape, bs, dtype):
    """Portions that start anywhere: (rows already there, rows of the portion)."""
    H, G, D, V, maps = shape
    portions = [(0, 2), (0, 130), (99, 3), (100, 2), (61, 200), (250, 131), (127, 5)]
    lens = [a + n for a, n in portions]
    kv, qs = data(H, G, D, V, maps, lens, dtype, seed=2)
    (pages, table), scale = setup(kv, bs, dtype), 1.7 * D ** -0.5
    rows = torch.cat([x[a:] for x, (a, _) in zip(qs, portions)])
    q = rows.reshape(rows.shape[0], -1).to(dtype).to(DEV)
    n = [x for _, x in portions]
    tr, tq = build_prefill_tiles(n)
    start = [sum(n[:i]) for i in range(len(n) + 1)]
    for window in (100, 128, 37, 1, 0):
        want = torch.cat([plain(x[a:], k, v, list(range(a, a + m)), scale, window, maps)
                          for x, (k, v), (a, m) in zip(qs, kv, portions)])
        for any_size in (False, True):
            out = torch.full((rows.shape[0], H * V), float("nan"), dtype=dtype, device=DEV)
            A.prefill(q, pages, out, block_table=table, seq_lens=i32(lens), q_start=i32(start), num_reqs=len(n),
                      tile_req=i32(tr), tile_q0=i32(tq), scale=scale, window=window, any_size=any_size, **shape_args(shape, bs))
            d = (out.double().cpu().view_as(want) - want).norm(dim=-1) / want.norm(dim=-1)
            assert d.max() < TOL[dtype], (window, any_size, int(d.max(-1).values.argmax()))
        if dtype == F32:
            break
    kind = A.kernel_kind("prefill", q, pages, scale=scale, window=37, **shape_args(shape, bs))
    assert kind == ("tensor-core" if dtype == BF and D % 16 == 0 and V % 8 == 0 else "any-size")


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("window", [48, 33])
def test_edges_of_windows_and_pages(window, dtype):
    """One key of one map carries the whole weight: just inside and just outside a window, at the borders of
    pages, in decode and in prompts; the other map sees nothing of it."""
    H, G, D, V, n, bs = 2, 1, 64, 16, 150, 16
    for key in (0, 15, 16, 47, 48, 95, 101):
        kv, qs = data(H, G, D, V, 2, [n], dtype, seed=3)
        k, v = kv[0]
        k[key, :, 1] = 8.0
        v[key] = 5.0
        q = torch.full((n, H, D), 0.5)
        pages, table = setup([(k, v)], bs, dtype)
        want = plain(q, k, v, list(range(n)), 0.3, window, 2)
        seen = [i for i in range(n) if 0 <= i - key < window]
        assert all((want[i, 1].mean() > 4.9) == (i in seen) for i in range(n))
        qd = q.reshape(n, -1).to(dtype).to(DEV)
        out = torch.empty(n, H * V, dtype=dtype, device=DEV)
        tr, tq = build_prefill_tiles([n])
        args = shape_args((H, G, D, V, 2), bs)
        A.prefill(qd, pages, out, block_table=table, seq_lens=i32([n]), q_start=i32([0, n]), num_reqs=1, tile_req=i32(tr),
                  tile_q0=i32(tq), scale=0.3, window=window, **args)
        assert (out.double().cpu().view_as(want) - want).abs().max() < 0.05
        A.decode(qd, pages, out, block_table=table.expand(n, -1).contiguous(), seq_lens=i32(list(range(1, n + 1))),
                 scale=0.3, window=window, splits=2, **args)
        assert (out.double().cpu().view_as(want) - want).abs().max() < 0.05


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("shape", [(4, 2, 2, 64, 48, 64), (2, 2, 1, 24, 16, 10), (6, 2, 1, 100, 36, 48), (2, 4, 2, 128, 256, 128),
                                   (2, 2, 2, 16, 8, 0)])
def test_weighted_norm_rotation_and_cache(dtype, shape):
    """Query, key and value heads of different counts; neighbouring pairs stored half the rotation apart."""
    H, G, GV, dim, V, rot = shape
    D, T, bs, base, eps = (dim + 15) // 16 * 16, 77, 16, 5e4, 1e-5
    g = torch.Generator().manual_seed(4)
    x = torch.randn(T, H + G, dim, generator=g).to(dtype)
    v = torch.randn(T, GV * V, generator=g).to(dtype)
    w = torch.rand(2, dim, generator=g) + 0.5
    order = list(range(0, rot, 2)) + list(range(1, rot, 2)) + list(range(rot, dim))
    pad = lambda t: torch.cat([t[..., order], torch.zeros(*t.shape[:-1], D - dim, dtype=t.dtype)], -1)      # noqa: E731
    qkv = torch.cat([pad(x).flatten(1), v], 1)
    pos = torch.randint(0, 3000, (T,), generator=g)
    slots = torch.randperm(200, generator=g)[:T]
    slots[5] = -1
    freqs = R.linear_frequencies(base, rot, 3.0)
    weight = torch.cat([w[:1].expand(H, dim), w[1:].expand(G, dim)], 0).double()
    want = pad(R.rotate(R.rms(x.double(), eps) * weight, pos, freqs))
    table = None
    if rot:
        from vllm_cpp_b200 import ops
        table = ops.rope_table(torch.tensor(freqs, dtype=torch.float64, device=DEV), 3000)
    cache = torch.full((13, bs * (G * D + GV * V)), 9.0, dtype=dtype, device=DEV)
    q = torch.full((T, H * D), float("nan"), dtype=dtype, device=DEV)
    A.rotate_kv(qkv.to(DEV), pos.to(DEV), table, rot, eps, q, slots.to(DEV), cache, H=H, G=G, value_heads=GV, D=D, V=V, dim=dim,
                block_size=bs, q_w=pad(w)[0].to(DEV), k_w=pad(w)[1].to(DEV))
    tol = 3e-5 if dtype == F32 else 3e-2
    assert (q.double().cpu().view(T, H, D) - want[:, :H]).abs().max() < tol
    keys, vals = A.page_views(cache.cpu(), bs, G * D)
    for t in range(T):
        if slots[t] >= 0:
            b, o = divmod(int(slots[t]), bs)
            assert (keys[b, o].double().view(G, D) - want[t, H:]).abs().max() < tol
            assert torch.equal(vals[b, o], v[t])
    assert int((keys.reshape(-1, G * D) == 9.0).all(-1).sum()) == 13 * bs - (T - 1)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("shape", [(3, 40), (1, 128), (5, 256), (2, 7), (4, 600)])
def test_difference_of_maps(dtype, shape):
    H, vdim = shape
    V, T = (vdim + 15) // 16 * 16, 33
    g = torch.Generator().manual_seed(5)
    x = torch.zeros(T, H, 2, V)
    x[..., :vdim] = torch.randn(T, H, 2, vdim, generator=g)
    x = x.to(dtype)
    want = R.rms(x[:, :, 0, :vdim].double() - 0.7 * x[:, :, 1, :vdim].double(), 1e-3) * 0.6
    out = torch.full((T, H * V), float("nan"), dtype=dtype, device=DEV)
    A.diff_combine(x.reshape(T, -1).to(DEV), out, H=H, V=V, vdim=vdim, lam=0.7, eps=1e-3, scale=0.6)
    got = out.double().cpu().view(T, H, V)
    assert (got[..., :vdim] - want).abs().max() < (1e-5 if dtype == F32 else 2e-2)
    assert not got[..., vdim:].any()


def test_stream_takes_a_multiple_of_the_update():
    from vllm_cpp_b200.ops.stream import softcap_f32, stream_norm
    g = torch.Generator().manual_seed(6)
    for width in (40, 1024, 5000):
        x, a, w = torch.randn(9, width, generator=g), torch.randn(9, width, generator=g), torch.randn(width, generator=g)
        want = x.double() + 0.3 * a.double()
        s, out = x.to(DEV), torch.empty(9, width, device=DEV)
        stream_norm(s, w.to(DEV), 1e-5, out, width=width, a=a.to(DEV), norm_offset=0.0, mult=0.3)
        assert (s.double().cpu() - want).abs().max() < 1e-6
        assert (out.double().cpu() - R.rms(want, 1e-5) * w.double()).abs().max() < 2e-5
        z = (x * 40).to(DEV)
        softcap_f32(z, 30.0)
        assert (z.double().cpu() - R.softcap(x.double() * 40, 30.0)).abs().max() < 1e-4
