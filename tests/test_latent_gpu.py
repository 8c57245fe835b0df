"""Kernels of the latent attention (norms, rotation and cache write, absorbed decode, prompts over expanded
keys and values, any-size forms) against the plain implementation."""
from types import SimpleNamespace

import pytest
import torch

import tabupel_reference as R
from test_maps_attn_gpu import i32, scatter
from vllm_cpp_b200.models.backend import GpuBackend
from vllm_cpp_b200.ops import latent as L
from vllm_cpp_b200.ops.reference import build_prefill_tiles

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
TOL = {BF: 1.5e-2, F32: 2e-5}

# heads, unrotated, rotated, value, query latent, key latent; pieces of 128 from one to four, more heads than
# one CTA of the decode kernel takes, and sizes beyond it
SHAPES = [(5, 64, 16, 80, 72, 64), (3, 40, 16, 24, 24, 100), (20, 128, 64, 128, 256, 512), (2, 24, 2, 40, 13, 200),
          (5, 100, 50, 90, 33, 300), (1, 8, 6, 5, 7, 9), (3, 64, 80, 48, 40, 64), (2, 32, 16, 32, 16, 600)]


def make(shape, lens, dtype, seed=0):
    """Random latents c, rotated key parts and query heads (before their rotation) per request."""
    H, D, rot, V, _, rank = shape
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, m=1.0: (torch.randn(*s, generator=g) * m).to(dtype).float()      # noqa: E731
    reqs = [(r(n, rank), r(n, rot), r(n, H, D + rot)) for n in lens]
    return reqs, r(H * D, rank, m=rank ** -0.5), r(H * V, rank, m=rank ** -0.5), [r(n, H) for n in lens]


def plain(c, kr, q, gate, uk, uv, at, scale, window, D):
    """-> [n, H, V] in float64 of the queries (rotated) at positions ``at``."""
    f, H = torch.float64, q.shape[1]
    k, v = (R.linear(c.to(f), w.to(f)).view(c.shape[0], H, -1) for w in (uk, uv))
    i, j = torch.tensor(at)[:, None], torch.arange(c.shape[0])[None]
    seen = (j <= i) & (i - j < window) if window else j <= i
    out = []
    for h in range(H):
        s = (q[:, h, :D].to(f) @ k[:, h].T + q[:, h, D:].to(f) @ kr.to(f).T) * scale
        out.append(torch.softmax(s.masked_fill(~seen, float("-inf")), -1) @ v[:, h] * torch.sigmoid(gate[:, h, None].to(f)))
    return torch.stack(out, 1)


def apart(x):
    """The rotated part's neighbouring pairs, half of it apart."""
    return torch.cat([x[..., 0::2], x[..., 1::2]], -1)


def run(shape, reqs, uk, uv, gates, portions, dtype, bs, scale, window, splits=1, expand=True):
    """The portions (rows already there, rows) of the requests; decode rows (one row) first."""
    H, D, rot, V, qr, rank = shape
    s, be = L.LatentShape(H=H, dim=D, rot=rot, vdim=V, q_rank=qr, rank=rank), GpuBackend(DEV)
    rows = []
    for (c, kr, _), (a, n) in zip(reqs, portions):
        x = torch.zeros(a + n, s.row)
        x[:, :rank], x[:, s.rankp: s.rankp + rot] = c[: a + n], apart(kr[: a + n])
        rows.append((x,))
    cache, table = scatter(rows, bs, dtype)
    if s.rankp > rank or s.rotp > rot:                       # (padding columns are zero in every page)
        v = cache.view(-1, bs, s.row)
        v[..., rank: s.rankp], v[..., s.rankp + rot:] = 0, 0
    nd = sum(n == 1 for _, n in portions)
    T = sum(n for _, n in portions)
    q = torch.zeros(T, H, s.qw)
    x = torch.cat([r[2][a: a + n] for r, (a, n) in zip(reqs, portions)])
    q[..., :D], q[..., s.qn: s.qn + rot] = x[..., :D], apart(x[..., D:])
    gate = torch.cat([y[a: a + n] for y, (a, n) in zip(gates, portions)]).to(dtype).to(DEV)
    w = {"uk_t": torch.zeros(H, s.rankp, s.qn), "uv": torch.zeros(H, s.V, s.rankp)}
    w["uk_t"][:, :rank, :D] = uk.view(H, D, rank).transpose(1, 2)
    w["uv"][:, :V, :rank] = uv.view(H, V, rank)
    kv = torch.zeros(H, s.D, s.rankp)
    kv[:, :D, :rank] = uk.view(H, D, rank)
    w["kv"] = torch.cat([kv.reshape(H * s.D, -1), w["uv"].reshape(H * s.V, -1)], 0)
    w = {k: v.to(dtype).to(DEV).contiguous() for k, v in w.items()}
    seq, n = [a + n for a, n in portions], [n for _, n in portions]
    pre = n[nd:]
    tr, tq = build_prefill_tiles(pre) if pre else ([0], [0])
    start = [sum(pre[:i]) for i in range(len(pre) + 1)]
    ctx = SimpleNamespace(num_decodes=nd, num_prefills=len(pre), num_tiles=len(tr) if pre else 0, seq_lens=i32(seq),
                          block_table=[table], prefill_q_start=i32(start), tile_req=i32(tr), tile_q0=i32(tq), decode_splits=splits,
                          extra={})

    def pages():
        first, base, total, bt = L.visible_pages(seq[nd:], pre, window, bs)
        return dict(first=i32(first.tolist()), base=i32(base.tolist()), total=total, table=torch.from_numpy(bt).to(DEV))
    expand = expand and L.prefill_kernel_fits(s, dtype, bs)
    new = lambda r, c: torch.zeros(r, c, dtype=dtype, device=DEV)                    # noqa: E731
    out = torch.full((T, H * s.V), float("nan"), dtype=dtype, device=DEV)
    pos = torch.cat([torch.arange(a, a + m) for a, m in portions]).to(DEV)
    turn = torch.cat([torch.ones(4096, rot // 2), torch.zeros(4096, rot // 2)], 1).to(DEV)     # (no rotation)
    be.latent_attention(q.reshape(T, -1).to(dtype).to(DEV), pos, turn, cache, w, s, ctx, 0, scale=scale, window=window,
                        block_size=bs, gate=gate, out=out, pages=pages if expand else None,
                        absorbed=lambda m: (new(m, H * s.row), new(m, H * s.rankp)), scratch=lambda _, r, c: new(r, c))
    got = out.double().cpu().view(T, H, s.V)
    assert not got[..., V:].any()
    want = torch.cat([plain(c[: a + m], kr[: a + m], x[a: a + m], y[a: a + m], uk, uv, list(range(a, a + m)), scale, window, D)
                      for (c, kr, x), y, (a, m) in zip(reqs, gates, portions)])
    return ((got[..., :V] - want).norm(dim=-1) / want.norm(dim=-1)).max().item()


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [BF, F32])
def test_decode(shape, dtype):
    lens = [1, 2, 64, 76, 77, 127, 128, 129, 200, 300, 411]
    reqs, uk, uv, gates = make(shape, lens, dtype, seed=1)
    for bs in (16, 64):
        for window, splits in ((0, 1), (76, 1), (76, 3), (128, 2), (129, 1), (1, 1), (0, 4)):
            e = run(shape, reqs, uk, uv, gates, [(n - 1, 1) for n in lens], dtype, bs, 0.8 * shape[1] ** -0.5, window, splits)
            assert e < TOL[dtype], (bs, window, splits)


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("bs", [8, 64, 256])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_portions_beside_decode_rows(shape, bs, dtype):
    portions = [(70, 1), (0, 1), (0, 2), (0, 130), (99, 3), (61, 200), (250, 131), (127, 5)]
    reqs, uk, uv, gates = make(shape, [a + n for a, n in portions], dtype, seed=2)
    for window in (76, 128, 1, 0):
        for expand in (True, False):
            if not expand and (dtype == F32 or window != 76):
                continue
            e = run(shape, reqs, uk, uv, gates, portions, dtype, bs, 0.8 * shape[1] ** -0.5, window, expand=expand)
            assert e < TOL[dtype], (window, expand)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_edges_of_windows(dtype):
    """One token's shared key part answers one query alone: just inside and just outside its window."""
    shape, n, window = (2, 32, 16, 16, 8, 48), 200, 50
    reqs, uk, uv, gates = make(shape, [n], dtype, seed=3)
    c, kr, q = reqs[0]
    for key in (0, 63, 64, 127, 128):
        k2, q2 = kr * 0.1, q.clone()
        k2[key] = 6.0
        at = key + window - 1
        q2[at: at + 2, :, 32:] = 1.0
        a, b = (plain(c, k2, q2, gates[0], uk, uv, list(range(n)), 0.5, w, 32) for w in (window, window - 1))
        assert (a[at] - b[at]).norm() > 0.3 * a[at].norm()
        for cut in (at, at + 1):
            for portions in ([(0, n)], [(cut, n - cut)], [(cut, 1)]):
                if portions[0][1] > 0:
                    assert run(shape, [(c, k2, q2)], uk, uv, gates, portions, dtype, 16, 0.5, window) < TOL[dtype]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [BF, F32])
def test_preparation(shape, dtype):
    H, D, rot, V, qr, rank = shape
    s, T, bs, eps = L.LatentShape(H=H, dim=D, rot=rot, vdim=V, q_rank=qr, rank=rank), 39, 8, 1e-5
    g = torch.Generator().manual_seed(4)
    freqs, mag = R.yarn_frequencies(3e3, rot, 5.0, 300, 20.0, 1.5)
    from vllm_cpp_b200 import ops
    table = ops.rope_table(torch.tensor(freqs, dtype=torch.float64, device=DEV), 900, mag)
    parts = [torch.randn(T, n, generator=g).to(dtype) for n in (qr, rank, rot, H)]
    down = torch.cat([torch.cat([apart(x) if i == 2 else x, torch.zeros(T, w - x.shape[1], dtype=dtype)], 1)
                      for i, (x, w) in enumerate(zip(parts, s.down))], 1)
    pad = lambda x, n: torch.cat([x, torch.zeros(n - x.numel())]).to(DEV)            # noqa: E731
    w1, w2 = torch.rand(qr, generator=g) + 0.5, torch.rand(rank, generator=g) + 0.5
    w = {"q_norm": pad(w1, s.down[0]), "kv_norm": pad(w2, s.down[1])}
    pos, slots = torch.randint(0, 900, (T,), generator=g), torch.randperm(96, generator=g)[:T]
    slots[3] = -1
    cq, cache = torch.full((T, s.down[0]), float("nan"), dtype=dtype, device=DEV), torch.zeros(12, bs * s.row, dtype=dtype, device=DEV)
    L.prepare(down.to(DEV), pos.to(DEV), table, w, s, eps, cq, slots.to(DEV), cache)
    tol = 2e-5 if dtype == F32 else 3e-2
    assert (cq.double().cpu()[:, :qr] - R.rms(parts[0].double(), eps) * w1.double()).abs().max() < tol
    assert not cq[:, qr:].any()
    turned = apart(R.rotate(parts[2].double()[:, None], pos, freqs, mag)[:, 0])
    latent = R.rms(parts[1].double(), eps) * w2.double()
    flat = cache.double().cpu().view(-1, s.row)
    ok = slots >= 0
    assert (flat[slots[ok], :rank] - latent[ok]).abs().max() < tol
    assert (flat[slots[ok], s.rankp: s.rankp + rot] - turned[ok]).abs().max() < tol
    assert int(flat.any(-1).sum()) == T - 1 and not flat[:, rank: s.rankp].any() and not flat[:, s.rankp + rot:].any()
    # queries: the first rows into absorbed rows, the others in place
    q = torch.randn(T, H, s.qw, generator=g).to(dtype)
    want = apart(R.rotate(torch.stack([q[..., s.qn: s.qn + rot // 2], q[..., s.qn + rot // 2: s.qn + rot]], -1).flatten(-2).double(),
                          pos, freqs, mag))
    qd, qa = q.reshape(T, -1).to(DEV), torch.zeros(7, H * s.row, dtype=dtype, device=DEV)
    L.queries(qd, pos.to(DEV), table, s, qa, 7)
    assert (qa.double().cpu().view(7, H, s.row)[..., s.rankp: s.rankp + rot] - want[:7]).abs().max() < tol
    got = qd.double().cpu().view(T, H, s.qw)
    assert (got[7:, :, s.qn: s.qn + rot] - want[7:]).abs().max() < tol
    assert torch.equal(got[..., : s.qn], q[..., : s.qn].double()) and torch.equal(got[:7], q[:7].double())
