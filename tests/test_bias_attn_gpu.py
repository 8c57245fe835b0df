"""Kernels of the mixed-head attention with a distance bias, the fp32 stream and the clamped experts
against plain PyTorch, over sizes that take the tensor-core kernels and sizes that do not."""
import math
import random

import pytest
import torch

import nufusun_reference as R

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _status():
    from vllm_cpp_b200 import ops
    assert ops.read_status() == 0


# (H, G, dim, vdim, block_size, bias_max)
SHAPES = [(8, 4, 32, 48, 16, 40), (4, 1, 64, 64, 32, 200), (6, 3, 16, 24, 8, 30), (12, 2, 72, 136, 64, 90),
          (32, 4, 128, 128, 32, 1024), (20, 1, 96, 256, 128, 64),
          (96, 6, 40, 40, 32, 50), (16, 16, 64, 64, 64, 70), (24, 8, 160, 16, 32, 300), (40, 2, 64, 128, 16, 100), (5, 5, 20, 12, 16, 50), (3, 1, 7, 11, 16, 33)]


def _case(shape, lens, seed, dtype):
    """Paged cache with scattered pages, queries with one key that stands out for some rows."""
    H, G, D, V, bs, bmax = shape
    g = torch.Generator().manual_seed(seed)
    rnd = random.Random(seed)
    kw, vw = G * D, G * V
    need = [(n + bs - 1) // bs for n in lens]
    nb = sum(need) + 3
    pages = list(range(1, nb))
    rnd.shuffle(pages)
    bt = torch.zeros(len(lens), max(need) + 1, dtype=torch.int32)
    cache = torch.randn(nb, bs * (kw + vw), generator=g) * 0.7
    keys, vals = [], []
    for r, n in enumerate(lens):
        ids = [pages.pop() for _ in range(need[r])]
        bt[r, :len(ids)] = torch.tensor(ids, dtype=torch.int32)
    cache = cache.to(dtype)
    for r, n in enumerate(lens):
        pg = cache[bt[r, :need[r]].long()]
        keys.append(pg[:, : bs * kw].reshape(-1, kw)[:n].double())
        vals.append(pg[:, bs * kw:].reshape(-1, G, V)[:n].double())
    rel = torch.randn(2 * max(2, min(16, bmax // 4)), H, generator=g)
    return cache, bt, keys, vals, rel


def _oracle(q, keys, vals, pos, rel, bmax, G):
    """q [H, kw] mixed rows at ``pos`` -> [H * V]."""
    H = q.shape[0]
    s = q.double() @ keys[: pos + 1].T + R.distance_bias(pos, rel.double(), bmax)
    p = R.softmax_with_null(s)
    v = vals[: pos + 1][:, [h // (H // G) for h in range(H)]]
    return torch.einsum("hj,jhv->hv", p, v).reshape(-1)


def _q(rows, H, kw, keys_of, g, dtype):
    """Random query rows; every other row is pulled towards one key, so that a missed key shows."""
    q = torch.randn(rows, H, kw, generator=g) / math.sqrt(kw)
    for t in range(0, rows, 2):
        ks, pos = keys_of(t)
        j = int(torch.randint(0, pos + 1, (1,), generator=g))
        k = ks[j].float()
        q[t] += k * (12.0 / float(k @ k))
    return q.to(dtype)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("shape", SHAPES)
def test_decode(shape, dtype):
    from vllm_cpp_b200.ops import bias_attn as A
    H, G, D, V, bs, bmax = shape
    lens = [1, 2, bs - 1, bs, bs + 1, 31, 32, 33, 64, 65, bmax, bmax + 1, 257, 700]
    cache, bt, keys, vals, rel = _case(shape, lens, 1, dtype)
    g = torch.Generator().manual_seed(2)
    kw = G * D
    q = _q(len(lens), H, kw, lambda t: (keys[t], lens[t] - 1), g, dtype)
    want = torch.stack([_oracle(q[r], keys[r], vals[r], lens[r] - 1, rel, bmax, G) for r in range(len(lens))])
    bias = A.distance_bias_table(rel, bmax).to(DEV)
    cache, bt = cache.to(DEV), bt.to(DEV)
    ldq = (H * kw + 7) // 8 * 8
    qd = torch.zeros(len(lens) + 1, ldq, dtype=dtype, device=DEV)
    qd[:len(lens), :H * kw] = q.reshape(len(lens), -1).to(DEV)
    sl = torch.tensor(lens + [0], dtype=torch.int32, device=DEV)      # the last row is a padding row
    bt = torch.cat([bt, torch.zeros_like(bt[:1])])
    tol = 8e-3 if dtype == torch.bfloat16 else 2e-6
    for splits in (1, 3, 8):
        for any_size in (False, True):
            out = torch.full((len(lens) + 1, (H * V + 7) // 8 * 8), 7.0, dtype=dtype, device=DEV)
            A.decode(qd, cache, out, block_table=bt, seq_lens=sl, H=H, G=G, kw=kw, vdim=V, block_size=bs, bias=bias,
                     null_entry=True, splits=splits, any_size=any_size)
            got = out[:len(lens), :H * V].double().cpu()
            err = (got - want).norm(dim=1) / want.norm(dim=1)
            assert err.max() < tol, (splits, any_size, err.tolist())
            assert (out[len(lens), :H * V] == 0).all()
            assert (out[:, H * V:] == 7).all()
    _status()
    kind = A.kernel_kind("decode", qd, cache, H=H, G=G, kw=kw, vdim=V, block_size=bs)
    assert kind == ("tensor-core" if dtype == torch.bfloat16 and kw % 8 == 0 and V % 8 == 0 else "any-size")


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("shape", SHAPES)
def test_prefill(shape, dtype):
    from vllm_cpp_b200.ops import bias_attn as A
    H, G, D, V, bs, bmax = shape
    portions = [(0, 2), (0, 1), (5, 3), (bs - 1, 2), (63, 66), (0, 130), (200, 129), (bmax, 40)]     # (context, new)
    lens = [c + n for c, n in portions]
    cache, bt, keys, vals, rel = _case(shape, lens, 3, dtype)
    g = torch.Generator().manual_seed(4)
    kw = G * D
    row_of = [(r, c + i) for r, (c, n) in enumerate(portions) for i in range(n)]
    T = len(row_of)
    q = _q(T, H, kw, lambda t: (keys[row_of[t][0]], row_of[t][1]), g, dtype)
    check = sorted(set(list(range(0, T, 7)) + [i for i in range(T) if row_of[i][1] in (0, 1, bs - 1, bs, 63, 64, bmax, bmax + 1)]
                       + [T - 1]))
    want = torch.stack([_oracle(q[t], keys[row_of[t][0]], vals[row_of[t][0]], row_of[t][1], rel, bmax, G) for t in check])
    bias = A.distance_bias_table(rel, bmax).to(DEV)
    cache, bt = cache.to(DEV), bt.to(DEV)
    qd = torch.zeros(T, (H * kw + 7) // 8 * 8, dtype=dtype, device=DEV)
    qd[:, :H * kw] = q.reshape(T, -1).to(DEV)
    qs = [0]
    tr, tq = [], []
    for r, (_, n) in enumerate(portions):
        qs.append(qs[-1] + n)
        for x in range(0, n, 128):
            tr.append(r)
            tq.append(x)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)      # noqa: E731
    tol = 8e-3 if dtype == torch.bfloat16 else 2e-6
    for any_size in (False, True):
        out = torch.full((T, (H * V + 7) // 8 * 8), 7.0, dtype=dtype, device=DEV)
        A.prefill(qd, cache, out, block_table=bt, seq_lens=i32(lens), q_start=i32(qs), num_reqs=len(lens),
                  tile_req=i32(tr), tile_q0=i32(tq), H=H, G=G, kw=kw, vdim=V, block_size=bs, bias=bias,
                  null_entry=True, any_size=any_size)
        got = out[:, :H * V].double().cpu()[check]
        err = (got - want).norm(dim=1) / want.norm(dim=1)
        assert err.max() < tol, (any_size, err.max(), check[int(err.argmax())], row_of[check[int(err.argmax())]])
        assert (out[:, H * V:] == 7).all()
    _status()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("shape,T", [((8, 4, 32, 48, 16, 0), 3), ((32, 4, 128, 128, 32, 0), 700), ((3, 1, 7, 11, 16, 0), 9),
                                     ((12, 6, 20, 12, 8, 0), 301)])
def test_head_mix_and_cache_write(shape, T, dtype):
    from vllm_cpp_b200.ops import bias_attn as A
    H, G, D, V, bs, _ = shape
    g = torch.Generator().manual_seed(5)
    kw, vw = G * D, G * V
    n8 = (H * D + kw + vw + 7) // 8 * 8
    qkv = torch.randn(T, n8, generator=g)
    mix = torch.randn(H, H, generator=g)
    nb = (T + bs - 1) // bs + 2
    slots = torch.randperm(nb * bs, generator=g)[:T]
    slots[T // 2] = -1
    cache = torch.zeros(nb, bs * (kw + vw), dtype=dtype, device=DEV)
    q_out = torch.zeros(T, (H * kw + 7) // 8 * 8, dtype=dtype, device=DEV)
    A.head_mix_kv(qkv.to(DEV), mix.to(DEV), q_out, slots.to(DEV), cache, H=H, G=G, dim=D, vdim=V, block_size=bs)
    q = qkv[:, :H * D].double().view(T, H, D)
    keys = torch.randn(G, D, generator=g).double()
    # the defining property: one dot product with a full key row is the mixed score
    want = torch.einsum("hg,tg->th", mix.double(), torch.einsum("tgd,gd->tg", q, keys[[h // (H // G) for h in range(H)]]))
    got = torch.einsum("thk,k->th", q_out[:, :H * kw].double().cpu().view(T, H, kw), keys.reshape(-1))
    tol = 1e-2 if dtype == torch.bfloat16 else 1e-5
    assert (got - want).norm() / want.norm() < tol
    flat = cache.cpu()
    k = flat[:, :bs * kw].reshape(nb * bs, kw)
    v = flat[:, bs * kw:].reshape(nb * bs, vw)
    ok = slots >= 0
    assert torch.equal(k[slots[ok]], qkv[ok, H * D:H * D + kw].to(dtype))
    assert torch.equal(v[slots[ok]], qkv[ok, H * D + kw:H * D + kw + vw].to(dtype))
    untouched = torch.ones(nb * bs, dtype=torch.bool)
    untouched[slots[ok]] = False
    assert (k[untouched] == 0).all() and (v[untouched] == 0).all()
    _status()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("T,W", [(1, 100), (5, 192), (33, 2048), (3, 5000)])
def test_stream_norm(T, W, dtype):
    from vllm_cpp_b200.ops.stream import stream_norm
    g = torch.Generator().manual_seed(6)
    C, k, eps = (W + 7) // 8 * 8, 3, 1e-4

    def pad(x):
        out = torch.zeros(*x.shape[:-1], C, dtype=x.dtype)
        out[..., :W] = x
        return out

    table, w = torch.randn(50, W, generator=g).to(dtype), torch.randn(W, generator=g) * 0.3
    ids = torch.randint(0, 50, (T,), generator=g)
    stream = torch.full((T, C), 9.0, device=DEV)
    out = torch.empty(T, C, dtype=dtype, device=DEV)
    tol = 6e-3 if dtype == torch.bfloat16 else 1e-6
    stream_norm(stream, pad(w).to(DEV), eps, out, width=W, ids=ids.to(DEV), table=pad(table).to(DEV), scale=1.7)
    x = table[ids].double() * 1.7
    assert torch.allclose(stream[:, :W].double().cpu(), x, atol=1e-6)
    assert (out[:, :W].double().cpu() - R.rms_norm(x, w.double(), eps)).norm() / W ** 0.5 / T ** 0.5 < tol
    a, y = torch.randn(T, W, generator=g), torch.randn(T * k, W, generator=g).to(dtype)
    pos = torch.randperm(T * k, generator=g).view(T, k).int()
    pos[0, 1] = -1
    pw = torch.rand(T, k, generator=g)
    for weights in (None, pw):
        stream_norm(stream, pad(w).to(DEV), eps, out, width=W, a=pad(a).to(DEV), y=pad(y).to(DEV), pair_pos=pos.to(DEV),
                    pair_w=None if weights is None else weights.to(DEV))
        wt = (torch.ones(T, k) if weights is None else weights).double() * (pos >= 0)
        x = x + a.double() + (y.double()[pos.long().clamp(min=0)] * wt[..., None]).sum(1)
        assert (stream[:, :W].double().cpu() - x).abs().max() < 1e-5
        assert (out[:, :W].double().cpu() - R.rms_norm(x, w.double(), eps)).norm() / W ** 0.5 / T ** 0.5 < tol
    assert (stream[:, W:] == 0).all() and (out[:, W:] == 0).all()
    _status()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("T,W,F,E,top", [(1, 64, 40, 3, 1), (70, 192, 96, 5, 2), (513, 256, 136, 16, 4), (9, 128, 64, 1, 1)])
def test_clamped_experts(T, W, F, E, top, dtype):
    from vllm_cpp_b200.ops import moe as M
    g = torch.Generator().manual_seed(7)
    limit = 0.9
    h = torch.randn(T, W, generator=g).to(dtype)
    router = torch.randn(E, W, generator=g).div(W ** 0.25).to(dtype)      # some scores round to 1 in fp32
    gate, up = (torch.randn(E, F, W, generator=g).div(W ** 0.5).to(dtype) for _ in range(2))
    down = torch.randn(E, W, F, generator=g).div(F ** 0.5).to(dtype)
    logits = (h.float() @ router.float().T).to(DEV)
    ids, w = M.router_topk(logits, top, renorm=False, scoring="sigmoid")
    want_ids, want_w = R.route(h.double(), router.double(), top)
    assert torch.equal(ids.cpu().long(), want_ids) and (w.cpu() - want_w).abs().max() < 1e-5
    saturated = torch.tensor([[30.0, 31.0, 29.0, 40.0, 33.0]], device=DEV)
    assert M.router_topk(saturated, 2, renorm=False, scoring="sigmoid")[0].tolist() == [[3, 4]]
    ws = M.MoeWorkspace(DEV, T, top, E, W, F, dtype)
    y = M.clamped_experts(h.to(DEV), ids, w, torch.cat([gate, up], 1).to(DEV), down.to(DEV), ws, limit=limit,
                          alpha=1.702, up_offset=1.0)
    got = y[ws.pair_pos[: T * top].long()].view(T, top, W).double().sum(1).cpu()
    tensors = {"router": router}
    for e in range(E):
        tensors.update({f"e{e}.gate": gate[e], f"e{e}.up": up[e], f"e{e}.down": down[e]})
    want = R.experts(h.double(), lambda n: tensors[n].double(),
                     {"router": {"experts": E, "top": top}, "expert": {"limit": limit}})
    assert (got - want).norm() / want.norm() < (6e-3 if dtype == torch.bfloat16 else 1e-6)
    _status()


def test_fp32_product():
    from vllm_cpp_b200.ops.stream import gemm_f32
    g = torch.Generator().manual_seed(8)
    for M, N, K in ((1, 8, 8), (65, 130, 33), (200, 64, 1000)):
        a, w, b = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g), torch.randn(N, generator=g)
        got = gemm_f32(a.to(DEV), w.to(DEV), b.to(DEV)).double().cpu()
        want = a.double() @ w.double().T + b.double()
        assert (got - want).norm() / want.norm() < 1e-6
