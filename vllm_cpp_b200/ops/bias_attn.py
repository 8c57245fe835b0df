"""Attention over pages ``[block_size, kw] keys | [block_size, G * vdim] values``: grouped heads (each reads
the key columns of its group) or heads mixed before the softmax, with an optional distance bias, null
softmax entry and limit to the query's chunk or window of positions. With two ``maps`` every head has two
queries and every group two keys over the same values (``diff_combine`` joins the two outputs).

The mix of the heads is moved to the query side (``head_mix_kv``): head ``h`` reads the whole key
row of a token with the query row ``[sum_{g in group 0} M[h, g] q_g | sum_{g in group 1} ... ]``."""
from __future__ import annotations

import ctypes
import math
from typing import NamedTuple, Optional

import torch

from . import _lib
from ._lib import check, lib, ptr, stream_ptr

_P, _L, _I = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int


class BiasAttnArgs(ctypes.Structure):
    _fields_ = [("q", _P), ("ldq", _L), ("out", _P), ("ldo", _L), ("cache", _P), ("num_blocks", _L),
                ("block_table", _P), ("seq_lens", _P), ("q_start", _P), ("bias", _P), ("tmp_o", _P),
                ("tmp_lse", _P), ("tile_req", _P), ("tile_q0", _P),
                ("max_blocks", _I), ("num_reqs", _I), ("rows", _I), ("H", _I), ("G", _I), ("kw", _I), ("vdim", _I),
                ("block_size", _I), ("bias_len", _I), ("null_entry", _I), ("f32", _I), ("splits", _I),
                ("num_tiles", _I), ("grouped", _I), ("chunk", _I), ("scale", ctypes.c_float),
                ("window", _I), ("maps", _I), ("values_in_keys", _I), ("shared", _I), ("gate", _P), ("ldg", _L),
                ("keys", _P), ("values", _P), ("shared_keys", _P), ("ldk", _L), ("ldv", _L), ("lds", _L),
                ("sink", _P), ("key_at", _I), ("out_scale", ctypes.c_float)]


class SplitRows(NamedTuple):
    """Key and value rows outside a page tensor, ``block_size`` consecutive rows to a page, and key columns that
    every head shares (a head's query row: its own columns padded to whole 64-wide chunks, then these)."""
    keys: torch.Tensor
    values: torch.Tensor
    shared: Optional[torch.Tensor] = None


_declared = False


def _declare():
    global _declared
    if _declared:
        return
    P, I, L = _lib.P, _lib.I, ctypes.c_longlong
    A = ctypes.POINTER(BiasAttnArgs)
    _lib.declare("b200_head_mix_kv", [P, L, P, P, L, P, P, I, I, I, I, I, I, I, P], I)
    _lib.declare("b200_rotate_kv", [P, L, P, P, I, _lib.F, P, P, P, L, P, P, I, I, I, I, I, I, I, I, I, P], I)
    _lib.declare("b200_rotate_tied", [P, L, P, P, I, P, L, P, P, I, I, I, I, I, I, P], I)
    _lib.declare("b200_diff_combine", [P, L, P, L, I, I, I, I, _lib.F, _lib.F, _lib.F, I, P], I)
    _lib.declare("b200_bias_attn_kernel", [A, I], I)
    _lib.declare("b200_bias_attn_decode", [A, I, P], I)
    _lib.declare("b200_bias_attn_prefill", [A, I, P], I)
    lib()
    _declared = True


def head_mix_kv(qkv, mix, q_out, slots, cache, *, H, G, dim, vdim, block_size):
    """fp32 ``qkv`` rows ``[q | k | v]`` -> mixed query rows ``q_out`` [T, H * G * dim] and this
    step's keys and values in ``cache`` (slot < 0: none), in the type of ``q_out``."""
    _declare()
    assert qkv.dtype == torch.float32 and mix.dtype == torch.float32 and q_out.dtype == cache.dtype
    check(lib().b200_head_mix_kv(ptr(qkv), qkv.stride(0), ptr(mix), ptr(q_out), q_out.stride(0), ptr(slots),
                                 ptr(cache), H, G, dim, vdim, block_size, qkv.shape[0],
                                 int(q_out.dtype == torch.float32), stream_ptr()), "head_mix_kv")


def rotate_kv(qkv, positions, table, rot, eps, q_out, slots, cache, *, H, G, D, V, dim, block_size, q_w=None, k_w=None,
              value_heads=None):
    """Rows ``[q | k | v]`` (``G`` 0: q alone) -> q and k heads rotated over their first ``rot`` dimensions
    (pairs half of ``rot`` apart, ``table`` [positions, cos | sin]) and divided by their root mean square
    over ``dim``; q to ``q_out`` [T, H * D], k and v to ``cache`` (slot < 0: none). With weights ``q_w`` /
    ``k_w`` fp32 [D] the heads are normed and weighted first, then rotated. ``value_heads``: as many as ``G``."""
    _declare()
    assert qkv.dtype == q_out.dtype and (cache is None or cache.dtype == q_out.dtype)
    check(lib().b200_rotate_kv(ptr(qkv), qkv.stride(0), ptr(positions), ptr(table), rot, eps, ptr(q_w), ptr(k_w), ptr(q_out),
                               q_out.stride(0), ptr(slots), ptr(cache), H, G, G if value_heads is None else value_heads, D, V,
                               dim, block_size, qkv.shape[0], int(q_out.dtype == torch.float32), stream_ptr()), "rotate_kv")


class TiedShape(NamedTuple):
    """Keys and values from one projection: a group's cache row is ``[first, not rotated | rest | first, rotated]``, the value
    is its first ``D`` columns and the key its last ``D``. ``rot`` dimensions are rotated, ``r8`` is that padded to 8s."""
    H: int
    G: int
    dim: int
    rot: int

    @property
    def r8(self) -> int:
        return (self.rot + 7) // 8 * 8

    @property
    def D(self) -> int:
        return (self.r8 + self.dim - self.rot + 15) // 16 * 16

    @property
    def pitch(self) -> int:
        return self.D + self.r8

    def spread(self, t: torch.Tensor, heads: int, axis: int = 0) -> torch.Tensor:
        """Each head's rows (or columns) of a projection in the order ``[first | rest]`` with the padding in place."""
        t = t.transpose(0, axis).reshape(heads, self.dim, -1)
        out = torch.zeros((heads, self.D, t.shape[2]), dtype=t.dtype, device=t.device)
        out[:, : self.rot], out[:, self.r8: self.r8 + self.dim - self.rot] = t[:, : self.rot], t[:, self.rot:]
        return out.reshape(heads * self.D, -1).transpose(0, axis)


def rotate_tied(qk, positions, table, q_out, slots, cache, s: TiedShape, *, block_size):
    """Rows ``[q heads | k heads]`` of ``s.D`` columns each (:meth:`TiedShape.spread`) -> rotated queries ``[rest | first]`` to
    ``q_out`` [T, H * D] and this step's cache rows (slot < 0: none). The rotated pairs lie half of ``rot`` apart."""
    _declare()
    assert qk.dtype == q_out.dtype == cache.dtype
    check(lib().b200_rotate_tied(ptr(qk), qk.stride(0), ptr(positions), ptr(table), s.rot, ptr(q_out), q_out.stride(0), ptr(slots),
                                 ptr(cache), s.H, s.G, s.D, block_size, qk.shape[0], int(q_out.dtype == torch.float32),
                                 stream_ptr()), "rotate_tied")


def diff_combine(maps, out, *, H, V, vdim, lam, eps, scale):
    """``maps`` [T, H * 2 * V] -> per head o = first - ``lam`` second, over its root mean square over ``vdim``,
    times ``scale``; ``out`` [T, H * V]."""
    _declare()
    check(lib().b200_diff_combine(ptr(maps), maps.stride(0), ptr(out), out.stride(0), H, V, vdim, maps.shape[0], lam, eps, scale,
                                  int(out.dtype == torch.float32), stream_ptr()), "diff_combine")
    return out


def _args(q, cache, out, block_table, seq_lens, H, G, kw, vdim, block_size, bias, null_entry, scale, chunk, window,
          maps, grouped, gate, values_in_keys, rows=None, sink=None, key_at=0, out_scale=1.0) -> BiasAttnArgs:
    a = BiasAttnArgs()
    a.sink, a.key_at, a.out_scale = ptr(sink), key_at, out_scale
    a.q, a.ldq, a.out, a.ldo = ptr(q), q.stride(0), ptr(out), out.stride(0)
    if rows is None:
        a.cache, a.num_blocks = ptr(cache), cache.shape[0]
    else:
        a.num_blocks = rows.keys.shape[0] // block_size
        a.keys, a.ldk, a.values, a.ldv = ptr(rows.keys), rows.keys.stride(0), ptr(rows.values), rows.values.stride(0)
        if rows.shared is not None:
            a.shared_keys, a.lds, a.shared = ptr(rows.shared), rows.shared.stride(0), q.shape[1] // H - -(-kw // G // 64) * 64
    a.block_table, a.max_blocks, a.seq_lens = ptr(block_table), block_table.stride(0), ptr(seq_lens)
    a.bias, a.bias_len = ptr(bias), bias.shape[1] if bias is not None else 0
    a.rows, a.num_reqs = q.shape[0], q.shape[0]
    a.H, a.G, a.kw, a.vdim, a.block_size = H, G, kw, vdim, block_size
    a.null_entry, a.f32, a.splits = int(null_entry), int(q.dtype == torch.float32), 1
    a.scale, a.chunk, a.window, a.maps, a.grouped = scale, chunk, window, maps, int(grouped)
    a.values_in_keys = int(values_in_keys)
    a.gate, a.ldg = ptr(gate), gate.stride(0) if gate is not None else 0
    return a


def decode(q, cache, out, *, block_table, seq_lens, H, G, kw, vdim, block_size, bias=None, null_entry=False,
           splits=1, tmp=None, any_size=False, scale=1.0, chunk=0, window=0, maps=1, grouped=False, gate=None,
           values_in_keys=False, sink=None, key_at=0, out_scale=1.0):
    """One query row per request, at its last position. ``gate`` [rows, H]: the outputs times its sigmoid (any-size
    kernel); ``values_in_keys``: values are the first ``vdim`` columns of a group's key row, its key the columns from
    ``key_at`` on. ``sink`` fp32 [H]: the softmax counts one more entry of that score without a value. The outputs are
    multiplied by ``out_scale``."""
    _declare()
    a = _args(q, cache, out, block_table, seq_lens, H, G, kw, vdim, block_size, bias, null_entry, scale, chunk, window, maps,
              grouped, gate, values_in_keys, None, sink, key_at, out_scale)
    if splits > 1:
        if tmp is None:
            tmp = (torch.empty(a.rows * H * splits * vdim, dtype=torch.float32, device=q.device),
                   torch.empty(a.rows * H * splits, dtype=torch.float32, device=q.device))
        assert tmp[0].numel() >= a.rows * H * splits * vdim and tmp[1].numel() >= a.rows * H * splits
        a.splits, a.tmp_o, a.tmp_lse = splits, ptr(tmp[0]), ptr(tmp[1])
    check(lib().b200_bias_attn_decode(ctypes.byref(a), int(any_size), stream_ptr()), "bias_attn_decode")
    return out


def prefill(q, cache, out, *, block_table, seq_lens, q_start, num_reqs, tile_req, tile_q0, H, G, kw, vdim,
            block_size, bias=None, null_entry=False, any_size=False, scale=1.0, chunk=0, window=0, maps=1, grouped=False,
            gate=None, values_in_keys=False, rows=None, sink=None, key_at=0, out_scale=1.0):
    """Portions of prompts; ``tile_req`` / ``tile_q0`` list their 128-row query tiles. ``rows``
    (:class:`SplitRows`, tensor-core kernel only) stands for ``cache``."""
    _declare()
    a = _args(q, cache, out, block_table, seq_lens, H, G, kw, vdim, block_size, bias, null_entry, scale, chunk, window, maps,
              grouped, gate, values_in_keys, rows, sink, key_at, out_scale)
    a.q_start, a.num_reqs = ptr(q_start), num_reqs
    a.tile_req, a.tile_q0, a.num_tiles = ptr(tile_req), ptr(tile_q0), tile_req.numel()
    check(lib().b200_bias_attn_prefill(ctypes.byref(a), int(any_size), stream_ptr()), "bias_attn_prefill")
    return out


def kernel_kind(phase: str, q, cache, *, H, G, kw, vdim, block_size, scale=1.0, chunk=0, window=0, maps=1,
                grouped=False, values_in_keys=False, key_at=0) -> str:
    """Which kernel serves a shape: "tensor-core" or "any-size"."""
    _declare()
    a = BiasAttnArgs()
    a.q, a.ldq, a.out, a.ldo, a.cache = ptr(q), q.stride(0), ptr(q), H * vdim, ptr(cache)
    a.H, a.G, a.kw, a.vdim, a.block_size = H, G, kw, vdim, block_size
    a.scale, a.chunk, a.window, a.maps, a.grouped = scale, chunk, window, maps, int(grouped)
    a.f32, a.tile_req = int(q.dtype == torch.float32), ptr(q)
    a.values_in_keys, a.key_at, a.out_scale = int(values_in_keys), key_at, 1.0
    return {2: "tensor-core", 1: "any-size"}[lib().b200_bias_attn_kernel(ctypes.byref(a), int(phase == "prefill"))]


def decode_splits(batch: int, max_seq_len: int, num_sms: int) -> int:
    """KV splits of the decode kernel (one CTA per request and split, one CTA per SM at real sizes;
    fixed per batch size, because the count is baked into a captured graph)."""
    return max(1, min(num_sms // max(1, batch), -(-max_seq_len // 128), 32))


def grouped_decode_splits(batch: int, groups: int, max_keys: int, num_sms: int) -> int:
    """KV splits of a grouped decode batch: one wave of two CTAs per SM, no split below 128 keys."""
    return max(1, min(2 * num_sms // max(1, batch * groups), -(-max_keys // 128), 32))


# ------------------------------------------------------------------------- tables built at load time
def bucket_of_distance(n: int, num_buckets: int, max_distance: int) -> int:
    """Distances below half the table have a bucket each; beyond, buckets are spaced evenly in the
    logarithm up to ``max_distance``, and the last bucket takes the rest."""
    half = num_buckets // 2
    if n < half:
        return n
    if max_distance <= half or n >= max_distance:
        return num_buckets - 1
    # (an exact boundary must not fall into the bucket below through the rounding of the logarithms)
    x = math.log(n / half) / math.log(max_distance / half) * (num_buckets - half)
    return min(num_buckets - 1, half + int(math.floor(x + 1e-9)))


def distance_bias_table(rel: torch.Tensor, max_distance: int) -> torch.Tensor:
    """``rel`` [buckets, H] -> fp32 [H, L]: the bias of every distance up to the first from which
    it no longer changes (the last column)."""
    B = rel.shape[0]
    idx = [bucket_of_distance(n, B, max_distance) for n in range(max(max_distance, B // 2) + 1)]
    while len(idx) > 1 and idx[-2] == idx[-1] == B - 1:
        idx.pop()
    return rel.float()[torch.tensor(idx, device=rel.device)].t().contiguous()


# ------------------------------------------------------------------------------ restatements
def page_views(cache, block_size, kw):
    """(keys [num_blocks, block_size, kw], values [num_blocks, block_size, vw]) of a page tensor."""
    nb = cache.shape[0]
    flat = cache.view(nb, -1)
    k = flat[:, : block_size * kw].view(nb, block_size, kw)
    v = flat[:, block_size * kw:].view(nb, block_size, -1)
    return k, v


def ref_head_mix_kv(qkv, mix, q_out, slots, cache, *, H, G, dim, vdim, block_size):
    T, kw, vw = qkv.shape[0], G * dim, G * vdim
    q = qkv[:, : H * dim].float().view(T, G, H // G, dim)
    m = torch.einsum("hgr,tgrd->thgd", mix.view(H, G, H // G), q)
    q_out[:T, : H * kw] = m.reshape(T, H * kw).to(q_out.dtype)
    keys, vals = page_views(cache, block_size, kw)
    ok = slots >= 0
    b, o = slots[ok] // block_size, slots[ok] % block_size
    keys[b, o] = qkv[ok, H * dim: H * dim + kw].to(cache.dtype)
    vals[b, o] = qkv[ok, H * dim + kw: H * dim + kw + vw].to(cache.dtype)


def ref_rotate_kv(qkv, positions, table, rot, eps, q_out, slots, cache, *, H, G, D, V, dim, block_size, q_w=None, k_w=None,
                  value_heads=None):
    T, half, GV = qkv.shape[0], rot // 2, G if value_heads is None else value_heads
    x = qkv[:, : (H + G) * D].float().view(T, H + G, D).clone()

    def norm(x):
        return x / torch.sqrt((x * x).sum(-1, keepdim=True) / dim + eps)
    if q_w is not None:
        x = norm(x) * torch.cat([q_w.expand(H, D), k_w.expand(G, D)], 0)
    if table is not None:
        cs = table[positions.long()]
        c, s = cs[:, None, :half], cs[:, None, half:]
        u, v = x[..., :half].clone(), x[..., half:rot].clone()
        x[..., :half], x[..., half:rot] = u * c - v * s, v * c + u * s
    if q_w is None:
        x = norm(x)
    q_out[:T, : H * D] = x[:, :H].reshape(T, -1).to(q_out.dtype)
    if G:
        keys, vals = page_views(cache, block_size, G * D)
        ok = slots >= 0
        b, o = slots[ok] // block_size, slots[ok] % block_size
        keys[b, o] = x[ok, H:].reshape(-1, G * D).to(cache.dtype)
        vals[b, o] = qkv[ok, (H + G) * D: (H + G) * D + GV * V].to(cache.dtype)


def ref_rotate_tied(qk, positions, table, q_out, slots, cache, s: TiedShape, *, block_size):
    T, half = qk.shape[0], s.rot // 2
    x = qk[:, : (s.H + s.G) * s.D].float().view(T, s.H + s.G, s.D)
    first, rest = x[..., : s.r8], x[..., s.r8:]
    turned = first.clone()
    if table is not None:
        cs = table[positions.long()]
        c, n = cs[:, None, :half], cs[:, None, half:]
        u, v = first[..., :half], first[..., half: s.rot]
        turned[..., :half], turned[..., half: s.rot] = u * c - v * n, v * c + u * n
    key = torch.cat([rest, turned], -1)
    q_out[:T, : s.H * s.D] = key[:, : s.H].reshape(T, -1).to(q_out.dtype)
    page = cache.view(cache.shape[0], -1)[:, : block_size * s.G * s.pitch].view(cache.shape[0], block_size, s.G * s.pitch)
    ok = slots >= 0
    page[slots[ok] // block_size, slots[ok] % block_size] = torch.cat([first, key], -1)[ok, s.H:].reshape(-1, s.G * s.pitch).to(cache.dtype)


def ref_diff_combine(maps, out, *, H, V, vdim, lam, eps, scale):
    T = maps.shape[0]
    x = maps[:, : H * 2 * V].float().view(T, H, 2, V)
    o = x[:, :, 0] - lam * x[:, :, 1]
    o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / vdim + eps) * scale
    out[:T, : H * V] = o.reshape(T, -1).to(out.dtype)
    return out


def ref_bias_attention(q, cache, out, *, block_table, seq_lens, q_start, H, G, kw, vdim, block_size, bias=None,
                       null_entry=False, scale=1.0, chunk=0, window=0, maps=1, grouped=False, gate=None, values_in_keys=False,
                       sink=None, key_at=0, out_scale=1.0):
    keys, vals = page_views(cache, block_size, kw)
    qs, R = q_start.tolist(), H // G
    for r, sl in enumerate(seq_lens.tolist()):
        t0, t1 = qs[r], qs[r + 1]
        if t1 <= t0 or sl <= 0:
            continue
        blocks = block_table[r, : (sl + block_size - 1) // block_size].long()
        k = keys[blocks].reshape(-1, kw)[:sl].float()
        v = k.view(sl, G, -1)[..., :vdim] if values_in_keys else vals[blocks].reshape(-1, G, vdim)[:sl].float()
        if key_at:
            k = k.view(sl, G, -1)[..., key_at:].reshape(sl, -1)
        v = v.repeat_interleave(R, 1)
        if grouped:                          # (head h reads map h % maps of its group)
            kg = k.view(sl, G, 1, maps, -1).expand(-1, -1, R // maps, -1, -1).reshape(sl, H, -1)
            s = torch.einsum("qhd,khd->hqk", q[t0:t1, : H * kg.shape[-1]].float().view(t1 - t0, H, -1), kg) * scale
        else:
            s = torch.einsum("qhd,kd->hqk", q[t0:t1, : H * kw].float().view(t1 - t0, H, kw), k) * scale
        at, key = torch.arange(sl - (t1 - t0), sl)[:, None], torch.arange(sl)[None]
        dist = at - key
        if bias is not None:
            s = s + bias[:, dist.clamp(0, bias.shape[1] - 1)]
        hidden = dist < 0
        if chunk:
            hidden = hidden | (at // chunk != key // chunk)
        if window:
            hidden = hidden | (dist >= window)
        s = s.masked_fill(hidden, -math.inf)
        m = s.amax(-1, keepdim=True)
        if null_entry:
            m = m.clamp(min=0)
        if sink is not None:
            m = torch.maximum(m, sink.view(-1, 1, 1))
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True) + (torch.exp(-m) if null_entry else 0.0)
        if sink is not None:
            den = den + torch.exp(sink.view(-1, 1, 1) - m)
        o = torch.einsum("hqk,khd->qhd", e / den, v) * out_scale
        if gate is not None:
            o = o * torch.sigmoid(gate[t0:t1, :H].float())[..., None]
        out[t0:t1, : H * vdim] = o.reshape(t1 - t0, H * vdim).to(out.dtype)
    return out
