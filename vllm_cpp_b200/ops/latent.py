"""Latent attention with per-layer sizes: preparation (norms of the query and key latents, rotation, cache
write), queries, and attention over pages of latent rows ``[latent (rankp) | rotated part (rotp)]``, with the
PyTorch restatements the CPU back end runs.

Decode rows take the absorbed form: queries through the key projection, every head over the same rows, values
= the latent, the value projection afterwards. Prompt portions expand the visible rows into keys and values
of every head (bf16 on the tensor cores) and run the prompt kernel of ``bias_attn.py``; sizes beyond these
kernels and the fp32 mode run the absorbed form on the any-size kernel."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from . import bias_attn as A
from ._lib import check, lib, ptr, stream_ptr

_P, _L, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float


def _pad(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class LatentShape:
    H: int
    dim: int
    rot: int
    vdim: int
    q_rank: int
    rank: int

    @property
    def qn(self) -> int:
        """Columns of a head's unrotated query part (whole 64-wide chunks)."""
        return _pad(self.dim, 64)

    @property
    def qw(self) -> int:
        return self.qn + _pad(self.rot, 16)

    @property
    def D(self) -> int:
        return _pad(self.dim, 16)

    @property
    def V(self) -> int:
        return _pad(self.vdim, 16)

    @property
    def tensor_decode(self) -> bool:
        return self.rank <= 512 and self.rot <= 64

    @property
    def rankp(self) -> int:
        return _pad(self.rank, 128 if self.tensor_decode else 64)

    @property
    def rotp(self) -> int:
        return 64 if self.tensor_decode else _pad(self.rot, 16)

    @property
    def row(self) -> int:
        return self.rankp + self.rotp

    @property
    def down(self) -> tuple:
        """Widths of the down projection's parts: query latent, key latent, shared rotated part, gates."""
        return tuple(_pad(n, 8) for n in (self.q_rank, self.rank, self.rot, self.H))

    @property
    def gate_column(self) -> int:
        return sum(self.down[:3])


class LatentPrepArgs(ctypes.Structure):
    _fields_ = [("down", _P), ("ldd", _L), ("positions", _P), ("cos_sin", _P), ("q_norm", _P), ("kv_norm", _P),
                ("cq", _P), ("ldcq", _L), ("slots", _P), ("cache", _P), ("T", _I), ("q_rank", _I), ("rank", _I),
                ("rot", _I), ("kv_col", _I), ("rot_col", _I), ("rankp", _I), ("row", _I), ("f32", _I), ("eps", _F)]


_declared = False


def _declare():
    global _declared
    if _declared:
        return
    P, I, L, F = _lib.P, _lib.I, ctypes.c_longlong, _lib.F
    _lib.declare("b200_latent_prepare", [ctypes.POINTER(LatentPrepArgs), P], I)
    _lib.declare("b200_latent_queries", [P, L, P, P, I, I, I, I, P, I, I, I, I, I, P], I)
    _lib.declare("b200_latent_decode", [P, P, I, P, L, I, I, I, I, P, I, P, I, F, I, P, L, I, P, P, P], I)
    _lib.declare("b200_latent_gather", [P, P, I, P, P, P, I, I, P, I, I, P], I)
    _lib.declare("b200_gemm_f32_batched", [P, I, I, P, I, P, I, L, I, I, I, I, P], I)
    lib()
    _declared = True


def prepare(down, positions, table, w, s: LatentShape, eps, cq, slots, cache):
    """Rows ``down`` -> normed query latents ``cq``, and this step's rows of ``cache`` (slot < 0: none): the
    normed key latent and the rotated part (pairs half of it apart, ``table`` [positions, cos | sin])."""
    _declare()
    a = LatentPrepArgs()
    a.down, a.ldd, a.positions, a.cos_sin = ptr(down), down.stride(0), ptr(positions), ptr(table)
    a.q_norm, a.kv_norm, a.cq, a.ldcq = ptr(w["q_norm"]), ptr(w["kv_norm"]), ptr(cq), cq.stride(0)
    a.slots, a.cache, a.T = ptr(slots), ptr(cache), down.shape[0]
    a.q_rank, a.rank, a.rot, a.kv_col, a.rot_col = s.q_rank, s.rank, s.rot, s.down[0], s.down[0] + s.down[1]
    a.rankp, a.row, a.f32, a.eps = s.rankp, s.row, int(down.dtype == torch.float32), eps
    check(lib().b200_latent_prepare(ctypes.byref(a), stream_ptr()), "latent_prepare")


def queries(q, positions, table, s: LatentShape, qabs, absorbed: int):
    """Rotates the rotated part of every head of ``q`` [T, H * qw]: in place, or for the first ``absorbed``
    rows into ``qabs`` [absorbed, H * row]."""
    _declare()
    check(lib().b200_latent_queries(ptr(q), q.stride(0), ptr(positions), ptr(table), s.H, s.qn, s.qw, s.rot, ptr(qabs),
                                    s.rankp, s.row, absorbed, q.shape[0], int(q.dtype == torch.float32), stream_ptr()),
          "latent_queries")


def heads_product(a, a_cols, w, out, out_cols, M):
    """out[m, h * out_cols + n] = sum_k a[m, h * a_cols + k] w[h, n, k] for every head h."""
    _declare()
    H, N, K = w.shape
    if a.dtype == torch.float32:
        check(lib().b200_gemm_f32_batched(ptr(a), a.stride(0), a_cols, ptr(w), K, ptr(out), out.stride(0), out_cols, M, N, K,
                                          H, stream_ptr()), "gemm_f32_batched")
    else:
        from .mla import gemm_batched
        gemm_batched(a, a_cols, w, out, out_cols, M, N, K, H)


def decode(qabs, cache, out, s: LatentShape, *, block_table, seq_lens, scale, window, block_size, gate, splits=1, tmp=None):
    """Absorbed rows ``qabs`` [B, H * row] over the pages -> latent outputs ``out`` [B, H * rankp]; ``gate``
    [B, H]: each head's output times sigmoid(gate)."""
    _declare()
    B = qabs.shape[0]
    if splits > 1 and tmp is None:
        tmp = (torch.empty(B * s.H * splits * s.rankp, dtype=torch.float32, device=qabs.device),
               torch.empty(B * s.H * splits, dtype=torch.float32, device=qabs.device))
    if splits > 1:
        assert tmp[0].numel() >= B * s.H * splits * s.rankp and tmp[1].numel() >= B * s.H * splits
    check(lib().b200_latent_decode(ptr(qabs), ptr(out), out.stride(0), ptr(cache), cache.shape[0], block_size, s.H,
                                   s.rankp, s.rotp, ptr(block_table), block_table.stride(0), ptr(seq_lens), B, scale,
                                   window, ptr(gate), gate.stride(0) if gate is not None else 0, splits,
                                   ptr(tmp[0]) if splits > 1 else None, ptr(tmp[1]) if splits > 1 else None,
                                   stream_ptr()), "latent_decode")
    return out


def decode_splits(batch: int, heads: int, max_keys: int, num_sms: int) -> int:
    """KV splits of a decode batch: one CTA per SM and wave, no split below 128 keys."""
    return max(1, min(num_sms // max(1, batch * -(-heads // 16)), -(-max_keys // 128), 16))


def visible_pages(seq_lens, q_lens, window: int, block_size: int):
    """Which pages of each portion its prompt kernel reads (whole 128-key tiles), packed one after the other:
    (first page per portion, first packed page per portion, pages in all, packed block table)."""
    import numpy as np
    seq, qn = np.asarray(seq_lens, dtype=np.int64), np.asarray(q_lens, dtype=np.int64)
    lo = np.maximum(seq - qn - window + 1, 0) if window else np.zeros_like(seq)
    first = lo // 128 * 128 // block_size
    n = (seq + block_size - 1) // block_size - first
    base = np.concatenate([[0], np.cumsum(n)[:-1]])
    bt = np.zeros((len(seq), int((first + n).max())), dtype=np.int32)
    for i in range(len(seq)):
        bt[i, first[i]: first[i] + n[i]] = base[i] + np.arange(n[i])
    return first.astype(np.int32), base.astype(np.int32), int(n.sum()), bt


def gather(cache, block_table, seq_lens, first, base, block_size, dense, num_reqs, max_pages):
    """The pages of :func:`visible_pages` one after the other in ``dense`` [rows, row]."""
    _declare()
    check(lib().b200_latent_gather(ptr(cache), ptr(block_table), block_table.stride(0), ptr(seq_lens), ptr(first), ptr(base),
                                   block_size, dense.shape[1] * dense.element_size(), ptr(dense), num_reqs, max_pages,
                                   stream_ptr()), "latent_gather")


def prefill_kernel_fits(s: LatentShape, dtype, block_size: int) -> bool:
    return dtype == torch.bfloat16 and s.V <= 256 and s.qw <= 512 and \
        (128 % block_size == 0 and block_size >= 8 or block_size % 128 == 0)


def prefill_expanded(q, kv, dense, out, s: LatentShape, *, block_table, seq_lens, q_start, num_reqs, tile_req, tile_q0, scale,
                     window, block_size, gate):
    """Prompt portions over expanded rows ``kv`` [rows, H * (D + V)] = [keys | values] and the rotated parts
    at the end of the rows ``dense``."""
    return A.prefill(q, kv, out, block_table=block_table, seq_lens=seq_lens, q_start=q_start, num_reqs=num_reqs,
                     tile_req=tile_req, tile_q0=tile_q0, H=s.H, G=s.H, kw=s.H * s.D, vdim=s.V, block_size=block_size,
                     scale=scale, window=window, grouped=True, gate=gate,
                     rows=A.SplitRows(kv[:, : s.H * s.D], kv[:, s.H * s.D:], dense[:, s.rankp:]))


def absorbed_any_size(qabs, cache, out, s: LatentShape, *, decode_rows, block_size, scale, window, gate, **rows):
    kw = dict(H=s.H, G=1, kw=s.row, vdim=s.rankp, block_size=block_size, scale=scale, window=window, gate=gate,
              any_size=True, values_in_keys=True)
    return A.decode(qabs, cache, out, **kw, **rows) if decode_rows else A.prefill(qabs, cache, out, **kw, **rows)


# ------------------------------------------------------------------------------ restatements
def _turn(x, positions, table):
    half = x.shape[-1] // 2
    if not half:
        return x
    cs = table[positions.long()].view(-1, *([1] * (x.dim() - 2)), 2 * half)
    c, s, u, v = cs[..., :half], cs[..., half:], x[..., :half], x[..., half:]
    return torch.cat([u * c - v * s, v * c + u * s], -1)


def ref_prepare(down, positions, table, w, s: LatentShape, eps, cq, slots, cache):
    x = down.float()

    def normed(y, weight):
        return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps) * weight
    cq[: x.shape[0], : s.q_rank] = normed(x[:, : s.q_rank], w["q_norm"][: s.q_rank]).to(cq.dtype)
    k0 = s.down[0]
    r0 = k0 + s.down[1]
    flat, ok = cache.view(-1, s.row), slots >= 0
    flat[slots[ok], : s.rank] = normed(x[:, k0: k0 + s.rank], w["kv_norm"][: s.rank])[ok].to(cache.dtype)
    flat[slots[ok], s.rankp: s.rankp + s.rot] = _turn(x[:, r0: r0 + s.rot], positions, table)[ok].to(cache.dtype)


def ref_latent_attention(q, positions, table, cache, w, s: LatentShape, *, block_table, seq_lens, q_start, scale, window,
                         block_size, gate, out):
    """Absorbed form; ``q`` before its rotation."""
    T = q.shape[0]
    x = q.float().view(T, s.H, s.qw)
    qa = torch.zeros(T, s.H, s.row)
    qa[..., : s.rankp] = torch.einsum("thd,hrd->thr", x[..., : s.qn], w["uk_t"].float())
    qa[..., s.rankp: s.rankp + s.rot] = _turn(x[..., s.qn: s.qn + s.rot], positions, table)
    o = torch.zeros(T, s.H * s.rankp)
    A.ref_bias_attention(qa.view(T, -1), cache, o, block_table=block_table, seq_lens=seq_lens, q_start=q_start, H=s.H, G=1,
                         kw=s.row, vdim=s.rankp, block_size=block_size, scale=scale, window=window, grouped=True,
                         values_in_keys=True, gate=gate)
    y = torch.einsum("thr,hvr->thv", o.view(T, s.H, s.rankp), w["uv"].float())
    out[:T, : s.H * s.V] = y.reshape(T, -1).to(out.dtype)
    return out
