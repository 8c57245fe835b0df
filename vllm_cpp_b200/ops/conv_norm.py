"""Start of an fp32 stream from token and token-pair embeddings, and the pass between layers of models whose
sublayers read short convolutions of a normed stream: stream update, norm in equal parts and one convolution per
sublayer in one kernel. With the PyTorch restatements the CPU back end runs.

A convolution over w * xhat (xhat: the stream with each part over its root mean square) plus w * xhat itself is one
convolution over xhat with the norm weight in its taps, so both sublayers carry the same past rows of xhat."""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from ._lib import check, lib, ptr, stream_ptr
from .rglru import RowArgs, _portions, _rows

_P, _L, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float


class EmbedPairsArgs(ctypes.Structure):
    _fields_ = [("rows", RowArgs), ("stream", _P), ("lds", _L), ("ids", _P), ("table", _P), ("bigram", _P), ("prev", _P),
                ("norm_w", _P), ("vocab", _L), ("buckets", _L), ("mul_prev", _L), ("mul_cur", _L),
                ("width", _I), ("cols", _I), ("groups", _I), ("f32", _I), ("scale", _F), ("eps", _F)]


class NormConvArgs(ctypes.Structure):
    _fields_ = [("rows", RowArgs), ("src", _P), ("dst", _P), ("lds", _L), ("a", _P), ("lda", _L), ("y", _P), ("ldy", _L),
                ("pair_pos", _P), ("pair_w", _P), ("w1", _P), ("w2", _P), ("out1", _P), ("out2", _P), ("ldo", _L),
                ("state", _P), ("width", _I), ("cols", _I), ("groups", _I), ("taps", _I), ("k", _I), ("f32", _I), ("eps", _F)]


_declared = False


def _declare():
    global _declared
    if _declared:
        return
    _lib.declare("b200_embed_pairs", [ctypes.POINTER(EmbedPairsArgs), _P], _I)
    _lib.declare("b200_norm_conv", [ctypes.POINTER(NormConvArgs), _P], _I)
    lib()
    _declared = True


def conv_weights(norm_w, canon):
    """fp32 [taps, cols] of h + conv(h), h = norm_w * xhat, as one convolution over xhat; ``canon`` [cols, taps]."""
    w = canon.float().t().clone()
    w[-1] += 1.0
    return (w * norm_w.float()).contiguous()


def embed_pairs(stream, ids, table, ctx, *, width, scale, norm_w, groups, eps, bigram=None, prev=None, spec=None):
    """``stream`` [T, cols] = norm(table[ids] * scale + bigram[row of (token before, token)]), the norm in
    ``groups`` equal parts of ``width``, weighted with ``norm_w`` fp32 [cols]. ``prev`` int64 [slots]: each request's
    last token, advanced; a first token takes the last row of ``bigram``. ``spec``: buckets, mul_prev, mul_cur."""
    _declare()
    a = EmbedPairsArgs()
    T, cols = stream.shape
    _rows(a.rows, ctx, T)
    a.stream, a.lds, a.ids, a.table, a.vocab = ptr(stream), stream.stride(0), ptr(ids), ptr(table), table.shape[0]
    a.norm_w, a.width, a.cols, a.groups = ptr(norm_w), width, cols, groups
    a.f32, a.scale, a.eps = int(table.dtype == torch.float32), scale, eps
    if bigram is not None:
        a.bigram, a.prev = ptr(bigram), ptr(prev)
        a.buckets, a.mul_prev, a.mul_cur = spec.buckets, spec.mul_prev, spec.mul_cur
        if bigram.shape[0] != spec.buckets + 1:
            raise ValueError(f"{bigram.shape[0]} rows of token pairs, not {spec.buckets + 1}")
    check(lib().b200_embed_pairs(ctypes.byref(a), stream_ptr()), "embed_pairs")
    return stream


def norm_conv(src, ctx, weights, outs, *, width, groups, eps, state=None, dst=None, a=None, y=None, pair_pos=None, pair_w=None):
    """x = ``src`` + ``a`` + sum_j ``pair_w`` [:, j] * ``y`` [``pair_pos`` [:, j]] (all but ``src`` optional), kept in
    ``dst`` (not ``src``); each of ``groups`` equal parts of its ``width`` values over its root mean square; ``outs`` [i] = the
    causal convolution of those rows with ``weights`` [i] fp32 [taps, cols]. ``state`` fp32 [slots, taps - 1, cols]: each
    request's last such rows, advanced; a request's first rows start from zeros."""
    _declare()
    T, cols = src.shape
    assert src.dtype == torch.float32 and (a is None or a.dtype == torch.float32) and 1 <= len(outs) == len(weights) <= 2
    assert dst is None or (dst.stride(0) == src.stride(0) and dst.data_ptr() != src.data_ptr())
    n = NormConvArgs()
    _rows(n.rows, ctx, T)
    n.src, n.dst, n.lds = ptr(src), ptr(dst), src.stride(0)
    n.a, n.lda = ptr(a), a.stride(0) if a is not None else 0
    n.y, n.ldy = ptr(y), y.stride(0) if y is not None else 0
    n.pair_pos, n.pair_w, n.k = ptr(pair_pos), ptr(pair_w), pair_pos.shape[1] if pair_pos is not None else 0
    n.w1, n.out1, n.ldo = ptr(weights[0]), ptr(outs[0]), outs[0].stride(0)
    if len(outs) > 1:
        assert outs[1].stride(0) == outs[0].stride(0)
        n.w2, n.out2 = ptr(weights[1]), ptr(outs[1])
    n.state, n.width, n.cols, n.groups, n.taps = ptr(state), width, cols, groups, weights[0].shape[0]
    n.f32, n.eps = int(outs[0].dtype == torch.float32), eps
    check(lib().b200_norm_conv(ctypes.byref(n), stream_ptr()), "norm_conv")


# ------------------------------------------------------------------------------ restatements
def _parts_over_rms(x, width, groups, eps):
    p = x[:, :width].reshape(x.shape[0], groups, -1)
    out = torch.zeros_like(x)
    out[:, :width] = (p / torch.sqrt((p * p).mean(-1, keepdim=True) + eps)).reshape(x.shape[0], width)
    return out


def ref_embed_pairs(stream, ids, table, ctx, *, width, scale, norm_w, groups, eps, bigram=None, prev=None, spec=None):
    x = table[ids].float() * scale
    if bigram is not None:
        row = torch.full_like(ids, spec.buckets)
        for t0, t1, slot, fresh in _portions(ctx):
            before = torch.cat([prev[slot: slot + 1], ids[t0: t1 - 1]])
            row[t0:t1] = (before * spec.mul_prev + ids[t0:t1] * spec.mul_cur) % spec.buckets
            if fresh:
                row[t0] = spec.buckets
            prev[slot] = ids[t1 - 1]
        x = x + bigram[row].float()
    stream.copy_(_parts_over_rms(x, width, groups, eps) * norm_w)
    return stream


def ref_norm_conv(src, ctx, weights, outs, *, width, groups, eps, state=None, dst=None, a=None, y=None, pair_pos=None, pair_w=None):
    x = src.clone()
    if a is not None:
        x += a
    if pair_pos is not None:
        for j in range(pair_pos.shape[1]):
            x += y[pair_pos[:, j].long()].float() * pair_w[:, j, None]
    if dst is not None:
        dst.copy_(x)
    x = _parts_over_rms(x, width, groups, eps)
    taps = weights[0].shape[0]
    if taps == 1:
        for w, o in zip(weights, outs):
            o.copy_(x * w[0])
        return
    for t0, t1, slot, fresh in _portions(ctx):
        n = t1 - t0
        xs = torch.cat([torch.zeros_like(state[slot]) if fresh else state[slot], x[t0:t1]], 0)
        for w, o in zip(weights, outs):
            o[t0:t1] = sum(xs[i: i + n] * w[i] for i in range(taps)).to(o.dtype)
        state[slot] = xs[n:]
