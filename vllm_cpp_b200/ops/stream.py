"""fp32 residual stream (update + RMSNorm in one kernel) and true fp32 products, with the PyTorch
restatements the CPU back end runs."""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from ._lib import check, lib, ptr, stream_ptr

_P, _L, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float


class StreamNormArgs(ctypes.Structure):
    _fields_ = [("stream", _P), ("ids", _P), ("table", _P), ("a", _P), ("y", _P), ("pair_pos", _P), ("pair_w", _P),
                ("norm_w", _P), ("post_w", _P), ("ident", _P), ("out", _P), ("lds", _L), ("lda", _L), ("ldy", _L),
                ("ldi", _L), ("ldo", _L), ("vocab", _L),
                ("T", _I), ("width", _I), ("cols", _I), ("k", _I), ("f32", _I), ("a_f32", _I),
                ("scale", _F), ("eps", _F), ("norm_offset", _F), ("mult", _F)]


class ClampedGate(ctypes.Structure):
    """g = min(gate, limit), u = clamp(up, -limit, limit): g * sigmoid(alpha g) * (u + up_offset)."""
    _fields_ = [("limit", _F), ("alpha", _F), ("up_offset", _F), ("row_w", _P)]


_declared = False


def _declare():
    global _declared
    if _declared:
        return
    P, I = _lib.P, _lib.I
    _lib.declare("b200_stream_norm", [ctypes.POINTER(StreamNormArgs), P], I)
    _lib.declare("b200_gated_act_f32", [P, I, P, I, I, I, I, P], I)
    _lib.declare("b200_gemm_f32", [P, I, P, I, P, I, P, I, I, I, I, P], I)
    _lib.declare("b200_softcap_f32", [P, ctypes.c_longlong, _lib.F, P], I)
    lib()
    _declared = True


def stream_norm(stream, norm_w, eps, out, *, width, ids=None, table=None, scale=1.0, a=None, y=None,
                pair_pos=None, pair_w=None, norm_offset=1.0, post_w=None, ident=None, mult=1.0):
    """``stream`` [T, cols] fp32 starts as ``table[ids] * scale`` or takes ``+= mult (a + sum_j w_j
    y[pair_pos[:, j]])`` (``ident`` rows where ``pair_pos`` < 0; may be ``out``), with ``post_w`` that sum
    over its rms times (post_w + norm_offset); ``out`` = stream / rms(stream) * (norm_w + norm_offset).
    ``cols`` is ``width`` padded with zeros."""
    _declare()
    T, cols = stream.shape
    s = StreamNormArgs()
    s.stream, s.norm_w, s.out = ptr(stream), ptr(norm_w), ptr(out)
    s.ids, s.table, s.a, s.y = ptr(ids), ptr(table), ptr(a), ptr(y)
    s.pair_pos, s.pair_w = ptr(pair_pos), ptr(pair_w)
    s.post_w, s.ident, s.ldi = ptr(post_w), ptr(ident), ident.stride(0) if ident is not None else 0
    s.lds, s.ldo = stream.stride(0), out.stride(0)
    s.lda = a.stride(0) if a is not None else 0
    s.ldy = y.stride(0) if y is not None else 0
    s.vocab = table.shape[0] if table is not None else 0
    s.T, s.width, s.cols, s.k = T, width, cols, pair_pos.shape[1] if pair_pos is not None else 0
    s.f32 = int(out.dtype == torch.float32)
    s.a_f32 = int(a is not None and a.dtype == torch.float32)
    s.scale, s.eps, s.norm_offset, s.mult = scale, eps, norm_offset, mult
    check(lib().b200_stream_norm(ctypes.byref(s), stream_ptr()), "stream_norm")
    return out


def gemm_f32(a, w, bias=None, out=None, act=0):
    """``act(a @ w.T (+ bias))`` in fp32 multiply-adds; ``act`` as in ``ops.gemm``."""
    _declare()
    M, K = a.shape
    N = w.shape[0]
    if out is None:
        out = torch.empty((M, N), dtype=torch.float32, device=a.device)
    check(lib().b200_gemm_f32(ptr(a), a.stride(0), ptr(w), w.stride(0), ptr(out), out.stride(0), ptr(bias), M, N, K,
                              act, stream_ptr()), f"gemm_f32 M={M} N={N} K={K}")
    return out


def softcap_f32(x, cap):
    """cap * tanh(x / cap) in place over fp32 rows [n, cols]."""
    _declare()
    check(lib().b200_softcap_f32(ptr(x), x.numel(), cap, stream_ptr()), "softcap_f32")
    return x


def gated_act_f32(gate_up, kind, out):
    """act(gate) * up of fp32 rows ``[gate | up]``; ``kind`` as in ``ops.act_and_mul``."""
    _declare()
    T, I = gate_up.shape[0], gate_up.shape[1] // 2
    check(lib().b200_gated_act_f32(ptr(gate_up), gate_up.stride(0), ptr(out), out.stride(0), T, I, kind, stream_ptr()),
          "gated_act_f32")
    return out


# ------------------------------------------------------------------------------ restatements
def ref_stream_norm(stream, norm_w, eps, out, *, width, ids=None, table=None, scale=1.0, a=None, y=None,
                    pair_pos=None, pair_w=None, norm_offset=1.0, post_w=None, ident=None, mult=1.0):
    if ids is not None:
        stream.copy_(table[ids].float() * scale)
    else:
        d = torch.zeros_like(stream)
        if a is not None:
            d += a.float()
        if pair_pos is not None:
            for j in range(pair_pos.shape[1]):
                yj = y[pair_pos[:, j].long().clamp(min=0)].float() * (pair_pos[:, j] >= 0)[:, None]
                if ident is not None:
                    yj = yj + ident.float() * (pair_pos[:, j] < 0)[:, None]
                d += yj * pair_w[:, j, None] if pair_w is not None else yj
        if post_w is not None:
            d = d / torch.sqrt((d * d).sum(-1, keepdim=True) / width + eps) * (post_w + norm_offset)
        stream += mult * d
    inv = 1.0 / torch.sqrt((stream * stream).sum(-1, keepdim=True) / width + eps)
    out.copy_(stream * inv * (norm_w + norm_offset))
    return out


def ref_clamped_gate(gate_up, limit, alpha, up_offset):
    """fp32 ``[gate | up]`` rows."""
    inter = gate_up.shape[-1] // 2
    g = gate_up[..., :inter].clamp(max=limit)
    u = gate_up[..., inter:].clamp(-limit, limit)
    return g * torch.sigmoid(alpha * g) * (u + up_offset)
