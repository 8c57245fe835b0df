"""Short causal convolutions and the real-gated linear recurrent unit, with the PyTorch restatements the CPU
back end runs.

Rows are an engine step's: decode rows first, then the prompt portions. Each of the ``blocks`` parts of the
channels is padded with zeros to ``B``, a multiple of 16."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from ._lib import check, lib, ptr, stream_ptr

_P, _L, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float


@dataclass(frozen=True)
class RglruShape:
    blocks: int
    size: int                                 # channels of a block
    taps: int

    @property
    def B(self) -> int:
        return (self.size + 15) // 16 * 16

    @property
    def C(self) -> int:
        return self.blocks * self.B

    @property
    def M(self) -> int:
        """Gate rows of a block, padded to whole 128-row tiles."""
        return (self.B + 127) // 128 * 128


class RowArgs(ctypes.Structure):
    """The rows of a step."""
    _fields_ = [("seq_lens", _P), ("slots", _P), ("q_start", _P), ("tile_req", _P), ("tile_q0", _P), ("nd", _I),
                ("num_prefills", _I), ("num_tiles", _I), ("T", _I)]


class ShortConvArgs(ctypes.Structure):
    _fields_ = [("rows", RowArgs), ("x", _P), ("ldx", _L), ("w", _P), ("bias", _P), ("state", _P), ("out", _P), ("ldo", _L),
                ("C", _I), ("taps", _I), ("act", _I), ("f32", _I)]


class RglruArgs(ctypes.Structure):
    _fields_ = [("rows", RowArgs), ("u", _P), ("ldu", _L), ("y", _P), ("ldy", _L), ("gates", _P), ("gate_bias", _P),
                ("rate", _P), ("state", _P), ("out", _P), ("ldo", _L), ("summary", _P), ("a", _P), ("b", _P),
                ("blocks", _I), ("B", _I), ("M", _I), ("slices", _I), ("f32", _I)]


_declared = False


def _declare():
    global _declared
    if _declared:
        return
    _lib.declare("b200_short_conv", [ctypes.POINTER(ShortConvArgs), _P], _I)
    _lib.declare("b200_rglru_fits", [ctypes.POINTER(RglruArgs)], _I)
    _lib.declare("b200_rglru_slices", [ctypes.POINTER(RglruArgs)], _I)
    _lib.declare("b200_rglru", [ctypes.POINTER(RglruArgs), _I, _P], _I)
    lib()
    _declared = True


def _rows(r, ctx, T):
    r.seq_lens, r.slots, r.q_start = ptr(ctx.seq_lens), ptr(ctx.state_slots), ptr(ctx.prefill_q_start)
    r.tile_req, r.tile_q0 = ptr(ctx.tile_req), ptr(ctx.tile_q0)
    r.nd, r.num_prefills, r.num_tiles, r.T = ctx.num_decodes, ctx.num_prefills, ctx.num_tiles, T


ACTIVATIONS = {None: 0, "silu": 1}


def short_conv(x, w, bias, state, ctx, out, act=None):
    """Causal convolution per channel over each request: ``x`` [T, C] (rows may be strided), ``w`` fp32
    [taps, C] (the last row is the current token's), ``state`` [slots, taps - 1, C] the inputs before this step,
    advanced in place; a request's first rows start from zeros."""
    _declare()
    a = ShortConvArgs()
    _rows(a.rows, ctx, x.shape[0])
    a.x, a.ldx, a.w, a.bias, a.state = ptr(x), x.stride(0), ptr(w), ptr(bias), ptr(state)
    a.out, a.ldo, a.C, a.taps = ptr(out), out.stride(0), x.shape[1], w.shape[0]
    a.act, a.f32 = ACTIVATIONS[act], int(x.dtype == torch.float32)
    check(lib().b200_short_conv(ctypes.byref(a), stream_ptr()), "short_conv")
    return out


def rglru_args(u, y, w, s: RglruShape, state, ctx, bufs, out) -> RglruArgs:
    _declare()
    a = RglruArgs()
    _rows(a.rows, ctx, u.shape[0])
    a.u, a.ldu, a.y, a.ldy = ptr(u), u.stride(0), ptr(y), y.stride(0)
    a.gates, a.gate_bias, a.rate, a.state = ptr(w["gates"]), ptr(w["gate_bias"]), ptr(w["rate"]), ptr(state)
    a.out, a.ldo = ptr(out), out.stride(0)
    a.summary, a.a, a.b = (ptr(bufs.get(n)) for n in ("summary", "a", "b"))
    a.blocks, a.B, a.M, a.f32 = s.blocks, s.B, s.M, int(u.dtype == torch.float32)
    return a


def run_rglru(a: RglruArgs, any_size: bool = False) -> None:
    check(lib().b200_rglru(ctypes.byref(a), int(any_size), stream_ptr()), "rglru")


def rglru(u, y, w, s: RglruShape, state, ctx, bufs, out, *, any_size=False):
    """Channels ``u`` [T, C] and gate branch ``y`` (before its GELU) -> ``out`` = state * gelu_tanh(y), the
    state fading by d = exp(rate * g0) and taking in g1 * u with weight sqrt(1 - d * d); g0 and g1 are sigmoids of
    ``gates`` [blocks, 2, M, B] over each block's channels plus ``gate_bias`` fp32 [2, C]. ``state`` fp32 [slots, C] is
    advanced; a request's first rows start from zero. ``bufs``: ``summary`` fp32 scratch (see
    :func:`summary_values`), or ``a`` / ``b`` fp32 [T, C] for the any-size kernels."""
    run_rglru(rglru_args(u, y, w, s, state, ctx, bufs, out), any_size)
    return out


MAX_SLICES = 64


def summary_values(s: RglruShape) -> int:
    """fp32 scratch values: state, decay and starting state of every slice and channel."""
    return 3 * MAX_SLICES * s.C


def tensor_core_size(s: RglruShape) -> bool:
    return s.B <= 256


# ------------------------------------------------------------------------------ restatements
def _portions(ctx):
    qs = ctx.query_start.tolist()
    for r, seq in enumerate(ctx.seq_lens.tolist()):
        slot = int(ctx.state_slots[r])
        if qs[r + 1] > qs[r] and slot >= 0:
            yield qs[r], qs[r + 1], slot, seq == qs[r + 1] - qs[r]


def ref_short_conv(x, w, bias, state, ctx, out, act=None):
    taps = w.shape[0]
    for t0, t1, slot, fresh in _portions(ctx):
        n = t1 - t0
        past = torch.zeros(taps - 1, x.shape[1]) if fresh else state[slot].float()
        xs = torch.cat([past, x[t0:t1].float()], 0)
        y = sum(xs[i: i + n] * w[i] for i in range(taps))
        if bias is not None:
            y = y + bias
        state[slot] = xs[n:].to(state.dtype)
        out[t0:t1] = (torch.nn.functional.silu(y) if act == "silu" else y).to(out.dtype)
    return out


def ref_rglru(u, y, w, s: RglruShape, state, ctx, bufs, out, **_):
    T = u.shape[0]
    x = u.float()
    logits = torch.einsum("tbc,bgoc->gtbo", x.view(T, s.blocks, s.B), w["gates"][:, :, : s.B].float())
    r, i = torch.sigmoid(logits.reshape(2, T, s.C) + w["gate_bias"][:, None])
    log_a = w["rate"] * r
    a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * i * x
    act = torch.nn.functional.gelu(y.float(), approximate="tanh")
    for t0, t1, slot, fresh in _portions(ctx):
        S = torch.zeros_like(state[slot]) if fresh else state[slot].clone()
        for t in range(t0, t1):
            S = a[t] * S + b[t]
            out[t] = (S * act[t]).to(out.dtype)
        state[slot] = S
    return out
