"""Gated delta rule with per-layer sizes: preparation (short convolutions, unit q / k, decay and write
strength), the recurrence and its gated norm, with the PyTorch restatements the CPU back end runs.

Rows are an engine step's: decode rows first, then the prompt portions. Sizes ``D`` / ``V`` are padded to
multiples of 16 with zeros, ``dim`` / ``vdim`` are the sizes the norms divide by."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from ._lib import check, lib, ptr, stream_ptr

_P, _L, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float


@dataclass(frozen=True)
class DeltaShape:
    G: int
    H: int
    D: int
    V: int
    dim: int
    vdim: int
    taps: int

    @property
    def channels(self) -> int:
        """q, k and v columns: those the convolutions run over."""
        return 2 * self.G * self.D + self.H * self.V

    @property
    def columns(self) -> int:
        """Columns of the projection ``[q | k | v | gate]``."""
        return self.channels + self.H * self.V


class DeltaArgs(ctypes.Structure):
    _fields_ = [("proj", _P), ("gate", _P), ("ldp", _L), ("ab", _P), ("ldab", _L), ("conv_w", _P), ("A", _P), ("dt", _P),
                ("norm_w", _P), ("conv_state", _P), ("state", _P), ("q", _P), ("k", _P), ("v", _P), ("g", _P),
                ("beta", _P), ("o", _P), ("out", _P), ("ldo", _L), ("seq_lens", _P), ("slots", _P), ("q_start", _P),
                ("tile_req", _P), ("tile_q0", _P), ("nd", _I), ("num_prefills", _I), ("num_tiles", _I), ("T", _I),
                ("G", _I), ("H", _I), ("D", _I), ("V", _I), ("dim", _I), ("vdim", _I), ("taps", _I), ("f32", _I), ("split", _I),
                ("eps", _F), ("q_scale", _F)]


_declared = False


def _declare():
    global _declared
    if _declared:
        return
    A = ctypes.POINTER(DeltaArgs)
    _lib.declare("b200_delta_prepare", [A, _P], _I)
    _lib.declare("b200_delta_rule", [A, _I, _P], _I)
    _lib.declare("b200_delta_norm", [A, _I, _P], _I)
    _lib.declare("b200_delta_chunk_fits", [A], _I)
    _lib.declare("b200_delta_chunk", [A, _P, _P, _P], _I)
    lib()
    _declared = True


def delta_args(proj, ab, w, shape: DeltaShape, conv_state, state, rows, bufs, out, eps, *, token_by_token=False) -> DeltaArgs:
    _declare()
    a, s = DeltaArgs(), shape
    a.proj, a.ldp, a.gate = ptr(proj), proj.stride(0), ptr(proj) + s.channels * proj.element_size()
    a.ab, a.ldab = ptr(ab), ab.stride(0)
    a.conv_w, a.A, a.dt, a.norm_w = ptr(w["conv_w"]), ptr(w["A"]), ptr(w["dt"]), ptr(w["norm"])
    a.conv_state, a.state = ptr(conv_state), ptr(state)
    for n in ("q", "k", "v", "g", "beta", "o"):
        setattr(a, n, ptr(bufs[n]))
    a.out, a.ldo = ptr(out), out.stride(0)
    a.seq_lens, a.slots, a.q_start = ptr(rows.seq_lens), ptr(rows.state_slots), ptr(rows.prefill_q_start)
    a.tile_req, a.tile_q0 = ptr(rows.tile_req), ptr(rows.tile_q0)
    a.nd, a.num_prefills, a.num_tiles, a.T = rows.num_decodes, rows.num_prefills, rows.num_tiles, proj.shape[0]
    a.G, a.H, a.D, a.V, a.dim, a.vdim, a.taps = s.G, s.H, s.D, s.V, s.dim, s.vdim, s.taps
    a.f32, a.eps, a.q_scale = int(proj.dtype == torch.float32), eps, s.dim ** -0.5
    a.split = int(bufs.get("chunks") is not None and a.num_prefills > 0 and not token_by_token
                  and lib().b200_delta_chunk_fits(ctypes.byref(a)))
    return a


def run_prepare(a: DeltaArgs) -> None:
    check(lib().b200_delta_prepare(ctypes.byref(a), stream_ptr()), "delta_prepare")


def run_rule(a: DeltaArgs, bufs) -> None:
    check(lib().b200_delta_rule(ctypes.byref(a), a.nd + (0 if a.split else a.num_prefills), stream_ptr()), "delta_rule")
    if a.split:
        tp, gc = bufs["chunks"]
        assert tp.numel() >= a.num_tiles * a.H * CHUNK_VALUES and gc.numel() >= a.num_tiles * a.H * 128
        check(lib().b200_delta_chunk(ctypes.byref(a), ptr(tp), ptr(gc), stream_ptr()), "delta_chunk")
        check(lib().b200_delta_norm(ctypes.byref(a), a.T - a.nd, stream_ptr()), "delta_norm")


def delta_mixer(proj, ab, w, shape: DeltaShape, conv_state, state, rows, bufs, out, eps, *, token_by_token=False):
    """``proj`` [T, columns] and ``ab`` fp32 [T, >= 2 H] -> ``out`` [T, H * V]. ``w``: conv_w fp32
    [taps, channels], A, dt, norm fp32. ``conv_state`` [slots, taps - 1, channels] and ``state`` fp32
    [slots, H, D, V] are advanced; a request's first rows start from zero. ``rows``: the step's
    :class:`StepContext`. ``bufs``: q, k, v, g, beta, o scratch of T rows, and for prompts ``chunks``
    (see :func:`chunk_workspace`). bf16 prompts run in chunks of 64 tokens on the tensor cores;
    ``token_by_token``, fp32 and sizes beyond them walk the tokens."""
    a = delta_args(proj, ab, w, shape, conv_state, state, rows, bufs, out, eps, token_by_token=token_by_token)
    run_prepare(a)
    run_rule(a, bufs)
    return out


CHUNK_VALUES = 2 * 4 * 64 * 64          # bf16 values per 128-row tile and head


def chunk_workspace(device, max_tiles: int, heads: int):
    """Scratch of the chunk kernels: (pair matrices, decay sums) for up to ``max_tiles`` 128-row tiles."""
    return (torch.empty(max_tiles * heads * CHUNK_VALUES, dtype=torch.bfloat16, device=device),
            torch.empty(max_tiles * heads * 128, dtype=torch.float32, device=device))


# ------------------------------------------------------------------------------ restatements
def ref_delta_mixer(proj, ab, w, shape: DeltaShape, conv_state, state, rows, bufs, out, eps, **_):
    s, T = shape, proj.shape[0]
    qs = rows.query_start.tolist()
    x = proj[:, : s.channels].float()
    z = proj[:, s.channels: s.columns].float().view(T, s.H, s.V)
    a, b = ab[:, : s.H].float(), ab[:, s.H: 2 * s.H].float()
    decay = torch.exp(-w["A"] * torch.nn.functional.softplus(a + w["dt"], threshold=1e9))
    beta = torch.sigmoid(b)
    for r, seq in enumerate(rows.seq_lens.tolist()):
        t0, t1 = qs[r], qs[r + 1]
        slot = int(rows.state_slots[r])
        if t1 <= t0 or slot < 0:
            continue
        n, fresh = t1 - t0, seq == t1 - t0
        past = torch.zeros(s.taps - 1, s.channels) if fresh else conv_state[slot].float()
        xs = torch.cat([past, x[t0:t1]], 0)
        y = torch.nn.functional.silu(sum(xs[i: i + n] * w["conv_w"][i] for i in range(s.taps)))
        conv_state[slot] = xs[n:].to(conv_state.dtype)
        gd = s.G * s.D
        q, k = (y[:, i * gd: (i + 1) * gd].view(n, s.G, s.D) for i in (0, 1))
        q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * s.dim ** -0.5
        k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        q, k = (v.repeat_interleave(s.H // s.G, 1) for v in (q, k))
        v = y[:, 2 * gd:].view(n, s.H, s.V).to(proj.dtype).float()
        S = torch.zeros_like(state[slot]) if fresh else state[slot].clone()
        o = torch.empty(n, s.H, s.V)
        for i in range(n):
            S = S * decay[t0 + i].view(-1, 1, 1)
            u = beta[t0 + i].view(-1, 1) * (v[i] - torch.einsum("hdv,hd->hv", S, k[i]))
            S = S + k[i].unsqueeze(-1) * u.unsqueeze(1)
            o[i] = torch.einsum("hdv,hd->hv", S, q[i])
        state[slot] = S
        o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / s.vdim + eps) * w["norm"]
        out[t0:t1, : s.H * s.V] = (o * torch.nn.functional.silu(z[t0:t1])).reshape(n, -1).to(out.dtype)
    return out
