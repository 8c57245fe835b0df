"""Recurrences over outer products, S <- decay * S + k v^T, o = S^T q, with fp32 states: gated linear attention (a
decay per key channel, output normed per head and gated) and the state-space form of Mamba-2 (a decay per head that
comes with the step size, keys and queries shared by groups of heads, gated output normed in equal parts). With the
PyTorch restatements the CPU back end runs.

Rows are an engine step's: decode rows first, then the prompt portions. Sizes ``D`` / ``V`` are padded to multiples
of 16 with zeros, ``dim`` / ``vdim`` are the sizes themselves."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from ._lib import check, lib, ptr, stream_ptr
from .rglru import RowArgs, _portions, _rows

_P, _L, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float
CHANNEL, HEAD = 0, 1                          # what has a decay of its own


@dataclass(frozen=True)
class OuterShape:
    H: int                                    # states
    G: int                                    # keys and queries, shared by H / G states each
    dim: int
    vdim: int
    rank: int = 0                             # of the decay's product (channel decays), padded to a multiple of 16

    @property
    def D(self) -> int:
        return (self.dim + 15) // 16 * 16

    @property
    def V(self) -> int:
        return (self.vdim + 15) // 16 * 16

    @property
    def inner(self) -> int:
        return self.H * self.V


class OuterArgs(ctypes.Structure):
    _fields_ = [("rows", RowArgs), ("q", _P), ("k", _P), ("v", _P), ("ld", _L),
                ("a1", _P), ("a2", _P), ("a2b", _P), ("lda1", _L),
                ("dt", _P), ("dt_bias", _P), ("A", _P), ("lddt", _L),
                ("state", _P), ("o", _P), ("pairs", _P), ("factors", _P), ("ws", _P), ("ws_decay", _P), ("gate", _P), ("ldg", _L), ("norm_w", _P), ("skip", _P),
                ("out", _P), ("ldo", _L),
                ("kind", _I), ("H", _I), ("G", _I), ("D", _I), ("V", _I), ("dim", _I), ("vdim", _I), ("rank", _I), ("f32", _I),
                ("parts", _I), ("seg_tiles", _I), ("multi", _I), ("q_scale", _F), ("inv_tau", _F), ("eps", _F), ("out_scale", _F)]


_declared = False


def _declare():
    global _declared
    if _declared:
        return
    A = ctypes.POINTER(OuterArgs)
    _lib.declare("b200_outer_fits", [A], _I)
    _lib.declare("b200_outer_workspace", [_I, _I, ctypes.POINTER(_I)], None)
    _lib.declare("b200_outer_step", [A, _I, _P], _I)
    _lib.declare("b200_outer_chunk", [A, _P], _I)
    _lib.declare("b200_outer_norm", [A, _I, _I, _P], _I)
    lib()
    _declared = True


MIN_SEGMENT = 4                               # 128-row tiles


def segment_tiles(num_tiles: int, portions: int, ctas: int, num_sms: int) -> int:
    """Tiles per segment of a portion, or 0 for whole portions: where ``ctas`` per segment do not fill the GPU, a
    portion is cut into parts that run side by side (all but the first and last twice: once for the state behind
    them, once from the state before them)."""
    if portions <= 0:
        return 0
    cuts = num_sms // max(1, ctas * portions) + 1
    per = -(-num_tiles // portions)
    if cuts < 3 or per < 2 * MIN_SEGMENT:
        return 0
    return max(MIN_SEGMENT, -(-per // cuts))


class Workspace:
    """Scratch of the chunk kernels for steps of up to ``max_tokens`` rows in ``max_portions`` portions; it serves every shape
    that :meth:`reserve` has seen."""

    def __init__(self, device, max_tokens: int, max_portions: int):
        self.device, self.chunks = device, max_tokens // 64 + max_portions
        # (a cut portion has 2 MIN_SEGMENT tiles at least, the last of them partly filled)
        self.segments = 2 * (max_tokens * 8 // (7 * 128 * MIN_SEGMENT) + 2)
        self.sizes = [0, 0, 0, 0]
        self.buffers: dict = {}

    def reserve(self, s: OuterShape, kind: int) -> None:
        _declare()
        v = (_I * 2)()
        lib().b200_outer_workspace(kind, s.D, v)
        need = (self.chunks * s.H * v[0], self.chunks * s.H * v[1], self.segments * s.H * s.D * s.V, self.segments * s.H * s.D)
        self.sizes = [max(a, b) for a, b in zip(self.sizes, need)]

    def allocate(self) -> dict:
        f32 = torch.float32
        self.buffers = {n: torch.empty(z, dtype=t, device=self.device) for n, z, t in
                        zip(("pairs", "factors", "states", "decays"), self.sizes, (torch.bfloat16, f32, f32, f32))}
        return self.buffers


def outer_args(s: OuterShape, q, k, v, state, ctx, bufs, out, *, eps, q_scale=1.0, out_scale=1.0, channel=None, head=None, gate=None,
               norm_w=None, skip=None, parts=0) -> OuterArgs:
    """``channel``: (a1 [T, rank], a2 [H * D, rank], bias fp32 [H * D], tau); ``head``: (dt [T, H], bias, A fp32 [H])."""
    _declare()
    a = OuterArgs()
    _rows(a.rows, ctx, q.shape[0])
    a.q, a.k, a.v, a.ld = ptr(q), ptr(k), ptr(v), q.stride(0)
    assert q.stride(0) == k.stride(0) == v.stride(0)
    if channel is not None:
        a1, a2, bias, tau = channel
        a.kind, a.a1, a.lda1, a.a2, a.a2b, a.inv_tau = CHANNEL, ptr(a1), a1.stride(0), ptr(a2), ptr(bias), 1.0 / tau
    else:
        dt, bias, A = head
        a.kind, a.dt, a.lddt, a.dt_bias, a.A = HEAD, ptr(dt), dt.stride(0), ptr(bias), ptr(A)
    a.state, a.o, a.ws, a.ws_decay = ptr(state), ptr(bufs["o"]), ptr(bufs.get("states")), ptr(bufs.get("decays"))
    a.pairs, a.factors = ptr(bufs.get("pairs")), ptr(bufs.get("factors"))
    a.gate, a.ldg, a.norm_w, a.skip = ptr(gate), gate.stride(0), ptr(norm_w), ptr(skip)
    a.out, a.ldo = ptr(out), out.stride(0)
    a.H, a.G, a.D, a.V, a.dim, a.vdim, a.rank = s.H, s.G, s.D, s.V, s.dim, s.vdim, s.rank
    a.f32, a.parts, a.q_scale, a.eps, a.out_scale = int(q.dtype == torch.float32), parts, q_scale, eps, out_scale
    return a


def run(a: OuterArgs, ctx, bufs, *, token_by_token=False, seg_tiles=None) -> None:
    """Recurrence and norm of all rows."""
    chunks = a.rows.num_prefills > 0 and not token_by_token and bool(lib().b200_outer_fits(ctypes.byref(a)))
    reqs = a.rows.nd + (0 if chunks else a.rows.num_prefills)
    if reqs:
        check(lib().b200_outer_step(ctypes.byref(a), reqs, stream_ptr()), "outer_step")
    if chunks:
        if seg_tiles is None:
            from . import num_sms
            seg_tiles = segment_tiles(a.rows.num_tiles, a.rows.num_prefills, a.H * -(-a.V // 64), num_sms())
        a.seg_tiles, a.multi = seg_tiles or 1 << 20, int(seg_tiles > 0 and a.rows.num_tiles > seg_tiles)
        if a.multi:
            most = 2 * (a.rows.num_tiles // seg_tiles + 1)
            assert bufs["states"].numel() >= most * a.H * a.D * a.V and bufs["decays"].numel() >= most * a.H * a.D
        v = (_I * 2)()
        lib().b200_outer_workspace(a.kind, a.D, v)
        most = a.H * ((a.rows.T - a.rows.nd) // 64 + a.rows.num_prefills)
        assert bufs["pairs"].numel() >= most * v[0] and bufs["factors"].numel() >= most * v[1]
        check(lib().b200_outer_chunk(ctypes.byref(a), stream_ptr()), "outer_chunk")
    # (decode rows of the channel kind are normed by the step kernel where it holds whole heads)
    check(lib().b200_outer_norm(ctypes.byref(a), reqs, int(chunks), stream_ptr()), "outer_norm")


def gated_linear_attention(q, k, v, gate, a1, w, s: OuterShape, state, ctx, bufs, out, *, tau, eps, token_by_token=False,
                           seg_tiles=None):
    """``q`` / ``k`` [T, H * D], ``v`` / ``gate`` [T, H * V], ``a1`` [T, rank] (columns of one projection) -> ``out`` [T, H * V].
    The state fades per key channel by sigmoid(a2 a1 + bias)^(1 / tau), ``w``: a2 [H * D, rank], a2_bias fp32 [H * D],
    norm fp32 [V]. ``state`` fp32 [slots, H, D, V] is advanced; a request's first rows start from zero. ``bufs``: o fp32
    [T, H * V], and for prompts the buffers of a :class:`Workspace`. bf16 prompts run in chunks of 64 tokens
    on the tensor cores; ``token_by_token``, fp32 and sizes beyond them walk the tokens."""
    a = outer_args(s, q, k, v, state, ctx, bufs, out, eps=eps, q_scale=s.dim ** -0.5, channel=(a1, w["a2"], w["a2_bias"], tau),
                   gate=gate, norm_w=w["norm"])
    run(a, ctx, bufs, token_by_token=token_by_token, seg_tiles=seg_tiles)
    return out


def state_space(u, z, dt, w, s: OuterShape, state, ctx, bufs, out, *, parts, eps, scale=1.0, token_by_token=False, seg_tiles=None):
    """``u`` [T, x | B | C] (convolved), gate ``z`` [T, H * V], ``dt`` [T, H] -> ``out`` [T, H * V] = scale * norm in ``parts``
    equal parts of (y + D x) silu(z). ``w``: dt_bias, A (= exp(A_log)), D fp32 [H], norm fp32 [H * V]."""
    gd = s.G * s.D
    x, B, C = u[:, : s.inner], u[:, s.inner: s.inner + gd], u[:, s.inner + gd: s.inner + 2 * gd]
    a = outer_args(s, C, B, x, state, ctx, bufs, out, eps=eps, out_scale=scale, head=(dt, w["dt_bias"], w["A"]), gate=z,
                   norm_w=w["norm"], skip=w["D"], parts=parts)
    run(a, ctx, bufs, token_by_token=token_by_token, seg_tiles=seg_tiles)
    return out


# ------------------------------------------------------------------------------ restatements
def _ref_recurrence(q, k, v, decay, state, ctx):
    """q, k, decay [T, H, D], v [T, H, V] -> o [T, H, V]."""
    o = torch.zeros_like(v)
    for t0, t1, slot, fresh in _portions(ctx):
        S = torch.zeros_like(state[slot]) if fresh else state[slot].clone()
        for t in range(t0, t1):
            S = S * decay[t].unsqueeze(-1) + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        state[slot] = S
    return o


def ref_gated_linear_attention(q, k, v, gate, a1, w, s: OuterShape, state, ctx, bufs, out, *, tau, eps, **_):
    T = q.shape[0]
    z = a1.float() @ w["a2"].float().t() + w["a2_bias"]
    decay = torch.exp(torch.nn.functional.logsigmoid(z) / tau).view(T, s.H, s.D)
    o = _ref_recurrence(q.float().reshape(T, s.H, s.D) * s.dim ** -0.5, k.float().reshape(T, s.H, s.D),
                        v.float().reshape(T, s.H, s.V), decay, state, ctx)
    o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / s.vdim + eps) * w["norm"]
    out.copy_(o.reshape(T, -1) * torch.nn.functional.silu(gate.float()))
    return out


def ref_state_space(u, z, dt, w, s: OuterShape, state, ctx, bufs, out, *, parts, eps, scale=1.0, **_):
    T, gd = u.shape[0], s.G * s.D
    x = u[:, : s.inner].float().reshape(T, s.H, s.V)
    B, C = (u[:, s.inner + i * gd: s.inner + (i + 1) * gd].float().reshape(T, s.G, s.D).repeat_interleave(s.H // s.G, 1) for i in (0, 1))
    step = torch.nn.functional.softplus(dt.float()[:, : s.H] + w["dt_bias"], threshold=1e9)
    decay = torch.exp(-w["A"] * step).unsqueeze(-1).expand(T, s.H, s.D)
    y = _ref_recurrence(C, B, x * step.unsqueeze(-1), decay, state, ctx) + w["D"][:, None] * x
    y = (y * torch.nn.functional.silu(z.float().reshape(T, s.H, s.V)))[..., : s.vdim].reshape(T, parts, -1)
    y = (y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)).reshape(T, s.H, s.vdim)
    res = torch.zeros(T, s.H, s.V)
    res[..., : s.vdim] = y
    out.copy_(scale * res.reshape(T, -1) * w["norm"])
    return out
