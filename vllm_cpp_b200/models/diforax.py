"""Diforax decoders: delta-rule and chunked-attention blocks in any order over an fp32 residual stream.

A sublayer f (mixer, then feed-forward) sits between two norms:  x += n2(f(n1(x))).

* Delta mixer (``ops/delta.py``): short convolutions, unit q / k, one decay and one write strength per
  head; the fp32 state and the convolutions' last inputs are kept per request slot (``recurrent.py``).
* Attention mixer (``ops/bias_attn.py``): q and k are rotated, then divided by their root mean square;
  a query sees its own chunk of positions. A block may read the keys and values of an earlier block.
* Feed-forward: a GELU gated unit, or experts chosen by corrected softmax scores among the best groups;
  identity experts return their input. The expert sum, the norm after it, the residual sum and the next
  norm are one kernel (``ops/stream.py``).

Every block has its own sizes. Storage is padded with zeros (head sizes to multiples of 16, other widths to
multiples of 8), so any size goes through the kernels; ``cfg.dtype == "float32"`` runs the same forward in
32 bits."""
from __future__ import annotations

import torch

from ..config import DenseSpec, ExpertSpec
from ..ops.bias_attn import grouped_decode_splits
from ..ops.delta import DeltaShape
from .base import StepContext
from .listed import ListedModel, pad as _pad, pad_heads as _pad_heads
from .recurrent import RecurrentState


def _delta_shape(d) -> DeltaShape:
    return DeltaShape(G=d.kv_heads, H=d.heads, D=_pad(d.dim, 16), V=_pad(d.vdim, 16), dim=d.dim, vdim=d.vdim, taps=d.conv)


class DiforaxModel(ListedModel):
    def __init__(self, cfg, *args, **kw):
        super().__init__(cfg, *args, **kw)
        self.delta_layers = [l for l, b in enumerate(cfg.blocks) if b.delta is not None]
        self.kv_layers = [l for l, b in enumerate(cfg.blocks) if b.attention is not None and b.attention.kv_from is None]
        self.moe_ws: dict = {}
        self.chunks = None                    # scratch of the chunked delta rule

    # ------------------------------------------------------------------ weights
    def init_random(self, seed: int = 0, std: float = 0.02) -> None:
        c, W = self.cfg, self.width
        big = sum(b.mlp.experts * b.mlp.ff * 3 * W for b in c.blocks if isinstance(b.mlp, ExpertSpec)) > 5e8
        gdev = self.device if (self.device.type == "cuda" and big) else torch.device("cpu")
        g = torch.Generator(device=gdev).manual_seed(seed)

        def full(*shape, s=std, mean=0.0):
            return torch.empty(shape, dtype=torch.float32, device=gdev).normal_(mean, s, generator=g).to(torch.bfloat16)

        def gen():
            yield "embed", full(c.vocab_size, W)
            for l, b in enumerate(c.blocks):
                m, d, f = b.attention or b.delta, b.delta, b.mlp
                norms = ("norm1", "norm1b") if f is None else ("norm1", "norm1b", "norm2", "norm2b")
                for n in norms:
                    yield f"l{l}.{n}", full(W, s=0.1, mean=1.0)
                own = d is not None or b.attention.kv_from is None
                vheads = m.heads if d is not None else m.kv_heads
                qheads = m.kv_heads if d is not None else m.heads
                rows = {"q": qheads * m.dim, "k": m.kv_heads * m.dim, "v": vheads * m.vdim}
                for n in ("q", "k", "v") if own else ("q",):
                    yield f"l{l}.mix.{n}", full(rows[n], W)
                    if d is not None:
                        yield f"l{l}.mix.{n}.conv", full(rows[n], d.conv, s=0.5)
                yield f"l{l}.mix.o", full(W, m.heads * m.vdim)
                if d is not None:
                    yield f"l{l}.mix.g", full(m.heads * m.vdim, W)
                    for n in ("a", "b"):
                        yield f"l{l}.mix.{n}", full(m.heads, W)
                    yield f"l{l}.mix.A_log", full(m.heads, s=0.5)
                    yield f"l{l}.mix.dt_bias", full(m.heads, s=0.5, mean=-2.0)
                    yield f"l{l}.mix.norm", full(m.vdim, s=0.1, mean=1.0)
                units = [""] if isinstance(f, DenseSpec) else [f"e{e}." for e in range(f.experts)] if f is not None else []
                for u in units:
                    yield f"l{l}.mlp.{u}gate", full(f.ff, W)
                    yield f"l{l}.mlp.{u}up", full(f.ff, W)
                    yield f"l{l}.mlp.{u}down", full(W, f.ff)
                if isinstance(f, ExpertSpec):
                    yield f"l{l}.mlp.router", full(f.experts + f.identity, W)
                    yield f"l{l}.mlp.correction", full(f.experts + f.identity, s=0.01)
            yield "final.norm", full(W, s=0.1, mean=1.0)
            yield "head", full(c.vocab_size, W)

        self.load_weights(gen())

    def load_weights(self, named_tensors) -> None:
        c, C, dev, dt, put = self.cfg, self.cols, self.device, self.dtype, self.put
        self.layers = [dict() for _ in c.blocks]
        for L, b in zip(self.layers, c.blocks):
            if isinstance(b.mlp, ExpertSpec):
                f8 = _pad(b.mlp.ff)
                L["w_gate_up"] = torch.zeros((b.mlp.experts, 2 * f8, C), dtype=dt, device=dev)
                L["w_down"] = torch.zeros((b.mlp.experts, C, f8), dtype=dt, device=dev)
        pend: list[dict] = [dict() for _ in c.blocks]
        for name, t in named_tensors:
            if not self._take_shared(name, t):
                l, rest = self._block_of(name)
                L, f, part = self.layers[l], c.blocks[l].mlp, rest.split(".")
                if isinstance(f, ExpertSpec) and part[0] == "mlp" and len(part) == 3:
                    e, f8 = int(part[1][1:]), _pad(f.ff)
                    if part[2] == "down":
                        L["w_down"][e, : self.width, : f.ff] = t.to(dev, dt)
                    else:
                        r0 = {"gate": 0, "up": f8}[part[2]]
                        L["w_gate_up"][e, r0: r0 + f.ff, : self.width] = t.to(dev, dt)
                pend[l][rest] = None if "w_gate_up" in L and len(part) == 3 and part[0] == "mlp" else t
        for l, (L, b, p) in enumerate(zip(self.layers, c.blocks, pend)):
            self._expect(l, self._tensor_names(b), set(p))
            for n in ("norm1", "norm1b", "norm2", "norm2b"):
                if n in p:
                    L[n] = put(p[n], C, dtype=torch.float32)
            (self._load_delta if b.delta is not None else self._load_attention)(L, b, {n[4:]: t for n, t in p.items()}, put)
            f = b.mlp
            if isinstance(f, DenseSpec):
                self._load_dense(L, f, p)
            elif f is not None:
                L["router"] = put(p["mlp.router"], _pad(f.experts + f.identity), C)
                L["correction"] = put(p["mlp.correction"], dtype=torch.float32)
        self._expect_shared()

    @staticmethod
    def _tensor_names(b) -> set:
        d, f = b.delta, b.mlp
        names = {"norm1", "norm1b", "mix.q", "mix.o"}
        if d is not None or b.attention.kv_from is None:
            names |= {"mix.k", "mix.v"}
        if d is not None:
            names |= {"mix." + n for n in ("q.conv", "k.conv", "v.conv", "g", "a", "b", "A_log", "dt_bias", "norm")}
        if f is not None:
            names |= {"norm2", "norm2b"}
        units = [""] if isinstance(f, DenseSpec) else [f"e{e}." for e in range(f.experts)] if f is not None else []
        names |= {f"mlp.{u}{n}" for u in units for n in ("gate", "up", "down")}
        return names | ({"mlp.router", "mlp.correction"} if isinstance(f, ExpertSpec) else set())

    def _load_delta(self, L, b, p, put) -> None:
        d, s, f32 = b.delta, _delta_shape(b.delta), dict(dtype=torch.float32)
        heads = {"q": (s.G, s.D), "k": (s.G, s.D), "v": (s.H, s.V), "g": (s.H, s.V)}
        rows = {n: _pad_heads(p[n], *heads[n]) for n in heads}
        L["shape"] = s
        L["proj"] = put(torch.cat(list(rows.values()), 0), s.columns, self.cols)
        L["ab"] = put(torch.cat([p["a"], p["b"]], 0), _pad(2 * s.H), self.cols)
        L["conv_w"] = put(torch.cat([_pad_heads(p[n + ".conv"], *heads[n]) for n in ("q", "k", "v")], 0).t(), **f32)
        L["A"], L["dt"] = torch.exp(put(p["A_log"], **f32)), put(p["dt_bias"], **f32)
        L["norm"] = put(p["norm"], s.V, **f32)
        L["o"] = put(_pad_heads(p["o"], d.heads, s.V, axis=1), self.cols, s.H * s.V)

    def _load_attention(self, L, b, p, put) -> None:
        a = b.attention
        D, V = _pad(a.dim, 16), _pad(a.vdim, 16)
        rows = [_pad_heads(p["q"], a.heads, D)]
        if a.kv_from is None:
            rows += [_pad_heads(p["k"], a.kv_heads, D), _pad_heads(p["v"], a.kv_heads, V)]
        q = torch.cat(rows, 0)
        L["proj"] = put(q, q.shape[0], self.cols)
        L["o"] = put(_pad_heads(p["o"], a.heads, V, axis=1), self.cols, a.heads * V)
        key = (a.rot_dims, a.rot_base)
        if a.rot_dims and key not in self.rope:
            i = torch.arange(0, a.rot_dims, 2, dtype=torch.float64)
            self.rope[key] = self.be.rope_table(a.rot_base ** (-i / a.rot_dims), self.max_position + 8)

    # ------------------------------------------------------------------ caches and state
    def _kv_row(self, l: int) -> int:
        a = self.cfg.blocks[l].attention
        return a.kv_heads * (_pad(a.dim, 16) + _pad(a.vdim, 16))

    def kv_cache_groups(self, block_size: int):
        """One group: blocks that all see the same chunks give back the pages behind the current one."""
        att = [b.attention for b in self.cfg.blocks if b.attention is not None]
        chunks = {a.chunk for a in att}
        big = max((self.cfg.blocks[l].attention for l in self.kv_layers), key=lambda a: a.kv_heads * (a.dim + a.vdim),
                  default=None)
        spec = dict(kind="full", block_size=block_size, num_kv_heads=big.kv_heads if big else 1,
                    head_size=big.dim if big else 8, head_size_v=big.vdim if big else 8, dtype_bytes=self.dtype.itemsize)
        if len(chunks) == 1 and chunks != {0}:
            spec.update(kind="chunked", attention_chunk_size=chunks.pop())
        return [(list(self.kv_layers), spec)]

    def alloc_kv_cache(self, num_blocks: int, block_size: int):
        """One tensor per block with keys of its own: a page holds ``block_size`` key rows, then value rows."""
        self.block_size = block_size
        self.kv_caches = [torch.zeros((num_blocks, block_size * self._kv_row(l)), dtype=self.dtype, device=self.device)
                          for l in self.kv_layers]
        self.cache_of = dict(zip(self.kv_layers, self.kv_caches))
        for l, b in enumerate(self.cfg.blocks):
            if b.attention is not None and b.attention.kv_from is not None:
                self.cache_of[l] = self.cache_of[b.attention.kv_from]
        self.layer_group = [0] * len(self.cfg.blocks)
        return self.kv_caches

    def kv_bytes_per_block(self, block_size: int) -> int:
        return max(1, sum(block_size * self._kv_row(l) for l in self.kv_layers) * self.dtype.itemsize)

    def state_bytes_per_request(self) -> int:
        n = 0
        for l in self.delta_layers:
            s = _delta_shape(self.cfg.blocks[l].delta)
            n += (s.taps - 1) * s.channels * self.dtype.itemsize + s.H * s.D * s.V * 4
        return n

    def decode_workspace(self, batch: int, max_seq_len: int, block_size: int):
        """(KV splits, split buffers) of a decode batch; one pair of buffers serves every block."""
        att = [b.attention for b in self.cfg.blocks if b.attention is not None]
        if self.device.type != "cuda" or not att:
            return 1, None
        from .. import ops
        keys = max(min(a.chunk or max_seq_len, max_seq_len) for a in att)
        s = grouped_decode_splits(batch, min(a.kv_heads for a in att), keys, ops.num_sms())
        if s == 1:
            return 1, None
        heads, out = max(a.heads for a in att), max(a.heads * _pad(a.vdim, 16) for a in att)
        return s, (torch.empty(batch * s * out, dtype=torch.float32, device=self.device),
                   torch.empty(batch * s * heads, dtype=torch.float32, device=self.device))

    # ------------------------------------------------------------------ buffers
    def _delta_buffers(self, s: DeltaShape, T: int):
        f32 = torch.float32
        proj = self.bufs.get(f"proj{s.columns}", T, s.columns, self.dtype)
        ab = self.bufs.get(f"ab{_pad(2 * s.H)}", T, _pad(2 * s.H), f32)
        sizes = {"q": (s.G * s.D, f32), "k": (s.G * s.D, f32), "v": (s.H * s.V, self.dtype), "g": (s.H, f32),
                 "beta": (s.H, f32), "o": (s.H * s.V, f32)}
        bufs = {n: self.bufs.get(f"delta_{n}{w}", T, w, t) for n, (w, t) in sizes.items()}
        bufs["chunks"] = self.chunks
        return proj, ab, bufs, self.bufs.get(f"heads{s.H * s.V}", T, s.H * s.V, self.dtype)

    def _attention_buffers(self, a, T: int):
        D, V = _pad(a.dim, 16), _pad(a.vdim, 16)
        n = a.heads * D + (a.kv_heads * (D + V) if a.kv_from is None else 0)
        return (self.bufs.get(f"proj{n}", T, n, self.dtype), self.bufs.get(f"q{a.heads * D}", T, a.heads * D, self.dtype),
                self.bufs.get(f"heads{a.heads * V}", T, a.heads * V, self.dtype))

    def reserve_buffers(self, max_tokens: int, max_reqs: int) -> None:
        self._reserve_rows(max_tokens, max_reqs)
        self.recurrent = RecurrentState()
        heads = max([self.cfg.blocks[l].delta.heads for l in self.delta_layers], default=0)
        if heads and self._bf16_kernels():
            from ..ops.delta import chunk_workspace
            self.chunks = chunk_workspace(self.device, (max_tokens + 127) // 128 + max_reqs, heads)
        for l, b in enumerate(self.cfg.blocks):
            f = b.mlp
            if b.delta is not None:
                s = _delta_shape(b.delta)
                self._delta_buffers(s, max_tokens)
                self.state[l] = (self.recurrent.add((max_reqs, s.taps - 1, s.channels), self.dtype, self.device),
                                 self.recurrent.add((max_reqs, s.H, s.D, s.V), torch.float32, self.device))
            else:
                self._attention_buffers(b.attention, max_tokens)
            if isinstance(f, DenseSpec):
                self._dense_buffers(f, max_tokens)
            elif f is not None:
                n, key = _pad(f.experts + f.identity), (f.experts, f.top, f.ff)
                self.bufs.reserve(f"router{n}", max_tokens, n, torch.float32)
                if self.device.type == "cuda" and key not in self.moe_ws:
                    from ..ops.moe import MoeWorkspace
                    self.moe_ws[key] = MoeWorkspace(self.device, max_tokens, f.top, f.experts, self.cols, _pad(f.ff),
                                                    self.dtype)

    # ------------------------------------------------------------------ forward
    def _delta(self, h, l, L, ctx, T, out):
        be, s = self.be, L["shape"]
        proj, ab, bufs, heads = self._delta_buffers(s, T)
        be.gemm(h, L["proj"], out=proj, out_dtype=self.dtype)
        be.gemm(h, L["ab"], out=ab, out_dtype=torch.float32)
        be.delta_mixer(proj, ab, L, s, *self.state[l], ctx, bufs, heads, self.cfg.rms_norm_eps)
        be.gemm(heads, L["o"], out=out, out_dtype=torch.float32)

    def _attention(self, h, l, L, a, ctx, T, out):
        be, D, V = self.be, _pad(a.dim, 16), _pad(a.vdim, 16)
        proj, q, heads = self._attention_buffers(a, T)
        be.gemm(h, L["proj"], out=proj, out_dtype=self.dtype)
        grp, cache = self.layer_group[l], self.cache_of[l]
        be.rotate_kv(proj, ctx.positions[:T], self.rope.get((a.rot_dims, a.rot_base)), a.rot_dims, self.cfg.rms_norm_eps,
                     q, ctx.slot_mapping[grp][:T], cache, H=a.heads, G=a.kv_heads if a.kv_from is None else 0, D=D, V=V,
                     dim=a.dim, block_size=self.block_size)
        be.bias_attention(q, cache, ctx, grp, out=heads, H=a.heads, G=a.kv_heads, kw=a.kv_heads * D, vdim=V,
                          block_size=self.block_size, scale=a.scale, chunk=a.chunk, grouped=True)
        be.gemm(heads, L["o"], out=out, out_dtype=torch.float32)

    def _feed_forward(self, h, L, f, T, out):
        """-> what ``stream_norm`` adds: a product, or expert outputs and where to find them."""
        be = self.be
        if isinstance(f, DenseSpec):
            return dict(a=self._dense(h, L, f, "gelu_tanh", T, out))
        n = f.experts + f.identity
        logits = self.bufs.get(f"router{_pad(n)}", T, _pad(n), torch.float32)
        be.gemm(h, L["router"], out=logits, out_dtype=torch.float32)
        y, pos, w = be.routed_experts(h, logits[:, :n], L["w_gate_up"], L["w_down"],
                                      self.moe_ws.get((f.experts, f.top, f.ff)), top=f.top, correction=L["correction"],
                                      groups=f.groups, keep=f.keep)
        return dict(y=y, pair_pos=pos, pair_w=w, ident=h if f.identity else None)

    def forward(self, ctx: StepContext) -> torch.Tensor:
        """Returns fp32 logits ``[num_logits, vocab]`` for the rows in ``ctx.logits_indices``."""
        c, be, T = self.cfg, self.be, ctx.num_tokens
        eps, norm = c.rms_norm_eps, dict(width=self.width, norm_offset=0.0)
        stream = self.bufs.get("stream", T, self.cols, torch.float32)
        h = self.bufs.get("normed", T, self.cols, self.dtype)
        mixed = self.bufs.get("mixed", T, self.cols, torch.float32)
        be.stream_norm(stream, self.layers[0]["norm1"], eps, h, ids=ctx.input_ids[:T], table=self.w["embed"], **norm)
        for l, (L, b) in enumerate(zip(self.layers, c.blocks)):
            if b.delta is not None:
                self._delta(h, l, L, ctx, T, mixed)
            else:
                self._attention(h, l, L, b.attention, ctx, T, mixed)
            nw = self.layers[l + 1]["norm1"] if l + 1 < len(self.layers) else self.w["final_norm"]
            be.stream_norm(stream, nw if b.mlp is None else L["norm2"], eps, h, a=mixed, post_w=L["norm1b"], **norm)
            if b.mlp is not None:
                add = self._feed_forward(h, L, b.mlp, T, mixed)
                be.stream_norm(stream, nw, eps, h, post_w=L["norm2b"], **add, **norm)
        return self._logits(ctx, h)
