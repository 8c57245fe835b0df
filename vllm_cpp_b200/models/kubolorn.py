"""Kubolorn decoders: gated-linear-attention blocks and blocks with softmax attention beside a state-space mixer, in
any order over an fp32 residual stream, with layers that run several times in a row.

Mixer and feed-forward read the same stream,  x += mixer(c1(norm1(x))) + ff(c2(norm2(x))):  norms in equal parts of
a row, then the input plus a short convolution of it. One kernel (``ops/conv_norm.py``) adds up the stream, norms it
and runs both convolutions; one product takes the outputs of mixer and dense feed-forward side by side, so that their
sum is never formed apart.

* Gated linear attention and the state-space mixer are recurrences over outer products (``ops/outer.py``).
* Attention (``ops/bias_attn.py``): the values are the keys before their rotation, so a cache row holds the shared
  columns once; a learned sink per head joins the softmax.
* Feed-forward: ungated units, dense or as routed experts.
* The stream starts as a normed sum of a token's and a token pair's embedding; the head is the embedding table.

Per request slot (``recurrent.py``): fp32 states, the convolutions' past rows, the last token. A pass of a looped layer
is a block of its own with the weights of the first pass. Storage is padded with zeros (head sizes to multiples of 16,
other widths to multiples of 8), so any size goes through the kernels; ``cfg.dtype == "float32"`` runs the same forward
in 32 bits."""
from __future__ import annotations

import torch

from ..config import DenseSpec, ExpertSpec
from ..ops.bias_attn import TiedShape, grouped_decode_splits
from ..ops.conv_norm import conv_weights
from ..ops.outer import CHANNEL, HEAD, OuterShape, Workspace
from .base import StepContext
from .listed import ListedModel, pad, pad_heads, padded
from .recurrent import RecurrentState


def tied_shape(a) -> TiedShape:
    return TiedShape(H=a.heads, G=a.kv_heads, dim=a.dim, rot=a.rot_dims)


def gla_shape(g, rank: int) -> OuterShape:
    return OuterShape(H=g.heads, G=g.heads, dim=g.dim, vdim=g.vdim, rank=pad(rank, 16))


def ssm_shape(r) -> OuterShape:
    return OuterShape(H=r.heads, G=r.groups, dim=r.state, vdim=r.vdim)


class KubolornModel(ListedModel):
    def __init__(self, cfg, *args, **kw):
        super().__init__(cfg, *args, **kw)
        self.kv_layers = [l for l, b in enumerate(cfg.blocks) if b.attention is not None]
        self.own = [l for l, b in enumerate(cfg.blocks) if b.weights_of is None]
        self.number = {l if cfg.blocks[l].layer is None else cfg.blocks[l].layer: l for l in self.own}
        self.moe_ws: dict = {}
        self.scratch: dict = {}

    # ------------------------------------------------------------------ weights
    def init_random(self, seed: int = 0, std: float = 0.02) -> None:
        c, W = self.cfg, self.width
        size = sum(f.ff * 2 * W * getattr(f, "experts", 1) for f in (c.blocks[l].mlp for l in self.own) if f is not None)
        gdev = self.device if (self.device.type == "cuda" and size > 2e8) else torch.device("cpu")
        g = torch.Generator(device=gdev).manual_seed(seed)

        def full(*shape, s=std, mean=0.0):
            return torch.empty(shape, dtype=torch.float32, device=gdev).normal_(mean, s, generator=g).to(torch.bfloat16)

        def norm(n):
            return full(n, s=0.1, mean=1.0)

        def gen():
            yield "embed", full(c.vocab_size, W)
            if c.bigram is not None:
                yield "bigram", full(c.bigram.buckets + 1, W)
            yield "embed.norm", norm(W)
            yield "final.norm", norm(W)
            for n, l in self.number.items():
                b, p = c.blocks[l], f"l{n}."
                for i in (1, 2) if b.mlp is not None else (1,):
                    yield f"{p}norm{i}", norm(W)
                    if c.input_conv:
                        yield f"{p}canon{i}", full(W, c.input_conv, s=0.2)
                a, r, la = b.attention, b.ssm, b.gla
                if la is not None:
                    for k, rows in (("q", la.dim), ("k", la.dim), ("v", la.vdim), ("g", la.vdim)):
                        yield f"{p}mix.{k}", full(la.heads * rows, W)
                    yield p + "mix.a1", full(la.rank, W)
                    yield p + "mix.a2", full(la.heads * la.dim, la.rank)
                    yield p + "mix.a2.b", full(la.heads * la.dim, s=1.0)
                    yield p + "mix.norm", norm(la.vdim)
                    yield p + "mix.o", full(W, la.heads * la.vdim)
                else:
                    q = p + "mix.left."
                    yield q + "q", full(a.heads * a.dim, W)
                    yield q + "k", full(a.kv_heads * a.dim, W)
                    yield q + "sink", full(a.heads, s=1.0)
                    yield q + "o", full(W, a.heads * a.vdim)
                    q, inner, gn = p + "mix.right.", r.heads * r.vdim, r.groups * r.state
                    yield q + "in", full(2 * inner + 2 * gn + r.heads, W)
                    yield q + "conv", full(inner + 2 * gn, r.conv, s=0.5)
                    yield q + "conv.b", full(inner + 2 * gn)
                    for k, m in (("dt_bias", -2.0), ("A_log", 1.0), ("D", 1.0)):
                        yield q + k, full(r.heads, s=0.5, mean=m)
                    yield q + "norm", norm(inner)
                    yield q + "o", full(W, inner)
                f = b.mlp
                for u in self._units(f):
                    yield f"{p}mlp.{u}up", full(f.ff, W)
                    yield f"{p}mlp.{u}down", full(W, f.ff)
                if isinstance(f, ExpertSpec):
                    yield p + "mlp.router", full(f.experts, W)

        self.load_weights(gen())

    GLA = ("q", "k", "v", "g", "a1", "a2", "a2.b", "norm", "o")
    LEFT = ("q", "k", "sink", "o")
    RIGHT = ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")

    @staticmethod
    def _units(f) -> list:
        return [] if f is None else [""] if isinstance(f, DenseSpec) else [f"e{e}." for e in range(f.experts)]

    def _tensor_names(self, b) -> set:
        names = {"mix." + n for n in self.GLA} if b.gla is not None else \
            {"mix.left." + n for n in self.LEFT} | {"mix.right." + n for n in self.RIGHT}
        for i in "12" if b.mlp is not None else "1":
            names |= {"norm" + i, "canon" + i} if self.cfg.input_conv else {"norm" + i}
        names |= {f"mlp.{u}{n}" for u in self._units(b.mlp) for n in ("up", "down")}
        return names | ({"mlp.router"} if isinstance(b.mlp, ExpertSpec) else set())

    def _take_shared(self, name: str, t: torch.Tensor) -> bool:
        if name == "embed":                            # (rows past the vocabulary are never looked up)
            self.w["embed"] = self.w["lm_head"] = self.put(t, pad(t.shape[0]), self.cols)
        elif name == "bigram" and self.cfg.bigram is not None:
            self.w["bigram"] = self.put(t, t.shape[0], self.cols)
        elif name in ("embed.norm", "final.norm"):
            self.w[name.replace(".", "_")] = self.put(t, self.cols, dtype=torch.float32)
        else:
            return False
        return True

    def load_weights(self, named_tensors) -> None:
        blocks = self.cfg.blocks
        self.layers = [dict() for _ in blocks]
        pend: dict[int, dict] = {l: {} for l in self.own}
        for name, t in named_tensors:
            if self._take_shared(name, t):
                continue
            layer, _, rest = name.partition(".")
            l = self.number.get(int(layer[1:])) if layer[:1] == "l" and layer[1:].isdigit() else None
            if l is None:
                raise ValueError(f"unexpected tensor {name!r}")
            pend[l][rest] = t
        for n, l in self.number.items():
            L, b, p = self.layers[l], blocks[l], pend.pop(l)
            spare = {"norm2", "canon2"} if b.mlp is None else set()      # (of a feed-forward that is not there)
            self._expect(n, self._tensor_names(b), set(p) - spare)
            reads = []
            for i in "12" if b.mlp is not None else "1":
                w = self.put(p["norm" + i], self.cols, dtype=torch.float32)
                taps = p.get("canon" + i)
                reads.append(w[None] if taps is None else
                             conv_weights(w, padded(taps.to(self.device, torch.float32), self.cols, taps.shape[1])))
            L["reads"] = reads
            mix = {k[4:]: t for k, t in p.items() if k.startswith("mix.")}
            outs = self._load_gla(L, b.gla, mix) if b.gla is not None else self._load_parallel(L, b, mix)
            f = b.mlp
            if isinstance(f, DenseSpec):
                L["up"] = self.put(p["mlp.up"], pad(f.ff, 16), self.cols)
                outs.append(self.put(p["mlp.down"], self.cols, pad(f.ff, 16)))
            elif f is not None:
                ff = pad(f.ff)
                L["router"] = self.put(p["mlp.router"], pad(f.experts), self.cols)
                L["w_up"] = torch.stack([self.put(p[f"mlp.e{e}.up"], ff, self.cols) for e in range(f.experts)])
                L["w_down"] = torch.stack([self.put(p[f"mlp.e{e}.down"], self.cols, ff) for e in range(f.experts)])
            L["o"] = torch.cat(outs, 1).contiguous()     # one product over [mixer outputs | feed-forward]
        for l, b in enumerate(blocks):
            if b.weights_of is not None:
                self.layers[l] = self.layers[b.weights_of]
        self._expect_shared()
        for k in ["embed_norm"] + (["bigram"] if self.cfg.bigram is not None else []):
            if k not in self.w:
                raise ValueError(f"{k} is missing from the checkpoint")

    def _load_gla(self, L, g, p) -> list:
        s, f32 = gla_shape(g, p["a1"].shape[0]), dict(dtype=torch.float32)
        L["shape"] = s
        parts = [pad_heads(p[n], s.H, w) for n, w in (("q", s.D), ("k", s.D), ("v", s.V), ("g", s.V))]
        proj = torch.cat(parts + [padded(p["a1"], s.rank, p["a1"].shape[1])], 0)
        L["proj"] = self.put(proj, proj.shape[0], self.cols)
        L["a2"] = self.put(pad_heads(p["a2"], s.H, s.D), s.H * s.D, s.rank)
        L["a2_bias"] = self.put(pad_heads(p["a2.b"], s.H, s.D), **f32)
        L["norm"] = self.put(p["norm"], s.V, **f32)
        return [self.put(pad_heads(p["o"], s.H, s.V, axis=1), self.cols, s.inner)]

    def _load_parallel(self, L, b, p) -> list:
        a, r, f32 = b.attention, b.ssm, dict(dtype=torch.float32)
        L["tied"], L["shape"] = t, s = tied_shape(a), ssm_shape(r)
        left, right = ({k[len(x):]: v for k, v in p.items() if k.startswith(x)} for x in ("left.", "right."))
        inner, gn = r.heads * r.vdim, r.groups * r.state
        z, x, B, C, dt = torch.split(right["in"], [inner, inner, gn, gn, r.heads], 0)
        spread = lambda v, n, w: pad_heads(v, n, w)                                              # noqa: E731
        rows = [t.spread(left["q"], t.H), t.spread(left["k"], t.G), spread(z, s.H, s.V), spread(x, s.H, s.V),
                spread(B, s.G, s.D), spread(C, s.G, s.D), dt]
        proj = torch.cat(rows, 0)
        L["proj"] = self.put(proj, pad(proj.shape[0]), self.cols)

        def channels(v):
            x, B, C = torch.split(v, [inner, gn, gn], 0)
            return torch.cat([spread(x, s.H, s.V), spread(B, s.G, s.D), spread(C, s.G, s.D)], 0)
        L["conv_w"] = self.put(channels(right["conv"]).t(), **f32)
        L["conv_b"] = self.put(channels(right["conv.b"]), **f32)
        L["dt_bias"], L["D"] = self.put(right["dt_bias"], **f32), self.put(right["D"], **f32)
        L["A"] = torch.exp(self.put(right["A_log"], **f32))
        L["norm"] = self.put(spread(right["norm"], s.H, s.V), **f32)
        L["sink"] = self.put(left["sink"], **f32)
        L["rope"] = self._rope_table(a.rot_base, a.rot_dims, a.rot_scaling)
        return [self.put(t.spread(left["o"], t.H, axis=1), self.cols, t.H * t.D),
                self.put(pad_heads(right["o"], s.H, s.V, axis=1), self.cols, s.inner)]

    # ------------------------------------------------------------------ caches and state
    def _row(self, l: int) -> int:
        """Cache values of a token."""
        t = tied_shape(self.cfg.blocks[l].attention)
        return t.G * t.pitch

    def kv_cache_groups(self, block_size: int):
        row = max((self._row(l) for l in self.kv_layers), default=16)
        return [(list(self.kv_layers), dict(kind="full", block_size=block_size, num_kv_heads=1, head_size=row - row // 2,
                                            head_size_v=row // 2, dtype_bytes=self.dtype.itemsize))]

    def alloc_kv_cache(self, num_blocks: int, block_size: int):
        """One tensor per attention: a page holds ``block_size`` rows of ``[first | rest | first rotated]`` per group."""
        self.block_size = block_size
        self.kv_caches = [torch.zeros((num_blocks, block_size * self._row(l)), dtype=self.dtype, device=self.device)
                          for l in self.kv_layers]
        self.cache_of = dict(zip(self.kv_layers, self.kv_caches))
        self.layer_group = [0] * len(self.cfg.blocks)
        return self.kv_caches

    def kv_bytes_per_block(self, block_size: int) -> int:
        return max(1, sum(block_size * self._row(l) for l in self.kv_layers) * self.dtype.itemsize)

    def _state_shapes(self, b):
        """(convolved channels and their past rows, states) of a block's mixer."""
        s = gla_shape(b.gla, 0) if b.gla is not None else ssm_shape(b.ssm)
        conv = None if b.gla is not None else (b.ssm.conv - 1, s.inner + 2 * s.G * s.D)
        return conv, (s.H, s.D, s.V)

    def state_bytes_per_request(self) -> int:
        n = 8
        for b in self.cfg.blocks:
            conv, (H, D, V) = self._state_shapes(b)
            n += H * D * V * 4 + max(0, self.cfg.input_conv - 1) * self.cols * 4
            n += conv[0] * conv[1] * self.dtype.itemsize if conv else 0
        return n

    def decode_workspace(self, batch: int, max_seq_len: int, block_size: int):
        """(KV splits, split buffers) of a decode batch; one pair of buffers serves every block."""
        if self.device.type != "cuda" or not self.kv_layers:
            return 1, None
        from .. import ops
        att = [tied_shape(self.cfg.blocks[l].attention) for l in self.kv_layers]
        s = max(grouped_decode_splits(batch, t.G * -(-t.H // t.G // 16), max_seq_len, ops.num_sms()) for t in att)
        if s == 1:
            return 1, None
        return s, (torch.empty(batch * s * max(t.H * t.D for t in att), dtype=torch.float32, device=self.device),
                   torch.empty(batch * s * max(t.H for t in att), dtype=torch.float32, device=self.device))

    # ------------------------------------------------------------------ buffers
    def _outer_buffers(self, s: OuterShape, T: int) -> dict:
        return {"o": self.bufs.get(f"outer{s.inner}", T, s.inner, torch.float32), **self.scratch}

    def _buffers(self, b, L, T: int):
        """(projection, [mixer outputs | dense feed-forward], columns of the mixer outputs)."""
        heads = L["shape"].inner + (L["tied"].H * L["tied"].D if b.attention is not None else 0)
        n, cat = L["proj"].shape[0], L["o"].shape[1]
        return (self.bufs.get(f"proj{n}", T, n, self.dtype), self.bufs.get(f"cat{cat}", T, cat, self.dtype), heads)

    def _parallel_buffers(self, L, T: int):
        t, s = L["tied"], L["shape"]
        n = s.inner + 2 * s.G * s.D
        return self.bufs.get(f"q{t.H * t.D}", T, t.H * t.D, self.dtype), self.bufs.get(f"conv{n}", T, n, self.dtype)

    def reserve_buffers(self, max_tokens: int, max_reqs: int) -> None:
        self._reserve_rows(max_tokens, max_reqs)
        for n, t in (("stream2", torch.float32), ("normed2", self.dtype)):
            self.bufs.reserve(n, max_tokens, self.cols, t)
        self.recurrent = RecurrentState()
        self.prev = self.recurrent.add((max_reqs,), torch.int64, self.device) if self.cfg.bigram is not None else None
        work = Workspace(self.device, max_tokens, max_reqs) if self._bf16_kernels() else None
        for l, b in enumerate(self.cfg.blocks):
            L, f = self.layers[l], b.mlp
            s = L["shape"]
            self._buffers(b, L, max_tokens)
            self._outer_buffers(s, max_tokens)
            if b.attention is not None:
                self._parallel_buffers(L, max_tokens)
            conv, state = self._state_shapes(b)
            rows = None
            if self.cfg.input_conv > 1:
                rows = self.recurrent.add((max_reqs, self.cfg.input_conv - 1, self.cols), torch.float32, self.device)
            self.state[l] = (rows, self.recurrent.add((max_reqs, *conv), self.dtype, self.device) if conv else None,
                             self.recurrent.add((max_reqs, *state), torch.float32, self.device))
            if work is not None:
                work.reserve(s, CHANNEL if b.gla is not None else HEAD)
            if isinstance(f, ExpertSpec):
                n, key = pad(f.experts), (f.experts, f.top, f.ff)
                self.bufs.reserve(f"router{n}", max_tokens, n, torch.float32)
                if self.device.type == "cuda" and key not in self.moe_ws:
                    from ..ops.moe import MoeWorkspace
                    self.moe_ws[key] = MoeWorkspace(self.device, max_tokens, f.top, f.experts, self.cols, pad(f.ff), self.dtype)
        if work is not None:
            self.scratch = work.allocate()

    # ------------------------------------------------------------------ forward
    def _gla(self, h, l, L, g, ctx, T, proj, out):
        s = L["shape"]
        self.be.gemm(h, L["proj"], out=proj, out_dtype=self.dtype)
        q, k, v, gate, a1 = torch.split(proj, [s.H * s.D, s.H * s.D, s.inner, s.inner, s.rank], 1)
        self.be.gated_linear_attention(q, k, v, gate, a1, L, s, self.state[l][2], ctx, self._outer_buffers(s, T), out, tau=g.tau,
                                       eps=self.cfg.rms_norm_eps)

    def _parallel(self, h, l, L, b, ctx, T, proj, out):
        be, a, t, s = self.be, b.attention, L["tied"], L["shape"]
        be.gemm(h, L["proj"], out=proj, out_dtype=self.dtype)
        qk = t.H * t.D + t.G * t.D
        z, u, dt = (proj[:, qk: qk + s.inner], proj[:, qk + s.inner: qk + 2 * s.inner + 2 * s.G * s.D],
                    proj[:, qk + 2 * s.inner + 2 * s.G * s.D:])
        q, conv = self._parallel_buffers(L, T)
        grp, cache = self.layer_group[l], self.cache_of[l]
        be.rotate_tied(proj[:, :qk], ctx.positions[:T], L["rope"], q, ctx.slot_mapping[grp][:T], cache, t, block_size=self.block_size)
        be.bias_attention(q, cache, ctx, grp, out=out[:, : t.H * t.D], H=t.H, G=t.G, kw=t.G * t.pitch, vdim=t.D,
                          block_size=self.block_size, scale=a.scale, grouped=True, values_in_keys=True, key_at=t.r8,
                          sink=L["sink"], out_scale=b.scales[0])
        be.short_conv(u, L["conv_w"], L["conv_b"], self.state[l][1], ctx, conv, act="silu")
        be.state_space(conv, z, dt, L, s, self.state[l][2], ctx, self._outer_buffers(s, T), out[:, t.H * t.D:],
                       parts=b.ssm.norm_groups, eps=self.cfg.rms_norm_eps, scale=b.scales[1])

    def _experts(self, h, L, f, T):
        logits = self.bufs.get(f"router{pad(f.experts)}", T, pad(f.experts), torch.float32)
        self.be.gemm(h, L["router"], out=logits, out_dtype=torch.float32)
        y, pos, w = self.be.plain_experts(h, logits[:, : f.experts], L["w_up"], L["w_down"],
                                          self.moe_ws.get((f.experts, f.top, f.ff)), top=f.top, act=f.plain)
        return dict(y=y, pair_pos=pos, pair_w=w)

    def forward(self, ctx: StepContext) -> torch.Tensor:
        """Returns fp32 logits ``[num_logits, vocab]`` for the rows in ``ctx.logits_indices``."""
        c, be, T = self.cfg, self.be, ctx.num_tokens
        norm = dict(width=self.width, groups=c.norm_groups, eps=c.rms_norm_eps)
        f32 = torch.float32
        x, x2, mixed = (self.bufs.get(n, T, self.cols, f32) for n in ("stream", "stream2", "mixed"))
        h1, h2 = (self.bufs.get(n, T, self.cols, self.dtype) for n in ("normed", "normed2"))
        be.embed_pairs(x, ctx.input_ids[:T], self.w["embed"], ctx, scale=c.embed_scale, norm_w=self.w["embed_norm"],
                       bigram=self.w.get("bigram"), prev=self.prev, spec=c.bigram, **norm)
        add: dict = {}
        for l, (L, b) in enumerate(zip(self.layers, c.blocks)):
            f = b.mlp
            be.norm_conv(x, ctx, L["reads"], (h1, h2)[: len(L["reads"])], state=self.state[l][0], dst=x2 if add else None, **add, **norm)
            if add:
                x, x2 = x2, x
            proj, cat, heads = self._buffers(b, L, T)
            if b.gla is not None:
                self._gla(h1, l, L, b.gla, ctx, T, proj, cat[:, :heads])
            else:
                self._parallel(h1, l, L, b, ctx, T, proj, cat[:, :heads])
            if isinstance(f, DenseSpec):
                be.plain_unit(h2, L["up"], f.plain, cat[:, heads:])
            be.gemm(cat, L["o"], out=mixed, out_dtype=f32)
            add = dict(a=mixed)
            if isinstance(f, ExpertSpec):
                add.update(self._experts(h2, L, f, T))
        be.norm_conv(x, ctx, [self.w["final_norm"][None]], [h1], **add, **norm)
        return self._logits(ctx, h1)
