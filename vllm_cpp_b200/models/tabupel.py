"""Tabupel decoders: differential-attention, latent-attention and gated-linear-recurrence blocks in any order
over an fp32 residual stream.

A sublayer f (mixer, then feed-forward) adds  x += m f(norm(x)).

* Differential attention (``ops/bias_attn.py``): q and k are normed and weighted per head and map, then
  rotated; a query sees a window of positions. The two maps of a head are two query heads over the same
  values, joined by ``diff_combine``.
* Latent attention (``ops/latent.py``): the cache holds a normed latent and one rotated key part per token.
  Decode rows run the absorbed form, prompt portions expanded keys and values.
* Recurrence (``ops/rglru.py``): a short convolution and a gated linear recurrence per channel; the fp32
  state and the convolution's last inputs are kept per request slot (``recurrent.py``).

A block may run with the weights of another one; its cache or state is its own. Every block has its own sizes.
Storage is padded with zeros (head sizes and recurrent blocks to multiples of 16, other widths to multiples of
8), so any size goes through the kernels; ``cfg.dtype == "float32"`` runs the same forward in 32 bits. The
rotated pairs (2i, 2i + 1) are stored half of the rotated size apart: the rows of the query and key
projections are put in that order when they are loaded, and no score notices."""
from __future__ import annotations

import torch

from ..ops.bias_attn import grouped_decode_splits
from ..ops.latent import LatentShape, decode_splits, prefill_kernel_fits
from ..ops.rglru import RglruShape, summary_values, tensor_core_size
from .base import StepContext
from .listed import ListedModel, pad, pad_heads
from .recurrent import RecurrentState

RATE = 8.0                                # log a = -RATE r softplus(lam)


def pairs_apart(t: torch.Tensor, heads: int, at: int, dims: int) -> torch.Tensor:
    """Rows ``at`` + 2i of each head to ``at`` + i, rows ``at`` + 2i + 1 to ``at`` + dims / 2 + i."""
    if not dims:
        return t
    x = t.reshape(heads, -1, *t.shape[1:]).clone()
    x[:, at: at + dims] = torch.cat([x[:, at: at + dims: 2], x[:, at + 1: at + dims: 2]], 1)
    return x.reshape(t.shape)


def latent_shape(a) -> LatentShape:
    return LatentShape(H=a.heads, dim=a.dim, rot=a.rot_dim, vdim=a.vdim, q_rank=a.q_rank, rank=a.kv_rank)


def rglru_shape(r) -> RglruShape:
    return RglruShape(blocks=r.blocks, size=r.width // r.blocks, taps=r.conv)


class TabupelModel(ListedModel):
    def __init__(self, cfg, *args, **kw):
        super().__init__(cfg, *args, **kw)
        self.kv_layers = [l for l, b in enumerate(cfg.blocks) if b.rglru is None]
        self._pages: dict[str, torch.Tensor] = {}

    # ------------------------------------------------------------------ weights
    def init_random(self, seed: int = 0, std: float = 0.02) -> None:
        c, W = self.cfg, self.width
        big = sum(b.mlp.ff * 3 * W for b in c.blocks if b.mlp is not None) > 2e8
        gdev = self.device if (self.device.type == "cuda" and big) else torch.device("cpu")
        g = torch.Generator(device=gdev).manual_seed(seed)

        def full(*shape, s=std, mean=0.0):
            return torch.empty(shape, dtype=torch.float32, device=gdev).normal_(mean, s, generator=g).to(torch.bfloat16)

        def norm(n):
            return full(n, s=0.1, mean=1.0)

        def gen():
            yield "embed", full(c.vocab_size, W)
            for l, b in enumerate(c.blocks):
                if b.weights_of is not None:
                    continue
                p, a, la, r = f"l{l}.mix.", b.attention, b.latent, b.rglru
                yield f"l{l}.norm1", norm(W)
                if a is not None:
                    for n, rows in (("q", a.heads * 2 * a.dim), ("k", a.kv_heads * 2 * a.dim), ("v", a.kv_heads * a.vdim)):
                        yield p + n, full(rows, W)
                    for n in ("q.norm", "k.norm"):
                        yield p + n, norm(a.dim)
                    for n in ("lq1", "lk1", "lq2", "lk2"):
                        yield p + n, full(a.dim, s=0.1)
                    yield p + "o", full(W, a.heads * a.vdim)
                elif la is not None:
                    yield p + "dq", full(la.q_rank, W)
                    yield p + "dq.norm", norm(la.q_rank)
                    yield p + "uq", full(la.heads * (la.dim + la.rot_dim), la.q_rank)
                    yield p + "dkv", full(la.kv_rank + la.rot_dim, W)
                    yield p + "dkv.norm", norm(la.kv_rank)
                    yield p + "uk", full(la.heads * la.dim, la.kv_rank)
                    yield p + "uv", full(la.heads * la.vdim, la.kv_rank)
                    yield p + "g", full(la.heads, W)
                    yield p + "o", full(W, la.heads * la.vdim)
                else:
                    n = r.width // r.blocks
                    for k in ("y", "x"):
                        yield p + k, full(r.width, W)
                        yield p + k + ".b", full(r.width)
                    yield p + "conv", full(r.width, r.conv, s=0.5)
                    yield p + "conv.b", full(r.width)
                    for k in ("ra", "ri"):
                        yield p + k, full(r.blocks, n, n)
                        yield p + k + ".b", full(r.blocks, n)
                    yield p + "lam", full(r.width, s=0.5, mean=-4.0)
                    yield p + "o", full(W, r.width)
                if b.mlp is not None:
                    yield f"l{l}.norm2", norm(W)
                    yield f"l{l}.mlp.gate", full(b.mlp.ff, W)
                    yield f"l{l}.mlp.up", full(b.mlp.ff, W)
                    yield f"l{l}.mlp.down", full(W, b.mlp.ff)
            yield "final.norm", norm(W)
            yield "head", full(c.vocab_size, W)

        self.load_weights(gen())

    MIXER = {"attention": ("q", "k", "v", "q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2", "o"),
             "latent": ("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "g", "o"),
             "rglru": ("y", "y.b", "x", "x.b", "conv", "conv.b", "ra", "ra.b", "ri", "ri.b", "lam", "o")}

    def load_weights(self, named_tensors) -> None:
        blocks = self.cfg.blocks
        self.layers = [dict() for _ in blocks]
        pend: list[dict] = [dict() for _ in blocks]
        for name, t in named_tensors:
            if not self._take_shared(name, t):
                l, rest = self._block_of(name)
                pend[l][rest] = t
        for l, (L, b, p) in enumerate(zip(self.layers, blocks, pend)):
            kind = next(k for k in self.MIXER if getattr(b, k) is not None)
            want = {"norm1"} | {"mix." + n for n in self.MIXER[kind]}
            if b.mlp is not None:
                want |= {"norm2", "mlp.gate", "mlp.up", "mlp.down"}
            self._expect(l, want if b.weights_of is None else set(), set(p))
            if b.weights_of is not None:
                continue
            for n in ("norm1", "norm2"):
                if n in p:
                    L[n] = self.put(p[n], self.cols, dtype=torch.float32)
            getattr(self, "_load_" + kind)(L, getattr(b, kind), {n[4:]: t for n, t in p.items()})
            if b.mlp is not None:
                self._load_dense(L, b.mlp, p)
            pend[l] = {}
        for l, b in enumerate(blocks):
            if b.weights_of is not None:
                self.layers[l] = self.layers[b.weights_of]
        self._expect_shared()

    def _load_attention(self, L, a, p) -> None:
        D, V, f32 = pad(a.dim, 16), pad(a.vdim, 16), dict(dtype=torch.float32)
        turn = lambda t, heads: pairs_apart(t, heads, 0, a.rot_dims)                         # noqa: E731
        rows = [pad_heads(turn(p[n], 2 * h), 2 * h, D) for n, h in (("q", a.heads), ("k", a.kv_heads))]
        q = torch.cat(rows + [pad_heads(p["v"], a.kv_heads, V)], 0)
        L["proj"] = self.put(q, q.shape[0], self.cols)
        L["q_norm"], L["k_norm"] = (self.put(turn(p[n], 1), D, **f32) for n in ("q.norm", "k.norm"))
        dots = [torch.exp((p["lq" + i].double() * p["lk" + i].double()).sum()).item() for i in "12"]
        L["lam"] = dots[0] - dots[1] + a.diff
        L["o"] = self.put(pad_heads(p["o"], a.heads, V, axis=1), self.cols, a.heads * V)
        L["rope"] = self._rope_table(a.rot_base, a.rot_dims, a.rot_scaling)

    def _load_latent(self, L, a, p) -> None:
        s, f32 = latent_shape(a), dict(dtype=torch.float32)
        L["shape"], H = s, s.H
        q8, k8, r8, g8 = s.down
        dkv = p["dkv"]
        parts = ((p["dq"], q8), (dkv[: s.rank], k8), (pairs_apart(dkv[s.rank:], 1, 0, s.rot), r8), (p["g"], g8))
        L["down_proj"] = torch.cat([self.put(t, n, self.cols) for t, n in parts], 0)
        L["q_norm"], L["kv_norm"] = (self.put(p[n], w, **f32) for n, w in (("dq.norm", q8), ("dkv.norm", k8)))
        uq = p["uq"].reshape(H, s.dim + s.rot, -1)
        turned = pairs_apart(uq[:, s.dim:].reshape(H * s.rot, uq.shape[2]), H, 0, s.rot).reshape(H, s.rot, uq.shape[2])
        uq = torch.cat([self.put(uq[:, : s.dim], H, s.qn, q8), self.put(turned, H, s.qw - s.qn, q8)], 1)
        L["uq"] = uq.reshape(H * s.qw, q8).contiguous()
        uk, uv = p["uk"].reshape(H, s.dim, -1), p["uv"].reshape(H, s.vdim, -1)
        L["uk_t"] = self.put(uk.transpose(1, 2), H, s.rankp, s.qn)
        L["uv"] = self.put(uv, H, s.V, s.rankp)
        if self._bf16_kernels():
            L["kv"] = torch.cat([self.put(uk, H, s.D, s.rankp).reshape(H * s.D, -1), L["uv"].reshape(H * s.V, -1)], 0)
        L["o"] = self.put(pad_heads(p["o"], H, s.V, axis=1), self.cols, H * s.V)
        L["rope"] = self._rope_table(a.rot_base, a.rot_dim, a.rot_scaling)

    def _load_rglru(self, L, r, p) -> None:
        s, f32 = rglru_shape(r), dict(dtype=torch.float32)
        L["shape"] = s
        spread = lambda t: pad_heads(t, s.blocks, s.B)                                       # noqa: E731
        L["proj"] = self.put(torch.cat([spread(p["y"]), spread(p["x"])], 0), 2 * s.C, self.cols)
        L["bias"] = self.put(torch.cat([spread(p["y.b"]), spread(p["x.b"])], 0))
        L["conv_w"] = self.put(spread(p["conv"]).t(), **f32)
        L["conv_b"] = self.put(spread(p["conv.b"]), **f32)
        L["gates"] = torch.stack([self.put(p[n], s.blocks, s.M, s.B) for n in ("ra", "ri")], 1).contiguous()
        L["gate_bias"] = torch.stack([self.put(spread(p[n + ".b"].reshape(-1)), **f32) for n in ("ra", "ri")])
        lam = p["lam"].to(self.device, torch.float64)
        L["rate"] = self.put(spread(-RATE * torch.nn.functional.softplus(lam, threshold=1e9)), **f32)
        L["o"] = self.put(pad_heads(p["o"], s.blocks, s.B, axis=1), self.cols, s.C)

    # ------------------------------------------------------------------ caches and state
    def _row(self, b) -> int:
        """Cache values of a token."""
        if b.latent is not None:
            return latent_shape(b.latent).row
        a = b.attention
        return a.kv_heads * (2 * pad(a.dim, 16) + pad(a.vdim, 16))

    def kv_cache_groups(self, block_size: int):
        """One group: where every block has a window, pages behind the widest are given back."""
        mix = [self.cfg.blocks[l].mixer for l in self.kv_layers]
        row = max((self._row(self.cfg.blocks[l]) for l in self.kv_layers), default=16)
        spec = dict(kind="full", block_size=block_size, num_kv_heads=1, head_size=row - row // 2, head_size_v=row // 2,
                    dtype_bytes=self.dtype.itemsize)
        if mix and all(m.window for m in mix):
            spec.update(kind="sliding", sliding_window=max(m.window for m in mix))
        return [(list(self.kv_layers), spec)]

    def alloc_kv_cache(self, num_blocks: int, block_size: int):
        """One tensor per block: a page holds ``block_size`` latent rows, or key rows, then value rows."""
        self.block_size = block_size
        self.kv_caches = [torch.zeros((num_blocks, block_size * self._row(self.cfg.blocks[l])), dtype=self.dtype,
                                      device=self.device) for l in self.kv_layers]
        self.cache_of = dict(zip(self.kv_layers, self.kv_caches))
        self.layer_group = [0] * len(self.cfg.blocks)
        return self.kv_caches

    def kv_bytes_per_block(self, block_size: int) -> int:
        return max(1, sum(block_size * self._row(self.cfg.blocks[l]) for l in self.kv_layers) * self.dtype.itemsize)

    def state_bytes_per_request(self) -> int:
        shapes = [rglru_shape(b.rglru) for b in self.cfg.blocks if b.rglru is not None]
        return sum(s.C * ((s.taps - 1) * self.dtype.itemsize + 4) for s in shapes)

    def decode_workspace(self, batch: int, max_seq_len: int, block_size: int):
        """(KV splits, split buffers) of a decode batch; one pair of buffers serves every block."""
        mix = [self.cfg.blocks[l].mixer for l in self.kv_layers]
        if self.device.type != "cuda" or not mix:
            return 1, None
        from .. import ops
        keys = max(min(m.window or max_seq_len, max_seq_len) for m in mix)
        s, heads, out = 1, 1, 1
        for b in (self.cfg.blocks[l] for l in self.kv_layers):
            if b.latent is not None:
                sh = latent_shape(b.latent)
                n, h, o = decode_splits(batch, sh.H, keys, ops.num_sms()), sh.H, sh.H * sh.rankp
            else:
                a = b.attention
                n, h, o = grouped_decode_splits(batch, a.kv_heads, keys, ops.num_sms()), 2 * a.heads, 2 * a.heads * pad(a.vdim, 16)
            s, heads, out = max(s, n), max(heads, h), max(out, o)
        if s == 1:
            return 1, None
        return s, (torch.empty(batch * s * out, dtype=torch.float32, device=self.device),
                   torch.empty(batch * s * heads, dtype=torch.float32, device=self.device))

    # ------------------------------------------------------------------ buffers
    def _attention_buffers(self, a, T: int):
        D, V = pad(a.dim, 16), pad(a.vdim, 16)
        n = 2 * (a.heads + a.kv_heads) * D + a.kv_heads * V
        return (self.bufs.get(f"proj{n}", T, n, self.dtype), self.bufs.get(f"q{2 * a.heads * D}", T, 2 * a.heads * D, self.dtype),
                self.bufs.get(f"maps{2 * a.heads * V}", T, 2 * a.heads * V, self.dtype),
                self.bufs.get(f"heads{a.heads * V}", T, a.heads * V, self.dtype))

    def _latent_buffers(self, s: LatentShape, T: int):
        n = sum(s.down)
        # (padding columns of the query latent meet zero weights and must be finite)
        return (self.bufs.get(f"down{n}", T, n, self.dtype), self.bufs.get(f"cq{s.q_rank}", T, s.down[0], self.dtype, zero=True),
                self.bufs.get(f"q{s.H * s.qw}", T, s.H * s.qw, self.dtype),
                self.bufs.get(f"heads{s.H * s.V}", T, s.H * s.V, self.dtype))

    def _absorbed_buffers(self, s: LatentShape, n: int):
        return (self.bufs.get(f"absorbed{s.H}_{s.row}", n, s.H * s.row, self.dtype, zero=True),
                self.bufs.get(f"latent{s.H * s.rankp}", n, s.H * s.rankp, self.dtype))

    def _rglru_buffers(self, s: RglruShape, T: int):
        bufs = {}
        if self.device.type == "cuda":
            if self.dtype == torch.bfloat16 and tensor_core_size(s):
                bufs["summary"] = self.bufs.get(f"summary{s.C}", 1, summary_values(s), torch.float32)
            else:
                bufs.update({n: self.bufs.get(f"rglru_{n}{s.C}", T, s.C, torch.float32) for n in "ab"})
        return (self.bufs.get(f"proj{2 * s.C}", T, 2 * s.C, self.dtype), self.bufs.get(f"conv{s.C}", T, s.C, self.dtype),
                bufs, self.bufs.get(f"heads{s.C}", T, s.C, self.dtype))

    def _expands(self, s: LatentShape) -> bool:
        """Whether prompt portions run on expanded keys and values."""
        return self.device.type == "cuda" and prefill_kernel_fits(s, self.dtype, self.block_size)

    def reserve_buffers(self, max_tokens: int, max_reqs: int) -> None:
        self._reserve_rows(max_tokens, max_reqs)
        self.recurrent = RecurrentState()
        for l, b in enumerate(self.cfg.blocks):
            if b.rglru is not None:
                s = rglru_shape(b.rglru)
                self._rglru_buffers(s, max_tokens)
                self.state[l] = (self.recurrent.add((max_reqs, s.taps - 1, s.C), self.dtype, self.device),
                                 self.recurrent.add((max_reqs, s.C), torch.float32, self.device))
            elif b.latent is not None:
                s = latent_shape(b.latent)
                self._latent_buffers(s, max_tokens)
                self._absorbed_buffers(s, max_reqs if self._expands(s) else max_tokens)
            else:
                self._attention_buffers(b.attention, max_tokens)
            if b.mlp is not None:
                self._dense_buffers(b.mlp, max_tokens)

    def _page_buffer(self, name: str, rows: int, cols: int) -> torch.Tensor:
        """Scratch rows that start as zeros (a tile may look at rows nobody wrote; they must be finite)."""
        t = self._pages.get(name)
        if t is None or t.shape[0] < rows or t.shape[1] != cols:
            t = self._pages[name] = torch.zeros((rows, cols), dtype=self.dtype, device=self.device)
        return t[:rows]

    # ------------------------------------------------------------------ forward
    def _attention(self, h, l, L, a, ctx, T, out):
        be, D, V, H, G = self.be, pad(a.dim, 16), pad(a.vdim, 16), a.heads, a.kv_heads
        proj, q, maps, heads = self._attention_buffers(a, T)
        be.gemm(h, L["proj"], out=proj, out_dtype=self.dtype)
        grp, cache, eps = self.layer_group[l], self.cache_of[l], self.cfg.rms_norm_eps
        be.rotate_kv(proj, ctx.positions[:T], L["rope"], a.rot_dims, eps, q, ctx.slot_mapping[grp][:T], cache, H=2 * H,
                     G=2 * G, value_heads=G, D=D, V=V, dim=a.dim, block_size=self.block_size, q_w=L["q_norm"], k_w=L["k_norm"])
        be.bias_attention(q, cache, ctx, grp, out=maps, H=2 * H, G=G, kw=2 * G * D, vdim=V, block_size=self.block_size,
                          scale=a.scale, window=a.window, maps=2, grouped=True)
        be.diff_combine(maps, heads, H=H, V=V, vdim=a.vdim, lam=L["lam"], eps=eps, scale=1.0 - a.diff)
        be.gemm(heads, L["o"], out=out, out_dtype=torch.float32)

    def _visible_pages(self, ctx: StepContext, window: int) -> dict:
        """``ops.latent.visible_pages`` of the step's portions on the device, once per step and window."""
        key = ("pages", window)
        if key not in ctx.extra:
            from ..ops.latent import visible_pages
            nd, P, host = ctx.num_decodes, ctx.num_prefills, ctx.extra.get("host")
            seq = (host["seq_lens"] if host is not None else ctx.seq_lens.cpu())[nd: nd + P].numpy()
            start = (host["prefill_q_start"] if host is not None else ctx.prefill_q_start.cpu())[: P + 1].numpy()
            first, base, total, bt = visible_pages(seq, start[1:] - start[:-1], window, self.block_size)
            flat = torch.cat([torch.from_numpy(x).reshape(-1) for x in (first, base, bt)]).to(self.device)
            ctx.extra[key] = dict(first=flat[:P], base=flat[P: 2 * P], total=total, table=flat[2 * P:].view(P, -1))
        return ctx.extra[key]

    def _latent(self, h, l, L, a, ctx, T, out):
        be, s, eps = self.be, L["shape"], self.cfg.rms_norm_eps
        down, cq, q, heads = self._latent_buffers(s, T)
        be.gemm(h, L["down_proj"], out=down, out_dtype=self.dtype)
        grp, cache, pos = self.layer_group[l], self.cache_of[l], ctx.positions[:T]
        be.latent_prepare(down, pos, L["rope"], L, s, eps, cq, ctx.slot_mapping[grp][:T], cache)
        be.gemm(cq, L["uq"], out=q, out_dtype=self.dtype)
        be.latent_attention(q, pos, L["rope"], cache, L, s, ctx, grp, scale=a.scale, window=a.window, block_size=self.block_size,
                            gate=down[:, s.gate_column:], out=heads,
                            pages=(lambda: self._visible_pages(ctx, a.window)) if self._expands(s) else None,
                            absorbed=lambda n: self._absorbed_buffers(s, n), scratch=self._page_buffer)
        be.gemm(heads, L["o"], out=out, out_dtype=torch.float32)

    def _rglru(self, h, l, L, ctx, T, out):
        be, s = self.be, L["shape"]
        proj, u, bufs, heads = self._rglru_buffers(s, T)
        be.gemm(h, L["proj"], bias=L["bias"], out=proj, out_dtype=self.dtype)
        conv_state, state = self.state[l]
        be.short_conv(proj[:, s.C:], L["conv_w"], L["conv_b"], conv_state, ctx, u)
        be.rglru(u, proj[:, : s.C], L, s, state, ctx, bufs, heads)
        be.gemm(heads, L["o"], out=out, out_dtype=torch.float32)

    def forward(self, ctx: StepContext) -> torch.Tensor:
        """Returns fp32 logits ``[num_logits, vocab]`` for the rows in ``ctx.logits_indices``."""
        c, be, T = self.cfg, self.be, ctx.num_tokens
        eps, norm = c.rms_norm_eps, dict(width=self.width, norm_offset=0.0)
        stream = self.bufs.get("stream", T, self.cols, torch.float32)
        h = self.bufs.get("normed", T, self.cols, self.dtype)
        mixed = self.bufs.get("mixed", T, self.cols, torch.float32)
        be.stream_norm(stream, self.layers[0]["norm1"], eps, h, ids=ctx.input_ids[:T], table=self.w["embed"], **norm)
        norm["mult"] = c.residual_multiplier
        for l, (L, b) in enumerate(zip(self.layers, c.blocks)):
            if b.rglru is not None:
                self._rglru(h, l, L, ctx, T, mixed)
            elif b.latent is not None:
                self._latent(h, l, L, b.latent, ctx, T, mixed)
            else:
                self._attention(h, l, L, b.attention, ctx, T, mixed)
            nw = self.layers[l + 1]["norm1"] if l + 1 < len(self.layers) else self.w["final_norm"]
            be.stream_norm(stream, nw if b.mlp is None else L["norm2"], eps, h, a=mixed, **norm)
            if b.mlp is not None:
                self._dense(h, L, b.mlp, "silu", T, mixed)
                be.stream_norm(stream, nw, eps, h, a=mixed, **norm)
        return self._logits(ctx, h)
