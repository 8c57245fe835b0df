"""Nufusun decoders: parallel blocks over an fp32 residual stream.

Per block, with h = RMSNorm(x) (weights stored around zero):  x += mixer(h) + experts(h).

* Mixer: biased q / k / v projections, no rotation; scores take a per-head temperature and a learned
  distance bias, are mixed across all heads, and the softmax counts one null entry of score 0.
  Temperature, score scale and head mix are one [H, H] matrix applied to the queries
  (``ops/bias_attn.py``), and the mixed bias is one fp32 table per head and distance, both built when
  the weights are loaded.
* Experts: sigmoid router, the score scales the expert's input, clamped gated unit; the expert
  outputs are summed by the kernel that updates the stream and applies the next block's norm.

Every block has its own sizes. Storage is padded to multiples of 8 (zeros), so any size goes through
the GEMM kernels; ``cfg.dtype == "float32"`` runs the same forward in 32 bits."""
from __future__ import annotations

import torch

from ..config import ModelConfig, ParallelConfig
from ..ops.bias_attn import decode_splits, distance_bias_table
from .backend import make_backend
from .base import BufferPool, StepContext
from .dense import DenseModel

GATE_ALPHA, UP_OFFSET = 1.702, 1.0


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _padded(t: torch.Tensor, *shape: int) -> torch.Tensor:
    if tuple(t.shape) == shape:
        return t
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


class NufusunModel(DenseModel):
    DTYPES = ("bfloat16", "float32")

    def __init__(self, cfg: ModelConfig, device="cuda", parallel: ParallelConfig | None = None,
                 comm=None, max_position: int | None = None):
        # (the dense constructor sets up rotary tables and shards this family does not have)
        self.cfg, self.device = cfg, torch.device(device)
        self.par = parallel or ParallelConfig()
        if self.par.tensor_parallel_size > 1:
            raise ValueError("Nufusun runs on one rank: its heads are mixed with one another")
        self.tp, self.rank, self.comm = 1, 0, comm
        self.be = make_backend(self.device)
        self.dtype = torch.float32 if cfg.dtype == "float32" else torch.bfloat16
        self.hq, self.hkv, self.D = cfg.num_heads, cfg.num_kv_heads, cfg.head_dim
        self.max_position = max_position or cfg.max_position_embeddings
        self.width, self.cols = cfg.hidden_size, _pad8(cfg.hidden_size)
        self.vocab_shard, self.vocab_start = cfg.vocab_size, 0
        self.bufs = BufferPool(self.device)
        self.moe_ws: dict = {}
        self.w: dict[str, torch.Tensor] = {}
        self.layers: list[dict] = []

    # ------------------------------------------------------------------ weights
    def init_random(self, seed: int = 0, std: float = 0.02) -> None:
        c, W = self.cfg, self.width
        big = sum(b.mlp.experts * b.mlp.ff * 3 * W for b in c.blocks if b.mlp) > 5e8
        gdev = self.device if (self.device.type == "cuda" and big) else torch.device("cpu")
        g = torch.Generator(device=gdev).manual_seed(seed)

        def full(*shape, s=std, mean=0.0):
            return torch.empty(shape, dtype=torch.float32, device=gdev).normal_(mean, s, generator=g).to(torch.bfloat16)

        def gen():
            yield "embed", full(c.vocab_size, W)
            for l, b in enumerate(c.blocks):
                a, m = b.attention, b.mlp
                yield f"l{l}.norm1", full(W, s=0.1)
                for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                    yield f"l{l}.mix.{n}", full(rows, W)
                    yield f"l{l}.mix.{n}.b", full(rows)
                yield f"l{l}.mix.rel", full(32, a.heads, s=0.5)
                yield f"l{l}.mix.talk", (torch.eye(a.heads, device=gdev) + full(a.heads, a.heads, s=0.2).float()).to(torch.bfloat16)
                yield f"l{l}.mix.temp", full(a.heads, s=0.1, mean=1.0)
                yield f"l{l}.mix.o", full(W, a.heads * a.vdim)
                yield f"l{l}.mix.o.b", full(W)
                if m is None:
                    continue
                yield f"l{l}.mlp.router", full(m.experts, W)
                for e in range(m.experts):
                    yield f"l{l}.mlp.e{e}.gate", full(m.ff, W)
                    yield f"l{l}.mlp.e{e}.up", full(m.ff, W)
                    yield f"l{l}.mlp.e{e}.down", full(W, m.ff)
            yield "final.norm", full(W, s=0.1)
            yield "head", full(c.vocab_size, W)

        self.load_weights(gen())

    def load_weights(self, named_tensors) -> None:
        c, C, dev, dt = self.cfg, self.cols, self.device, self.dtype

        def put(t, *shape, dtype=None):
            return _padded(t.to(dev, dtype or dt), *(shape or t.shape)).contiguous()

        self.layers = [dict() for _ in c.blocks]
        for L, b in zip(self.layers, c.blocks):
            if b.mlp is not None:
                m, f8 = b.mlp, _pad8(b.mlp.ff)
                L["w_gate_up"] = torch.zeros((m.experts, 2 * f8, C), dtype=dt, device=dev)
                L["w_down"] = torch.zeros((m.experts, C, f8), dtype=dt, device=dev)
        pend: list[dict] = [dict() for _ in c.blocks]
        for name, t in named_tensors:
            if name == "embed":
                self.w["embed"] = put(t, t.shape[0], C)
            elif name == "head":
                self.w["lm_head"] = put(t, _pad8(t.shape[0]), C)
            elif name == "final.norm":
                self.w["final_norm"] = put(t, C, dtype=torch.float32)
            else:
                layer, _, rest = name.partition(".")
                if not (layer.startswith("l") and layer[1:].isdigit() and int(layer[1:]) < len(c.blocks)):
                    raise ValueError(f"unexpected tensor {name!r}")
                l = int(layer[1:])
                L, m = self.layers[l], c.blocks[l].mlp
                part = rest.split(".")
                if rest == "norm1":
                    L["norm"] = put(t, C, dtype=torch.float32)
                elif part[0] == "mix":
                    pend[l][rest[4:]] = t
                elif rest == "mlp.router" and m is not None:
                    L["router"] = put(t, _pad8(m.experts), C)
                elif part[0] == "mlp" and m is not None and len(part) == 3 and part[1][:1] == "e" and part[1][1:].isdigit():
                    e, f8 = int(part[1][1:]), _pad8(m.ff)
                    if part[2] == "down":
                        L["w_down"][e, : self.width, : m.ff] = t.to(dev, dt)
                    else:
                        r0 = {"gate": 0, "up": f8}[part[2]]
                        L["w_gate_up"][e, r0: r0 + m.ff, : self.width] = t.to(dev, dt)
                else:
                    raise ValueError(f"unexpected tensor {name!r}")
        for l, (L, b, p) in enumerate(zip(self.layers, c.blocks, pend)):
            missing = [n for n in ("q", "q.b", "k", "k.b", "v", "v.b", "rel", "talk", "temp", "o", "o.b") if n not in p]
            if missing or "norm" not in L or (b.mlp is not None and "router" not in L):
                raise ValueError(f"layer {l}: tensors missing from the checkpoint {missing}")
            a = b.attention
            n = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim)
            f32 = dict(dtype=torch.float32)
            L["qkv"] = put(torch.cat([p["q"], p["k"], p["v"]], 0), _pad8(n), C)
            L["qkv_bias"] = put(torch.cat([p["q.b"], p["k.b"], p["v.b"]], 0), _pad8(n))
            L["o"] = put(p["o"], C, _pad8(a.heads * a.vdim))
            L["o_bias"] = put(p["o.b"], C)
            talk, temp = put(p["talk"], **f32), put(p["temp"], **f32)
            L["mix"] = (talk * (temp * a.scale)[None]).contiguous()
            L["bias"] = (talk @ distance_bias_table(put(p["rel"], **f32), a.bias_max)).contiguous()
        for k in ("embed", "lm_head", "final_norm"):
            if k not in self.w:
                raise ValueError(f"{k} is missing from the checkpoint")

    def quantize_weights(self, method: str = "nvfp4") -> None:
        raise ValueError("Nufusun checkpoints are served in bfloat16 or float32")

    # ------------------------------------------------------------------ KV cache
    def kv_cache_groups(self, block_size: int):
        a = max((b.attention for b in self.cfg.blocks), key=lambda x: x.kv_heads * (x.dim + x.vdim))
        return [(list(range(len(self.cfg.blocks))),
                 dict(kind="full", block_size=block_size, num_kv_heads=a.kv_heads, head_size=a.dim, head_size_v=a.vdim,
                      dtype_bytes=self.dtype.itemsize))]

    def alloc_kv_cache(self, num_blocks: int, block_size: int):
        """One page tensor per layer: a page holds ``block_size`` key rows, then as many value rows."""
        self.block_size = block_size
        self.kv_caches = [torch.zeros((num_blocks, block_size * a.kv_heads * (a.dim + a.vdim)), dtype=self.dtype,
                                      device=self.device) for a in (b.attention for b in self.cfg.blocks)]
        self.layer_group = [0] * len(self.cfg.blocks)
        return self.kv_caches

    def kv_bytes_per_block(self, block_size: int) -> int:
        return sum(block_size * b.attention.kv_heads * (b.attention.dim + b.attention.vdim)
                   for b in self.cfg.blocks) * self.dtype.itemsize

    def decode_workspace(self, batch: int, max_seq_len: int, block_size: int):
        """(KV splits, split buffers) of a decode batch; one pair of buffers serves every layer."""
        if self.device.type != "cuda":
            return 1, None
        from .. import ops
        s = decode_splits(batch, max_seq_len, ops.num_sms())
        if s == 1:
            return 1, None
        heads = max(b.attention.heads for b in self.cfg.blocks)
        out = max(b.attention.heads * b.attention.vdim for b in self.cfg.blocks)
        return s, (torch.empty(batch * s * out, dtype=torch.float32, device=self.device),
                   torch.empty(batch * s * heads, dtype=torch.float32, device=self.device))

    # ------------------------------------------------------------------ buffers
    def _layer_buffers(self, a, T: int):
        qkv = self.bufs.get(f"qkv{_pad8(a.heads * a.dim + a.kv_heads * (a.dim + a.vdim))}", T,
                            _pad8(a.heads * a.dim + a.kv_heads * (a.dim + a.vdim)), torch.float32)
        q = self.bufs.get(f"q{_pad8(a.heads * a.kv_heads * a.dim)}", T, _pad8(a.heads * a.kv_heads * a.dim), self.dtype)
        # the padding columns of the output projection's input meet zero weights and must be finite
        attn = self.bufs.get(f"attn{a.heads * a.vdim}", T, _pad8(a.heads * a.vdim), self.dtype, zero=True)
        return qkv, q, attn

    def reserve_buffers(self, max_tokens: int, max_reqs: int) -> None:
        self.bufs.reserve("stream", max_tokens, self.cols, torch.float32)
        self.bufs.reserve("mixed", max_tokens, self.cols, torch.float32)
        self.bufs.reserve("normed", max_tokens, self.cols, self.dtype)
        self.bufs.reserve("last", max_reqs, self.cols, self.dtype)
        self.bufs.reserve("logits", max_reqs, _pad8(self.cfg.vocab_size), torch.float32)
        for b in self.cfg.blocks:
            self._layer_buffers(b.attention, max_tokens)
            m = b.mlp
            if m is None:
                continue
            self.bufs.reserve(f"router{_pad8(m.experts)}", max_tokens, _pad8(m.experts), torch.float32)
            key = (m.experts, m.top, m.ff)
            if self.device.type == "cuda" and key not in self.moe_ws:
                from ..ops.moe import MoeWorkspace
                self.moe_ws[key] = MoeWorkspace(self.device, max_tokens, m.top, m.experts, self.cols, _pad8(m.ff),
                                                self.dtype)

    def fused_tp_supported(self) -> bool:
        return False

    # ------------------------------------------------------------------ forward
    def _experts(self, h, L, m, T):
        be = self.be
        logits = self.bufs.get(f"router{_pad8(m.experts)}", T, _pad8(m.experts), torch.float32)
        be.gemm(h, L["router"], out=logits, out_dtype=torch.float32)
        return be.clamped_experts(h, logits[:, : m.experts], L["w_gate_up"], L["w_down"],
                                  self.moe_ws.get((m.experts, m.top, m.ff)), top=m.top, limit=m.limit,
                                  alpha=GATE_ALPHA, up_offset=UP_OFFSET)

    def forward(self, ctx: StepContext) -> torch.Tensor:
        """Returns fp32 logits ``[num_logits, vocab]`` for the rows in ``ctx.logits_indices``."""
        c, be, T = self.cfg, self.be, ctx.num_tokens
        eps, norm = c.rms_norm_eps, dict(width=self.width)
        stream = self.bufs.get("stream", T, self.cols, torch.float32)
        h = self.bufs.get("normed", T, self.cols, self.dtype)
        mixed = self.bufs.get("mixed", T, self.cols, torch.float32)
        be.stream_norm(stream, self.layers[0]["norm"], eps, h, ids=ctx.input_ids[:T], table=self.w["embed"],
                       scale=c.embed_scale, **norm)
        for l, (L, b) in enumerate(zip(self.layers, c.blocks)):
            a = b.attention
            qkv, q, attn = self._layer_buffers(a, T)
            be.gemm(h, L["qkv"], bias=L["qkv_bias"], out=qkv, out_dtype=torch.float32)
            grp = self.layer_group[l]
            be.head_mix_kv(qkv, L["mix"], q, ctx.slot_mapping[grp][:T], self.kv_caches[l], H=a.heads, G=a.kv_heads,
                           dim=a.dim, vdim=a.vdim, block_size=self.block_size)
            be.bias_attention(q, self.kv_caches[l], ctx, grp, out=attn, H=a.heads, G=a.kv_heads,
                              kw=a.kv_heads * a.dim, vdim=a.vdim, block_size=self.block_size, bias=L["bias"],
                              null_entry=True)
            be.gemm(attn, L["o"], bias=L["o_bias"], out=mixed, out_dtype=torch.float32)
            y = pair_pos = None
            if b.mlp is not None:
                y, pair_pos = self._experts(h, L, b.mlp, T)
            nw = self.layers[l + 1]["norm"] if l + 1 < len(self.layers) else self.w["final_norm"]
            be.stream_norm(stream, nw, eps, h, a=mixed, y=y, pair_pos=pair_pos, **norm)
        if ctx.decode_only_full_logits:
            n, last = T, h
        else:
            n = ctx.num_logits
            last = be.gather_rows(h, ctx.logits_indices[:n], out=self.bufs.get("last", n, self.cols, self.dtype))
        logits = self.bufs.get("logits", n, self.w["lm_head"].shape[0], torch.float32)
        be.gemm(last, self.w["lm_head"], out=logits, out_dtype=torch.float32)
        return logits[:, : c.vocab_size]
