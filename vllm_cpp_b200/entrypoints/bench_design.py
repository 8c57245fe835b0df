"""Throughput of a design with listed layers beside the closest other model of this package at equal layer
sizes, and its kernels beside the like kernels of that model, each against its roofline.

``bench.py --design nufusun`` (beside Qwen3-MoE), ``--design diforax`` (beside the Qwen3.5 MoE hybrids),
``--design tabupel`` (beside the dense Qwen3.5 hybrids, its latent kernels beside DeepSeek-V2's) or ``--design kubolorn``
(beside the Qwen3.5 hybrids, dense or with experts) runs it and prints one JSON line. Random weights; device time (CUDA events); kernels are timed with an L2 flush
between iterations, median of several."""
from __future__ import annotations

import json
import os

import torch

# name -> width, heads, kv heads, head size, experts, top, expert size, layers
FIELDS = ("width", "heads", "kv_heads", "head", "experts", "top", "expert", "layers")
NUFUSUN_SIZES = {
    "30b-a3b layers": (2048, 32, 4, 128, 128, 8, 768, 4),
    "small layers": (1024, 16, 4, 64, 32, 4, 512, 6),
    "8 kv heads": (2048, 32, 8, 64, 64, 4, 1024, 4),
    "wide layers": (4096, 32, 8, 128, 16, 2, 2048, 3),
}


# name -> those, then delta value heads, delta key heads (of 128 x 128)
DIFORAX_SIZES = {
    "30b-a3b layers": (2048, 32, 4, 128, 128, 8, 768, 4, 32, 16),
    "wide heads": (2048, 16, 2, 256, 64, 4, 1024, 4, 32, 16),
    "small layers": (1024, 16, 4, 128, 32, 4, 512, 8, 16, 8),
    "wide layers": (4096, 32, 8, 128, 16, 2, 2048, 4, 48, 16),
}


# width, dense size, layers; differential heads, kv heads, size (values twice as wide); latent heads, query and
# key latent; recurrent width, its blocks
TABUPEL_FIELDS = ("width", "ff", "layers", "heads", "kv_heads", "head", "latent_heads", "q_rank", "kv_rank", "recurrent", "blocks")
TABUPEL_SIZES = {
    "2b layers": (2560, 7680, 6, 20, 4, 64, 16, 1536, 512, 2560, 10),
    "wide heads": (2048, 6144, 6, 8, 2, 128, 16, 1024, 512, 2048, 8),
    "small layers": (1024, 3072, 12, 8, 4, 64, 8, 512, 512, 1024, 8),
    "wide layers": (4096, 12288, 6, 32, 8, 64, 16, 1536, 512, 4096, 16),
}


# width, attention heads, kv heads, size, experts (0: dense), top, expert or dense size, layers, linear-attention heads and
# state-space heads (states of 128 x 128 and 128 x 64)
KUBOLORN_FIELDS = FIELDS + ("gla_heads", "ssm_heads")
KUBOLORN_SIZES = {
    "2b layers": (2048, 16, 4, 128, 0, 0, 8192, 8, 16, 32),
    "30b-a3b layers": (2048, 32, 4, 128, 128, 8, 768, 4, 16, 32),
    "small layers": (1024, 16, 4, 64, 32, 4, 512, 8, 8, 16),
    "wide layers": (4096, 32, 8, 128, 0, 0, 12288, 4, 32, 64),
}


def kubolorn_configs(size):
    """Three linear-attention layers to one layer with attention beside a state-space mixer. The other model: as many
    delta-rule heads of 128 x 128, one attention layer in four; its gated units are two thirds as wide, so that the
    feed-forwards hold as many weights."""
    from ..config import (AttentionSpec, BigramSpec, BlockSpec, DenseSpec, ExpertSpec, GlaSpec, ModelConfig, RopeConfig, RotaryScaling,
                          SsmSpec, model_config_of_blocks)
    W, H, G, D, E, top, ff, layers, gh, sh = size
    mlp = ExpertSpec(experts=E, top=top, ff=ff * 3 // 2, plain="relu2") if E else DenseSpec(ff, plain="gelu_tanh")
    g = BlockSpec(None, mlp, gla=GlaSpec(heads=gh, dim=128, vdim=128, tau=16.0))
    a = AttentionSpec(heads=H, kv_heads=G, dim=D, vdim=D, scale=D ** -0.5, rot_dims=D // 2, rot_base=1e6, rot_scaling=RotaryScaling(8.0, 8192),
                      sink=True, tied=True)
    p = BlockSpec(a, mlp, ssm=SsmSpec(heads=sh, groups=4, state=128, vdim=64, conv=4, norm_groups=4), scales=(0.7, 0.7))
    mine = model_config_of_blocks("Kubolorn", [p if l % 4 == 3 else g for l in range(layers)], vocab=32000, width=W, eps=1e-6,
                                  embed_scale=1.0, norm_groups=4, input_conv=4, bigram=BigramSpec(32749, 31337, 7919))
    dense = dict(architecture="Qwen3_5ForConditionalGeneration", intermediate_size=ff * 2 // 3 // 128 * 128)
    moe = dict(architecture="Qwen3_5MoeForConditionalGeneration", intermediate_size=3 * W, num_experts=E, num_experts_per_tok=top,
               moe_intermediate_size=ff, norm_topk_prob=True)
    other = ModelConfig(vocab_size=32000, hidden_size=W, num_layers=layers, num_heads=H, num_kv_heads=G, head_dim=D,
                        max_position_embeddings=32768, qk_norm=True, gemma_norm=True, attn_output_gate=True, rope=RopeConfig(theta=1e6),
                        layer_types=["full_attention" if l % 4 == 3 else "linear_attention" for l in range(layers)],
                        linear_num_key_heads=gh, linear_num_value_heads=gh, linear_key_head_dim=128, linear_value_head_dim=128,
                        linear_conv_kernel_dim=4, **(moe if E else dense))
    return {"kubolorn": mine, "qwen3.5": other}


def tabupel_configs(size):
    """Two recurrent layers to one attention layer, latent and differential in turn; windows longer than the
    prompts, as the other model's attention has no limit. The other model: the same pattern of delta-rule layers
    and attention layers with heads as wide as a head's two maps."""
    from ..config import (AttentionSpec, BlockSpec, DenseSpec, LatentSpec, ModelConfig, RglruSpec, RopeConfig, RotaryScaling,
                          model_config_of_blocks)
    W, ff, layers, H, G, D, LH, qr, kr, rec, nb = size
    mlp, win = DenseSpec(ff), 1 << 15
    r = BlockSpec(None, mlp, rglru=RglruSpec(width=rec, blocks=nb, conv=4))
    a = BlockSpec(None, mlp, latent=LatentSpec(heads=LH, dim=128, rot_dim=64, vdim=128, q_rank=qr, kv_rank=kr, scale=192 ** -0.5,
                                               window=win, rot_base=1e4, rot_scaling=RotaryScaling(40.0, 4096)))
    d = BlockSpec(AttentionSpec(heads=H, kv_heads=G, dim=D, vdim=2 * D, scale=D ** -0.5, rot_dims=D, rot_base=1e6,
                                rot_scaling=RotaryScaling(8.0), window=win, diff=0.5), mlp)
    mine = model_config_of_blocks("Tabupel", [(r, r, a, r, r, d)[l % 6] for l in range(layers)], vocab=32000, width=W, eps=1e-6,
                                  residual_mult=0.5, logit_softcap=30.0)
    other = ModelConfig(architecture="Qwen3_5ForConditionalGeneration", vocab_size=32000, hidden_size=W, intermediate_size=ff,
                        num_layers=layers, num_heads=H, num_kv_heads=G, head_dim=2 * D, max_position_embeddings=32768, qk_norm=True,
                        gemma_norm=True, attn_output_gate=True, rope=RopeConfig(theta=1e6),
                        layer_types=["full_attention" if l % 3 == 2 else "linear_attention" for l in range(layers)],
                        linear_num_key_heads=max(1, rec // 256), linear_num_value_heads=max(2, rec // 128), linear_key_head_dim=128,
                        linear_value_head_dim=128, linear_conv_kernel_dim=4)
    return {"tabupel": mine, "qwen3.5": other}


def diforax_configs(size):
    """Three delta blocks to one attention block; chunks longer than the prompts, as the other model's
    attention has no limit; an eighth as many identity experts (at least four), which the other model does not have."""
    from ..config import AttentionSpec, BlockSpec, DeltaSpec, ExpertSpec, ModelConfig, RopeConfig, model_config_of_blocks
    W, H, G, D, E, top, ff, layers, dh, dk = size
    moe = ExpertSpec(experts=E, top=top, ff=ff, identity=max(4, E // 8), groups=4, keep=2)
    att = AttentionSpec(heads=H, kv_heads=G, dim=D, vdim=D, scale=D ** -0.5, rot_dims=D, rot_base=1e6, chunk=1 << 15)
    delta = BlockSpec(None, moe, DeltaSpec(heads=dh, kv_heads=dk, dim=128, vdim=128, conv=4))
    blocks = [BlockSpec(att, moe) if l % 4 == 3 else delta for l in range(layers)]
    mine = model_config_of_blocks("Diforax", blocks, vocab=32000, width=W, eps=1e-6)
    other = ModelConfig(architecture="Qwen3_5MoeForConditionalGeneration", vocab_size=32000, hidden_size=W,
                        intermediate_size=3 * W, num_layers=layers, num_heads=H, num_kv_heads=G, head_dim=D,
                        max_position_embeddings=32768, qk_norm=True, gemma_norm=True, attn_output_gate=True,
                        rope=RopeConfig(theta=1e6), layer_types=["full_attention" if l % 4 == 3 else "linear_attention"
                                                                 for l in range(layers)],
                        linear_num_key_heads=dk, linear_num_value_heads=dh, linear_key_head_dim=128,
                        linear_value_head_dim=128, linear_conv_kernel_dim=4, num_experts=E, num_experts_per_tok=top,
                        moe_intermediate_size=ff, norm_topk_prob=True)
    return {"diforax": mine, "qwen3.5-moe": other}


def nufusun_configs(size):
    from ..config import AttentionSpec, BlockSpec, ExpertSpec, ModelConfig, RopeConfig, model_config_of_blocks
    W, H, G, D, E, top, ff, layers = size
    block = BlockSpec(AttentionSpec(heads=H, kv_heads=G, dim=D, vdim=D, scale=D ** -0.5, bias_max=1024),
                      ExpertSpec(experts=E, top=top, ff=ff, limit=7.0))
    mine = model_config_of_blocks("Nufusun", [block] * layers, vocab=32000, width=W, eps=1e-6, embed_scale=1.0)
    other = ModelConfig(architecture="Qwen3MoeForCausalLM", vocab_size=32000, hidden_size=W, intermediate_size=3 * W,
                        num_layers=layers, num_heads=H, num_kv_heads=G, head_dim=D, max_position_embeddings=32768,
                        qk_norm=True, rope=RopeConfig(theta=1e6), num_experts=E, num_experts_per_tok=top,
                        moe_intermediate_size=ff, norm_topk_prob=True)
    return {"nufusun": mine, "qwen3-moe": other}


def throughput(cfg, prompt: int, batch: int, decode_steps: int, prompt_steps: int) -> dict:
    """Prompt tokens/s over full-budget steps and decoded tokens/s of a full batch, device time."""
    from ..config import EngineArgs
    from ..engine import LLM, SamplingParams
    budget, block = 8192, 32
    max_len = prompt + decode_steps + 64
    llm = LLM(EngineArgs(model_config=cfg, device="cuda", block_size=block, max_model_len=max_len, max_num_seqs=batch,
                         max_num_batched_tokens=budget, num_blocks=batch * (max_len // block + 2) + 8,
                         enable_prefix_caching=False))
    llm.runner.warmup_graphs([s for s in llm.runner.graph_sizes if s >= batch][:1])
    g = torch.Generator().manual_seed(1)
    rng = lambda n: torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist()      # noqa: E731

    def run(n_req, out, skip):
        for _ in range(n_req):
            llm.add_request(rng(prompt), SamplingParams(temperature=0.0, max_tokens=out, ignore_eos=True))
        for _ in range(skip):
            llm.step()

    per_step = max(1, budget // prompt)
    run(per_step * 3, 1, 3)                                         # warm-up
    run(per_step * prompt_steps, 1, 0)
    llm.runner.device_step_ms()
    llm.runner.time_steps = True
    tokens = 0
    while llm.has_unfinished_requests():
        llm.step()
        tokens += llm.step_stats()["scheduled_tokens"]
    prefill = tokens / llm.runner.device_step_ms() * 1e3
    llm.runner.time_steps = False
    run(batch, decode_steps + 8, -(-batch * prompt // budget) + 4)  # prompts in, a few decode steps
    llm.runner.device_step_ms()
    llm.runner.time_steps = True
    for _ in range(decode_steps - 8):
        llm.step()
    ms = llm.runner.device_step_ms() / (decode_steps - 8)
    status = llm.runner.ops.read_status()
    return {"prefill_tok_s": round(prefill), "decode_tok_s": round(batch / ms * 1e3), "decode_step_ms": round(ms, 4),
            "status": status}


# ------------------------------------------------------------------------------ kernels
def _peaks():
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return p["hbm_gbs"], p["bf16_tflops"], "measured"
    except (OSError, KeyError, ValueError):
        return 6650.0, 1590.0, "fallback"


class KernelBench:
    def __init__(self, size):
        self.W, self.H, self.G, self.D, self.E, self.top, self.ff = size[:7]
        self.dev = torch.device("cuda")
        self.hbm, self.tflops, _ = _peaks()
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=self.dev)
        self.rows: list = []

    def time(self, fn, iters=9):
        from ..ops.bench import _time
        return _time(fn, iters=iters, warmup=3, flush=self.flush)

    def add(self, name, whose, fn, nbytes=0.0, flops=0.0, note=None, full_us=None):
        """The roofline is the slower of the bytes at the measured copy rate and the tensor FLOPs at
        the measured GEMM rate. ``full_us``: the roofline with work that ``flops`` leaves out."""
        ms = self.time(fn)
        best = max(nbytes / (self.hbm * 1e6), flops / (self.tflops * 1e9))
        row = {"kernel": name, "model": whose, "us": round(ms * 1e3, 1), "roofline_us": round(best * 1e3, 1),
               "fraction": round(best / ms, 3)}
        if full_us is not None:
            row.update(full_roofline_us=round(full_us, 1), full_fraction=round(full_us / (ms * 1e3), 3))
        if note:
            row["note"] = note
        self.rows.append(row)

    def rnd(self, *shape, dtype=torch.bfloat16, s=1.0):
        return (torch.randn(*shape, device=self.dev, dtype=torch.float32) * s).to(dtype)

    def i32(self, x):
        return torch.tensor(x, dtype=torch.int32, device=self.dev)


class NufusunKernels(KernelBench):
    def run(self):
        self.attention(B=4, prompt=2048, decode_batch=64, ctx=4096)
        self.attention(B=8, prompt=1024, decode_batch=8, ctx=16384)
        for T in (64, 8192):
            self.rest(T)

    def attention(self, B, prompt, decode_batch, ctx, bs=32):
        from .. import ops
        from ..ops import bias_attn as A
        from ..ops.reference import build_prefill_tiles
        H, G, D, kw = self.H, self.G, self.D, self.G * self.D
        bias = self.rnd(H, 1024, dtype=torch.float32)
        # ---- prompts of equal length
        nb, T = prompt // bs, B * prompt
        bt = torch.arange(1, B * nb + 1, device=self.dev, dtype=torch.int32).view(B, nb)
        sl, qs = self.i32([prompt] * B), self.i32([i * prompt for i in range(B + 1)])
        tr, tq = (self.i32(x) for x in build_prefill_tiles([prompt] * B))
        pairs = B * prompt * (prompt + 1) / 2
        flops = 2 * pairs * H * 2 * D
        q = self.rnd(T, H * kw, s=kw ** -0.5)
        pages = self.rnd(B * nb + 1, bs * 2 * kw)
        out = torch.empty(T, H * D, dtype=torch.bfloat16, device=self.dev)
        shape = dict(H=H, G=G, kw=kw, vdim=D, block_size=bs)
        kind = A.kernel_kind("prefill", q, pages, **shape)
        # mixing the heads costs H multiply-adds per head and pair in fp32 (128 lanes an SM), or products
        # kw wide instead of D; the cheaper of the two
        sms, mhz = torch.cuda.get_device_properties(0).multi_processor_count, 1965.0
        full = min(max(flops / self.tflops / 1e6, pairs * H * H / (sms * 128 * mhz)),
                   2 * pairs * H * (kw + D) / self.tflops / 1e6)
        self.add(f"attention, {B} x {prompt} prompt", "nufusun",
                 lambda: A.prefill(q, pages, out, block_table=bt, seq_lens=sl, q_start=qs, num_reqs=B, tile_req=tr,
                                   tile_q0=tq, bias=bias, null_entry=True, **shape), flops=flops, full_us=full,
                 note=f"{kind}; multiplies {kw} + {D} wide, {(kw + D) / (2 * D):.2f} x the counted FLOPs")
        q2, kv = self.rnd(T, H * D), self.rnd(B * nb + 1, 2, bs, G, D)
        self.add(f"attention, {B} x {prompt} prompt", "qwen3-moe",
                 lambda: ops.attn_prefill(q2, kv, block_table=bt, seq_lens=sl, q_start=qs, tile_req=tr, tile_q0=tq,
                                          num_q_heads=H, num_kv_heads=G, head_dim=D, block_size=bs, scale=D ** -0.5,
                                          out=out), flops=flops)
        # ---- head mix + cache write against qk-norm + rotation + cache write
        qkv = self.rnd(T, (H + 2 * G) * D, dtype=torch.float32)
        slots = (bt.long()[:, :, None] * bs + torch.arange(bs, device=self.dev)).reshape(-1)
        mix = self.rnd(H, H, dtype=torch.float32)
        self.add(f"query preparation + cache write, {T} tokens", "nufusun",
                 lambda: A.head_mix_kv(qkv, mix, q, slots, pages, H=H, G=G, dim=D, vdim=D, block_size=bs),
                 nbytes=T * ((H + 2 * G) * D * 4 + (H * kw + 2 * G * D) * 2))
        qkvb, pos = qkv.to(torch.bfloat16), torch.arange(T, device=self.dev) % prompt
        table = self.rnd(prompt, D, dtype=torch.float32)
        nw = self.rnd(D)
        self.add(f"query preparation + cache write, {T} tokens", "qwen3-moe",
                 lambda: ops.rope_kv(qkvb, pos, table, num_q_heads=H, num_kv_heads=G, head_dim=D, q_norm=nw, k_norm=nw,
                                     slot_mapping=slots, kv_cache=kv, block_size=bs),
                 nbytes=T * ((H + 2 * G) * D * 2 + (H + 4 * G) * D * 2 - 2 * G * D))
        # ---- decode
        B, nb = decode_batch, ctx // bs
        bt = torch.arange(1, B * nb + 1, device=self.dev, dtype=torch.int32).view(B, nb)
        sl = self.i32([ctx] * B)
        pages, kv = self.rnd(B * nb + 1, bs * 2 * kw), self.rnd(B * nb + 1, 2, bs, G, D)
        q, q2 = self.rnd(B, H * kw, s=kw ** -0.5), self.rnd(B, H * D)
        nbytes = B * ctx * 2 * kw * 2
        splits = A.decode_splits(B, ctx, ops.num_sms())
        out = torch.empty(B, H * D, dtype=torch.bfloat16, device=self.dev)
        self.add(f"attention, decode {B} x {ctx}", "nufusun",
                 lambda: A.decode(q, pages, out, block_table=bt, seq_lens=sl, bias=bias, null_entry=True, splits=splits,
                                  **shape), nbytes=nbytes, note=A.kernel_kind("decode", q, pages, **shape))
        self.add(f"attention, decode {B} x {ctx}", "qwen3-moe",
                 lambda: ops.attn_decode(q2, kv, block_table=bt, seq_lens=sl, num_q_heads=H, num_kv_heads=G, head_dim=D,
                                         block_size=bs, scale=D ** -0.5, out=out), nbytes=nbytes)

    def rest(self, T):
        from .. import ops
        from ..ops import moe as M
        from ..ops.stream import stream_norm
        W, E, top, ff = self.W, self.E, self.top, self.ff
        P = T * top
        ws = M.MoeWorkspace(self.dev, T, top, E, W, ff)
        x, wgu, wd = self.rnd(T, W), self.rnd(E, 2 * ff, W, s=0.05), self.rnd(E, W, ff, s=0.05)
        logits = self.rnd(T, E, dtype=torch.float32)
        ids, w = M.router_topk(logits, top, renorm=False, scoring="sigmoid")
        used = min(E, int(ids.unique().numel()))
        chunks = min(ws.max_chunks, E + (P + 255) // 256)
        M.moe_sort(ids, 0, E, ws)
        M.moe_gather(x, ws, E, P)
        act = M.ClampedGate(7.0, 1.702, 1.0, M.ptr(ws.row_w))
        nbytes = used * 2 * ff * W * 2 + P * (W + ff) * 2
        args = (M.ptr(ws.chunk_expert), M.ptr(ws.chunk_row0), M.ptr(ws.chunk_n), M.ptr(ws.meta), chunks)
        import ctypes
        self.add(f"gated expert products, {T} tokens", "nufusun",
                 lambda: M.check(M.lib().b200_moe_grouped_gemm_clamped(M.ptr(ws.xs), P, M.ptr(wgu), E, 2 * ff, W, M.ptr(ws.act),
                                                                       *args, ctypes.byref(act), M.stream_ptr()), "clamped"),
                 nbytes=nbytes, flops=2.0 * P * 2 * ff * W)
        self.add(f"gated expert products, {T} tokens", "qwen3-moe",
                 lambda: M.grouped_gemm_gated(ws.xs, wgu, ws.act, ws, P, chunks), nbytes=nbytes, flops=2.0 * P * 2 * ff * W)
        out, stream = torch.empty_like(x), self.rnd(T, W, dtype=torch.float32)
        a, nw = self.rnd(T, W, dtype=torch.float32), self.rnd(W, dtype=torch.float32)
        pos = ws.pair_pos[:P].view(T, top)
        self.add(f"expert sum + residual + norm, {T} tokens", "nufusun",
                 lambda: stream_norm(stream, nw, 1e-6, out, width=W, a=a, y=ws.y, pair_pos=pos),
                 nbytes=T * W * (4 + 4 + 4 + 2 * top + 2))
        o2, res, nwb = torch.empty_like(x), self.rnd(T, W), nw.to(torch.bfloat16)

        def two():
            M.combine(ws.y, ws, w, o2)
            ops.rmsnorm(o2, nwb, 1e-6, residual=res, out=out)
        self.add(f"expert sum + residual + norm, {T} tokens", "qwen3-moe", two, nbytes=T * W * 2 * (top + 1 + 1 + 2 + 1),
                 note="two kernels")


class DiforaxKernels(KernelBench):
    def __init__(self, size):
        super().__init__(size)
        self.dh, self.dk = size[8:]

    def run(self):
        self.attention(B=4, prompt=2048, decode_batch=64, ctx=4096)
        self.attention(B=8, prompt=1024, decode_batch=8, ctx=16384)
        self.delta(B=4, n=2048)
        self.delta(B=8, n=1024)
        self.delta(B=1, n=8192)
        for B in (16, 64, 256):
            self.delta(B=B, n=1)
        for T in (64, 8192):
            self.rest(T)

    def attention(self, B, prompt, decode_batch, ctx, bs=32):
        from .. import ops
        from ..ops import bias_attn as A
        from ..ops.reference import build_prefill_tiles
        H, G, D, kw = self.H, self.G, self.D, self.G * self.D
        shape = dict(H=H, G=G, kw=kw, vdim=D, block_size=bs, grouped=True)
        nb, T = prompt // bs, B * prompt
        bt = torch.arange(1, B * nb + 1, device=self.dev, dtype=torch.int32).view(B, nb)
        sl, qs = self.i32([prompt] * B), self.i32([i * prompt for i in range(B + 1)])
        tr, tq = (self.i32(x) for x in build_prefill_tiles([prompt] * B))
        q, pages = self.rnd(T, H * D), self.rnd(B * nb + 1, bs * 2 * kw)
        kv, out = self.rnd(B * nb + 1, 2, bs, G, D), torch.empty(T, H * D, dtype=torch.bfloat16, device=self.dev)
        for chunk in (0, 512):
            n, last = divmod(prompt, chunk or prompt)
            size = chunk or prompt
            pairs = B * (n * size * (size + 1) / 2 + last * (last + 1) / 2)
            self.add(f"attention, {B} x {prompt} prompt" + (f", chunks of {chunk}" if chunk else ""), "diforax",
                     lambda: A.prefill(q, pages, out, block_table=bt, seq_lens=sl, q_start=qs, num_reqs=B, tile_req=tr,
                                       tile_q0=tq, scale=D ** -0.5, chunk=chunk, **shape), flops=2 * pairs * H * 2 * D,
                     note=A.kernel_kind("prefill", q, pages, scale=D ** -0.5, chunk=chunk, **shape))
            self.add(f"attention, {B} x {prompt} prompt" + (f", chunks of {chunk}" if chunk else ""), "qwen3.5-moe",
                     lambda: ops.attn_prefill(q, kv, block_table=bt, seq_lens=sl, q_start=qs, tile_req=tr, tile_q0=tq,
                                              num_q_heads=H, num_kv_heads=G, head_dim=D, block_size=bs, scale=D ** -0.5,
                                              window=-chunk, out=out), flops=2 * pairs * H * 2 * D)
        qkv, pos = self.rnd(T, (H + 2 * G) * D), torch.arange(T, device=self.dev) % prompt
        slots = (bt.long()[:, :, None] * bs + torch.arange(bs, device=self.dev)).reshape(-1)
        table, nw = self.rnd(prompt, D, dtype=torch.float32), self.rnd(D)
        nbytes = T * 2 * (H + 2 * G) * D * 2
        self.add(f"query preparation + cache write, {T} tokens", "diforax",
                 lambda: A.rotate_kv(qkv, pos, table, D, 1e-6, q, slots, pages, H=H, G=G, D=D, V=D, dim=D, block_size=bs),
                 nbytes=nbytes)
        self.add(f"query preparation + cache write, {T} tokens", "qwen3.5-moe",
                 lambda: ops.rope_kv(qkv, pos, table, num_q_heads=H, num_kv_heads=G, head_dim=D, q_norm=nw, k_norm=nw,
                                     slot_mapping=slots, kv_cache=kv, block_size=bs, q_out=q), nbytes=nbytes)
        B, nb = decode_batch, ctx // bs
        bt = torch.arange(1, B * nb + 1, device=self.dev, dtype=torch.int32).view(B, nb)
        sl = self.i32([ctx] * B)
        pages, kv, q = self.rnd(B * nb + 1, bs * 2 * kw), self.rnd(B * nb + 1, 2, bs, G, D), self.rnd(B, H * D)
        out = torch.empty(B, H * D, dtype=torch.bfloat16, device=self.dev)
        splits = A.grouped_decode_splits(B, G, ctx, ops.num_sms())
        tmp = (torch.empty(B * H * splits * D, dtype=torch.float32, device=self.dev),
               torch.empty(B * H * splits, dtype=torch.float32, device=self.dev))
        nbytes = B * ctx * 2 * kw * 2
        self.add(f"attention, decode {B} x {ctx}", "diforax",
                 lambda: A.decode(q, pages, out, block_table=bt, seq_lens=sl, splits=splits, tmp=tmp, scale=D ** -0.5,
                                  **shape), nbytes=nbytes, note=A.kernel_kind("decode", q, pages, scale=D ** -0.5, **shape))
        self.add(f"attention, decode {B} x {ctx}", "qwen3.5-moe",
                 lambda: ops.attn_decode(q, kv, block_table=bt, seq_lens=sl, num_q_heads=H, num_kv_heads=G, head_dim=D,
                                         block_size=bs, scale=D ** -0.5, out=out), nbytes=nbytes)

    def delta(self, B, n):
        """``B`` prompts of ``n`` tokens, or (n 1) a decode batch: preparation, then recurrence with norm and gate."""
        import ctypes
        from types import SimpleNamespace
        from ..ops import delta as X
        from ..ops import gdn as Q
        from ..ops.reference import build_prefill_tiles
        G, H, D, T = self.dk, self.dh, 128, B * n
        s = X.DeltaShape(G=G, H=H, D=D, V=D, dim=D, vdim=D, taps=4)
        f32 = dict(dtype=torch.float32)
        proj, ab = self.rnd(T, s.columns), self.rnd(T, 2 * H, **f32)
        w = {"conv_w": self.rnd(4, s.channels, **f32), "A": self.rnd(H, **f32).abs(), "dt": self.rnd(H, **f32),
             "norm": self.rnd(D, **f32)}
        conv, state = self.rnd(B, 3, s.channels), torch.zeros(B, H, D, D, device=self.dev)
        tr, tq = build_prefill_tiles([n] * B) if n > 1 else ([], [])
        rows = SimpleNamespace(seq_lens=self.i32([n + 5] * B), state_slots=self.i32(list(range(B))),
                               prefill_q_start=self.i32([i * n for i in range(B + 1)]), tile_req=self.i32(tr or [0]),
                               tile_q0=self.i32(tq or [0]), num_decodes=B if n == 1 else 0, num_prefills=0 if n == 1 else B,
                               num_tiles=len(tr))
        bufs = {"q": self.rnd(T, G, D, **f32), "k": self.rnd(T, G, D, **f32), "v": self.rnd(T, H, D), "g": self.rnd(T, H, **f32),
                "beta": self.rnd(T, H, **f32), "o": self.rnd(T, H, D, **f32), "chunks": X.chunk_workspace(self.dev, len(tr) + 1, H)}
        out = torch.empty(T, H * D, dtype=torch.bfloat16, device=self.dev)
        a = X.delta_args(proj, ab, w, s, conv, state, rows, bufs, out, 1e-6)
        what = f"{B} x {n} prompt" if n > 1 else f"decode {B}"
        prep = T * (2 * s.channels * 2 + 2 * H * 4)
        step = T * (2 * G * D + 3 * H * D) * 2 + B * H * D * D * 4 * 2
        flops = T * H * (6.0 * D * D + 4 * 64 * D) if n > 1 else 0
        self.add(f"delta preparation, {what}", "diforax", lambda: X.run_prepare(a), nbytes=prep)
        self.add(f"delta rule + gated norm, {what}", "diforax", lambda: X.run_rule(a, bufs), nbytes=step, flops=flops,
                 note="state, q and k in 32 bits")
        # the other model's kernels
        cw, cst = w["conv_w"].t().contiguous().to(torch.bfloat16), self.rnd(B, s.channels, 3)
        xc, st2 = self.rnd(T, s.channels), torch.zeros(B, H, D, D, device=self.dev)
        mixed, z = proj[:, : s.channels], proj[:, s.channels:]
        abb, slots, core = ab.to(torch.bfloat16), rows.state_slots, torch.empty_like(out)
        a2, b2, nw = abb[:, :H], abb[:, H:], w["norm"].to(torch.bfloat16)
        if n == 1:
            self.add(f"delta preparation, {what}", "qwen3.5-moe", lambda: Q.conv1d_update(mixed, cw, cst, slots, xc), nbytes=prep,
                     note="convolution only")

            def theirs():
                Q.packed_decode(xc, a2, b2, w["A"], w["dt"], st2, slots, core.view(T, H, D), G, H)
                Q.rmsnorm_gated(core, z, nw, core, heads=H)
        else:
            q, k = self.rnd(T, G, D), self.rnd(T, G, D)
            g, beta, init = self.rnd(T, H, **f32), self.rnd(T, H, **f32).abs(), self.i32([1] * B)
            ws, qsl = Q.GdnWorkspace(self.dev, T, B, H), rows.prefill_q_start
            host = [i * n for i in range(B + 1)]
            t0, ln, s0 = Q.build_chunk_table(host)
            table = (self.i32(t0.tolist()), self.i32(ln.tolist()), self.i32(s0.tolist()))

            def theirs_prep():
                Q.conv1d_fwd(mixed, cw, cst, qsl, slots, init, xc)
                Q.post_conv(xc, G, H, a2, b2, w["A"], w["dt"], q, k, g, beta)
            self.add(f"delta preparation, {what}", "qwen3.5-moe", theirs_prep, nbytes=prep)

            def theirs():
                Q.chunk_scan(q, k, xc, g, beta, st2, host, slots, init, core.view(T, H, D), ws, v_col0=2 * G * D, table=table)
                Q.rmsnorm_gated(core, z, nw, core, heads=H)
        self.add(f"delta rule + gated norm, {what}", "qwen3.5-moe", theirs, nbytes=step, flops=flops)

    def rest(self, T):
        import ctypes
        from .. import ops
        from ..ops import moe as M
        from ..ops.stream import stream_norm
        W, E, top, ff = self.W, self.E, self.top, self.ff
        P, I = T * top, max(4, E // 8)
        ws = M.MoeWorkspace(self.dev, T, top, E, W, ff)
        x, wgu, wd = self.rnd(T, W), self.rnd(E, 2 * ff, W, s=0.05), self.rnd(E, W, ff, s=0.05)
        logits, corr = self.rnd(T, E + I, dtype=torch.float32), self.rnd(E + I, dtype=torch.float32, s=0.01)
        choose = lambda: M.router_topk(logits, top, renorm=False, e_bias=corr, n_group=4, topk_group=2, group_best=1)  # noqa: E731
        self.add(f"router, {T} tokens", "diforax", choose, nbytes=T * ((E + I) * 4 + top * 8))
        plain = logits[:, :E].contiguous()
        self.add(f"router, {T} tokens", "qwen3.5-moe", lambda: M.router_topk(plain, top), nbytes=T * (E * 4 + top * 8))
        for who, (ids, w) in (("diforax", choose()), ("qwen3.5-moe", M.router_topk(plain, top))):
            real = ids < E
            used, pairs = int(ids[real].unique().numel()), int(real.sum())
            chunks = min(ws.max_chunks, E + (P + 255) // 256)
            M.moe_sort(ids, 0, E, ws)
            M.moe_gather(x, ws, E, P)
            nbytes, fl = used * 2 * ff * W * 2 + pairs * (W + ff) * 2, 2.0 * pairs * 2 * ff * W
            if who == "diforax":
                act = M.ClampedGate(float("inf"), 1.0, 0.0, None)
                args = (M.ptr(ws.chunk_expert), M.ptr(ws.chunk_row0), M.ptr(ws.chunk_n), M.ptr(ws.meta), chunks)
                fn = lambda: M.check(M.lib().b200_moe_grouped_gemm_clamped(M.ptr(ws.xs), P, M.ptr(wgu), E, 2 * ff, W,  # noqa: E731
                                                                           M.ptr(ws.act), *args, ctypes.byref(act), M.stream_ptr()), "gemm")
            else:
                fn = lambda: M.grouped_gemm_gated(ws.xs, wgu, ws.act, ws, P, chunks)                    # noqa: E731
            self.add(f"gated expert products, {T} tokens", who, fn, nbytes=nbytes, flops=fl)
            self.add(f"down expert products, {T} tokens", who, lambda: M.grouped_gemm(ws.act, wd, ws.y, ws, P, chunks),
                     nbytes=used * ff * W * 2 + pairs * (W + ff) * 2, flops=fl / 2)
            out, stream = torch.empty_like(x), self.rnd(T, W, dtype=torch.float32)
            nw = self.rnd(W, dtype=torch.float32)
            if who == "diforax":
                pos = ws.pair_pos[:P].view(T, top)
                self.add(f"expert sum + norms + residual, {T} tokens", who,
                         lambda: stream_norm(stream, nw, 1e-6, out, width=W, y=ws.y, pair_pos=pos, pair_w=w, post_w=nw, ident=out,
                                             norm_offset=0.0), nbytes=T * W * (4 + 4 + 2 * top + 2), note="a norm more")
                mixed = self.rnd(T, W, dtype=torch.float32)
                self.add(f"norms + residual, {T} tokens", who,
                         lambda: stream_norm(stream, nw, 1e-6, out, width=W, a=mixed, post_w=nw, norm_offset=0.0),
                         nbytes=T * W * (4 + 4 + 4 + 2), note="a norm more")
                continue
            o2, res, nwb = torch.empty_like(x), self.rnd(T, W), nw.to(torch.bfloat16)

            def two():
                M.combine(ws.y, ws, w, o2)
                ops.rmsnorm(o2, nwb, 1e-6, residual=res, out=out)
            self.add(f"expert sum + norms + residual, {T} tokens", who, two, nbytes=T * W * 2 * (top + 1 + 1 + 2 + 1), note="two kernels")
            self.add(f"norms + residual, {T} tokens", who, lambda: ops.rmsnorm(o2, nwb, 1e-6, residual=res, out=out),
                     nbytes=T * W * 2 * 4)


class TabupelKernels(KernelBench):
    def __init__(self, size):
        super().__init__((size[0], *size[3:6], 1, 1, size[1]))
        self.LH, self.qr, self.kr, self.rec, self.nb = size[6:]

    def run(self):
        self.attention(B=4, prompt=2048, decode_batch=64, ctx=4096)
        self.attention(B=8, prompt=1024, decode_batch=8, ctx=16384)
        self.latent(B=4, prompt=2048, decode_batch=64, ctx=4096)
        self.latent(B=8, prompt=1024, decode_batch=8, ctx=16384)
        for B, n in ((4, 2048), (8, 1024), (1, 8192), (16, 1), (64, 1), (256, 1)):
            self.recurrence(B, n)
        for T in (64, 8192):
            self.rest(T)

    def step_rows(self, B, prompt, bs):
        from ..ops.reference import build_prefill_tiles
        nb = prompt // bs
        bt = torch.arange(1, B * nb + 1, device=self.dev, dtype=torch.int32).view(B, nb)
        tr, tq = (self.i32(x) for x in build_prefill_tiles([prompt] * B))
        return bt, dict(seq_lens=self.i32([prompt] * B), q_start=self.i32([i * prompt for i in range(B + 1)]), tile_req=tr, tile_q0=tq)

    @staticmethod
    def pairs(B, n, window):
        w = min(window or n, n)
        return B * (w * (w + 1) / 2 + (n - w) * w)

    def attention(self, B, prompt, decode_batch, ctx, bs=32):
        from .. import ops
        from ..ops import bias_attn as A
        H, G, D = self.H, self.G, self.D
        V, T = 2 * D, B * prompt
        row = G * (2 * D + V)
        bt, rows = self.step_rows(B, prompt, bs)
        shape = dict(H=2 * H, G=G, kw=2 * G * D, vdim=V, block_size=bs, grouped=True, maps=2, scale=D ** -0.5)
        q, pages = self.rnd(T, 2 * H * D), self.rnd(B * prompt // bs + 1, bs * row)
        maps = torch.empty(T, 2 * H * V, dtype=torch.bfloat16, device=self.dev)
        q2, kv = self.rnd(T, H * V), self.rnd(B * prompt // bs + 1, 2, bs, G, V)
        out = torch.empty(T, H * V, dtype=torch.bfloat16, device=self.dev)
        for window in (0, 512):
            what = f"attention, {B} x {prompt} prompt" + (f", window {window}" if window else "")
            n = self.pairs(B, prompt, window)
            self.add(what, "tabupel", lambda: A.prefill(q, pages, maps, block_table=bt, num_reqs=B, window=window, **rows, **shape),
                     flops=2 * n * 2 * H * (D + V), note=A.kernel_kind("prefill", q, pages, window=window, **shape))
            self.add(what, "qwen3.5", lambda: ops.attn_prefill(q2, kv, block_table=bt, num_q_heads=H, num_kv_heads=G, head_dim=V,
                                                               block_size=bs, scale=V ** -0.5, window=window, out=out, **rows),
                     flops=2 * n * H * 2 * V)
        qkv, pos = self.rnd(T, 2 * (H + G) * D + G * V), torch.arange(T, device=self.dev) % prompt
        slots = (bt.long()[:, :, None] * bs + torch.arange(bs, device=self.dev)).reshape(-1)
        table, nw = self.rnd(prompt, D, dtype=torch.float32), self.rnd(D, dtype=torch.float32)
        nbytes = T * 2 * (2 * (H + G) * D + G * V) * 2
        self.add(f"query preparation + cache write, {T} tokens", "tabupel",
                 lambda: A.rotate_kv(qkv, pos, table, D, 1e-6, q, slots, pages, H=2 * H, G=2 * G, value_heads=G, D=D, V=V, dim=D,
                                     block_size=bs, q_w=nw, k_w=nw), nbytes=nbytes)
        qkv2, nw2 = self.rnd(T, (H + 2 * G) * V), self.rnd(V)
        table2 = self.rnd(prompt, V, dtype=torch.float32)
        self.add(f"query preparation + cache write, {T} tokens", "qwen3.5",
                 lambda: ops.rope_kv(qkv2, pos, table2, num_q_heads=H, num_kv_heads=G, head_dim=V, q_norm=nw2, k_norm=nw2,
                                     slot_mapping=slots, kv_cache=kv, block_size=bs, q_out=q2), nbytes=T * 2 * (H + 2 * G) * V * 2)
        from ..ops import gdn as Q
        self.add(f"difference of the maps + norm, {T} tokens", "tabupel",
                 lambda: A.diff_combine(maps, out, H=H, V=V, vdim=V, lam=0.4, eps=1e-6, scale=0.5), nbytes=T * 3 * H * V * 2)
        a, b = self.rnd(T, H * 128), self.rnd(T, H * 128)
        core, nw3 = torch.empty_like(a), self.rnd(128)
        self.add(f"difference of the maps + norm, {T} tokens", "qwen3.5",
                 lambda: Q.rmsnorm_gated(a, b, nw3, core, heads=H), nbytes=T * 3 * H * 128 * 2, note="norm and gate of two rows")
        B, nb = decode_batch, ctx // bs
        bt = torch.arange(1, B * nb + 1, device=self.dev, dtype=torch.int32).view(B, nb)
        sl = self.i32([ctx] * B)
        pages, kv, q, q2 = self.rnd(B * nb + 1, bs * row), self.rnd(B * nb + 1, 2, bs, G, V), self.rnd(B, 2 * H * D), self.rnd(B, H * V)
        maps, out = (torch.empty(B, n * H * V, dtype=torch.bfloat16, device=self.dev) for n in (2, 1))
        splits = A.grouped_decode_splits(B, G, ctx, ops.num_sms())
        tmp = (torch.empty(B * 2 * H * splits * V, dtype=torch.float32, device=self.dev),
               torch.empty(B * 2 * H * splits, dtype=torch.float32, device=self.dev))
        nbytes = B * ctx * row * 2
        self.add(f"attention, decode {B} x {ctx}", "tabupel",
                 lambda: A.decode(q, pages, maps, block_table=bt, seq_lens=sl, splits=splits, tmp=tmp, **shape), nbytes=nbytes,
                 note=A.kernel_kind("decode", q, pages, **shape))
        self.add(f"attention, decode {B} x {ctx}", "qwen3.5",
                 lambda: ops.attn_decode(q2, kv, block_table=bt, seq_lens=sl, num_q_heads=H, num_kv_heads=G, head_dim=V,
                                         block_size=bs, scale=V ** -0.5, out=out), nbytes=nbytes)

    def latent(self, B, prompt, decode_batch, ctx, bs=32):
        from .. import ops
        from ..ops import latent as L
        from ..ops import mla as M
        H, T = self.LH, B * prompt
        s = L.LatentShape(H=H, dim=128, rot=64, vdim=128, q_rank=self.qr, rank=self.kr)
        scale, gate = 192 ** -0.5, self.rnd(T, s.down[3])
        bt, rows = self.step_rows(B, prompt, bs)
        cache, q = self.rnd(B * prompt // bs + 1, bs * s.row), self.rnd(T, H * s.qw)
        out = torch.empty(T, H * s.V, dtype=torch.bfloat16, device=self.dev)
        wkv = self.rnd(H * (s.D + s.V), s.rankp, s=0.05)
        dense, kvb = self.rnd(T, s.row), self.rnd(T, H * (s.D + s.V))
        n = self.pairs(B, prompt, 0)
        first, base, total, table = L.visible_pages([prompt] * B, [prompt] * B, 0, bs)
        first, base, table = self.i32(first.tolist()), self.i32(base.tolist()), torch.from_numpy(table).to(self.dev)
        flops = 2 * n * H * (192 + 128)
        self.add(f"latent attention, {B} x {prompt} prompt", "tabupel",
                 lambda: L.prefill_expanded(q, kvb, dense, out, s, block_table=table, num_reqs=B, scale=scale, window=0,
                                            block_size=bs, gate=gate, **rows), flops=flops)
        qpad, pages = self.rnd(T, H * 256), self.rnd(T // bs, 2, bs, H, 256)
        attn = torch.empty(T, H * 256, dtype=torch.bfloat16, device=self.dev)
        sl, qs, tr, tq = (rows[k] for k in ("seq_lens", "q_start", "tile_req", "tile_q0"))
        ident = torch.arange(T // bs, device=self.dev, dtype=torch.int32).view(B, -1)
        theirs = H <= 16 and self.kr == 512
        self.add(f"latent attention, {B} x {prompt} prompt", "deepseek-v2",
                 lambda: ops.attn_prefill(qpad, pages, block_table=ident, num_q_heads=H, num_kv_heads=H, head_dim=256, block_size=bs,
                                          scale=scale, out=attn, **rows), flops=flops, note="heads padded to 256")

        def expand():
            L.gather(cache, bt, sl, first, base, bs, dense, B, table.shape[1])
            ops.gemm(dense[:, : s.rankp], wkv, out=kvb, const_w=True)

        def their_expand():
            M.gather_latent(cache, bt, sl, base * bs, bs, dense, B, prompt // bs)
            ops.gemm(dense[:, :512], wkv, out=kvb)
            M.assemble_kv(kvb, dense, pages, T, H, bs)
            M.pad_q(q, qpad, T, H)
        nbytes = T * (2 * s.row + H * (s.D + s.V)) * 2
        fl = 2.0 * T * s.rankp * H * (s.D + s.V)
        self.add(f"latent rows to keys and values, {T} tokens", "tabupel", expand, nbytes=nbytes, flops=fl, note="gather, product")
        if theirs:
            self.add(f"latent rows to keys and values, {T} tokens", "deepseek-v2", their_expand, nbytes=nbytes, flops=fl,
                     note="gather, product, assembly of keys, padding of queries")
        # ---- preparation
        down, cq = self.rnd(T, sum(s.down)), torch.empty(T, s.down[0], dtype=torch.bfloat16, device=self.dev)
        f32 = dict(dtype=torch.float32)
        w = {"q_norm": self.rnd(s.down[0], **f32), "kv_norm": self.rnd(s.down[1], **f32)}
        pos, tab = torch.arange(T, device=self.dev) % prompt, self.rnd(prompt, 64, **f32)
        slots = (bt.long()[:, :, None] * bs + torch.arange(bs, device=self.dev)).reshape(-1)
        self.add(f"latent preparation, {T} tokens", "tabupel",
                 lambda: L.prepare(down, pos, tab, w, s, 1e-6, cq, slots, cache), nbytes=T * 2 * (sum(s.down[:3]) * 2))
        self.add(f"latent queries, {T} tokens", "tabupel", lambda: L.queries(q, pos, tab, s, None, 0), nbytes=T * H * 64 * 2 * 2)
        qa = self.rnd(T, H * 192 + 576)
        kvn, cache3 = self.rnd(512), self.rnd(B * prompt // bs + 1, bs, 576)
        kvc, kpe = qa[:, H * 192: H * 192 + 512], qa[:, H * 192 + 512:]

        def their_prep():
            ops.rope_kv(qa, pos, tab, num_q_heads=H, num_kv_heads=1, head_dim=64, rot_dim=64, neox=False, q_head_stride=192,
                        offsets=(128, H * 192 + 512, 0))
            ops.rmsnorm(kvc, kvn, 1e-6, out=kvc)
            ops.concat_and_cache_mla(kvc, kpe, slots, cache3)
        self.add(f"latent preparation and queries, {T} tokens", "deepseek-v2", their_prep, nbytes=T * 2 * (H * 64 * 2 + 576 * 2),
                 note="three kernels, no query latent")
        # ---- decode
        B, nb = decode_batch, ctx // bs
        bt = torch.arange(1, B * nb + 1, device=self.dev, dtype=torch.int32).view(B, nb)
        sl, cache = self.i32([ctx] * B), self.rnd(B * nb + 1, bs * s.row)
        qabs, olat = self.rnd(B, H * s.row), torch.empty(B, H * s.rankp, dtype=torch.bfloat16, device=self.dev)
        splits = L.decode_splits(B, H, ctx, ops.num_sms())
        tmp = (torch.empty(B * H * splits * s.rankp, dtype=torch.float32, device=self.dev),
               torch.empty(B * H * splits, dtype=torch.float32, device=self.dev))
        for window in (0, 1024):
            keys = min(window or ctx, ctx)
            what = f"latent attention, decode {B} x {ctx}" + (f", window {window}" if window else "")
            self.add(what, "tabupel", lambda: L.decode(qabs, cache, olat, s, block_table=bt, seq_lens=sl, scale=scale, window=window,
                                                       block_size=bs, gate=gate[:B], splits=splits, tmp=tmp),
                     nbytes=B * keys * s.row * 2)
        if theirs:
            q3, c3 = qabs.view(B, H, 576), cache.view(-1, bs, 576)
            self.add(f"latent attention, decode {B} x {ctx}", "deepseek-v2",
                     lambda: M.mla_decode(q3, c3, bt, sl, olat, scale, bs, splits=splits,
                                          tmp=(tmp[0].view(B, H, splits, 512), tmp[1].view(B, H, splits))), nbytes=B * ctx * 576 * 2)

    def recurrence(self, B, n):
        """``B`` prompts of ``n`` tokens, or (n 1) a decode batch: convolution, then gates and recurrence."""
        from types import SimpleNamespace
        from ..ops import gdn as Q
        from ..ops import rglru as G
        from ..ops.reference import build_prefill_tiles
        s, T, C = G.RglruShape(blocks=self.nb, size=self.rec // self.nb, taps=4), B * n, self.rec
        f32 = dict(dtype=torch.float32)
        tr, tq = build_prefill_tiles([n] * B) if n > 1 else ([], [])
        rows = SimpleNamespace(seq_lens=self.i32([n + 5] * B), state_slots=self.i32(list(range(B))),
                               prefill_q_start=self.i32([i * n for i in range(B + 1)]), tile_req=self.i32(tr or [0]),
                               tile_q0=self.i32(tq or [0]), num_decodes=B if n == 1 else 0, num_prefills=0 if n == 1 else B,
                               num_tiles=len(tr))
        proj, u, out = self.rnd(T, 2 * C), self.rnd(T, C), torch.empty(T, C, dtype=torch.bfloat16, device=self.dev)
        w = {"gates": self.rnd(s.blocks, 2, s.M, s.B, s=0.05), "gate_bias": self.rnd(2, C, **f32), "rate": -self.rnd(C, **f32).abs()}
        cw, cb, conv = self.rnd(4, C, **f32), self.rnd(C, **f32), self.rnd(B, 3, C)
        state, bufs = torch.zeros(B, C, device=self.dev), {"summary": torch.empty(G.summary_values(s), device=self.dev)}
        what = f"{B} x {n} prompt" if n > 1 else f"decode {B}"
        self.add(f"convolution, {what}", "tabupel", lambda: G.short_conv(proj[:, C:], cw, cb, conv, rows, u),
                 nbytes=(T * 2 + B * 6) * C * 2)
        a = G.rglru_args(u, proj[:, :C], w, s, state, rows, bufs, out)
        self.add(f"gates + recurrence, {what}", "tabupel", lambda: G.run_rglru(a),
                 nbytes=T * C * 6 + B * C * 8 + 2 * C * s.B * 2, flops=2.0 * T * C * 2 * s.B)
        # the delta rule of as many channels
        H, K, D = max(2, C // 128), max(1, C // 256), 128
        CC = 2 * K * D + H * D
        x, xc, cw2, cst = self.rnd(T, CC), self.rnd(T, CC), self.rnd(CC, 4), self.rnd(B, CC, 3)
        st2, z, core = torch.zeros(B, H, D, D, device=self.dev), self.rnd(T, H * D), torch.empty(T, H * D, dtype=torch.bfloat16, device=self.dev)
        slots, init, nw = rows.state_slots, self.i32([1] * B), self.rnd(D)
        A, dt = self.rnd(H, **f32).abs(), self.rnd(H, **f32)
        if n == 1:
            ab = self.rnd(T, 2 * H)
            self.add(f"convolution, {what}", "qwen3.5", lambda: Q.conv1d_update(x, cw2, cst, slots, xc), nbytes=(T * 2 + B * 6) * CC * 2)

            def theirs():
                Q.packed_decode(xc, ab[:, :H], ab[:, H:], A, dt, st2, slots, core.view(T, H, D), K, H)
                Q.rmsnorm_gated(core, z, nw, core, heads=H)
        else:
            q, k = self.rnd(T, K, D), self.rnd(T, K, D)
            g, beta = -self.rnd(T, H, **f32).abs(), self.rnd(T, H, **f32).abs()
            ws, host = Q.GdnWorkspace(self.dev, T, B, H), [i * n for i in range(B + 1)]
            table = tuple(self.i32(x.tolist()) for x in Q.build_chunk_table(host))
            self.add(f"convolution, {what}", "qwen3.5", lambda: Q.conv1d_fwd(x, cw2, cst, rows.prefill_q_start, slots, init, xc),
                     nbytes=(T * 2 + B * 6) * CC * 2)

            def theirs():
                Q.chunk_scan(q, k, xc, g, beta, st2, host, slots, init, core.view(T, H, D), ws, v_col0=2 * K * D, table=table)
                Q.rmsnorm_gated(core, z, nw, core, heads=H)
        self.add(f"gates + recurrence, {what}", "qwen3.5", theirs,
                 nbytes=T * (2 * K * D + 3 * H * D) * 2 + B * H * D * D * 8, flops=T * H * (6.0 * D * D + 4 * 64 * D) if n > 1 else 0,
                 note="delta rule + norm")

    def rest(self, T):
        from .. import ops
        from ..ops.stream import softcap_f32, stream_norm
        W = self.W
        out, stream, mixed, nw = self.rnd(T, W), self.rnd(T, W, dtype=torch.float32), self.rnd(T, W, dtype=torch.float32), self.rnd(W, dtype=torch.float32)
        self.add(f"residual + norm, {T} tokens", "tabupel",
                 lambda: stream_norm(stream, nw, 1e-6, out, width=W, a=mixed, norm_offset=0.0, mult=0.5), nbytes=T * W * (4 + 4 + 4 + 2))
        o2, res, nwb = torch.empty_like(out), self.rnd(T, W), nw.to(torch.bfloat16)
        self.add(f"residual + norm, {T} tokens", "qwen3.5", lambda: ops.rmsnorm(o2, nwb, 1e-6, residual=res, out=out), nbytes=T * W * 2 * 4)
        if T <= 64:
            logits = self.rnd(T, 32000, dtype=torch.float32)
            self.add(f"logit cap, {T} rows", "tabupel", lambda: softcap_f32(logits, 30.0), nbytes=T * 32000 * 8)


class KubolornKernels(KernelBench):
    def __init__(self, size):
        super().__init__(size)
        self.gh, self.sh = size[8:]

    def run(self):
        self.attention(B=4, prompt=2048, decode_batch=64, ctx=4096)
        self.attention(B=8, prompt=1024, decode_batch=8, ctx=16384)
        for B, n in ((4, 2048), (8, 1024), (1, 8192), (16, 1), (64, 1), (256, 1)):
            self.recurrences(B, n)
        for T in (64, 8192):
            self.rest(T)

    def attention(self, B, prompt, decode_batch, ctx, bs=32):
        from .. import ops
        from ..ops import bias_attn as A
        from ..ops.reference import build_prefill_tiles
        H, G, D = self.H, self.G, self.D
        s, T, nb, scale = A.TiedShape(H, G, D, D // 2), B * prompt, prompt // bs, D ** -0.5
        row = G * s.pitch
        shape = dict(H=H, G=G, kw=row, vdim=s.D, block_size=bs, grouped=True, values_in_keys=True, key_at=s.r8, scale=scale)
        sink = self.rnd(H, dtype=torch.float32)
        bt = torch.arange(1, B * nb + 1, device=self.dev, dtype=torch.int32).view(B, nb)
        tr, tq = (self.i32(x) for x in build_prefill_tiles([prompt] * B))
        rows = dict(seq_lens=self.i32([prompt] * B), q_start=self.i32([i * prompt for i in range(B + 1)]), tile_req=tr, tile_q0=tq)
        q, pages, kv = self.rnd(T, H * D), self.rnd(B * nb + 1, bs * row), self.rnd(B * nb + 1, 2, bs, G, D)
        out = torch.empty(T, H * D, dtype=torch.bfloat16, device=self.dev)
        flops = 2 * B * (prompt * (prompt + 1) / 2) * H * 2 * D
        what = f"attention, {B} x {prompt} prompt"
        self.add(what, "kubolorn", lambda: A.prefill(q, pages, out, block_table=bt, num_reqs=B, sink=sink, **rows, **shape), flops=flops,
                 note=A.kernel_kind("prefill", q, pages, **shape))
        self.add(what, "qwen3.5", lambda: ops.attn_prefill(q, kv, block_table=bt, num_q_heads=H, num_kv_heads=G, head_dim=D, block_size=bs,
                                                           scale=scale, out=out, **rows), flops=flops)
        qk, pos = self.rnd(T, (H + G) * D), torch.arange(T, device=self.dev) % prompt
        slots = (bt.long()[:, :, None] * bs + torch.arange(bs, device=self.dev)).reshape(-1)
        table, qkv, nw = self.rnd(prompt, D, dtype=torch.float32), self.rnd(T, (H + 2 * G) * D), self.rnd(D)
        half = table[:, : D // 2].contiguous()
        what = f"query preparation + cache write, {T} tokens"
        self.add(what, "kubolorn", lambda: A.rotate_tied(qk, pos, half, q, slots, pages, s, block_size=bs),
                 nbytes=T * 2 * ((H + G) * D + H * D + row))
        self.add(what, "qwen3.5", lambda: ops.rope_kv(qkv, pos, table, num_q_heads=H, num_kv_heads=G, head_dim=D, q_norm=nw, k_norm=nw,
                                                      slot_mapping=slots, kv_cache=kv, block_size=bs, q_out=q), nbytes=T * 2 * (H + 2 * G) * D * 2)
        B, nb = decode_batch, ctx // bs
        bt = torch.arange(1, B * nb + 1, device=self.dev, dtype=torch.int32).view(B, nb)
        sl, pages, kv, q = self.i32([ctx] * B), self.rnd(B * nb + 1, bs * row), self.rnd(B * nb + 1, 2, bs, G, D), self.rnd(B, H * D)
        out = torch.empty(B, H * D, dtype=torch.bfloat16, device=self.dev)
        splits = A.grouped_decode_splits(B, G, ctx, ops.num_sms())
        tmp = (torch.empty(B * H * splits * D, dtype=torch.float32, device=self.dev), torch.empty(B * H * splits, dtype=torch.float32, device=self.dev))
        what = f"attention, decode {B} x {ctx}"
        self.add(what, "kubolorn", lambda: A.decode(q, pages, out, block_table=bt, seq_lens=sl, splits=splits, tmp=tmp, sink=sink, **shape),
                 nbytes=B * ctx * row * 2, note=A.kernel_kind("decode", q, pages, **shape))
        self.add(what, "qwen3.5", lambda: ops.attn_decode(q, kv, block_table=bt, seq_lens=sl, num_q_heads=H, num_kv_heads=G, head_dim=D,
                                                          block_size=bs, scale=scale, out=out), nbytes=B * ctx * 2 * G * D * 2)

    def recurrences(self, B, n):
        """``B`` prompts of ``n`` tokens, or (n 1) a decode batch: both recurrences with their norms, and the convolution of the
        state-space mixer; beside the delta rule of as many heads."""
        from types import SimpleNamespace
        from ..ops import gdn as Q
        from ..ops import outer as O
        from ..ops import rglru as R
        from ..ops.reference import build_prefill_tiles
        T, f32, H = B * n, dict(dtype=torch.float32), self.gh
        tr, tq = build_prefill_tiles([n] * B) if n > 1 else ([], [])
        rows = SimpleNamespace(seq_lens=self.i32([n + 5] * B), state_slots=self.i32(list(range(B))),
                               prefill_q_start=self.i32([i * n for i in range(B + 1)]), tile_req=self.i32(tr or [0]),
                               tile_q0=self.i32(tq or [0]), num_decodes=B if n == 1 else 0, num_prefills=0 if n == 1 else B, num_tiles=len(tr))
        what = f"{B} x {n} prompt" if n > 1 else f"decode {B}"

        def buffers(s, kind):
            work = O.Workspace(self.dev, T, B)
            work.reserve(s, kind)
            return {"o": self.rnd(T, s.inner, **f32), **work.allocate()}
        # (a chunk of 64: products with the state, pairs of tokens, their products with v, the update)
        flops = lambda s: T * s.H * (4.0 * s.D * s.V + 64.0 * (s.D + s.V)) if n > 1 else 0.0                # noqa: E731
        s = O.OuterShape(H=H, G=H, dim=128, vdim=128, rank=16)
        proj = self.rnd(T, 4 * H * 128 + 16)
        parts = torch.split(proj, [H * 128] * 4 + [16], 1)
        w = {"a2": self.rnd(H * 128, 16, s=0.25), "a2_bias": self.rnd(H * 128, **f32), "norm": self.rnd(128, **f32)}
        state, out, bufs = torch.zeros(B, H, 128, 128, device=self.dev), self.rnd(T, H * 128), buffers(s, O.CHANNEL)
        self.add(f"linear attention + gated norm, {what}", "kubolorn",
                 lambda: O.gated_linear_attention(*parts, w, s, state, rows, bufs, out, tau=16.0, eps=1e-6),
                 nbytes=T * (5 * H * 128 + 16) * 2 + B * H * 128 * 128 * 8, flops=flops(s))
        m = O.OuterShape(H=self.sh, G=4, dim=128, vdim=64)
        C = m.inner + 2 * m.G * m.D
        row, u, z = self.rnd(T, C + m.inner + 64), self.rnd(T, C), self.rnd(T, m.inner)
        cw, cb, conv = self.rnd(4, C, **f32), self.rnd(C, **f32), self.rnd(B, 3, C)
        self.add(f"convolution, {what}", "kubolorn", lambda: R.short_conv(row[:, m.inner: m.inner + C], cw, cb, conv, rows, u, act="silu"),
                 nbytes=(T * 2 + B * 6) * C * 2)
        wm = {"dt_bias": self.rnd(m.H, **f32), "A": self.rnd(m.H, **f32).abs(), "D": self.rnd(m.H, **f32), "norm": self.rnd(m.inner, **f32)}
        stm, outm, bufm, dt = torch.zeros(B, m.H, 128, 64, device=self.dev), self.rnd(T, m.inner), buffers(m, O.HEAD), row[:, -64:]
        self.add(f"state space + gated norm, {what}", "kubolorn",
                 lambda: O.state_space(u, z, dt, wm, m, stm, rows, bufm, outm, parts=4, eps=1e-6),
                 nbytes=T * (C + 2 * m.inner + m.H) * 2 + B * m.H * 128 * 64 * 8, flops=flops(m))
        K, D = H, 128                                        # the delta rule
        CC = 2 * K * D + H * D
        x, xc, cw2, cst = self.rnd(T, CC), self.rnd(T, CC), self.rnd(CC, 4), self.rnd(B, CC, 3)
        st2, z2, core = torch.zeros(B, H, D, D, device=self.dev), self.rnd(T, H * D), self.rnd(T, H * D)
        slots, init, nw = rows.state_slots, self.i32([1] * B), self.rnd(D)
        A, dtb = self.rnd(H, **f32).abs(), self.rnd(H, **f32)
        if n == 1:
            ab = self.rnd(T, 2 * H)
            self.add(f"convolution, {what}", "qwen3.5", lambda: Q.conv1d_update(x, cw2, cst, slots, xc), nbytes=(T * 2 + B * 6) * CC * 2)

            def theirs():
                Q.packed_decode(xc, ab[:, :H], ab[:, H:], A, dtb, st2, slots, core.view(T, H, D), K, H)
                Q.rmsnorm_gated(core, z2, nw, core, heads=H)
        else:
            q, k = self.rnd(T, K, D), self.rnd(T, K, D)
            g, beta = -self.rnd(T, H, **f32).abs(), self.rnd(T, H, **f32).abs()
            ws, host = Q.GdnWorkspace(self.dev, T, B, H), [i * n for i in range(B + 1)]
            table = tuple(self.i32(x.tolist()) for x in Q.build_chunk_table(host))
            self.add(f"convolution, {what}", "qwen3.5", lambda: Q.conv1d_fwd(x, cw2, cst, rows.prefill_q_start, slots, init, xc),
                     nbytes=(T * 2 + B * 6) * CC * 2)

            def theirs():
                Q.chunk_scan(q, k, xc, g, beta, st2, host, slots, init, core.view(T, H, D), ws, v_col0=2 * K * D, table=table)
                Q.rmsnorm_gated(core, z2, nw, core, heads=H)
        self.add(f"delta rule + gated norm, {what}", "qwen3.5", theirs,
                 nbytes=T * (2 * K * D + 3 * H * D) * 2 + B * H * D * D * 8, flops=T * H * (6.0 * D * D + 4 * 64 * D) if n > 1 else 0)

    def rest(self, T):
        from types import SimpleNamespace
        from .. import ops
        from ..config import BigramSpec
        from ..models.backend import GpuBackend
        from ..ops import conv_norm as N
        from ..ops import moe as M
        from ..ops.reference import build_prefill_tiles
        W, f32, be = self.W, dict(dtype=torch.float32), GpuBackend()
        B, n = (T, 1) if T <= 64 else (4, T // 4)
        tr, tq = build_prefill_tiles([n] * B) if n > 1 else ([], [])
        rows = SimpleNamespace(seq_lens=self.i32([n + 5] * B), state_slots=self.i32(list(range(B))),
                               prefill_q_start=self.i32([i * n for i in range(B + 1)]), tile_req=self.i32(tr or [0]),
                               tile_q0=self.i32(tq or [0]), num_decodes=B if n == 1 else 0, num_prefills=0 if n == 1 else B, num_tiles=len(tr))
        src, dst, mixed = (self.rnd(T, W, **f32) for _ in range(3))
        outs, taps = [self.rnd(T, W), self.rnd(T, W)], [self.rnd(4, W, **f32), self.rnd(4, W, **f32)]
        state = self.rnd(B, 3, W, **f32)
        norm = dict(width=W, groups=4, eps=1e-6)
        o2, res, nwb = self.rnd(T, W), self.rnd(T, W), self.rnd(W)
        what = f"residual + norm, {T} tokens"
        self.add(what, "kubolorn", lambda: N.norm_conv(src, rows, taps, outs, state=state, dst=dst, a=mixed, **norm),
                 nbytes=T * W * (4 + 4 + 4 + 4) + B * W * 24, note="two convolutions more")
        self.add(what, "qwen3.5", lambda: ops.rmsnorm(o2, nwb, 1e-6, residual=res, out=outs[0]), nbytes=T * W * 2 * 4)
        ids, table, big = torch.randint(0, 32000, (T,), device=self.dev), self.rnd(32000, W), self.rnd(32750, W)
        prev, nw = torch.zeros(B, dtype=torch.int64, device=self.dev), self.rnd(W, **f32)
        self.add(f"embedding, {T} tokens", "kubolorn",
                 lambda: N.embed_pairs(src, ids, table, rows, scale=1.0, norm_w=nw, bigram=big, prev=prev, spec=BigramSpec(32749, 31337, 7919),
                                       **norm), nbytes=T * W * 8, note="token pairs and norm")
        self.add(f"embedding, {T} tokens", "qwen3.5", lambda: ops.embedding(ids, table, out=o2), nbytes=T * W * 4)
        x = self.rnd(T, W)
        if not self.E:
            ff, fg = self.ff, self.ff * 2 // 3 // 128 * 128
            up, cat, gu = self.rnd(ff, W, s=0.05), self.rnd(T, ff + W), self.rnd(2 * fg, W, s=0.05)
            act, scratch = self.rnd(T, fg), self.rnd(T, 2 * fg)
            what = f"feed-forward, first product, {T} tokens"
            self.add(what, "kubolorn", lambda: be.plain_unit(x, up, "gelu_tanh", cat[:, W:]), nbytes=(ff * W + T * (W + ff)) * 2, flops=2.0 * T * ff * W)
            self.add(what, "qwen3.5", lambda: be.gated_unit(x, gu, 0, act, scratch), nbytes=(2 * fg * W + T * (W + fg)) * 2, flops=2.0 * T * 2 * fg * W)
            wo, out = self.rnd(W, ff + W, s=0.05), self.rnd(T, W, **f32)
            what = f"feed-forward, second product, {T} tokens"
            self.add(what, "kubolorn", lambda: be.gemm(cat, wo, out=out, out_dtype=torch.float32), nbytes=((ff + W) * W + T * (W + ff)) * 2 + T * W * 4,
                     flops=2.0 * T * (ff + W) * W, note="with the mixer's, fp32")
            wd = self.rnd(W, fg, s=0.05)
            self.add(what, "qwen3.5", lambda: be.gemm(act, wd, out=o2), nbytes=(fg * W + T * (W + fg)) * 2, flops=2.0 * T * fg * W)
            return
        E, top, ff = self.E, self.top, self.ff
        P, fp = T * top, ff * 3 // 2
        ws, wg = M.MoeWorkspace(self.dev, T, top, E, W, fp), M.MoeWorkspace(self.dev, T, top, E, W, ff)
        ids, w = M.router_topk(self.rnd(T, E, **f32), top)
        used, chunks = int(ids.unique().numel()), min(ws.max_chunks, E + (P + 255) // 256)
        wu, wd, wgu, wgd = self.rnd(E, fp, W, s=0.05), self.rnd(E, W, fp, s=0.05), self.rnd(E, 2 * ff, W, s=0.05), self.rnd(E, W, ff, s=0.05)
        for z in (ws, wg):
            M.moe_sort(ids, 0, E, z)
            M.moe_gather(x, z, E, P)
        args = (M.ptr(ws.chunk_expert), M.ptr(ws.chunk_row0), M.ptr(ws.chunk_n), M.ptr(ws.meta), chunks, M.PLAIN["relu2"], M.stream_ptr())
        what = f"experts, first products, {T} tokens"
        self.add(what, "kubolorn", lambda: M.check(M.lib().b200_moe_grouped_gemm_act(M.ptr(ws.xs), P, M.ptr(wu), E, fp, W, M.ptr(ws.act), *args), "gemm"),
                 nbytes=(used * fp * W + P * (W + fp)) * 2, flops=2.0 * P * fp * W)
        self.add(what, "qwen3.5", lambda: M.grouped_gemm_gated(wg.xs, wgu, wg.act, wg, P, chunks), nbytes=(used * 2 * ff * W + P * (W + ff)) * 2,
                 flops=2.0 * P * 2 * ff * W)
        what = f"experts, second products, {T} tokens"
        self.add(what, "kubolorn", lambda: M.grouped_gemm(ws.act, wd, ws.y, ws, P, chunks), nbytes=(used * fp * W + P * (W + fp)) * 2,
                 flops=2.0 * P * fp * W)
        self.add(what, "qwen3.5", lambda: M.grouped_gemm(wg.act, wgd, wg.y, wg, P, chunks), nbytes=(used * ff * W + P * (W + ff)) * 2,
                 flops=2.0 * P * ff * W)
        pos = ws.pair_pos[:P].view(T, top)
        what = f"expert sum + residual + norm, {T} tokens"
        self.add(what, "kubolorn", lambda: N.norm_conv(src, rows, taps, outs, state=state, dst=dst, a=mixed, y=ws.y, pair_pos=pos, pair_w=w, **norm),
                 nbytes=T * W * (4 + 4 + 4 + 4 + 2 * top) + B * W * 24, note="two convolutions more")

        def two():
            M.combine(wg.y, wg, w, o2)
            ops.rmsnorm(o2, nwb, 1e-6, residual=res, out=outs[0])
        self.add(what, "qwen3.5", two, nbytes=T * W * 2 * (top + 1 + 1 + 2 + 1), note="two kernels")


DESIGNS = {"nufusun": (NUFUSUN_SIZES, nufusun_configs, NufusunKernels), "diforax": (DIFORAX_SIZES, diforax_configs, DiforaxKernels),
           "tabupel": (TABUPEL_SIZES, tabupel_configs, TabupelKernels),
           "kubolorn": (KUBOLORN_SIZES, kubolorn_configs, KubolornKernels)}


def run(design="nufusun", sizes=None, kernels=True) -> dict:
    table, configs, bench = DESIGNS[design]
    hbm, tf, how = _peaks()
    res = {"metric": "design_layer_throughput", "unit": "tok/s", "impl": "ours", "design": design, "dtype": "bf16",
           "data": "synthetic (uniform-random prompt ids, random-init weights)",
           "roofline": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": how}, "models": {}, "kernels": {}}
    names = TABUPEL_FIELDS if design == "tabupel" else KUBOLORN_FIELDS if design == "kubolorn" else FIELDS + (("delta_heads", "delta_key_heads") if design == "diforax" else ())
    for name, size in table.items():
        if sizes and name not in sizes:
            continue
        res["models"][name] = {"layers": dict(zip(names, size))}
        for prompt, batch in ((1024, 64), (4096, 16)):
            r = {}
            for who, cfg in configs(size).items():
                r[who] = throughput(cfg, prompt, batch, decode_steps=40, prompt_steps=4)
                torch.cuda.empty_cache()
            res["models"][name][f"prompt {prompt}, decode batch {batch}"] = r
        if kernels:
            k = bench(size)
            k.run()
            res["kernels"][name] = k.rows
            del k
            torch.cuda.empty_cache()
    return res
