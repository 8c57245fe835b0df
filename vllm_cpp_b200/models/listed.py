"""What the families with listed layers (``ModelConfig.blocks``) and per-layer sizes share: padded storage, the
dense feed-forward, caches by block, recurrent state, logits."""
from __future__ import annotations

import torch

from ..config import ModelConfig, ParallelConfig, RopeConfig
from .backend import make_backend
from .base import BufferPool, StepContext
from .dense import ACT_KIND, DenseModel
from .recurrent import RecurrentState
from .rope import rope_parameters


def pad(n: int, m: int = 8) -> int:
    return (n + m - 1) // m * m


def padded(t: torch.Tensor, *shape: int) -> torch.Tensor:
    if tuple(t.shape) == shape:
        return t
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


def pad_heads(t: torch.Tensor, heads: int, padded: int, axis: int = 0) -> torch.Tensor:
    """Each head's rows (or columns) padded with zeros."""
    t = t.transpose(0, axis)
    out = torch.zeros((heads, padded, *t.shape[1:]), dtype=t.dtype, device=t.device)
    out[:, : t.shape[0] // heads] = t.reshape(heads, -1, *t.shape[1:])
    return out.reshape(heads * padded, *t.shape[1:]).transpose(0, axis)


class ListedModel(DenseModel):
    DTYPES = ("bfloat16", "float32")

    def __init__(self, cfg: ModelConfig, device="cuda", parallel: ParallelConfig | None = None,
                 comm=None, max_position: int | None = None):
        # (the dense constructor sets up the one rotary table and the shards of uniform layers)
        self.cfg, self.device = cfg, torch.device(device)
        self.par = parallel or ParallelConfig()
        if self.par.tensor_parallel_size > 1:
            raise ValueError(f"{cfg.architecture} runs on one rank")
        self.tp, self.rank, self.comm = 1, 0, comm
        self.be = make_backend(self.device)
        self.dtype = torch.float32 if cfg.dtype == "float32" else torch.bfloat16
        self.hq, self.hkv, self.D = cfg.num_heads, cfg.num_kv_heads, pad(cfg.head_dim, 16)
        self.max_position = max_position or cfg.max_position_embeddings
        self.width, self.cols = cfg.hidden_size, pad(cfg.hidden_size)
        self.vocab_shard, self.vocab_start = cfg.vocab_size, 0
        self.bufs = BufferPool(self.device)
        self.recurrent = RecurrentState()
        self.state: dict[int, tuple] = {}
        self.rope: dict[tuple, torch.Tensor] = {}
        self.w: dict[str, torch.Tensor] = {}
        self.layers: list[dict] = []

    def quantize_weights(self, method: str = "nvfp4") -> None:
        raise ValueError(f"{self.cfg.architecture} checkpoints are served in bfloat16 or float32")

    def fused_tp_supported(self) -> bool:
        return False

    # ------------------------------------------------------------------ weights
    def put(self, t: torch.Tensor, *shape: int, dtype=None) -> torch.Tensor:
        """On the device in the model's type (or ``dtype``), padded with zeros to ``shape``."""
        return padded(t.to(self.device, dtype or self.dtype), *(shape or t.shape)).contiguous()

    def _take_shared(self, name: str, t: torch.Tensor) -> bool:
        """The tensors that belong to no block."""
        if name == "embed":
            self.w["embed"] = self.put(t, t.shape[0], self.cols)
        elif name == "head":
            self.w["lm_head"] = self.put(t, pad(t.shape[0]), self.cols)
        elif name == "final.norm":
            self.w["final_norm"] = self.put(t, self.cols, dtype=torch.float32)
        else:
            return False
        return True

    def _block_of(self, name: str) -> tuple[int, str]:
        """(block, rest of the name) of a block's tensor."""
        layer, _, rest = name.partition(".")
        if not (layer.startswith("l") and layer[1:].isdigit() and int(layer[1:]) < len(self.cfg.blocks)):
            raise ValueError(f"unexpected tensor {name!r}")
        return int(layer[1:]), rest

    @staticmethod
    def _expect(l: int, want: set, have: set) -> None:
        if want != have:
            raise ValueError(f"layer {l}: tensors missing from the checkpoint {sorted(want - have)}, "
                             f"unexpected {sorted(have - want)}")

    def _expect_shared(self) -> None:
        for k in ("embed", "lm_head", "final_norm"):
            if k not in self.w:
                raise ValueError(f"{k} is missing from the checkpoint")

    def _bf16_kernels(self) -> bool:
        return self.device.type == "cuda" and self.dtype == torch.bfloat16

    def _ff_padded(self, ff: int) -> int:
        """(the gated product takes gate and up rows in blocks of 128)"""
        return pad(ff, 128 if self._bf16_kernels() else 8)

    def _load_dense(self, L: dict, f, p: dict) -> None:
        ff = self._ff_padded(f.ff)
        gate, up = (self.put(p["mlp." + n], ff, self.cols) for n in ("gate", "up"))
        if self._bf16_kernels():
            from ..ops import interleave_gate_up
            L["gate_up"] = interleave_gate_up(gate, up).contiguous()
        else:
            L["gate_up"] = torch.cat([gate, up], 0)
        L["down"] = self.put(p["mlp.down"], self.cols, ff)

    def _rope_table(self, base, dims, scaling):
        """Table of one rotation; blocks with the same rotation share it."""
        if not dims:
            return None
        key = (base, dims, repr(scaling))
        if key not in self.rope:
            cfg = scaling.rope(base, dims) if scaling is not None else RopeConfig(theta=base, rotary_dim=dims)
            inv, magnitude, _ = rope_parameters(cfg, dims, self.max_position)
            self.rope[key] = self.be.rope_table(inv, self.max_position + 8, magnitude)
        return self.rope[key]

    # ------------------------------------------------------------------ state
    def snapshot_state(self, slots: list) -> None:
        self.recurrent.snapshot(slots)

    def restore_state(self, slots: list) -> None:
        self.recurrent.restore(slots)

    # ------------------------------------------------------------------ buffers and forward
    def _reserve_rows(self, max_tokens: int, max_reqs: int) -> None:
        self.bufs.reserve("stream", max_tokens, self.cols, torch.float32)
        self.bufs.reserve("mixed", max_tokens, self.cols, torch.float32)
        self.bufs.reserve("normed", max_tokens, self.cols, self.dtype)
        self.bufs.reserve("last", max_reqs, self.cols, self.dtype)
        self.bufs.reserve("logits", max_reqs, pad(self.cfg.vocab_size), torch.float32)

    def _dense_buffers(self, f, T: int):
        ff = self._ff_padded(f.ff)
        return (self.bufs.get(f"act{ff}", T, ff, self.dtype), self.bufs.get(f"gate_up{ff}", T, 2 * ff, self.dtype))

    def _dense(self, h, L: dict, f, act_name: str, T: int, out):
        act, gate_up = self._dense_buffers(f, T)
        self.be.gated_unit(h, L["gate_up"], ACT_KIND[act_name], act, gate_up)
        return self.be.gemm(act, L["down"], out=out, out_dtype=torch.float32)

    def _logits(self, ctx: StepContext, h) -> torch.Tensor:
        """fp32 logits ``[num_logits, vocab]`` of the normed rows asked for in ``ctx.logits_indices``."""
        if ctx.decode_only_full_logits:
            n, last = ctx.num_tokens, h
        else:
            n = ctx.num_logits
            last = self.be.gather_rows(h, ctx.logits_indices[:n], out=self.bufs.get("last", n, self.cols, self.dtype))
        logits = self.bufs.get("logits", n, self.w["lm_head"].shape[0], torch.float32)
        self.be.gemm(last, self.w["lm_head"], out=logits, out_dtype=torch.float32)
        if self.cfg.final_logit_softcap > 0:
            self.be.softcap_f32(logits, self.cfg.final_logit_softcap)
        return logits[:, : self.cfg.vocab_size]
