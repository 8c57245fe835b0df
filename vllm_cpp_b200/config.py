"""Typed configuration: model architecture (from a HF ``config.json`` or a named synthetic
shape), engine arguments and the parallel layout.

Reference surface: ``include/vllm/transformers_utils/hf_config.h`` (typed config incl.
``text_config`` nesting and RoPE parameter normalisation), ``include/vllm/entrypoints/
model_loader.h:36-75`` (EngineParams) and ``include/vllm/config/scheduler.h``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Any, Optional


@dataclass
class RopeConfig:
    theta: float = 10000.0
    rotary_dim: Optional[int] = None          # None => head_dim
    neox: bool = True                         # False => GPT-J (interleaved pairs)
    scaling_type: Optional[str] = None        # llama3 | yarn | deepseek_yarn | linear | dynamic | longrope | mrope
    factor: float = 1.0
    low_freq_factor: float = 1.0
    high_freq_factor: float = 4.0
    original_max_position: int = 8192
    beta_fast: float = 32.0
    beta_slow: float = 1.0
    mscale: float = 1.0
    mscale_all_dim: float = 0.0
    attn_factor: float = 1.0
    short_factor: Optional[list] = None       # longrope
    long_factor: Optional[list] = None
    mrope_section: Optional[list] = None
    alpha: Optional[float] = None             # dynamic NTK alpha
    config_max_position: int = 0              # the checkpoint's max_position_embeddings (longrope magnitude scale)
    short_mscale: Optional[float] = None      # longrope: explicit magnitude scales, when the checkpoint gives them
    long_mscale: Optional[float] = None
    truncate: bool = True                     # YaRN: round the correction range outward to whole dimensions
    extrapolation_factor: float = 1.0         # YaRN: weight of the unscaled frequencies inside the ramp
    apply_yarn_scaling: bool = True           # YaRN: False keeps only attn_factor as the magnitude scale


@dataclass
class RotaryScaling:
    """Frequencies divided by ``factor``; with ``original`` (the length before scaling) YaRN, which divides the
    slow ones only: those of at most ``slow`` turns within it, ramped up to ``fast`` turns."""
    factor: float
    original: float = 0
    fast: float = 32.0
    slow: float = 1.0

    def rope(self, base: float, dims: int) -> RopeConfig:
        import math
        if not self.original:
            return RopeConfig(theta=base, rotary_dim=dims, scaling_type="linear", factor=self.factor)
        return RopeConfig(theta=base, rotary_dim=dims, scaling_type="yarn", factor=self.factor,
                          original_max_position=self.original, beta_fast=self.fast, beta_slow=self.slow,
                          apply_yarn_scaling=False, attn_factor=0.1 * math.log(self.factor) + 1.0)


@dataclass
class AttentionSpec:
    """Softmax mixer of one decoder block: grouped heads with separate key and value sizes. Positions
    enter through a distance bias that saturates at ``bias_max`` (0: none) or a rotation of the first
    ``rot_dims`` dimensions (0: none). With ``diff`` every head has two maps over the same values and
    subtracts the second, weighted by a learned number that starts around ``diff``. ``sink``: a learned
    number per head whose exponential joins the softmax's denominator; ``tied``: the values are the keys
    before their rotation."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: int = 0
    rot_dims: int = 0
    rot_base: float = 10000.0
    chunk: int = 0                            # > 0: a query sees the keys of its own chunk of this many positions
    kv_from: Optional[int] = None             # block whose keys and values are read (None: its own)
    window: int = 0                           # > 0: a query sees itself and the window - 1 positions before it
    rot_scaling: Optional[RotaryScaling] = None
    diff: Optional[float] = None
    sink: bool = False
    tied: bool = False


@dataclass
class LatentSpec:
    """Latent softmax mixer of one decoder block: ``heads`` heads whose keys (``dim``) and values (``vdim``)
    are projections of one normed latent of ``kv_rank`` values per token, beside ``rot_dim`` rotated key
    dimensions shared by the heads; queries come from a normed latent of ``q_rank`` values; each head's output
    has a sigmoid gate."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int = 0
    rot_base: float = 10000.0
    rot_scaling: Optional[RotaryScaling] = None


@dataclass
class RglruSpec:
    """Real-gated linear recurrent mixer of one decoder block: ``width`` channels behind a short convolution of
    ``conv`` taps, gates from ``blocks`` square matrices over equal parts of them."""
    width: int
    blocks: int
    conv: int


@dataclass
class DeltaSpec:
    """Gated-delta-rule mixer of one decoder block: ``heads`` states of ``dim`` x ``vdim``, queries and
    keys shared by ``heads / kv_heads`` heads each, short convolutions of ``conv`` taps."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass
class GlaSpec:
    """Gated-linear-attention mixer of one decoder block: ``heads`` states of ``dim`` x ``vdim`` whose key
    channels fade by sigmoid(z)^(1 / ``tau``), z a product of rank ``rank`` (a checkpoint's tensors say which)."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 16


@dataclass
class SsmSpec:
    """State-space mixer (Mamba-2) of one decoder block: ``heads`` states of ``state`` x ``vdim``, input and
    output vectors shared by ``heads / groups`` heads each, a short convolution of ``conv`` taps, the gated output
    normed in ``norm_groups`` equal parts."""
    heads: int
    groups: int
    state: int
    vdim: int
    conv: int
    norm_groups: int


@dataclass
class DenseSpec:
    """Feed-forward of one decoder block: one gated unit, or with ``plain`` one ungated unit with that
    activation."""
    ff: int
    plain: Optional[str] = None


@dataclass
class ExpertSpec:
    """Feed-forward of one decoder block: ``top`` of ``experts`` gated units (clamped at ``limit``) and
    ``identity`` experts that return their input; the choice is made among the ``keep`` best of
    ``groups`` groups of neighbours."""
    experts: int
    top: int
    ff: int
    limit: float = float("inf")
    identity: int = 0
    groups: int = 1
    keep: int = 1
    plain: Optional[str] = None


@dataclass
class BlockSpec:
    attention: Optional[AttentionSpec] = None
    mlp: "Optional[ExpertSpec | DenseSpec]" = None
    delta: Optional[DeltaSpec] = None         # set instead of ``attention``, as the next two
    latent: Optional[LatentSpec] = None
    rglru: Optional[RglruSpec] = None
    weights_of: Optional[int] = None          # block whose weights this one runs with (None: its own)
    gla: Optional[GlaSpec] = None             # set instead of ``attention``
    ssm: Optional[SsmSpec] = None             # beside ``attention``: the sum of both, times ``scales``
    scales: tuple = (1.0, 1.0)
    layer: Optional[int] = None               # number of its tensors in the checkpoint (None: its place)

    @property
    def mixer(self):
        return self.attention or self.delta or self.latent or self.rglru or self.gla or self.ssm


@dataclass
class BigramSpec:
    """Embedding of token pairs: row (before * ``mul_prev`` + token * ``mul_cur``) mod ``buckets`` of a table, row
    ``buckets`` for a first token."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class LoopSpec:
    """Layers ``start`` .. ``stop`` - 1 run ``times`` times in a row with the same weights."""
    start: int
    stop: int
    times: int


@dataclass
class ModelConfig:
    architecture: str = "LlamaForCausalLM"
    vocab_size: int = 32000
    hidden_size: int = 4096
    intermediate_size: int = 11008
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 32
    head_dim: int = 128
    rms_norm_eps: float = 1e-6
    max_position_embeddings: int = 8192
    tie_word_embeddings: bool = False
    rope: RopeConfig = field(default_factory=RopeConfig)
    qk_norm: bool = False                     # per-head RMSNorm on q and k (Qwen3)
    attention_bias: bool = False
    mlp_bias: bool = False
    hidden_act: str = "silu"
    sliding_window: int = 0
    attention_chunk_size: int = 0             # chunked-local attention ("chunked_attention" layers)
    # layer pattern / extras for the non-plain families
    layer_types: Optional[list] = None        # per-layer "full_attention" | "sliding_attention" | "chunked_attention" | "linear_attention"
    attn_logit_softcap: float = 0.0
    final_logit_softcap: float = 0.0
    embed_scale: float = 1.0
    gemma_norm: bool = False                  # (1 + w) RMSNorm weights
    sandwich_norm: bool = False               # post-attention / post-mlp norms (Gemma2/3, GLM4)
    post_norm: bool = False                   # OLMo2-style: norm after the block, not before
    residual_multiplier: float = 1.0          # Granite
    attention_multiplier: Optional[float] = None
    logits_scaling: float = 1.0
    # MoE
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True
    num_shared_experts: int = 0
    shared_expert_intermediate_size: int = 0
    shared_expert_gate: bool = False
    first_k_dense_replace: int = 0
    routed_scaling_factor: float = 1.0
    scoring_func: str = "softmax"
    topk_method: str = "greedy"
    n_group: int = 1
    mtp_num_hidden_layers: int = 0            # decoder blocks of the multi-token-prediction head (0: none in the checkpoint)
    topk_group: int = 1
    # MLA
    kv_lora_rank: int = 0
    q_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    # Gated DeltaNet (Qwen3.5 / 3.6)
    linear_num_key_heads: int = 0
    linear_num_value_heads: int = 0
    linear_key_head_dim: int = 0
    linear_value_head_dim: int = 0
    linear_conv_kernel_dim: int = 4
    full_attention_interval: int = 4
    attn_output_gate: bool = False
    partial_rotary_factor: float = 1.0
    # quantisation
    quant: Optional[str] = None               # None | "nvfp4" | "fp8"
    dtype: str = "bfloat16"
    eos_token_id: Optional[int] = None
    bos_token_id: Optional[int] = None
    # block-by-block sizes of the families whose config.json lists every layer (None: uniform)
    blocks: Optional[list] = None
    norm_groups: int = 1                      # norms divide this many equal parts of a row each by its own rms
    input_conv: int = 0                       # taps of the convolution over what a sublayer reads (0: none)
    bigram: Optional[BigramSpec] = None
    loop: Optional[LoopSpec] = None           # (already unrolled in ``blocks``)
    raw: dict = field(default_factory=dict)

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0

    @property
    def is_hybrid(self) -> bool:
        return bool(self.layer_types) and "linear_attention" in self.layer_types


def _rope_from_hf(cfg: dict, head_dim: int) -> RopeConfig:
    r = RopeConfig(theta=float(cfg.get("rope_theta", 10000.0)))
    prf = cfg.get("partial_rotary_factor")
    if prf is not None and prf < 1.0:
        r.rotary_dim = int(head_dim * prf)
    rs = cfg.get("rope_scaling") or cfg.get("rope_parameters") or None
    if rs:
        if "rope_theta" in rs:
            r.theta = float(rs["rope_theta"])
        if "partial_rotary_factor" in rs and rs["partial_rotary_factor"] < 1.0:
            r.rotary_dim = int(head_dim * rs["partial_rotary_factor"])
        t = rs.get("rope_type", rs.get("type"))
        if t and t != "default":
            r.scaling_type = t
        r.factor = float(rs.get("factor", 1.0))
        r.low_freq_factor = float(rs.get("low_freq_factor", 1.0))
        r.high_freq_factor = float(rs.get("high_freq_factor", 4.0))
        # Phi-3 keeps the original window beside rope_scaling, not inside it
        r.original_max_position = int(rs.get("original_max_position_embeddings",
                                             cfg.get("original_max_position_embeddings",
                                                     cfg.get("max_position_embeddings", 8192))))
        r.config_max_position = int(cfg.get("max_position_embeddings", 0) or 0)
        r.beta_fast = float(rs.get("beta_fast", 32.0))
        r.beta_slow = float(rs.get("beta_slow", 1.0))
        r.mscale = float(rs.get("mscale", 1.0))
        r.mscale_all_dim = float(rs.get("mscale_all_dim", 0.0))
        r.attn_factor = float(rs.get("attn_factor", 1.0))
        r.short_factor = rs.get("short_factor")
        r.long_factor = rs.get("long_factor")
        r.mrope_section = rs.get("mrope_section")
        r.alpha = rs.get("alpha")
        r.short_mscale, r.long_mscale = rs.get("short_mscale"), rs.get("long_mscale")
        r.truncate = bool(rs.get("truncate", True))
        r.extrapolation_factor = float(rs.get("extrapolation_factor", 1.0))
        r.apply_yarn_scaling = bool(rs.get("apply_yarn_scaling", True))
    return r


def model_config_from_hf(cfg: dict) -> ModelConfig:
    """Builds a ModelConfig from a HF ``config.json`` dict (``text_config`` nesting honoured)."""
    arch = (cfg.get("architectures") or ["LlamaForCausalLM"])[0]
    t = dict(cfg)
    if "text_config" in cfg:
        t.update(cfg["text_config"])
    hidden = int(t["hidden_size"])
    heads = int(t["num_attention_heads"])
    head_dim = int(t.get("head_dim") or hidden // heads)
    m = ModelConfig(
        architecture=arch, vocab_size=int(t["vocab_size"]), hidden_size=hidden,
        intermediate_size=int(t.get("intermediate_size", 4 * hidden)),
        num_layers=int(t["num_hidden_layers"]), num_heads=heads,
        num_kv_heads=int(t.get("num_key_value_heads", heads)), head_dim=head_dim,
        rms_norm_eps=float(t.get("rms_norm_eps", t.get("layer_norm_eps", 1e-6))),
        max_position_embeddings=int(t.get("max_position_embeddings", 8192)),
        tie_word_embeddings=bool(t.get("tie_word_embeddings", False)),
        rope=_rope_from_hf(t, head_dim), attention_bias=bool(t.get("attention_bias", False)),
        mlp_bias=bool(t.get("mlp_bias", False)), hidden_act=t.get("hidden_act", "silu"),
        sliding_window=int(t.get("sliding_window") or 0), layer_types=t.get("layer_types"),
        attention_chunk_size=int(t.get("attention_chunk_size") or 0),
        raw=cfg)
    eos = t.get("eos_token_id")
    m.eos_token_id = eos[0] if isinstance(eos, list) else eos
    m.bos_token_id = t.get("bos_token_id")
    a = arch
    if a in ("Qwen3ForCausalLM", "Qwen3MoeForCausalLM"):
        m.qk_norm = True
    if a in ("Qwen3MoeForCausalLM",):
        m.num_experts = int(t["num_experts"])
        m.num_experts_per_tok = int(t["num_experts_per_tok"])
        m.moe_intermediate_size = int(t["moe_intermediate_size"])
        m.norm_topk_prob = bool(t.get("norm_topk_prob", True))
    if a in ("DeepseekV2ForCausalLM", "DeepseekV3ForCausalLM", "Glm4MoeLiteForCausalLM"):
        m.kv_lora_rank = int(t["kv_lora_rank"])
        m.q_lora_rank = int(t.get("q_lora_rank") or 0)
        m.qk_nope_head_dim = int(t["qk_nope_head_dim"])
        m.qk_rope_head_dim = int(t["qk_rope_head_dim"])
        m.v_head_dim = int(t["v_head_dim"])
        m.num_experts = int(t.get("n_routed_experts", 0))
        m.num_experts_per_tok = int(t.get("num_experts_per_tok", 0))
        m.moe_intermediate_size = int(t.get("moe_intermediate_size", 0))
        m.num_shared_experts = int(t.get("n_shared_experts") or 0)
        m.first_k_dense_replace = int(t.get("first_k_dense_replace", 0))
        m.routed_scaling_factor = float(t.get("routed_scaling_factor", 1.0))
        m.norm_topk_prob = bool(t.get("norm_topk_prob", False))
        m.scoring_func = t.get("scoring_func", "softmax")
        m.topk_method = t.get("topk_method", "greedy")
        m.n_group = int(t.get("n_group") or 1)
        m.mtp_num_hidden_layers = int(t.get("mtp_num_hidden_layers") or 0)
        m.topk_group = int(t.get("topk_group") or 1)
        m.rope.neox = False
        if m.rope.scaling_type == "yarn":
            m.rope.scaling_type = "deepseek_yarn"
    if a.startswith("Gemma"):
        m.gemma_norm = True
        m.embed_scale = hidden ** 0.5
        m.hidden_act = "gelu_tanh"
        m.attn_logit_softcap = float(t.get("attn_logit_softcapping") or 0.0)
        m.final_logit_softcap = float(t.get("final_logit_softcapping") or 0.0)
        m.sandwich_norm = a in ("Gemma2ForCausalLM", "Gemma3ForCausalLM")
        m.qk_norm = a == "Gemma3ForCausalLM"
        if t.get("query_pre_attn_scalar"):
            m.attention_multiplier = float(t["query_pre_attn_scalar"]) ** -0.5
        m.tie_word_embeddings = True
    if a == "GraniteForCausalLM":
        m.residual_multiplier = float(t.get("residual_multiplier", 1.0))
        m.attention_multiplier = float(t.get("attention_multiplier", head_dim ** -0.5))
        m.embed_scale = float(t.get("embedding_multiplier", 1.0))
        m.logits_scaling = float(t.get("logits_scaling", 1.0))
    if a in ("Olmo2ForCausalLM", "Olmo3ForCausalLM"):
        m.post_norm = True
        m.qk_norm = True
    if a in ("Glm4ForCausalLM",):
        m.sandwich_norm = True
        m.rope.neox = False
        m.attention_bias = bool(t.get("attention_bias", True))
    if a in ("Qwen3_5ForConditionalGeneration", "Qwen3_5MoeForConditionalGeneration",
             "Qwen3NextForCausalLM"):
        m.qk_norm = True
        m.gemma_norm = True
        m.attn_output_gate = True
        m.linear_num_key_heads = int(t.get("linear_num_key_heads", 16))
        m.linear_num_value_heads = int(t.get("linear_num_value_heads", 32))
        m.linear_key_head_dim = int(t.get("linear_key_head_dim", 128))
        m.linear_value_head_dim = int(t.get("linear_value_head_dim", 128))
        m.linear_conv_kernel_dim = int(t.get("linear_conv_kernel_dim", 4))
        m.full_attention_interval = int(t.get("full_attention_interval", 4))
        if not m.layer_types:
            m.layer_types = ["full_attention" if (i + 1) % m.full_attention_interval == 0
                             else "linear_attention" for i in range(m.num_layers)]
        if "num_experts" in t and t["num_experts"]:
            m.num_experts = int(t["num_experts"])
            m.num_experts_per_tok = int(t["num_experts_per_tok"])
            m.moe_intermediate_size = int(t["moe_intermediate_size"])
            m.shared_expert_intermediate_size = int(t.get("shared_expert_intermediate_size", 0))
            m.num_shared_experts = 1 if m.shared_expert_intermediate_size else 0
            m.shared_expert_gate = True
    q = t.get("quantization_config") or {}
    if q:
        method = (q.get("quant_method") or "").lower()
        algo = (q.get("quant_algo") or "").lower()
        if "nvfp4" in json.dumps(q).lower() or algo == "nvfp4":
            m.quant = "nvfp4"
        elif method == "fp8" or algo == "fp8":
            m.quant = "fp8"
    return m


def model_config_from_blocks(cfg: dict) -> ModelConfig:
    """ModelConfig of a config.json that names one ``architecture`` and lists its ``layers``, each
    with a mixer and a feed-forward (or null)."""
    arch = cfg["architecture"]
    readers = {"Nufusun": _nufusun_block, "Diforax": _diforax_block, "Tabupel": _tabupel_block, "Kubolorn": _kubolorn_block}
    if arch not in readers:
        raise ValueError(f"no reader for the layer list of architecture {arch!r}")
    blocks = []
    for i, l in enumerate(cfg["layers"]):
        try:
            blocks.append(_checked(readers[arch](l), blocks))
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    loop = LoopSpec(**{k: int(cfg["loop"][k]) for k in ("start", "stop", "times")}) if cfg.get("loop") else None
    if loop is not None:
        blocks = unrolled(blocks, loop)
    for i, b in enumerate(blocks):
        if b.weights_of is not None:
            src = blocks[b.weights_of] if 0 <= b.weights_of < len(blocks) else None
            if src is None or src.weights_of is not None:
                raise ValueError(f"layer {i}: block {b.weights_of} has no weights of its own")
            if (src.mixer, src.mlp) != (b.mixer, b.mlp):
                raise ValueError(f"layer {i}: block {b.weights_of}, whose weights it uses, has other sizes")
    kw = dict(vocab=int(cfg["vocab"]), width=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), raw=cfg)
    if arch in ("Nufusun", "Kubolorn"):
        kw["embed_scale"] = float(cfg["embedding"]["scale"])
    if arch == "Kubolorn":
        bigram = cfg["embedding"].get("bigram")
        kw.update(norm_groups=int(cfg["norm"].get("groups") or 1), loop=loop,
                  input_conv=int((cfg.get("canon") or {}).get("taps") or 0),
                  bigram=BigramSpec(**{k: int(bigram[k]) for k in ("buckets", "mul_prev", "mul_cur")}) if bigram else None)
    if arch == "Tabupel":
        kw.update(residual_mult=float(cfg["residual_mult"]), logit_softcap=float(cfg["logit_softcap"]))
    m = model_config_of_blocks(arch, blocks, **kw)
    m.eos_token_id, m.bos_token_id = cfg.get("eos_token_id"), cfg.get("bos_token_id")
    return m


def _nufusun_block(l: dict) -> BlockSpec:
    if l["type"] != "attention":
        raise ValueError(f"unknown mixer {l['type']!r}")
    m, mlp = l["mixer"], None
    att = AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                        scale=float(m["scale"]), bias_max=int(m["bias_max"]))
    if l.get("mlp") is not None:
        f = l["mlp"]
        if f["kind"] != "moe":
            raise ValueError(f"unknown feed-forward {f['kind']!r}")
        mlp = ExpertSpec(experts=int(f["router"]["experts"]), top=int(f["router"]["top"]), ff=int(f["expert"]["ff"]),
                         limit=float(f["expert"]["limit"]))
    return BlockSpec(att, mlp)


def _diforax_block(l: dict) -> BlockSpec:
    m, f = l["mixer"], l.get("mlp")
    sizes = {k: int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim")}
    att = delta = mlp = None
    if l["type"] == "delta":
        delta = DeltaSpec(**sizes, conv=int(m["conv"]))
    elif l["type"] == "attention":
        rot, mask = m.get("rot") or {}, m.get("mask") or {}
        att = AttentionSpec(**sizes, scale=float(m["scale"]), rot_dims=int(rot.get("dims", 0)),
                            rot_base=float(rot.get("base", 1.0)), chunk=int(mask.get("size", 0)),
                            kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
    else:
        raise ValueError(f"unknown mixer {l['type']!r}")
    if f is not None and f["kind"] == "dense":
        mlp = DenseSpec(ff=int(f["ff"]))
    elif f is not None and f["kind"] == "moe":
        r = f["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        mlp = ExpertSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(f["expert"]["ff"]),
                         identity=int(r.get("identity") or 0), groups=int(g["count"]), keep=int(g["keep"]))
    elif f is not None:
        raise ValueError(f"unknown feed-forward {f['kind']!r}")
    return BlockSpec(att, mlp, delta)


def _tabupel_block(l: dict) -> BlockSpec:
    m, f, att, latent, rglru, mlp = l["mixer"], l.get("mlp"), None, None, None, None
    rot, mask = m.get("rot") or {}, m.get("mask") or {}
    scaling = rot.get("scaling")
    if scaling is not None:
        scaling = RotaryScaling(**{k: float(v) for k, v in scaling.items() if k in ("factor", "original", "fast", "slow")})
    where = dict(window=int(mask.get("size", 0)), rot_base=float(rot.get("base", 1.0)), rot_scaling=scaling)
    if l["type"] == "attention":
        att = AttentionSpec(**{k: int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim")}, scale=float(m["scale"]),
                            rot_dims=int(rot.get("dims", 0)), diff=float(m["diff"]), **where)
    elif l["type"] == "latent_attention":
        latent = LatentSpec(**{k: int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")},
                            scale=float(m["scale"]), **where)
        if int(rot.get("dims", latent.rot_dim)) != latent.rot_dim:
            raise ValueError(f"{rot['dims']} rotated dimensions of {latent.rot_dim}")
    elif l["type"] == "rglru":
        rglru = RglruSpec(**{k: int(m[k]) for k in ("width", "blocks", "conv")})
    else:
        raise ValueError(f"unknown mixer {l['type']!r}")
    if f is not None:
        if f["kind"] != "dense":
            raise ValueError(f"unknown feed-forward {f['kind']!r}")
        mlp = DenseSpec(ff=int(f["ff"]))
    src = l.get("weights_of")
    return BlockSpec(att, mlp, latent=latent, rglru=rglru, weights_of=None if src is None else int(src))


def _kubolorn_block(l: dict) -> BlockSpec:
    m, f, mlp = l["mixer"], l.get("mlp"), None
    if f is not None and f["kind"] == "dense":
        mlp = DenseSpec(ff=int(f["ff"]), plain="gelu_tanh")
    elif f is not None and f["kind"] == "moe":
        mlp = ExpertSpec(experts=int(f["router"]["experts"]), top=int(f["router"]["top"]), ff=int(f["expert"]["ff"]), plain="relu2")
    elif f is not None:
        raise ValueError(f"unknown feed-forward {f['kind']!r}")
    if l["type"] == "gla":
        return BlockSpec(None, mlp, gla=GlaSpec(**{k: int(m[k]) for k in ("heads", "dim", "vdim")}, tau=float(m["tau"])))
    if l["type"] != "parallel":
        raise ValueError(f"unknown mixer {l['type']!r}")
    a, r, rot = m["left"], m["right"], m["left"].get("rot") or {}
    if int(a.get("vdim", a["dim"])) != int(a["dim"]):
        raise ValueError(f"values that are keys of {a['dim']} cannot have {a['vdim']}")
    scaling = rot.get("scaling")
    if scaling is not None:
        scaling = RotaryScaling(**{k: float(scaling[k]) for k in ("factor", "original", "fast", "slow")})
    att = AttentionSpec(**{k: int(a[k]) for k in ("heads", "kv_heads", "dim")}, vdim=int(a["dim"]), scale=float(a["scale"]),
                        rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 1.0)), rot_scaling=scaling, sink=True,
                        tied=True)
    ssm = SsmSpec(**{k: int(r[k]) for k in ("heads", "groups", "state", "vdim", "conv", "norm_groups")})
    return BlockSpec(att, mlp, ssm=ssm, scales=(float(m["left_scale"]), float(m["right_scale"])))


def unrolled(blocks: list, loop: LoopSpec) -> list:
    """The blocks in the order they run; a pass after the first runs with the first one's weights."""
    from dataclasses import replace
    a, b, n = loop.start, loop.stop, loop.times
    if not (0 <= a < b <= len(blocks) and n >= 1):
        raise ValueError(f"layers {a} .. {b - 1} of {len(blocks)} cannot run {n} times")
    order = list(range(a)) + list(range(a, b)) * n + list(range(b, len(blocks)))
    first = {l: order.index(l) for l in order}
    return [replace(blocks[l], layer=l, weights_of=None if first[l] == i else first[l]) for i, l in enumerate(order)]


def _checked(b: BlockSpec, before: list) -> BlockSpec:
    """The sizes of a block fit together (``before``: the blocks ahead of it)."""
    m, a, f, lat = b.mixer, b.attention, b.mlp, b.latent
    if (a or b.delta) is not None and m.heads % m.kv_heads:
        raise ValueError(f"{m.heads} heads do not divide into {m.kv_heads} groups")
    if a is not None and (a.rot_dims % 2 or a.rot_dims > a.dim):
        raise ValueError(f"{a.rot_dims} rotated dimensions of {a.dim}")
    if lat is not None and lat.rot_dim % 2:
        raise ValueError(f"{lat.rot_dim} rotated dimensions")
    if (b.delta or b.rglru or b.ssm) is not None and (b.ssm or m).conv < 1:
        raise ValueError("a convolution has at least one tap")
    r = b.ssm
    if r is not None and (r.heads % r.groups or r.heads * r.vdim % r.norm_groups):
        raise ValueError(f"{r.heads} heads of {r.vdim} do not divide into {r.groups} groups and {r.norm_groups} normed parts")
    if b.rglru is not None and m.width % m.blocks:
        raise ValueError(f"{m.width} channels do not divide into {m.blocks} blocks")
    if a is not None and a.kv_from is not None:
        src = before[a.kv_from].attention if 0 <= a.kv_from < len(before) else None
        if src is None or src.kv_from is not None:
            raise ValueError(f"block {a.kv_from} has no keys of its own to read")
        if (src.kv_heads, src.dim, src.vdim) != (a.kv_heads, a.dim, a.vdim):
            raise ValueError(f"the keys of block {a.kv_from} have other sizes")
    if isinstance(f, ExpertSpec):
        n = f.experts + f.identity
        if n % f.groups or not 1 <= f.keep <= f.groups:
            raise ValueError(f"{n} experts in {f.groups} groups, {f.keep} kept")
        if not 1 <= f.top <= n // f.groups * f.keep:
            raise ValueError(f"{f.top} of {n // f.groups * f.keep} experts")
    return b


def model_config_of_blocks(arch: str, blocks: list, *, vocab: int, width: int, eps: float, embed_scale: float = 1.0,
                           residual_mult: float = 1.0, logit_softcap: float = 0.0, max_position: int = 32768,
                           norm_groups: int = 1, input_conv: int = 0, bigram: Optional[BigramSpec] = None,
                           loop: Optional[LoopSpec] = None, raw: Optional[dict] = None) -> ModelConfig:
    att = [b.attention for b in blocks if b.attention is not None]
    lat = [b.latent for b in blocks if b.latent is not None]
    moe = [b.mlp for b in blocks if isinstance(b.mlp, ExpertSpec)]
    dense = [b.mlp.ff for b in blocks if isinstance(b.mlp, DenseSpec)]
    m = ModelConfig(
        architecture=arch, vocab_size=vocab, hidden_size=width, num_layers=len(blocks),
        intermediate_size=max([m.ff * m.top for m in moe] + dense, default=0),
        num_heads=max([a.heads for a in att + lat], default=1), num_kv_heads=max([a.kv_heads for a in att], default=1),
        head_dim=max([a.dim for a in att + lat], default=8), v_head_dim=max([a.vdim for a in att + lat], default=8),
        rms_norm_eps=eps, embed_scale=embed_scale, norm_topk_prob=False,
        num_experts=max([m.experts for m in moe], default=0), num_experts_per_tok=max([m.top for m in moe], default=0),
        moe_intermediate_size=max([m.ff for m in moe], default=0), max_position_embeddings=max_position,
        blocks=blocks, norm_groups=norm_groups, input_conv=input_conv, bigram=bigram, loop=loop, raw=raw or {})
    if width % norm_groups:
        raise ValueError(f"a width of {width} does not divide into {norm_groups} normed parts")
    if arch == "Kubolorn":
        # (every block carries the last inputs of its convolutions, the embedding the last token)
        m.tie_word_embeddings, m.norm_topk_prob, m.hidden_act = True, True, "gelu_tanh"
        m.layer_types = ["linear_attention"] * len(blocks)
    elif arch == "Nufusun":
        m.gemma_norm, m.attention_bias, m.hidden_act, m.scoring_func = True, True, "clamped_gate", "sigmoid"
    elif arch == "Tabupel":
        m.hidden_act, m.residual_multiplier, m.final_logit_softcap = "silu", residual_mult, logit_softcap
        m.layer_types = ["linear_attention" if b.rglru is not None else "sliding_attention" if b.mixer.window
                         else "full_attention" for b in blocks]
    else:
        m.sandwich_norm, m.hidden_act = True, "gelu_tanh"
        m.layer_types = ["linear_attention" if b.delta is not None else "chunked_attention" if b.attention.chunk
                         else "full_attention" for b in blocks]
    return m


def block_config_dict(cfg: ModelConfig) -> dict:
    """config.json of a ModelConfig with ``blocks`` (the inverse of model_config_from_blocks)."""
    if cfg.architecture in ("Tabupel", "Kubolorn"):
        return (_tabupel_dict if cfg.architecture == "Tabupel" else _kubolorn_dict)(cfg)
    layers = []
    for b in cfg.blocks:
        m, a, f, mlp = b.attention or b.delta, b.attention, b.mlp, None
        mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim}
        if b.delta is not None:
            mixer["conv"] = m.conv
        else:
            mixer["scale"] = a.scale
            if a.bias_max:
                mixer["bias_max"] = a.bias_max
            if a.rot_dims:
                mixer["rot"] = {"base": a.rot_base, "dims": a.rot_dims}
            if a.chunk:
                mixer["mask"] = {"size": a.chunk}
            if a.kv_from is not None:
                mixer["kv_from"] = a.kv_from
        if isinstance(f, DenseSpec):
            mlp = {"kind": "dense", "ff": f.ff}
        elif f is not None:
            mlp = {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff}}
            if cfg.architecture == "Nufusun":
                mlp["expert"]["limit"] = f.limit
            else:
                mlp["router"].update(groups={"count": f.groups, "keep": f.keep}, identity=f.identity)
        layers.append({"type": "attention" if b.delta is None else "delta", "mixer": mixer, "mlp": mlp})
    out = {"architecture": cfg.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_size,
           "norm": {"eps": cfg.rms_norm_eps}, "layers": layers}
    if cfg.architecture == "Nufusun":
        out["embedding"] = {"scale": cfg.embed_scale}
    return out


def _tabupel_dict(cfg: ModelConfig) -> dict:
    from dataclasses import asdict
    layers = []
    for b in cfg.blocks:
        m = {k: v for k, v in asdict(b.mixer).items() if v is not None}
        kind = "rglru" if b.rglru is not None else "latent_attention" if b.latent is not None else "attention"
        if b.rglru is None:
            rot = {"base": m.pop("rot_base"), "dims": m.pop("rot_dims", m.get("rot_dim"))}
            s = m.pop("rot_scaling", None)
            if s is not None:
                rot["scaling"] = s if s["original"] else {"factor": s["factor"]}
            w = m.pop("window")
            m.update(rot=rot, **({"mask": {"size": w}} if w else {}))
            for k in ("bias_max", "chunk", "sink", "tied"):
                m.pop(k, None)
        l = {"type": kind, "mixer": m, "mlp": None if b.mlp is None else {"kind": "dense", "ff": b.mlp.ff}}
        if b.weights_of is not None:
            l["weights_of"] = b.weights_of
        layers.append(l)
    return {"architecture": cfg.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_size,
            "norm": {"eps": cfg.rms_norm_eps}, "residual_mult": cfg.residual_multiplier,
            "logit_softcap": cfg.final_logit_softcap, "layers": layers}


def _kubolorn_dict(cfg: ModelConfig) -> dict:
    from dataclasses import asdict
    layers = []
    for b in cfg.blocks:
        if b.weights_of is not None:
            continue
        f, mlp = b.mlp, None
        if isinstance(f, DenseSpec):
            mlp = {"kind": "dense", "ff": f.ff}
        elif f is not None:
            mlp = {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff}}
        if b.gla is not None:
            g = b.gla
            m = {"heads": g.heads, "dim": g.dim, "vdim": g.vdim, "tau": g.tau}
        else:
            a = b.attention
            left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
            if a.rot_dims:
                left["rot"] = {"base": a.rot_base, "dims": a.rot_dims}
                if a.rot_scaling is not None:
                    left["rot"]["scaling"] = asdict(a.rot_scaling)
            m = {"left": left, "right": asdict(b.ssm), "left_scale": b.scales[0], "right_scale": b.scales[1]}
        layers.append({"type": "gla" if b.gla is not None else "parallel", "mixer": m, "mlp": mlp})
    out = {"architecture": cfg.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_size, "layers": layers,
           "norm": {"eps": cfg.rms_norm_eps, "groups": cfg.norm_groups}, "embedding": {"scale": cfg.embed_scale},
           "canon": {"taps": cfg.input_conv}}
    if cfg.bigram is not None:
        out["embedding"]["bigram"] = asdict(cfg.bigram)
    if cfg.loop is not None:
        out["loop"] = asdict(cfg.loop)
    return out


def load_model_config(model_dir: str) -> ModelConfig:
    with open(os.path.join(model_dir, "config.json")) as f:
        raw = json.load(f)
    if "architecture" in raw and "layers" in raw:
        return model_config_from_blocks(raw)
    return model_config_from_hf(raw)


# ------------------------------------------------------------------ named synthetic shapes
def synthetic_config(name: str) -> ModelConfig:
    """Architectures of the benchmark configurations (random-init weights). A ``+fp8`` or ``+nvfp4``
    suffix selects that weight quantisation (``llama-3.1-8b+fp8``), ``+bf16`` none."""
    n = name.lower()
    if "+" in n:
        base, q = n.rsplit("+", 1)
        if q not in ("fp8", "nvfp4", "bf16"):
            raise ValueError(f"unknown quantisation suffix '+{q}'")
        cfg = synthetic_config(base)
        cfg.quant = None if q == "bf16" else q
        return cfg
    if n in ("qwen3-0.6b", "qwen3_0_6b"):
        return ModelConfig(architecture="Qwen3ForCausalLM", vocab_size=151936, hidden_size=1024,
                           intermediate_size=3072, num_layers=28, num_heads=16, num_kv_heads=8,
                           head_dim=128, rms_norm_eps=1e-6, max_position_embeddings=40960,
                           tie_word_embeddings=True, qk_norm=True, rope=RopeConfig(theta=1e6))
    if n in ("llama-3.1-8b", "llama3.1-8b", "llama_3_1_8b"):
        return ModelConfig(architecture="LlamaForCausalLM", vocab_size=128256, hidden_size=4096,
                           intermediate_size=14336, num_layers=32, num_heads=32, num_kv_heads=8,
                           head_dim=128, rms_norm_eps=1e-5, max_position_embeddings=131072,
                           rope=RopeConfig(theta=5e5, scaling_type="llama3", factor=8.0,
                                           low_freq_factor=1.0, high_freq_factor=4.0,
                                           original_max_position=8192))
    if n in ("qwen3-coder-30b-a3b", "qwen3-30b-a3b"):
        return ModelConfig(architecture="Qwen3MoeForCausalLM", vocab_size=151936, hidden_size=2048,
                           intermediate_size=6144, num_layers=48, num_heads=32, num_kv_heads=4,
                           head_dim=128, rms_norm_eps=1e-6, max_position_embeddings=262144,
                           qk_norm=True, rope=RopeConfig(theta=1e7), num_experts=128,
                           num_experts_per_tok=8, moe_intermediate_size=768, norm_topk_prob=True)
    if n in ("deepseek-v2-lite",):
        return ModelConfig(architecture="DeepseekV2ForCausalLM", vocab_size=102400,
                           hidden_size=2048, intermediate_size=10944, num_layers=27, num_heads=16,
                           num_kv_heads=16, head_dim=192, rms_norm_eps=1e-6,
                           max_position_embeddings=163840,
                           rope=RopeConfig(theta=10000.0, neox=False, scaling_type="deepseek_yarn",
                                           factor=40.0, original_max_position=4096, beta_fast=32,
                                           beta_slow=1, mscale=0.707, mscale_all_dim=0.707,
                                           rotary_dim=64),
                           num_experts=64, num_experts_per_tok=6, moe_intermediate_size=1408,
                           num_shared_experts=2, first_k_dense_replace=1, norm_topk_prob=False,
                           kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64,
                           v_head_dim=128)
    if n in ("qwen3.6-27b", "qwen3_6_27b"):
        L = 64
        return ModelConfig(architecture="Qwen3_5ForConditionalGeneration", vocab_size=248320,
                           hidden_size=5120, intermediate_size=17408, num_layers=L, num_heads=24,
                           num_kv_heads=4, head_dim=256, rms_norm_eps=1e-6,
                           max_position_embeddings=262144, qk_norm=True, gemma_norm=True,
                           attn_output_gate=True,
                           rope=RopeConfig(theta=1e7, rotary_dim=64),
                           layer_types=["full_attention" if (i + 1) % 4 == 0 else
                                        "linear_attention" for i in range(L)],
                           linear_num_key_heads=16, linear_num_value_heads=48,
                           linear_key_head_dim=128, linear_value_head_dim=128,
                           linear_conv_kernel_dim=4, quant="nvfp4")
    if n in ("nufusun-30b-a3b",):
        # the layer sizes of qwen3-coder-30b-a3b
        b = BlockSpec(AttentionSpec(heads=32, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, bias_max=1024),
                      ExpertSpec(experts=128, top=8, ff=768, limit=7.0))
        return model_config_of_blocks("Nufusun", [b] * 48, vocab=151936, width=2048, eps=1e-6, embed_scale=1.0,
                                      max_position=262144)
    if n == "tiny-nufusun":
        b = BlockSpec(AttentionSpec(heads=6, kv_heads=3, dim=32, vdim=48, scale=0.2, bias_max=60),
                      ExpertSpec(experts=5, top=2, ff=64, limit=2.0))
        return model_config_of_blocks("Nufusun", [b, BlockSpec(b.attention), b], vocab=500, width=192, eps=1e-5,
                                      embed_scale=2.0, max_position=2048)
    if n in ("diforax-30b-a3b",):
        # width, attention heads and experts of qwen3-coder-30b-a3b, three delta layers to one attention layer
        moe = ExpertSpec(experts=128, top=8, ff=768, identity=16, groups=8, keep=4)
        delta = BlockSpec(None, moe, DeltaSpec(heads=32, kv_heads=16, dim=128, vdim=128, conv=4))
        att = BlockSpec(AttentionSpec(heads=32, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, rot_dims=128,
                                      rot_base=1e6, chunk=8192), moe)
        return model_config_of_blocks("Diforax", [delta, delta, delta, att] * 12, vocab=151936, width=2048, eps=1e-6,
                                      max_position=262144)
    if n == "tiny-diforax":
        att = AttentionSpec(heads=6, kv_heads=3, dim=24, vdim=40, scale=0.3, rot_dims=16, rot_base=5e3, chunk=50)
        moe = ExpertSpec(experts=6, top=2, ff=64, identity=2, groups=4, keep=2)
        delta = DeltaSpec(heads=4, kv_heads=2, dim=24, vdim=16, conv=3)
        shared = AttentionSpec(**{**att.__dict__, "kv_from": 1, "chunk": 70})
        return model_config_of_blocks("Diforax", [BlockSpec(None, DenseSpec(96), delta), BlockSpec(att, moe),
                                                  BlockSpec(None, None, delta), BlockSpec(shared, DenseSpec(80))],
                                      vocab=500, width=192, eps=1e-5, max_position=2048)
    if n == "tabupel-3b":
        # two recurrent layers to one attention layer, latent and differential attention in turn
        ff, rec = DenseSpec(7680), RglruSpec(width=2560, blocks=10, conv=4)
        lat = LatentSpec(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512, scale=192 ** -0.5, window=2048,
                         rot_base=1e4, rot_scaling=RotaryScaling(40.0, 4096))
        att = AttentionSpec(heads=10, kv_heads=2, dim=128, vdim=256, scale=128 ** -0.5, rot_dims=128, rot_base=1e6,
                            rot_scaling=RotaryScaling(8.0), diff=0.6, window=2048)
        r, a, d = (BlockSpec(None, ff, rglru=rec), BlockSpec(None, ff, latent=lat), BlockSpec(att, ff))
        return model_config_of_blocks("Tabupel", [r, r, a, r, r, d] * 4 + [r, r], vocab=151936, width=2560, eps=1e-6,
                                      residual_mult=0.5, logit_softcap=30.0, max_position=131072)
    if n == "tiny-tabupel":
        ff = DenseSpec(96)
        rec = BlockSpec(None, ff, rglru=RglruSpec(width=80, blocks=5, conv=3))
        lat = LatentSpec(heads=3, dim=40, rot_dim=16, vdim=24, q_rank=56, kv_rank=48, scale=0.15, window=50, rot_base=5e3,
                         rot_scaling=RotaryScaling(3.0, 64))
        att = AttentionSpec(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.2, rot_dims=16, rot_base=5e3,
                            rot_scaling=RotaryScaling(2.0), diff=0.4, window=33)
        return model_config_of_blocks("Tabupel", [BlockSpec(None, None, latent=lat), rec, BlockSpec(att, DenseSpec(64)),
                                                  BlockSpec(None, ff, rglru=rec.rglru, weights_of=1)],
                                      vocab=500, width=192, eps=1e-5, residual_mult=0.7, logit_softcap=20.0, max_position=2048)
    if n == "kubolorn-3b":
        # three linear-attention layers to one parallel layer; the parallel layers carry the experts
        g = BlockSpec(None, DenseSpec(8192, plain="gelu_tanh"), gla=GlaSpec(heads=16, dim=128, vdim=128, tau=16.0))
        att = AttentionSpec(heads=32, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, rot_dims=64, rot_base=1e6,
                            rot_scaling=RotaryScaling(8.0, 8192), sink=True, tied=True)
        p = BlockSpec(att, ExpertSpec(experts=64, top=4, ff=1024, plain="relu2"), scales=(0.7, 0.7),
                      ssm=SsmSpec(heads=32, groups=4, state=128, vdim=64, conv=4, norm_groups=4))
        loop = LoopSpec(start=8, stop=16, times=2)
        return model_config_of_blocks("Kubolorn", unrolled([g, g, g, p] * 6, loop), vocab=151936, width=2048, eps=1e-6, embed_scale=45.0,
                                      norm_groups=4, input_conv=4, bigram=BigramSpec(65521, 31337, 7919), loop=loop,
                                      max_position=65536)
    if n == "tiny-kubolorn":
        att = AttentionSpec(heads=6, kv_heads=2, dim=40, vdim=40, scale=0.2, rot_dims=24, rot_base=5e3,
                            rot_scaling=RotaryScaling(3.0, 64), sink=True, tied=True)
        p = BlockSpec(att, ExpertSpec(experts=4, top=2, ff=48, plain="relu2"), scales=(0.9, 1.1),
                      ssm=SsmSpec(heads=6, groups=2, state=24, vdim=32, conv=3, norm_groups=4))
        g = BlockSpec(None, DenseSpec(96, plain="gelu_tanh"), gla=GlaSpec(heads=3, dim=24, vdim=40, tau=8.0, rank=8))
        loop = LoopSpec(start=0, stop=2, times=2)
        return model_config_of_blocks("Kubolorn", unrolled([g, p, BlockSpec(None, None, gla=g.gla)], loop), vocab=500, width=192, eps=1e-5,
                                      embed_scale=2.0, norm_groups=3, input_conv=2, bigram=BigramSpec(101, 7, 3), loop=loop,
                                      max_position=2048)
    if n.startswith("tiny"):
        # small shapes for tests: tiny-dense, tiny-moe, tiny-mla, tiny-gdn
        base = dict(vocab_size=512, hidden_size=256, intermediate_size=512, num_layers=2,
                    num_heads=4, num_kv_heads=2, head_dim=64, rms_norm_eps=1e-6,
                    max_position_embeddings=2048, rope=RopeConfig(theta=1e4))
        if n == "tiny-dense":
            return ModelConfig(architecture="LlamaForCausalLM", **base)
        if n == "tiny-qwen3":
            return ModelConfig(architecture="Qwen3ForCausalLM", qk_norm=True,
                               tie_word_embeddings=True, **base)
        if n == "tiny-opt":
            return ModelConfig(architecture="OPTForCausalLM", hidden_act="relu", tie_word_embeddings=True,
                               **{**base, "num_kv_heads": 4})
        if n == "tiny-mla":
            base.update(head_dim=192, num_heads=4, num_kv_heads=4)
            return ModelConfig(architecture="DeepseekV2ForCausalLM", num_experts=8, num_experts_per_tok=2,
                               moe_intermediate_size=128, num_shared_experts=1, first_k_dense_replace=1,
                               norm_topk_prob=False, kv_lora_rank=512, qk_nope_head_dim=128,
                               qk_rope_head_dim=64, v_head_dim=128,
                               **{**base, "rope": RopeConfig(theta=1e4, neox=False, rotary_dim=64)})
        if n == "tiny-gdn":
            base.update(num_layers=4, head_dim=256, num_heads=2, num_kv_heads=1)
            return ModelConfig(architecture="Qwen3_5ForConditionalGeneration", qk_norm=True,
                               gemma_norm=True, attn_output_gate=True,
                               layer_types=["full_attention" if (i + 1) % 4 == 0 else "linear_attention"
                                            for i in range(4)],
                               linear_num_key_heads=2, linear_num_value_heads=4,
                               linear_key_head_dim=128, linear_value_head_dim=128,
                               linear_conv_kernel_dim=4, tie_word_embeddings=True,
                               **{**base, "rope": RopeConfig(theta=1e4, rotary_dim=64)})
        if n == "tiny-gdn-moe":
            base.update(num_layers=4, head_dim=256, num_heads=2, num_kv_heads=1)
            return ModelConfig(architecture="Qwen3_5MoeForConditionalGeneration", qk_norm=True,
                               gemma_norm=True, attn_output_gate=True,
                               layer_types=["full_attention" if (i + 1) % 4 == 0 else "linear_attention"
                                            for i in range(4)],
                               linear_num_key_heads=2, linear_num_value_heads=4,
                               linear_key_head_dim=128, linear_value_head_dim=128,
                               linear_conv_kernel_dim=4, tie_word_embeddings=True,
                               num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128,
                               shared_expert_intermediate_size=256, num_shared_experts=1,
                               shared_expert_gate=True, norm_topk_prob=True,
                               **{**base, "rope": RopeConfig(theta=1e4, rotary_dim=64)})
        if n == "tiny-moe":
            return ModelConfig(architecture="Qwen3MoeForCausalLM", qk_norm=True, num_experts=8,
                               num_experts_per_tok=2, moe_intermediate_size=128, **base)
    raise KeyError(f"unknown synthetic model shape: {name}")


@dataclass
class ParallelConfig:
    tensor_parallel_size: int = 1
    enable_expert_parallel: bool = False
    rank: int = 0
    local_rank: int = 0
    fused_collectives: bool = True      # False => GEMM kernel + NCCL call (the baseline mode)
    # True: rank 0 owns the scheduler and publishes every step to the other ranks, which run
    # ``LLM.serve_as_worker()`` and never see a request (serving). False: every rank runs its own
    # scheduler and must be fed identical requests (offline batches driven by one script per rank).
    driver_worker: bool = False
    # Expert-parallel load balancing (parallel/eplb.py): redundant physical expert slots (the
    # total must divide over the ranks), steps between rebalances, steps of load history used.
    enable_eplb: bool = False
    eplb_redundant_experts: int = 0
    eplb_interval: int = 3000
    eplb_window: int = 1000
    # Decode context parallelism (KV of one sequence split over ranks). Only 1 is implemented:
    # long prompts are handled by chunked prefill over the paged cache. The field exists so that
    # KV-cache specs and attention metadata carry the degree (reference: dcp_world_size = 1 fixed
    # in src/vllm/v1/core/sched/scheduler.cpp:78-79).
    dcp_world_size: int = 1

    def __post_init__(self):
        if self.dcp_world_size != 1:
            raise ValueError("decode context parallelism is not implemented: dcp_world_size must be 1")

    @property
    def world_size(self) -> int:
        return self.tensor_parallel_size


@dataclass
class EngineArgs:
    model: Optional[str] = None                 # directory / .gguf, or None with model_config set
    model_config: Optional[ModelConfig] = None
    block_size: int = 32
    num_blocks: int = 0                         # 0 => size from gpu_memory_utilization
    gpu_memory_utilization: float = 0.90
    max_model_len: int = 0                      # 0 => config.max_position_embeddings
    max_num_seqs: int = 8
    max_num_batched_tokens: int = 0             # 0 => dense 2048 / MoE 4096 (8192 at >= 32 seqs)
    enable_prefix_caching: Optional[bool] = None  # None => on unless hybrid
    scheduling_policy: str = "fcfs"
    async_scheduling: Optional[bool] = None
    # spec_decode.SpeculativeConfig; method "ngram" is wired through the engine (prompt-lookup
    # drafts, argmax verification), the other methods have their building blocks only
    speculative_config: Optional[object] = None
    # device "cpu": "torch" = the fp32 PyTorch oracle the GPU path is compared with,
    # "native" = the C++ thread-pool backend (csrc/cpu)
    cpu_backend: str = "torch"
    # CPU only: keep the linear-layer weights in GGUF blocks ("q8_0" | "q4_0") and run the GEMMs on
    # the packed form (integer block dot products); None keeps bf16 weights
    cpu_weight_quant: Optional[str] = None
    enable_cuda_graphs: bool = True
    # "auto": the checkpoint's type (bf16). "float32": weights, activations, cache and products in
    # 32 bits, for the models that support it
    dtype: str = "auto"
    # logits rows per step for positions asked for with LLM.score_positions (besides the sampled ones)
    max_score_rows: int = 0
    seed: int = 0
    device: str = "cuda"
    parallel: ParallelConfig = field(default_factory=ParallelConfig)
    tokenizer: Optional[str] = None
    kv_transfer_config: Optional[dict] = None

    def resolve_max_num_batched_tokens(self, cfg: ModelConfig) -> int:
        if self.max_num_batched_tokens > 0:
            return self.max_num_batched_tokens
        if cfg.is_moe:
            return 8192 if self.max_num_seqs >= 32 else 4096
        return 2048

    def resolve_prefix_caching(self, cfg: ModelConfig) -> bool:
        if self.enable_prefix_caching is not None:
            return self.enable_prefix_caching
        return not cfg.is_hybrid
