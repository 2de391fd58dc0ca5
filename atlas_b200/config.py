"""Model / quantization / serving configuration.

`ModelConfig.from_hf` parses a HuggingFace ``config.json`` dictionary into one
flat dataclass that every layer reads.  It covers the decoder families the
engine serves: Llama/Mistral/Qwen2/Qwen3 dense, Qwen3-MoE, and the Qwen3-Next
hybrid (Gated-DeltaNet + gated attention + MoE + MTP head).

Reference parity: ``crates/avarok-core/src/config.rs`` (``ModelConfig::from_hf``),
``crates/avarok-core/src/config/dispatch.rs`` (model_type aliases) and
``crates/avarok-core/src/config/methods.rs:187`` (``local_expert_range``).
"""
from __future__ import annotations

import dataclasses
import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

# model_type spellings accepted from config.json -> canonical family.
_FAMILY_ALIASES = {
    "llama": "dense", "mistral": "dense", "qwen2": "dense", "qwen3": "dense", "gemma3_text": "dense", "gemma3": "dense",
    "qwen3_moe": "moe", "qwen3_vl_moe": "moe", "mixtral": "moe", "minimax_m2": "moe",
    "qwen3_next": "hybrid", "qwen3_5": "hybrid", "qwen35": "hybrid", "qwen3_5_text": "hybrid",
    "qwen3_5_moe": "hybrid", "qwen35_moe": "hybrid", "qwen3_6_moe": "hybrid", "qwen3_5_moe_text": "hybrid",
    "holo3_1_moe": "hybrid",
    "nemotron_h": "hybrid", "nemotron_h_puzzle": "hybrid",
    "deepseek_v2": "moe", "deepseek_v3": "moe", "deepseek_v32": "moe", "kimi_k2": "moe",
    "papidra": "hybrid", "tomizen": "hybrid", "kenovik": "hybrid", "bisudra": "hybrid",
}

# widths the attention kernels are instantiated for; heads of any other size are zero-padded to the next one
ATTENTION_WIDTHS = (64, 128, 256)


def padded_head_width(*dims: int) -> int:
    """Cache width of heads whose query / key / value sizes are ``dims``."""
    for w in ATTENTION_WIDTHS:
        if max(dims) <= w:
            return w
    raise ValueError(f"attention heads of {max(dims)} channels are not supported (at most {ATTENTION_WIDTHS[-1]})")


@dataclass
class LayerSpec:
    """One layer of a model whose layers differ in kind or size: the mixer's kind, whether a feed-forward sublayer
    follows, and the :class:`ModelConfig` fields that hold for this layer only.

    A layer that runs several times (looped models) has one entry per run, in the order of execution.  Runs after the first
    take the weights of an earlier entry and keep a cache or state of their own."""
    kind: str                              # a mixer kind of ``layers.MIXERS``
    has_mlp: bool = True
    overrides: Dict[str, Any] = field(default_factory=dict)
    weights_of: int = -1                   # entry whose weights this run takes (-1: it has its own)
    step: int = -1                         # >= 0: row of the model's step vectors added to the residual ahead of this run


@dataclass
class QuantConfig:
    """Weight / KV-cache quantization description.

    method:
      * ``"none"``      – weights stay in ``ModelConfig.dtype``.
      * ``"fp8_block"`` – FP8 e4m3 weights with one fp32 scale per 128x128 tile
        (``weight_scale_inv`` tensors), activations quantized per token per
        128-wide K group at run time.
      * ``"nvfp4"``     – packed E2M1 weights ``[N, K/2]``, e4m3 scale per 16
        elements ``[N, K/16]`` and one fp32 global scale ``weight_scale_2``.
    Reference parity: ``crates/spark-model/src/quant_format/{fp8_blockscaled,modelopt,compressed_tensors}.rs``.
    """
    method: str = "none"
    weight_block: Tuple[int, int] = (128, 128)
    group_size: int = 16
    kv_cache_dtype: str = "auto"  # auto | bf16 | fp8 | turbo8 (Hadamard-rotated fp8) | nvfp4
    # modules kept in high precision (substring match on parameter prefix)
    ignore: List[str] = field(default_factory=lambda: ["lm_head", "embed_tokens", "router", "gate."])
    # when method is nvfp4 for experts only (config 3: attention bf16, experts nvfp4)
    experts_only: bool = False

    @staticmethod
    def from_hf(qc: Optional[Dict[str, Any]]) -> "QuantConfig":
        if not qc:
            return QuantConfig()
        method = str(qc.get("quant_method", qc.get("quant_algo", ""))).lower()
        fmt = str(qc.get("fmt", qc.get("format", ""))).lower()
        if method == "fp8" or "fp8" in method:
            wb = qc.get("weight_block_size") or [128, 128]
            return QuantConfig(method="fp8_block", weight_block=(int(wb[0]), int(wb[1])),
                               kv_cache_dtype="fp8" if qc.get("kv_cache_scheme") else "auto")
        if "nvfp4" in method or "nvfp4" in fmt or method in ("modelopt", "modelopt_fp4"):
            gs = int(qc.get("group_size", 16))
            ign = list(qc.get("ignore", qc.get("exclude_modules", [])))
            out = QuantConfig(method="nvfp4", group_size=gs)
            if ign:
                out.ignore = ign
            return out
        if method == "compressed-tensors":
            groups = qc.get("config_groups", {})
            for g in groups.values():
                w = g.get("weights", {})
                if w.get("num_bits") == 4 and w.get("type") == "float":
                    return QuantConfig(method="nvfp4", group_size=int(w.get("group_size", 16)),
                                       ignore=list(qc.get("ignore", [])) or QuantConfig().ignore)
                if w.get("num_bits") == 8 and w.get("type") == "float":
                    return QuantConfig(method="fp8_block")
        return QuantConfig()


@dataclass
class ModelConfig:
    model_type: str = "llama"
    family: str = "dense"            # dense | moe | hybrid
    vocab_size: int = 32000
    hidden_size: int = 4096
    intermediate_size: int = 11008
    num_hidden_layers: int = 32
    num_attention_heads: int = 32
    num_key_value_heads: int = 32
    head_dim: int = 128
    rms_norm_eps: float = 1e-6
    rope_theta: float = 10000.0
    rope_scaling: Optional[Dict[str, Any]] = None
    partial_rotary_factor: float = 1.0
    max_position_embeddings: int = 32768
    tie_word_embeddings: bool = False
    attention_bias: bool = False
    qk_norm: bool = False             # Qwen3-style per-head RMSNorm on q and k
    attn_output_gate: bool = False    # Qwen3-Next gated attention (q_proj emits q and gate)
    sliding_window: Optional[int] = None
    norm_plus_one: bool = False       # (1 + weight) RMSNorm convention (Qwen3-Next, Gemma)
    qk_norm_plus_one: Optional[bool] = None   # the same for the q / k head norms (None = as the other norms)
    # MoE
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    shared_expert_intermediate_size: int = 0
    norm_topk_prob: bool = True
    router_scoring: str = "softmax"   # softmax | sigmoid | sqrtsoftplus
    router_f32: bool = False          # router logits leave their matrix product in fp32
    router_logit_bias: bool = False   # a learned number per expert joins the logits (selection and weights)
    routed_scaling_factor: float = 1.0
    router_n_group: int = 0           # group-limited routing (DeepSeek-V3): experts split into n_group groups ...
    router_topk_group: int = 0        # ... of which the topk_group best stay eligible
    router_selection_bias: bool = False   # per-expert e_score_correction_bias used for selection only
    num_hash_layers: int = 0          # first MoE layers select experts by a static token-id table (DeepSeek-V4)
    decoder_sparse_step: int = 1
    mlp_only_layers: List[int] = field(default_factory=list)
    # hybrid (Gated DeltaNet)
    layer_types: List[str] = field(default_factory=list)  # "full_attention" | "linear_attention"
    full_attention_interval: int = 4
    linear_num_key_heads: int = 0
    linear_num_value_heads: int = 0
    linear_key_head_dim: int = 128
    linear_value_head_dim: int = 128
    linear_conv_kernel_dim: int = 4
    # single-module blocks (Nemotron-H): per layer "mamba" | "attention" | "mlp"; empty for the other families
    block_types: List[str] = field(default_factory=list)
    # layers of different kinds and sizes, each with its own values of the fields of this class
    layer_specs: List[LayerSpec] = field(default_factory=list)
    # hyper-connections: number of residual streams (0 = one plain residual stream in the activations' dtype)
    residual_streams: int = 0
    # norms on the sublayers' outputs only: every sublayer reads the (fp32) residual stream itself
    output_norms: bool = False
    # norms on the sublayers' inputs, on an fp32 residual stream (models given by a list of layers)
    input_norms: bool = False
    loop_steps: int = 0               # passes of the looped layers that have a step vector
    # parts of a layer on normed outputs: layer norms (mean taken off, with a bias) in place of RMS norms, also ahead of the head;
    # sigmoid gates on the sublayers' results, computed from what the sublayer reads; a short causal convolution added to the
    # mixer's input (number of taps, 0 = off); a second embedding of the tokens that every layer takes its share of (numbers per
    # layer, 0 = off); every layer hands on a weighted sum of all layers' results so far
    layer_norms: bool = False
    sublayer_gates: bool = False
    input_conv_taps: int = 0
    token_side_dim: int = 0
    depth_average: bool = False
    mamba_num_heads: int = 0
    mamba_head_dim: int = 64
    ssm_state_size: int = 128
    mamba_n_groups: int = 8
    mamba_conv_kernel: int = 4
    mamba_dt_min: float = 0.0
    mamba_norm_groups: int = 0        # parts of the gated output norm (0 = one per B / C group)
    # RG-LRU recurrence (gated linear recurrent unit per channel)
    rglru_width: int = 0
    rglru_blocks: int = 0
    rglru_conv_kernel: int = 4
    # WKV recurrence (RWKV-style time mixing)
    wkv_num_heads: int = 0
    wkv_head_dim: int = 0
    # mLSTM (matrix memory with exponential gates)
    mlstm_num_heads: int = 0
    mlstm_head_dim: int = 0
    mlstm_value_dim: int = 0
    mlstm_gate_cap: float = 0.0       # bound on the raw gates (cap * tanh(. / cap))
    # silu_glu (gated SwiGLU) | relu2 (up -> relu^2 -> down) | clamped_glu | silu_unit (SwiGLU on alternating gate and up rows, the
    # form that the products' epilogues apply)
    mlp_activation: str = "silu_glu"
    mlp_bias: bool = False            # the dense feed-forward's projections have biases
    glu_limit: float = 0.0            # clamped_glu: bound on the gate (above) and on the up branch (both sides)
    glu_alpha: float = 1.702          # clamped_glu: slope inside the gate's sigmoid
    shared_glu_limit: float = 0.0     # the same bound for the shared expert
    # attention variants: chunked visibility (a token sees its own chunk only), a learned per-head sink in the softmax
    # denominator, the number of rotated dimensions when it is not a fraction of head_dim
    attn_chunk: int = 0
    attn_sinks: bool = False
    attn_sink_score: Optional[float] = None   # a fixed sink score of every head instead of learned ones (0: one is added)
    attn_softcap: float = 0.0         # scores become cap * tanh(score / cap) before the softmax (0 = off)
    attn_head_gate: bool = False      # every head's output times the sigmoid of one number per head
    # a learned bias per head and distance bucket joins the scores: rows of the table and the distance from which on all
    # keys share its last row (0 = off); the first half of the rows are single distances, the others logarithmic
    attn_distance_rows: int = 0
    attn_distance_reach: int = 0
    qk_norm_rows: bool = False        # q and k are normed over all heads at once, before they are split
    # differential attention: two maps per head over the same values, output of the first minus a learned multiple of the second,
    # with this constant in the multiple and 1 minus it on the result
    attn_diff: float = 0.0
    attn_query_temp: float = 0.0      # queries times 1 + c ln(floor((position + 1) / every) + 1) (0 = off)
    attn_query_temp_every: int = 1
    rotary_dims: Optional[int] = None
    attn_cache_width: int = 0         # padded width of cached heads (0 = head_dim)
    # multi-head latent attention (DeepSeek): 0 = plain GQA.  head_dim is then the padded cache width
    kv_lora_rank: int = 0
    q_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    rope_interleaved: bool = True     # checkpoint stores rotary columns as (even, odd) pairs
    first_k_dense_replace: int = 0    # leading layers with a dense FFN in an otherwise MoE model
    # Gemma: scaled embeddings, explicit attention scale, norms after the mixer and the FFN as well as before them, a
    # separate rotary base for sliding-window layers, soft-capped output logits
    embed_scale: float = 1.0
    attn_scale: float = 0.0           # 0 = head_dim ** -0.5
    sandwich_norms: bool = False
    rope_local_theta: float = 0.0     # rotary base of the sliding-window layers (0 = same table as the other layers)
    final_logit_softcapping: float = 0.0
    # multimodal: interleaved MRoPE sections (time, row, column), the image placeholder id and the vision tower's config
    mrope_section: List[int] = field(default_factory=list)
    image_token_id: int = -1
    vision: Any = None                # models.vision.VisionConfig
    # MTP speculative head
    mtp_num_layers: int = 0
    # numerics
    dtype: str = "bfloat16"
    quant: QuantConfig = field(default_factory=QuantConfig)
    bos_token_id: Optional[int] = None
    eos_token_id: Any = None

    # ------------------------------------------------------------------ helpers
    @property
    def q_size(self) -> int:
        return self.num_attention_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_key_value_heads * self.head_dim

    @property
    def rotary_dim(self) -> int:
        if self.rotary_dims is not None:
            return self.rotary_dims
        return int(self.head_dim * self.partial_rotary_factor)

    def for_layer(self, i: int) -> "ModelConfig":
        """The configuration as layer ``i`` sees it (its own sizes in place of the model's)."""
        if not self.layer_specs:
            return self
        return dataclasses.replace(self, layer_specs=[], **self.layer_specs[i].overrides)

    def layer_kind(self, i: int) -> str:
        """Mixer kind of layer ``i``: ``attention``, ``gdn``, ``none`` (an FFN-only block) or one of ``layers.MIXERS``."""
        if self.layer_specs:
            return self.layer_specs[i].kind
        if self.block_types:
            return {"mamba": "mamba2", "attention": "attention"}.get(self.block_types[i], "none")
        if self.family != "hybrid":
            return "attention"                # (Gemma's layer_types only choose the attention window)
        if self.layer_types:
            return "attention" if self.layer_types[i] == "full_attention" else "gdn"
        return "attention" if (i + 1) % self.full_attention_interval == 0 else "gdn"

    def is_moe_layer(self, i: int) -> bool:
        if self.layer_specs:
            return self.layer_specs[i].has_mlp and self.for_layer(i).num_experts > 0
        if self.block_types:
            return self.block_types[i] == "moe"
        if self.num_experts <= 0 or i in self.mlp_only_layers or i < self.first_k_dense_replace:
            return False
        return (i + 1) % max(1, self.decoder_sparse_step) == 0

    def local_expert_range(self, ep_rank: int, ep_size: int) -> Tuple[int, int]:
        """Contiguous expert slice owned by ``ep_rank`` (remainder to the low ranks)."""
        e = self.num_experts
        base, rem = divmod(e, ep_size)
        lo = ep_rank * base + min(ep_rank, rem)
        return lo, lo + base + (1 if ep_rank < rem else 0)

    def eos_ids(self) -> List[int]:
        if self.eos_token_id is None:
            return []
        if isinstance(self.eos_token_id, (list, tuple)):
            return [int(x) for x in self.eos_token_id]
        return [int(self.eos_token_id)]

    def param_count(self) -> int:
        h, L = self.hidden_size, self.num_hidden_layers
        n = self.vocab_size * h * (1 if self.tie_word_embeddings else 2)
        if self.layer_specs:
            return n + sum(self.for_layer(i)._spec_layer_params(s) for i, s in enumerate(self.layer_specs) if s.weights_of < 0)
        for i in range(L):
            if self.layer_kind(i) == "attention":
                qmul = 2 if self.attn_output_gate else 1
                n += h * (self.q_size * qmul + 2 * self.kv_size) + self.q_size * h
            elif self.layer_kind(i) == "mamba2":
                di = self.mamba_num_heads * self.mamba_head_dim
                n += h * (2 * di + 2 * self.mamba_n_groups * self.ssm_state_size + self.mamba_num_heads) + di * h
            elif self.layer_kind(i) == "none":
                pass
            else:
                kd = self.linear_num_key_heads * self.linear_key_head_dim
                vd = self.linear_num_value_heads * self.linear_value_head_dim
                n += h * (2 * kd + 2 * vd) + h * 2 * self.linear_num_value_heads + vd * h
            if self.is_moe_layer(i):
                n += self.num_experts * 3 * h * self.moe_intermediate_size + h * self.num_experts
                n += 3 * h * self.shared_expert_intermediate_size
            elif self.block_types:
                n += 2 * h * self.intermediate_size if self.block_types[i] == "mlp" else 0
            else:
                n += 3 * h * self.intermediate_size
        return n

    def _spec_layer_params(self, spec: LayerSpec) -> int:
        """Projection weights of one layer described by a :class:`LayerSpec` (``self`` is the layer's own view)."""
        h = self.hidden_size
        n = (2 if self.mlp_activation == "relu2" else 3) * h * self.intermediate_size if spec.has_mlp and not self.num_experts else 0
        if self.sublayer_gates:
            n += (2 if spec.has_mlp else 1) * h * h
        n += self.token_side_dim * (2 * h + self.vocab_size)
        if spec.has_mlp and self.num_experts:
            n += self.num_experts * (h + (2 if self.mlp_activation == "relu2" else 3) * h * self.moe_intermediate_size)
            n += 3 * h * self.shared_expert_intermediate_size
        if spec.kind in ("attention", "parallel"):
            dv = self.v_head_dim or self.head_dim
            n += h * (self.q_size + self.kv_size + self.num_key_value_heads * dv) + self.num_attention_heads * dv * h
        if spec.kind == "differential":
            dv, H = self.v_head_dim or self.head_dim, self.num_attention_heads
            n += h * (2 * self.q_size + 2 * self.kv_size + self.num_key_value_heads * dv) + (2 if self.attn_output_gate else 1) * H * dv * h
        if spec.kind in ("mamba2", "parallel"):
            di = self.mamba_num_heads * self.mamba_head_dim
            n += h * (2 * di + 2 * self.mamba_n_groups * self.ssm_state_size + self.mamba_num_heads) + di * h
        if spec.kind == "rglru":
            n += 3 * h * self.rglru_width + 2 * self.rglru_width * (self.rglru_width // self.rglru_blocks)
        if spec.kind == "wkv":
            n += 5 * h * self.wkv_num_heads * self.wkv_head_dim
        if spec.kind == "mlstm":
            n += h * self.mlstm_num_heads * (2 * self.mlstm_head_dim + 3 * self.mlstm_value_dim + 2)
        if spec.kind == "latent_attention":
            qk, H = self.qk_nope_head_dim + self.qk_rope_head_dim, self.num_attention_heads
            n += h * (H * qk + self.kv_lora_rank + self.qk_rope_head_dim + H * self.v_head_dim)
            n += self.kv_lora_rank * H * (self.qk_nope_head_dim + self.v_head_dim)
        return n

    # ------------------------------------------------------------------ parsing
    @staticmethod
    def from_hf(cfg: Dict[str, Any]) -> "ModelConfig":
        outer = cfg
        native = _NATIVE_ARCHITECTURES.get(str(cfg.get("architecture", "")).lower())
        if native is not None:
            c = native(cfg)
            c.validate()
            return c
        if "text_config" in cfg and isinstance(cfg["text_config"], dict):
            merged = dict(cfg["text_config"])
            for k in ("quantization_config", "torch_dtype"):
                if k in cfg and k not in merged:
                    merged[k] = cfg[k]
            cfg = merged
        mt = str(cfg.get("model_type", "llama")).lower()
        if mt not in _FAMILY_ALIASES:
            raise ValueError(f"Unsupported model_type '{mt}'. Supported: {sorted(_FAMILY_ALIASES)}")
        fam = _FAMILY_ALIASES[mt]
        nh = int(cfg["num_attention_heads"])
        hs = int(cfg["hidden_size"])
        rope_params = cfg.get("rope_parameters") or {}
        c = ModelConfig(
            model_type=mt, family=fam,
            vocab_size=int(cfg["vocab_size"]), hidden_size=hs,
            intermediate_size=int(cfg.get("intermediate_size", 0) or 0),
            num_hidden_layers=int(cfg.get("num_hidden_layers") or len(cfg.get("layers_block_type") or cfg.get("hybrid_override_pattern") or [])),
            num_attention_heads=nh,
            num_key_value_heads=int(cfg.get("num_key_value_heads", nh)),
            head_dim=int(cfg.get("head_dim") or hs // nh),
            rms_norm_eps=float(cfg.get("rms_norm_eps", 1e-6)),
            rope_theta=float(cfg.get("rope_theta", rope_params.get("rope_theta", 10000.0))),
            rope_scaling=cfg.get("rope_scaling") or (rope_params if rope_params.get("rope_type", "default") != "default" else None),
            partial_rotary_factor=float(cfg.get("partial_rotary_factor", rope_params.get("partial_rotary_factor", 1.0))),
            max_position_embeddings=int(cfg.get("max_position_embeddings", 32768)),
            tie_word_embeddings=bool(cfg.get("tie_word_embeddings", False)),
            attention_bias=bool(cfg.get("attention_bias", mt == "qwen2")),
            qk_norm=mt in ("qwen3", "qwen3_moe", "qwen3_vl_moe") or fam == "hybrid",
            attn_output_gate=fam == "hybrid" and bool(cfg.get("attn_output_gate", True)),
            sliding_window=cfg.get("sliding_window") if cfg.get("use_sliding_window", True) else None,
            norm_plus_one=fam == "hybrid",
            num_experts=int(cfg.get("num_experts", cfg.get("num_local_experts", 0)) or 0),
            num_experts_per_tok=int(cfg.get("num_experts_per_tok", 0) or 0),
            moe_intermediate_size=int(cfg.get("moe_intermediate_size", 0) or 0),
            shared_expert_intermediate_size=int(cfg.get("shared_expert_intermediate_size", 0) or 0),
            norm_topk_prob=bool(cfg.get("norm_topk_prob", True)),
            router_scoring=str(cfg.get("scoring_func", "softmax")),
            routed_scaling_factor=float(cfg.get("routed_scaling_factor", 1.0) or 1.0),
            router_n_group=int(cfg.get("n_group", 0) or 0),
            router_topk_group=int(cfg.get("topk_group", 0) or 0),
            router_selection_bias=bool(cfg.get("router_selection_bias", cfg.get("topk_method", "") == "noaux_tc")),
            num_hash_layers=int(cfg.get("num_hash_layers", 0) or 0),
            decoder_sparse_step=int(cfg.get("decoder_sparse_step", 1) or 1),
            mlp_only_layers=list(cfg.get("mlp_only_layers", []) or []),
            layer_types=list(cfg.get("layer_types", []) or []),
            full_attention_interval=int(cfg.get("full_attention_interval", 4) or 4),
            linear_num_key_heads=int(cfg.get("linear_num_key_heads", 0) or 0),
            linear_num_value_heads=int(cfg.get("linear_num_value_heads", 0) or 0),
            linear_key_head_dim=int(cfg.get("linear_key_head_dim", 128) or 128),
            linear_value_head_dim=int(cfg.get("linear_value_head_dim", 128) or 128),
            linear_conv_kernel_dim=int(cfg.get("linear_conv_kernel_dim", 4) or 4),
            mtp_num_layers=int(cfg.get("mtp_num_hidden_layers", cfg.get("num_nextn_predict_layers", 0)) or 0),
            dtype=str(cfg.get("torch_dtype", cfg.get("dtype", "bfloat16"))),
            quant=QuantConfig.from_hf(cfg.get("quantization_config")),
            bos_token_id=cfg.get("bos_token_id"), eos_token_id=cfg.get("eos_token_id"),
        )
        if mt in ("gemma3_text", "gemma3"):
            rp = cfg.get("rope_parameters") or {}
            glob, loc = rp.get("full_attention") or {}, rp.get("sliding_attention") or {}
            c.rope_theta = float(glob.get("rope_theta", cfg.get("rope_theta", 1e6)))
            c.rope_scaling = glob if glob.get("rope_type", "default") != "default" else cfg.get("rope_scaling")
            c.rope_local_theta = float(loc.get("rope_theta", cfg.get("rope_local_base_freq", 1e4)))
            c.partial_rotary_factor = 1.0
            c.norm_plus_one = c.qk_norm = c.sandwich_norms = True
            c.embed_scale = float(hs) ** 0.5
            c.attn_scale = float(cfg.get("query_pre_attn_scalar", c.head_dim)) ** -0.5
            c.mlp_activation = "gelu_tanh_glu"
            c.layer_types = list(cfg.get("layer_types") or [])
            c.sliding_window = cfg.get("sliding_window")
            c.final_logit_softcapping = float(cfg.get("final_logit_softcapping") or 0.0)
            c.tie_word_embeddings = bool(cfg.get("tie_word_embeddings", True))
            if cfg.get("attn_logit_softcapping"):
                raise ValueError("attention logit soft-capping (Gemma-2) is not supported")
        if mt == "mixtral":
            c.moe_intermediate_size = c.intermediate_size
        if mt.startswith("deepseek") or mt == "kimi_k2":
            c.num_experts = int(cfg.get("n_routed_experts", 0) or 0)
            c.shared_expert_intermediate_size = c.moe_intermediate_size * int(cfg.get("n_shared_experts", 0) or 0)
            c.first_k_dense_replace = int(cfg.get("first_k_dense_replace", 0) or 0)
            c.decoder_sparse_step = int(cfg.get("moe_layer_freq", 1) or 1)
            c.router_scoring = str(cfg.get("scoring_func", "sigmoid" if mt != "deepseek_v2" else "softmax"))
            c.router_selection_bias = mt != "deepseek_v2"
            c.num_key_value_heads = nh
            c.kv_lora_rank = int(cfg.get("kv_lora_rank", 512))
            c.q_lora_rank = int(cfg.get("q_lora_rank") or 0)
            c.qk_nope_head_dim = int(cfg.get("qk_nope_head_dim", 128))
            c.qk_rope_head_dim = int(cfg.get("qk_rope_head_dim", 64))
            c.v_head_dim = int(cfg.get("v_head_dim", 128))
            c.rope_interleaved = bool(cfg.get("rope_interleave", True))
            need = max(c.qk_nope_head_dim + c.qk_rope_head_dim, c.v_head_dim)
            c.head_dim = next((d for d in (64, 128, 256) if d >= need), need)
            c.partial_rotary_factor = c.qk_rope_head_dim / c.head_dim
            c.qk_norm = False
        if mt.startswith("nemotron_h"):
            blocks = cfg.get("layers_block_type")
            if not blocks and cfg.get("hybrid_override_pattern"):
                blocks = [{"M": "mamba", "*": "attention", "-": "mlp", "E": "moe"}[ch] for ch in cfg["hybrid_override_pattern"]]
            c.block_types = list(blocks or [])
            c.num_hidden_layers = len(c.block_types)
            c.mamba_num_heads = int(cfg.get("mamba_num_heads", 128))
            c.mamba_head_dim = int(cfg.get("mamba_head_dim", 64))
            c.ssm_state_size = int(cfg.get("ssm_state_size", 128))
            c.mamba_n_groups = int(cfg.get("n_groups", 8))
            c.mamba_conv_kernel = int(cfg.get("conv_kernel", 4))
            c.mamba_dt_min = float(cfg.get("time_step_min", 0.001))
            c.mlp_activation = "relu2"
            c.rms_norm_eps = float(cfg.get("layer_norm_epsilon", cfg.get("rms_norm_eps", 1e-5)))
            c.partial_rotary_factor = 0.0                     # attention blocks carry no positional rotation
            c.qk_norm = c.attn_output_gate = c.norm_plus_one = False
            c.num_experts = c.num_experts_per_tok = 0
            if "moe" in c.block_types:
                raise ValueError("nemotron_h checkpoints with MoE blocks are not supported")
        c.mrope_section = list(rope_params.get("mrope_section") or (cfg.get("rope_scaling") or {}).get("mrope_section") or [])
        if isinstance(outer.get("vision_config"), dict) and outer.get("image_token_id") is not None and fam == "hybrid":
            from .models.vision import VisionConfig
            c.vision = VisionConfig.from_hf(outer["vision_config"])
            c.image_token_id = int(outer["image_token_id"])
            if not c.mrope_section:
                c.mrope_section = [11, 11, 10]
        c.validate()
        return c

    @staticmethod
    def from_pretrained(path: str) -> "ModelConfig":
        with open(os.path.join(path, "config.json")) as f:
            cfg = json.load(f)
        c = ModelConfig.from_hf(cfg)
        side = os.path.join(path, "hf_quant_config.json")   # ModelOpt sidecar
        if c.quant.method == "none" and os.path.exists(side):
            with open(side) as f:
                q = json.load(f).get("quantization", {})
            c.quant = QuantConfig.from_hf(q)
        return c

    def validate(self) -> None:
        if self.num_attention_heads % max(1, self.num_key_value_heads):
            raise ValueError("num_attention_heads must be a multiple of num_key_value_heads")
        if self.num_experts and not self.num_experts_per_tok:
            raise ValueError("MoE config needs num_experts_per_tok")
        if self.family == "hybrid" and not self.linear_num_value_heads and not (self.block_types or self.layer_specs):
            raise ValueError("hybrid config needs linear_num_value_heads")

    def to_dict(self) -> Dict[str, Any]:
        return dataclasses.asdict(self)


# ---------------------------------------------------------------------------- configurations that list their layers
def _rotary_overrides(rot: Optional[Dict[str, Any]]) -> Dict[str, Any]:
    """``{dims, base, scaling}`` -> rotary fields; ``scaling`` is YaRN's ``{factor, original, fast, slow}`` or, with a factor alone,
    linear."""
    if not rot:
        return {"rotary_dims": 0}
    sc = rot.get("scaling")
    if sc and "original" not in sc:
        return {"rotary_dims": int(rot["dims"]), "rope_theta": float(rot["base"]),
                "rope_scaling": {"rope_type": "linear", "factor": float(sc["factor"])}}
    return {"rotary_dims": int(rot["dims"]), "rope_theta": float(rot["base"]),
            "rope_scaling": None if not sc else {
                "rope_type": "yarn", "factor": float(sc["factor"]), "original_max_position_embeddings": float(sc["original"]),
                "beta_fast": float(sc["fast"]), "beta_slow": float(sc["slow"]),
                "attention_factor": 0.1 * math.log(float(sc["factor"])) + 1.0}}


def _attention_overrides(m: Dict[str, Any]) -> Dict[str, Any]:
    d, dv = int(m["dim"]), int(m.get("vdim", m["dim"]))
    return {"num_attention_heads": int(m["heads"]), "num_key_value_heads": int(m["kv_heads"]), "head_dim": d, "v_head_dim": dv,
            "attn_cache_width": padded_head_width(d, dv), "attn_scale": float(m["scale"]), **_rotary_overrides(m.get("rot"))}


def _mamba2_overrides(m: Dict[str, Any]) -> Dict[str, Any]:
    return {"mamba_num_heads": int(m["heads"]), "mamba_head_dim": int(m["vdim"]), "ssm_state_size": int(m["state"]),
            "mamba_n_groups": int(m["groups"]), "mamba_norm_groups": int(m["norm_groups"]), "mamba_conv_kernel": int(m["conv"]),
            "mamba_dt_min": 0.0}


def _papidra_layer(lc: Dict[str, Any]) -> LayerSpec:
    kind, m, mlp = str(lc["type"]), lc["mixer"], lc.get("mlp")
    over: Dict[str, Any] = {}
    if kind == "wkv":
        over.update(wkv_num_heads=int(m["heads"]), wkv_head_dim=int(m["dim"]))
    elif kind == "parallel":
        over.update(_attention_overrides(m["left"]), attn_sinks=True, attn_chunk=int((m["left"].get("mask") or {}).get("size", 0)))
        over.update(_mamba2_overrides(m["right"]))
    else:
        raise ValueError(f"unsupported Papidra layer type '{kind}'")
    if mlp is not None:
        if mlp.get("kind", "dense") != "dense":
            raise ValueError(f"unsupported Papidra feed-forward '{mlp['kind']}'")
        over.update(intermediate_size=int(mlp["ff"]), glu_limit=float(mlp["limit"]), mlp_activation="clamped_glu")
    return LayerSpec(kind, mlp is not None, over)


def papidra_config(cfg: Dict[str, Any]) -> ModelConfig:
    """Papidra: WKV layers and layers with attention and Mamba-2 side by side, on hyper-connected residual streams."""
    specs = [_papidra_layer(lc) for lc in cfg["layers"]]
    c = ModelConfig(model_type="papidra", family="hybrid", vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]),
                    intermediate_size=max([s.overrides.get("intermediate_size", 0) for s in specs] + [1]),
                    num_hidden_layers=len(specs), num_attention_heads=1, num_key_value_heads=1, head_dim=64,
                    rms_norm_eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]),
                    residual_streams=int(cfg["streams"]), tie_word_embeddings=True, layer_specs=specs,
                    mlp_activation="clamped_glu", dtype=str(cfg.get("torch_dtype", cfg.get("dtype", "bfloat16"))),
                    quant=QuantConfig(kv_cache_dtype="bf16"), bos_token_id=cfg.get("bos_token_id"), eos_token_id=cfg.get("eos_token_id"))
    return _size_by_heads(c)


def _size_by_heads(c: ModelConfig) -> ModelConfig:
    """The model-wide view of a list of layers carries the head sizes of the first attention layer (it sizes buffers)."""
    for s in c.layer_specs:
        if "num_attention_heads" in s.overrides:
            for k in ("num_attention_heads", "num_key_value_heads", "head_dim"):
                setattr(c, k, s.overrides[k])
            break
    return c


def _latent_overrides(m: Dict[str, Any]) -> Dict[str, Any]:
    d, dr, dv = int(m["dim"]), int(m["rot_dim"]), int(m["vdim"])
    mask = m.get("mask")
    return {"num_attention_heads": int(m["heads"]), "num_key_value_heads": 1, "head_dim": d + dr, "qk_nope_head_dim": d,
            "qk_rope_head_dim": dr, "v_head_dim": dv, "kv_lora_rank": int(m["kv_rank"]), "attn_scale": float(m["scale"]),
            "attn_cache_width": padded_head_width(d + dr, dv), "sliding_window": int(mask["size"]) if mask else None,
            **_rotary_overrides(m.get("rot"))}


def _expert_overrides(mlp: Dict[str, Any]) -> Dict[str, Any]:
    if mlp.get("kind") != "moe":
        raise ValueError(f"unsupported Tomizen feed-forward '{mlp.get('kind')}'")
    r = mlp["router"]
    return {"num_experts": int(r["experts"]), "num_experts_per_tok": int(r["top"]), "moe_intermediate_size": int(mlp["expert"]["ff"]),
            "norm_topk_prob": False, "router_scoring": "softmax", "router_f32": True, "mlp_activation": "relu2"}


def _tomizen_layer(lc: Dict[str, Any]) -> LayerSpec:
    kind, m, mlp = str(lc["type"]), lc["mixer"], lc.get("mlp")
    if kind == "mlstm":
        over = {"mlstm_num_heads": int(m["heads"]), "mlstm_head_dim": int(m["dim"]), "mlstm_value_dim": int(m["vdim"]),
                "mlstm_gate_cap": float(m["gate_cap"])}
    elif kind == "latent_attention":
        over = _latent_overrides(m)
    elif kind == "attention":
        over = _attention_overrides(m)
        over.update(attn_softcap=float(m["softcap"]), attn_head_gate=True, qk_norm=True, qk_norm_plus_one=False)
    else:
        raise ValueError(f"unsupported Tomizen layer type '{kind}'")
    if mlp is not None:
        over.update(_expert_overrides(mlp))
    return LayerSpec(kind, mlp is not None, over)


def tomizen_config(cfg: Dict[str, Any]) -> ModelConfig:
    """Tomizen: mLSTM, latent-attention and soft-capped attention layers with experts, norms on the sublayers' outputs."""
    specs = [_tomizen_layer(lc) for lc in cfg["layers"]]
    widest = lambda k: max([s.overrides.get(k, 0) for s in specs] + [0])
    c = ModelConfig(model_type="tomizen", family="hybrid", vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]),
                    intermediate_size=max(1, widest("moe_intermediate_size")), num_hidden_layers=len(specs), num_attention_heads=1,
                    num_key_value_heads=1, head_dim=64, rms_norm_eps=float(cfg["norm"]["eps"]), norm_plus_one=True, output_norms=True,
                    layer_specs=specs, dtype=str(cfg.get("torch_dtype", cfg.get("dtype", "bfloat16"))),
                    quant=QuantConfig(kv_cache_dtype="bf16"), bos_token_id=cfg.get("bos_token_id"), eos_token_id=cfg.get("eos_token_id"))
    c.moe_intermediate_size = c.intermediate_size
    return _size_by_heads(c)


def _kenovik_ff(mlp: Dict[str, Any]) -> Dict[str, Any]:
    if mlp.get("kind", "dense") == "dense":
        return {"intermediate_size": int(mlp["ff"]), "mlp_activation": "silu_glu"}
    if mlp["kind"] != "moe":
        raise ValueError(f"unsupported Kenovik feed-forward '{mlp['kind']}'")
    r, shared = mlp["router"], mlp.get("shared")
    groups = r.get("groups") or {"count": 1, "keep": 1}
    if int(r["experts"]) % int(groups["count"]):
        raise ValueError(f"{r['experts']} experts do not form {groups['count']} equal groups")
    if int(r["top"]) > int(r["experts"]) // int(groups["count"]) * int(groups["keep"]):
        raise ValueError(f"{r['top']} experts per token do not fit into {groups['keep']} of {groups['count']} groups")
    return {"num_experts": int(r["experts"]), "num_experts_per_tok": int(r["top"]), "moe_intermediate_size": int(mlp["expert"]["ff"]),
            "mlp_activation": "clamped_glu", "glu_limit": float(mlp["expert"]["limit"]), "norm_topk_prob": True,
            "router_scoring": "sigmoid", "router_selection_bias": True, "router_f32": True, "routed_scaling_factor": float(r["scale"]),
            "router_n_group": int(groups["count"]), "router_topk_group": int(groups["keep"]),
            "shared_expert_intermediate_size": int(shared["ff"]) if shared else 0,
            "shared_glu_limit": float(shared["limit"]) if shared else 0.0}


def _kenovik_layer(lc: Dict[str, Any]) -> LayerSpec:
    kind, m, mlp = str(lc["type"]), lc["mixer"], lc.get("mlp")
    if kind == "rglru":
        over = {"rglru_width": int(m["width"]), "rglru_blocks": int(m["blocks"]), "rglru_conv_kernel": int(m["conv"])}
        if over["rglru_width"] % over["rglru_blocks"]:
            raise ValueError(f"{over['rglru_width']} channels do not form {over['rglru_blocks']} equal blocks")
    elif kind == "attention":
        over = {**_attention_overrides(m), "attention_bias": True, "attn_sinks": True, "attn_sink_score": 0.0}
    elif kind == "attention_2":
        temp = m.get("q_temp") or {"coef": 0.0, "every": 1}
        over = {**_attention_overrides(m), "qk_norm": True, "qk_norm_rows": True, "qk_norm_plus_one": False,
                "attn_query_temp": float(temp["coef"]), "attn_query_temp_every": int(temp["every"]),
                "attn_distance_rows": int(m.get("bias_rows", 32)), "attn_distance_reach": int(m["bias_max"])}
        kind = "attention"
    else:
        raise ValueError(f"unsupported Kenovik layer type '{kind}'")
    if mlp is not None:
        over.update(_kenovik_ff(mlp))
    return LayerSpec(kind, mlp is not None, over)


def _unrolled(specs: List[LayerSpec], loop: Optional[Dict[str, Any]]) -> List[LayerSpec]:
    """One entry per run of a layer: layers ``start .. stop - 1`` run ``times`` times in a row on the same weights, and the first
    one of every pass adds that pass's step vector."""
    if not loop:
        return list(specs)
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= a < b <= len(specs) or times < 1:
        raise ValueError(f"a loop over layers {a} .. {b - 1}, {times} times, does not fit a model of {len(specs)} layers")
    runs = list(specs[:a])
    for t in range(times):
        for i in range(a, b):
            runs.append(dataclasses.replace(specs[i], weights_of=i if t else -1, step=t if i == a else -1))
    return runs + list(specs[b:])


def kenovik_config(cfg: Dict[str, Any]) -> ModelConfig:
    """Kenovik: RG-LRU layers and two kinds of attention (biased projections with a fixed sink; distance bias with normed
    projections and a query temperature), dense or expert feed-forwards, some of the layers run several times."""
    loop = cfg.get("loop")
    specs = _unrolled([_kenovik_layer(lc) for lc in cfg["layers"]], loop)
    widest = lambda k: max([s.overrides.get(k, 0) for s in specs] + [0])
    c = ModelConfig(model_type="kenovik", family="hybrid", vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]),
                    intermediate_size=max(1, widest("intermediate_size"), widest("moe_intermediate_size")), num_hidden_layers=len(specs),
                    num_attention_heads=1, num_key_value_heads=1, head_dim=64, rms_norm_eps=float(cfg["norm"]["eps"]), input_norms=True,
                    embed_scale=float(cfg["embedding"]["scale"]), loop_steps=int(loop["times"]) if loop else 0, tie_word_embeddings=True,
                    layer_specs=specs, dtype=str(cfg.get("torch_dtype", cfg.get("dtype", "bfloat16"))),
                    quant=QuantConfig(kv_cache_dtype="bf16"), bos_token_id=cfg.get("bos_token_id"), eos_token_id=cfg.get("eos_token_id"))
    c.moe_intermediate_size = widest("moe_intermediate_size")
    return _size_by_heads(c)


def _bisudra_ff(mlp: Dict[str, Any]) -> Dict[str, Any]:
    if mlp.get("kind", "dense") == "dense":
        return {"intermediate_size": int(mlp["ff"]), "mlp_activation": "relu2", "mlp_bias": True}
    if mlp["kind"] != "moe":
        raise ValueError(f"unsupported Bisudra feed-forward '{mlp['kind']}'")
    r = mlp["router"]
    if not 1 <= int(r["top"]) <= int(r["experts"]):
        raise ValueError(f"{r['top']} of {r['experts']} experts per token")
    return {"num_experts": int(r["experts"]), "num_experts_per_tok": int(r["top"]), "moe_intermediate_size": int(mlp["expert"]["ff"]),
            "mlp_activation": "silu_unit", "norm_topk_prob": True, "router_scoring": "softmax", "router_f32": True, "router_logit_bias": True}


def _bisudra_layer(lc: Dict[str, Any]) -> LayerSpec:
    if lc["type"] != "attention":
        raise ValueError(f"unsupported Bisudra layer type '{lc['type']}'")
    m, mlp = lc["mixer"], lc.get("mlp")
    mask = m.get("mask")
    over = {**_attention_overrides(m), "attn_diff": float(m["diff"]), "attn_output_gate": True, "qk_norm": True, "qk_norm_plus_one": False,
            "sliding_window": int(mask["size"]) if mask else None}
    over["attn_cache_width"] = padded_head_width(2 * over["head_dim"], over["v_head_dim"])      # a cached key holds both maps' keys
    if mlp is not None:
        over.update(_bisudra_ff(mlp))
    return LayerSpec("differential", mlp is not None, over)


def bisudra_config(cfg: Dict[str, Any]) -> ModelConfig:
    """Bisudra: differential attention in a sliding window behind an input convolution, dense or expert feed-forwards, gated and
    layer-normed sublayer outputs, a token input per layer, depth averages."""
    specs = [_bisudra_layer(lc) for lc in cfg["layers"]]
    widest = lambda k: max([s.overrides.get(k, 0) for s in specs] + [0])
    c = ModelConfig(model_type="bisudra", family="hybrid", vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]),
                    intermediate_size=max(1, widest("intermediate_size"), widest("moe_intermediate_size")), num_hidden_layers=len(specs),
                    num_attention_heads=1, num_key_value_heads=1, head_dim=64, rms_norm_eps=float(cfg["norm"]["eps"]), output_norms=True,
                    layer_norms=True, sublayer_gates=True, input_conv_taps=int(cfg["canon"]["taps"]), token_side_dim=int(cfg["token_side"]["dim"]),
                    depth_average=True, tie_word_embeddings=True, layer_specs=specs, dtype=str(cfg.get("torch_dtype", cfg.get("dtype", "bfloat16"))),
                    quant=QuantConfig(kv_cache_dtype="bf16"), bos_token_id=cfg.get("bos_token_id"), eos_token_id=cfg.get("eos_token_id"))
    c.moe_intermediate_size = widest("moe_intermediate_size")
    return _size_by_heads(c)


# ``architecture`` of a config.json that lists its layers one by one -> its reader
_NATIVE_ARCHITECTURES = {"papidra": papidra_config, "tomizen": tomizen_config, "kenovik": kenovik_config, "bisudra": bisudra_config}


# ---------------------------------------------------------------------------- presets
def tiny_dense(dtype: str = "float32") -> ModelConfig:
    """2-layer plumbing model: hidden 256, 4q/2kv heads x 64, FFN 512, vocab 1024."""
    return ModelConfig(model_type="llama", family="dense", vocab_size=1024, hidden_size=256,
                       intermediate_size=512, num_hidden_layers=2, num_attention_heads=4,
                       num_key_value_heads=2, head_dim=64, rms_norm_eps=1e-6, rope_theta=1e6,
                       max_position_embeddings=4096, dtype=dtype)


def llama3_8b(quant: str = "fp8_block") -> ModelConfig:
    return ModelConfig(model_type="llama", family="dense", vocab_size=128256, hidden_size=4096,
                       intermediate_size=14336, num_hidden_layers=32, num_attention_heads=32,
                       num_key_value_heads=8, head_dim=128, rms_norm_eps=1e-5, rope_theta=5e5,
                       max_position_embeddings=8192,
                       quant=QuantConfig(method=quant, kv_cache_dtype="fp8" if quant != "none" else "auto"))


def llama3_70b(quant: str = "fp8_block") -> ModelConfig:
    return ModelConfig(model_type="llama", family="dense", vocab_size=128256, hidden_size=8192,
                       intermediate_size=28672, num_hidden_layers=80, num_attention_heads=64,
                       num_key_value_heads=8, head_dim=128, rms_norm_eps=1e-5, rope_theta=5e5,
                       max_position_embeddings=65536,
                       quant=QuantConfig(method=quant, kv_cache_dtype="fp8" if quant != "none" else "auto"))


def qwen3_30b_a3b(quant: str = "nvfp4") -> ModelConfig:
    return ModelConfig(model_type="qwen3_moe", family="moe", vocab_size=151936, hidden_size=2048,
                       intermediate_size=6144, num_hidden_layers=48, num_attention_heads=32,
                       num_key_value_heads=4, head_dim=128, rms_norm_eps=1e-6, rope_theta=1e6,
                       qk_norm=True, num_experts=128, num_experts_per_tok=8, moe_intermediate_size=768,
                       norm_topk_prob=True, max_position_embeddings=40960,
                       quant=QuantConfig(method=quant, experts_only=True, kv_cache_dtype="fp8"))


def qwen3_next_80b(quant: str = "fp8_block") -> ModelConfig:
    return ModelConfig(model_type="qwen3_next", family="hybrid", vocab_size=151936, hidden_size=2048,
                       intermediate_size=5120, num_hidden_layers=48, num_attention_heads=16,
                       num_key_value_heads=2, head_dim=256, rms_norm_eps=1e-6, rope_theta=1e7,
                       partial_rotary_factor=0.25, qk_norm=True, attn_output_gate=True, norm_plus_one=True,
                       num_experts=512, num_experts_per_tok=10, moe_intermediate_size=512,
                       shared_expert_intermediate_size=512, norm_topk_prob=True,
                       full_attention_interval=4, linear_num_key_heads=16, linear_num_value_heads=32,
                       linear_key_head_dim=128, linear_value_head_dim=128, linear_conv_kernel_dim=4,
                       mtp_num_layers=1, max_position_embeddings=262144,
                       quant=QuantConfig(method=quant, kv_cache_dtype="fp8"))


def tiny_moe(dtype: str = "float32") -> ModelConfig:
    return ModelConfig(model_type="qwen3_moe", family="moe", vocab_size=1024, hidden_size=256,
                       intermediate_size=512, num_hidden_layers=2, num_attention_heads=4,
                       num_key_value_heads=2, head_dim=64, rope_theta=1e6, qk_norm=True,
                       num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128,
                       max_position_embeddings=4096, dtype=dtype)


def tiny_hybrid(dtype: str = "float32") -> ModelConfig:
    return ModelConfig(model_type="qwen3_next", family="hybrid", vocab_size=1024, hidden_size=256,
                       intermediate_size=512, num_hidden_layers=4, num_attention_heads=4,
                       num_key_value_heads=2, head_dim=64, rope_theta=1e6, partial_rotary_factor=0.25,
                       qk_norm=True, attn_output_gate=True, norm_plus_one=True,
                       num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128,
                       shared_expert_intermediate_size=128, full_attention_interval=4,
                       linear_num_key_heads=2, linear_num_value_heads=4, linear_key_head_dim=32,
                       linear_value_head_dim=32, linear_conv_kernel_dim=4, mtp_num_layers=1,
                       max_position_embeddings=4096, dtype=dtype)


def tiny_nemotron_h(dtype: str = "float32") -> ModelConfig:
    """Nemotron-H style stack of single-module blocks: Mamba-2, position-free attention and relu^2 MLP."""
    return ModelConfig(model_type="nemotron_h", family="hybrid", vocab_size=1024, hidden_size=256, intermediate_size=512,
                       num_hidden_layers=6, num_attention_heads=4, num_key_value_heads=2, head_dim=64,
                       partial_rotary_factor=0.0, rms_norm_eps=1e-5,
                       block_types=["mamba", "mlp", "mamba", "attention", "mlp", "mamba"], mamba_num_heads=8,
                       mamba_head_dim=32, ssm_state_size=32, mamba_n_groups=2, mamba_conv_kernel=4, mamba_dt_min=0.001,
                       mlp_activation="relu2", max_position_embeddings=4096, dtype=dtype)


def tiny_deepseek(dtype: str = "float32") -> ModelConfig:
    """DeepSeek-V3 style: latent attention, a leading dense layer, then MoE layers with a group-limited sigmoid router,
    selection bias, weight scale and an ungated shared expert."""
    return ModelConfig(model_type="deepseek_v3", family="moe", vocab_size=1024, hidden_size=256, intermediate_size=512,
                       num_hidden_layers=3, num_attention_heads=4, num_key_value_heads=4, head_dim=64,
                       partial_rotary_factor=0.25, kv_lora_rank=64, q_lora_rank=96, qk_nope_head_dim=32, qk_rope_head_dim=16,
                       v_head_dim=32, num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128,
                       shared_expert_intermediate_size=128, first_k_dense_replace=1, router_scoring="sigmoid",
                       router_selection_bias=True, router_n_group=4, router_topk_group=2, routed_scaling_factor=2.5,
                       max_position_embeddings=4096, dtype=dtype)


def _papidra(vocab: int, width: int, ff: int, pattern: str, streams: int, wkv: tuple, attn: tuple, mamba: tuple, chunk: int,
             dtype: str) -> ModelConfig:
    """``pattern``: ``w`` = WKV layer without feed-forward, ``p`` = parallel layer with one; ``wkv`` (heads, dim), ``attn``
    (heads, kv heads, dim), ``mamba`` (heads, channels, state, groups)."""
    left = {"heads": attn[0], "kv_heads": attn[1], "dim": attn[2], "vdim": attn[2], "scale": attn[2] ** -0.5, "mask": {"size": chunk},
            "rot": {"base": 5e5, "dims": attn[2], "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}
    right = {"heads": mamba[0], "vdim": mamba[1], "state": mamba[2], "groups": mamba[3], "norm_groups": mamba[3], "conv": 4}
    layers = [{"type": "wkv", "mixer": {"heads": wkv[0], "dim": wkv[1]}, "mlp": None} if ch == "w" else
              {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": {"kind": "dense", "ff": ff, "limit": 7.0}}
              for ch in pattern]
    return papidra_config({"vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": width ** 0.5},
                           "streams": streams, "layers": layers, "dtype": dtype})


def tiny_papidra(dtype: str = "float32") -> ModelConfig:
    c = _papidra(1024, 256, 384, "wpwp", 2, (4, 64), (4, 2, 64), (8, 32, 32, 2), 48, dtype)
    c.max_position_embeddings = 4096
    return c


def papidra_8b(quant: str = "none") -> ModelConfig:
    """Layers of the size of an 8B decoder: width 4096, 32 heads of 128 (8 kv), 128 Mamba-2 heads of 64, 64 WKV heads of 64."""
    c = _papidra(131072, 4096, 14336, "wp" * 16, 4, (64, 64), (32, 8, 128), (128, 64, 128, 8), 4096, "bfloat16")
    c.quant = QuantConfig(method=quant, kv_cache_dtype="bf16")
    return c


def nemotron_h_8b(quant: str = "none") -> ModelConfig:
    pattern = "M-M-M-MM-M-M-M*-M-M-M*-M-M-M-M*-M-M-M-M*-M-MM-M-M-M-M-M-"
    blocks = [{"M": "mamba", "*": "attention", "-": "mlp"}[ch] for ch in pattern]
    return ModelConfig(model_type="nemotron_h", family="hybrid", vocab_size=131072, hidden_size=4096, intermediate_size=21504,
                       num_hidden_layers=len(blocks), num_attention_heads=32, num_key_value_heads=8, head_dim=128,
                       partial_rotary_factor=0.0, rms_norm_eps=1e-5, block_types=blocks, mamba_num_heads=128, mamba_head_dim=64,
                       ssm_state_size=128, mamba_n_groups=8, mamba_conv_kernel=4, mamba_dt_min=0.001, mlp_activation="relu2",
                       max_position_embeddings=8192, quant=QuantConfig(method=quant, kv_cache_dtype="fp8"))


def _tomizen(vocab: int, width: int, pattern: str, mlstm: tuple, latent: tuple, attn: tuple, experts: tuple, dtype: str) -> ModelConfig:
    """``pattern``: ``m`` = mLSTM, ``l`` = latent attention, ``a`` = attention; ``mlstm`` (heads, dim, vdim), ``latent`` (heads, dim,
    rot_dim, vdim, rank, window), ``attn`` (heads, kv heads, dim), ``experts`` (count, top, ff)."""
    lh, ld, lr, lv, rank, window = latent
    mixers = {
        "m": ("mlstm", {"heads": mlstm[0], "dim": mlstm[1], "vdim": mlstm[2], "gate_cap": 15.0}),
        "l": ("latent_attention", {"heads": lh, "dim": ld, "rot_dim": lr, "vdim": lv, "kv_rank": rank, "scale": (ld + lr) ** -0.5,
                                   "mask": {"size": window}, "rot": {"base": 5e5, "dims": lr, "scaling": {
                                       "factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}),
        "a": ("attention", {"heads": attn[0], "kv_heads": attn[1], "dim": attn[2], "vdim": attn[2], "scale": attn[2] ** -0.5, "softcap": 30.0})}
    mlp = {"kind": "moe", "expert": {"ff": experts[2]}, "router": {"experts": experts[0], "top": experts[1]}}
    return tomizen_config({"vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "dtype": dtype,
                           "layers": [{"type": mixers[ch][0], "mixer": mixers[ch][1], "mlp": mlp} for ch in pattern]})


def tiny_tomizen(dtype: str = "float32") -> ModelConfig:
    c = _tomizen(1024, 192, "mlam", (3, 32, 48), (6, 40, 24, 56, 96, 72), (6, 2, 64), (8, 3, 96), dtype)
    c.max_position_embeddings = 4096
    return c


def tomizen_16b(quant: str = "none") -> ModelConfig:
    """Layers of the size of a 16B mixture-of-experts decoder: width 2048, 16 mLSTM heads of 128 / 256, 16 latent heads on rank 512,
    16 attention heads of 128 (2 kv), 64 experts of 1408 (6 per token)."""
    c = _tomizen(131072, 2048, "mlam" * 8, (16, 128, 256), (16, 64, 64, 128, 512, 4096), (16, 2, 128), (64, 6, 1408), "bfloat16")
    c.quant = QuantConfig(method=quant, kv_cache_dtype="bf16")
    return c


def _kenovik(vocab: int, width: int, pattern: str, lru: tuple, attn: tuple, attn2: tuple, ff: int, experts: tuple, loop: Optional[tuple],
             dtype: str) -> ModelConfig:
    """``pattern``: ``r`` = RG-LRU, ``a`` = attention with a fixed sink, ``d`` = attention with a distance bias, each with experts;
    a capital letter has a dense feed-forward of ``ff`` instead.  ``lru`` (width, blocks), ``attn`` (heads, kv heads, dim, vdim,
    rotated), ``attn2`` (heads, kv heads, dim, vdim, reach), ``experts`` (count, top, ff, groups, kept), ``loop`` (start, stop, times)."""
    mixers = {
        "r": ("rglru", {"width": lru[0], "blocks": lru[1], "conv": 4}),
        "a": ("attention", {"heads": attn[0], "kv_heads": attn[1], "dim": attn[2], "vdim": attn[3], "scale": attn[2] ** -0.5,
                            "rot": {"base": 5e5, "dims": attn[4], "scaling": {"factor": 4.0}}}),
        "d": ("attention_2", {"heads": attn2[0], "kv_heads": attn2[1], "dim": attn2[2], "vdim": attn2[3], "scale": attn2[2] ** -0.5,
                              "bias_max": attn2[4], "q_temp": {"coef": 0.1, "every": 8192}})}
    e, top, eff, groups, keep = experts
    moe = {"kind": "moe", "expert": {"ff": eff, "limit": 7.0}, "shared": {"ff": eff, "limit": 7.0},
           "router": {"experts": e, "top": top, "scale": 2.5, "groups": {"count": groups, "keep": keep}}}
    layers = [{"type": mixers[ch.lower()][0], "mixer": mixers[ch.lower()][1], "mlp": {"kind": "dense", "ff": ff} if ch.isupper() else moe}
              for ch in pattern]
    return kenovik_config({"vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5}, "dtype": dtype,
                           "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "layers": layers})


def tiny_kenovik(dtype: str = "float32") -> ModelConfig:
    c = _kenovik(1024, 192, "Drad", (144, 3), (6, 2, 64, 48, 32), (4, 2, 48, 64, 100), 256, (8, 3, 96, 4, 2), (1, 3, 2), dtype)
    c.max_position_embeddings = 4096
    return c


def kenovik_20b(quant: str = "none") -> ModelConfig:
    """Layers of the size of a 20B mixture-of-experts decoder: width 2048, RG-LRU of 2560 channels in 10 blocks, 16 heads of 128
    (2 kv), 64 experts of 1408 (6 per token, 8 groups of which 4 stay open), the middle eight layers run twice."""
    c = _kenovik(131072, 2048, "R" + "radr" * 7 + "rad", (2560, 10), (16, 2, 128, 128, 64), (16, 2, 128, 128, 4096), 8192,
                 (64, 6, 1408, 8, 4), (12, 20, 2), "bfloat16")
    c.quant = QuantConfig(method=quant, kv_cache_dtype="bf16")
    return c


def _bisudra(vocab: int, width: int, pattern: str, attn: tuple, ff: int, experts: tuple, taps: int, side: int, dtype: str) -> ModelConfig:
    """``pattern``: ``d`` = layer with a dense feed-forward, ``e`` = with experts, ``n`` = without one; ``attn`` (heads, kv heads, dim,
    vdim, rotated, window), ``experts`` (count, top, ff)."""
    h, g, d, dv, rot, window = attn
    mlps = {"d": {"kind": "dense", "ff": ff}, "n": None,
            "e": {"kind": "moe", "expert": {"ff": experts[2]}, "router": {"experts": experts[0], "top": experts[1]}}}
    layers = [{"type": "attention", "mixer": {"heads": h, "kv_heads": g, "dim": d, "vdim": dv, "scale": d ** -0.5, "diff": min(0.8 - 0.6 * math.exp(-0.3 * i), 0.8),
                                              "mask": {"size": window}, "rot": {"base": 5e5, "dims": rot}}, "mlp": mlps[ch]}
              for i, ch in enumerate(pattern)]
    return bisudra_config({"vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "canon": {"taps": taps}, "token_side": {"dim": side},
                           "layers": layers, "dtype": dtype})


def tiny_bisudra(dtype: str = "float32") -> ModelConfig:
    c = _bisudra(1024, 192, "dedn", (6, 2, 24, 40, 16, 72), 256, (8, 3, 72), 4, 20, dtype)
    c.max_position_embeddings = 4096
    return c


def bisudra_8b(quant: str = "none") -> ModelConfig:
    """Layers of the size of an 8B mixture-of-experts decoder: width 2048, 16 heads of two maps of 64 and values of 128 (4 kv),
    64 experts of 1408 (6 per token) in every second layer."""
    c = _bisudra(131072, 2048, "de" * 12, (16, 4, 64, 128, 64, 4096), 8192, (64, 6, 1408), 4, 128, "bfloat16")
    c.quant = QuantConfig(method=quant, kv_cache_dtype="bf16")
    return c


PRESETS = {
    "tiny-dense": tiny_dense, "tiny-moe": tiny_moe, "tiny-hybrid": tiny_hybrid,
    "llama3-8b": llama3_8b, "llama3-70b": llama3_70b,
    "qwen3-30b-a3b": qwen3_30b_a3b, "qwen3-next-80b": qwen3_next_80b,
    "tiny-nemotron-h": tiny_nemotron_h, "nemotron-h-8b": nemotron_h_8b, "tiny-deepseek": tiny_deepseek,
    "tiny-papidra": tiny_papidra, "papidra-8b": papidra_8b, "tiny-tomizen": tiny_tomizen, "tomizen-16b": tomizen_16b,
    "tiny-kenovik": tiny_kenovik, "kenovik-20b": kenovik_20b, "tiny-bisudra": tiny_bisudra, "bisudra-8b": bisudra_8b,
}


@dataclass
class EngineConfig:
    """Serving knobs (same names/defaults as the reference's serve flags,
    ``crates/spark-server/src/cli/serve_args.rs``)."""
    max_seq_len: int = 32768
    block_size: int = 16
    kv_cache_dtype: str = "auto"
    sparse_attention_blocks: int = 0          # > 0: decode attention reads at most this many KV blocks per sequence
    async_decode: bool = True                 # lag-one decode pipeline for plain greedy decode steps (GPU, CUDA graphs)
    kv_high_precision_layers: tuple = ()      # attention layers that keep a 16-bit cache when kv_cache_dtype is fp8
    gpu_memory_utilization: float = 0.90
    num_kv_blocks: Optional[int] = None       # explicit override (tests / CPU)
    max_num_seqs: int = 128
    max_batch_size: int = 128                 # decode batch cap per step
    max_prefill_tokens: int = 8192
    scheduling_policy: str = "fifo"           # fifo | slai
    tbt_deadline_ms: float = 100.0
    enable_prefix_caching: bool = True
    speculative: bool = False
    num_drafts: int = 0
    mtp_gate: bool = True
    mtp_draft_vocab: int = 0                  # > 0: draft steps score this many rows of the lm_head (a quantised draft-only head)
    mtp_vocab_rank: str = "id"                # "id": the first rows; or the path of a ranked-ids table (utils/vocab_rank.py)
    dcut_ratio: float = 0.0                   # > 0: keep this fraction of the batch's draft rows, ranked by drafter confidence
    ngram_speculative: bool = False           # prompt-lookup drafts (no draft model); uses num_drafts
    self_speculative: bool = False            # layer-skipping drafts from the target model itself; uses num_drafts
    self_spec_keep: float = 0.5               # fraction of the layers the draft pass runs (first and last always kept)
    ngram_max: int = 4
    ngram_min: int = 2
    ssm_cache_slots: int = 16
    ssm_checkpoint_interval: int = 256
    swap_space_gb: float = 0.0
    disk_swap_gb: float = 0.0               # file-backed tier below the host tier (0 = off)
    disk_swap_path: str = ""                # directory of the swap file (default: the system temp directory)
    use_cuda_graphs: bool = True
    tp_size: int = 1
    ep_size: int = 1
    seed: int = 0
    admission_watermark_tokens: int = 256     # decode headroom reserved at admission
    request_timeout_s: float = 0.0
