"""Model and engine configuration.

Model hyper-parameters come from a checkpoint's ``config.json`` (``from_hf``) or
from a named preset (random-init benchmarking).  ``EngineConfig`` carries the
serving knobs that the CLI exposes.

Reference parity: pegainfer-qwen3/src/config.rs:213-262,465-506;
pegainfer-qwen35/src/config.rs:26-215; pegainfer-deepseek-v2-lite/src/config.rs:69-190;
pegainfer-kimi-k2/src/config.rs:16-140; pegainfer-frontend/src/model_line.rs:93-206
(shared serving flags).
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field, replace
from typing import Optional


@dataclass(frozen=True)
class MixerSpec:
    """Token mixer of one layer, for families whose layers are listed one by one.  ``kind``: ``"attention"`` (all fields but
    the recurrent and latent ones), ``"lightning"`` (fixed decay per head), ``"channel_delta"`` (gated delta rule with a decay
    per key channel; ``conv`` taps, low-rank decay and output-gate projections of the given ranks) or ``"latent"`` (attention
    over a cached latent of ``kv_rank`` columns and, with ``rot_dims``, a shared rotated key part; queries through a latent of
    ``q_rank``, or straight from the stream without one; a sliding window, an element-wise or per-head output gate and a sink
    are optional) or ``"wkv"`` (token-shift mixes, a decay per key channel from a low-rank projection of ``decay_rank``, a bonus
    for the current token), ``"ssd"`` (state-space duality: one decay per token and head, ``dim`` state rows, ``kv_heads`` groups
    of heads that share them, a convolution, a gate in front of a norm in ``norm_groups`` parts), ``"lru"`` (gated linear
    recurrence per channel over ``heads`` blocks of ``dim`` channels, a convolution, a GELU branch) or ``"parallel"`` (the mixers
    ``parts`` side by side over one input, each times its ``part_scales``)."""

    kind: str
    heads: int
    dim: int  # query / key size of a head
    vdim: int
    kv_heads: int = 0  # attention: KV heads; channel_delta: query / key heads
    scale: float = 1.0
    softcap: float = 0.0  # 0: no cap
    rot_dims: int = 0
    rot_base: float = 10000.0
    kv_from: int = -1  # attention: layer whose cache this layer reads (-1: its own)
    decay: tuple = ()
    conv: int = 0
    decay_rank: int = 0
    gate_rank: int = 0
    q_rank: int = 0
    kv_rank: int = 0
    window: int = 0  # a position sees itself and the window - 1 before it (0: all before it)
    out_gate: bool = False
    yarn: tuple = ()  # (factor, original, fast, slow) of the rotation, or none
    head_gate: bool = False  # latent: the sigmoid of one number per head multiplies the head's output
    sink: bool = False  # latent: a learned number per head in the softmax's denominator
    head_norm: bool = False  # attention: query and key norms per head (False: over the whole projection)
    values_are_keys: bool = False  # attention: no value projection, the values are the projected keys before their norm
    q_temp: tuple = ()  # attention: (coef, every): queries at position p times 1 + coef * ln(floor((p + 1) / every) + 1)
    bias: bool = False  # attention: query, key and value projections have biases
    head_temp: bool = False  # attention: a learned factor per head on the scores
    slopes: tuple = ()  # attention: per head, what the (capped) score loses per position of distance
    norm_groups: int = 0
    parts: tuple = ()
    part_scales: tuple = ()

    def flat(self) -> tuple:
        """The mixer, or those it has side by side."""
        return self.parts or (self,)


@dataclass(frozen=True)
class ExpertsSpec:
    """Mixture-of-experts feed-forward: ``scoring`` (softmax or sigmoid) over ``experts``, the ``top`` best of the ``keep`` best
    of ``groups`` groups of neighbours (a group counts as its best expert); with ``correction`` a learned number per expert is
    added for the choice only; the chosen scores are the weights, divided by their sum with ``norm`` and times ``scale``.  An
    expert of width ``ff`` is an up projection, the squared ReLU and a down projection (``act`` relu2), or gate and up
    projections with SiLU (``act`` swiglu).  ``shared_ff``: width of an expert that runs for every token, times the sigmoid of
    one number per token (0: none)."""

    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1
    scoring: str = "softmax"
    correction: bool = False
    norm: bool = False
    scale: float = 1.0
    act: str = "relu2"
    shared_ff: int = 0


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    ff: int = 0  # width of the gated feed-forward (0: the layer has none)
    moe: Optional[ExpertsSpec] = None
    act: str = "silu"  # of the feed-forward's gate: silu or gelu_tanh; xielu (two learned numbers): a feed-forward without gate


@dataclass
class ModelConfig:
    family: str = "qwen3"  # qwen3 | qwen35 | deepseek_v2 | kimi_k2 | glm_dsa | gemma4 | kimi_k3 | nemipel | vekalorn | zeripel | nonetar
    vocab_size: int = 1024
    hidden_size: int = 256
    num_layers: int = 2
    num_q_heads: int = 4
    num_kv_heads: int = 2
    head_dim: int = 64
    intermediate_size: int = 768
    rms_eps: float = 1e-6
    rope_theta: float = 1e6
    max_position: int = 4096
    tie_word_embeddings: bool = False
    eos_token_ids: tuple = ()
    qk_norm: bool = True
    # Qwen3.5 hybrid
    layer_types: tuple = ()  # "linear_attention" | "full_attention" per layer
    partial_rotary_factor: float = 1.0
    attn_output_gate: bool = False
    norm_weight_offset: bool = False  # (1 + w) RMSNorm
    gdn_num_k_heads: int = 0
    gdn_num_v_heads: int = 0
    gdn_head_dim: int = 128
    gdn_conv_kernel: int = 4
    # MLA
    q_lora_rank: int = 0
    kv_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    rope_scaling: Optional[dict] = None
    # MoE
    n_routed_experts: int = 0
    n_shared_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    first_k_dense_replace: int = 0
    scoring_func: str = "softmax"
    n_group: int = 1
    topk_group: int = 1
    norm_topk_prob: bool = False
    routed_scaling_factor: float = 1.0
    router_bias: bool = False
    expert_quant: str = "bf16"  # bf16 | int4_g32 | fp8_block128 | mxfp4 (Kimi-K3 checkpoints; dequantised to bf16 when loaded)
    quant_group_size: int = 32
    dense_quant: str = "bf16"  # bf16 | fp8_block128: projections outside the experts stay FP8 and run the FP8 GEMM
    # MTP
    num_mtp_layers: int = 0
    # sparse attention indexer (GLM-5 line): every query keeps its index_topk best-scoring keys
    index_topk: int = 0
    index_head_dim: int = 128
    index_n_heads: int = 0
    # Gemma 4 line: sliding-window layers (head_dim, num_kv_heads, rope_theta_local, full rotary) interleaved with global
    # layers (global_head_dim, num_global_kv_heads, rope_theta, partial_rotary_factor of the head rotated); layer_types
    # holds "sliding_attention" | "full_attention"
    sliding_window: int = 0
    global_head_dim: int = 0
    num_global_kv_heads: int = 0
    attention_k_eq_v: bool = False  # global layers have no v_proj: V is the key projection (before key norm and RoPE)
    final_logit_softcapping: float = 0.0
    rope_theta_local: float = 10000.0
    hidden_act: str = "silu"  # "silu" | "gelu_tanh" | "situ"
    # Kimi-K3 line: KDA linear-attention layers ("linear_attention", gdn_head_dim / gdn_conv_kernel give the head and the
    # short convolution) interleaved with NoPE MLA layers ("full_attention"), routed experts that work in a latent of
    # latent_moe_dim columns, and the attention-residual stream that snapshots the residual every attn_res_block layers
    latent_moe_dim: int = 0
    attn_res_block: int = 0
    kda_gate_rank: int = 0
    kda_gate_lower_bound: float = -5.0
    # families whose layers are listed one by one (Nemipel, Vekalorn, Zeripel, Nonetar lines): the mixer and feed-forward of every layer, the factor on
    # the stream in the norm after the sum; final_logit_softcapping caps the logits
    layer_specs: tuple = ()
    postln_alpha: float = 1.0
    # Zeripel line: factor on the token embedding, table of token pairs (buckets, mul_prev, mul_cur), factor on a sublayer's output
    embed_scale: float = 1.0
    bigram: tuple = ()
    residual_mult: float = 1.0
    # Nonetar line: copies of the residual stream, factor on the logits
    streams: int = 1
    logit_scale: float = 1.0

    # -- derived ---------------------------------------------------------------
    @property
    def q_size(self) -> int:
        return self.num_q_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    @property
    def rotary_dim(self) -> int:
        return int(self.head_dim * self.partial_rotary_factor)

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0

    @property
    def is_moe(self) -> bool:
        return self.n_routed_experts > 0

    @property
    def qk_head_dim(self) -> int:
        return self.qk_nope_head_dim + self.qk_rope_head_dim

    def layer_is_moe(self, i: int) -> bool:
        return self.is_moe and i >= self.first_k_dense_replace

    def layer_type(self, i: int) -> str:
        return self.layer_types[i] if self.layer_types else "full_attention"

    def mla_softmax_scale(self) -> float:
        scale = 1.0 / math.sqrt(self.qk_head_dim)
        rs = self.rope_scaling or {}
        if rs.get("type", rs.get("rope_type")) == "yarn":
            m = yarn_get_mscale(rs.get("factor", 1.0), rs.get("mscale_all_dim", 0.0))
            scale *= m * m
        return scale

    def param_count(self) -> int:
        """Approximate parameter count (for memory planning)."""
        h = self.hidden_size
        per_layer = 0
        if self.is_mla:
            q = (h * self.q_lora_rank + self.q_lora_rank * self.num_q_heads * self.qk_head_dim) if self.q_lora_rank else h * self.num_q_heads * self.qk_head_dim
            kv = h * (self.kv_lora_rank + self.qk_rope_head_dim) + self.kv_lora_rank * self.num_q_heads * (self.qk_nope_head_dim + self.v_head_dim)
            per_layer += q + kv + self.num_q_heads * self.v_head_dim * h
        else:
            per_layer += h * (self.q_size + 2 * self.kv_size) + self.q_size * h
        dense = 3 * h * self.intermediate_size
        moe = 3 * h * self.moe_intermediate_size * (self.n_routed_experts + self.n_shared_experts) + h * self.n_routed_experts
        n_moe = max(0, self.num_layers - self.first_k_dense_replace) if self.is_moe else 0
        total = self.num_layers * per_layer + (self.num_layers - n_moe) * dense + n_moe * moe
        total += self.vocab_size * h * (1 if self.tie_word_embeddings else 2)
        return total


def yarn_get_mscale(scale: float, mscale: float) -> float:
    """YaRN attention-scale correction (pegainfer-deepseek-v2-lite/src/host_ops.rs:377-386)."""
    if scale <= 1.0:
        return 1.0
    return 0.1 * mscale * math.log(scale) + 1.0


def _hybrid_pattern(n: int) -> tuple:
    return tuple("full_attention" if (i + 1) % 4 == 0 else "linear_attention" for i in range(n))


_YARN_DSV2 = {"type": "yarn", "factor": 40.0, "original_max_position_embeddings": 4096, "beta_fast": 32, "beta_slow": 1, "mscale": 0.707, "mscale_all_dim": 0.707}
_YARN_KIMI = {"type": "yarn", "factor": 64.0, "original_max_position_embeddings": 4096, "beta_fast": 32, "beta_slow": 1, "mscale": 1.0, "mscale_all_dim": 1.0}

PRESETS = {
    "tiny-qwen3": ModelConfig(),
    "qwen3-0.6b": ModelConfig(vocab_size=151936, hidden_size=1024, num_layers=28, num_q_heads=16, num_kv_heads=8, head_dim=128, intermediate_size=3072, max_position=40960, tie_word_embeddings=True),
    "qwen3-4b": ModelConfig(vocab_size=151936, hidden_size=2560, num_layers=36, num_q_heads=32, num_kv_heads=8, head_dim=128, intermediate_size=9728, max_position=40960, tie_word_embeddings=True),
    "qwen3-8b": ModelConfig(vocab_size=151936, hidden_size=4096, num_layers=36, num_q_heads=32, num_kv_heads=8, head_dim=128, intermediate_size=12288, max_position=40960),
    "tiny-qwen35": ModelConfig(family="qwen35", vocab_size=1024, hidden_size=256, num_layers=4, num_q_heads=4, num_kv_heads=2, head_dim=64, intermediate_size=512, layer_types=_hybrid_pattern(4), partial_rotary_factor=0.25, attn_output_gate=True, norm_weight_offset=True, gdn_num_k_heads=2, gdn_num_v_heads=4, gdn_head_dim=32, rope_theta=1e7),
    "qwen3.5-27b": ModelConfig(family="qwen35", vocab_size=248320, hidden_size=5120, num_layers=64, num_q_heads=24, num_kv_heads=4, head_dim=256, intermediate_size=17408, layer_types=_hybrid_pattern(64), partial_rotary_factor=0.25, attn_output_gate=True, norm_weight_offset=True, gdn_num_k_heads=16, gdn_num_v_heads=48, gdn_head_dim=128, rope_theta=1e7, max_position=262144),
    "tiny-dsv2": ModelConfig(family="deepseek_v2", vocab_size=1024, hidden_size=256, num_layers=3, num_q_heads=4, num_kv_heads=4, head_dim=48, intermediate_size=512, qk_norm=False, kv_lora_rank=64, qk_nope_head_dim=32, qk_rope_head_dim=16, v_head_dim=32, n_routed_experts=8, n_shared_experts=2, num_experts_per_tok=2, moe_intermediate_size=128, first_k_dense_replace=1, rope_theta=10000.0, rope_scaling=dict(_YARN_DSV2)),
    "small-dsv2": ModelConfig(family="deepseek_v2", vocab_size=4096, hidden_size=1024, num_layers=3, num_q_heads=16, num_kv_heads=16, head_dim=192, intermediate_size=2048, qk_norm=False, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128, n_routed_experts=16, n_shared_experts=2, num_experts_per_tok=4, moe_intermediate_size=256, first_k_dense_replace=1, rope_theta=10000.0, rope_scaling=dict(_YARN_DSV2), max_position=8192),
    "small-kimi": ModelConfig(family="kimi_k2", vocab_size=4096, hidden_size=1024, num_layers=3, num_q_heads=16, num_kv_heads=16, head_dim=192, intermediate_size=2048, qk_norm=False, q_lora_rank=512, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128, n_routed_experts=32, n_shared_experts=1, num_experts_per_tok=4, moe_intermediate_size=256, first_k_dense_replace=1, scoring_func="sigmoid", n_group=4, topk_group=2, norm_topk_prob=True, routed_scaling_factor=2.827, router_bias=True, expert_quant="int4_g32", rope_theta=50000.0, rope_scaling=dict(_YARN_KIMI), rms_eps=1e-5, max_position=8192, num_mtp_layers=1),
    "small-qwen35": ModelConfig(family="qwen35", vocab_size=4096, hidden_size=1024, num_layers=4, num_q_heads=8, num_kv_heads=2, head_dim=256, intermediate_size=2048, layer_types=_hybrid_pattern(4), partial_rotary_factor=0.25, attn_output_gate=True, norm_weight_offset=True, gdn_num_k_heads=4, gdn_num_v_heads=8, gdn_head_dim=128, rope_theta=1e7, max_position=8192),
    "dsv2-lite": ModelConfig(family="deepseek_v2", vocab_size=102400, hidden_size=2048, num_layers=27, num_q_heads=16, num_kv_heads=16, head_dim=192, intermediate_size=10944, qk_norm=False, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128, n_routed_experts=64, n_shared_experts=2, num_experts_per_tok=6, moe_intermediate_size=1408, first_k_dense_replace=1, rope_theta=10000.0, rope_scaling=dict(_YARN_DSV2), max_position=163840),
    "tiny-kimi": ModelConfig(family="kimi_k2", vocab_size=1024, hidden_size=256, num_layers=3, num_q_heads=4, num_kv_heads=4, head_dim=48, intermediate_size=512, qk_norm=False, q_lora_rank=96, kv_lora_rank=64, qk_nope_head_dim=32, qk_rope_head_dim=16, v_head_dim=32, n_routed_experts=16, n_shared_experts=1, num_experts_per_tok=4, moe_intermediate_size=128, first_k_dense_replace=1, scoring_func="sigmoid", n_group=4, topk_group=2, norm_topk_prob=True, routed_scaling_factor=2.827, router_bias=True, expert_quant="int4_g32", rope_theta=50000.0, rope_scaling=dict(_YARN_KIMI), rms_eps=1e-5, num_mtp_layers=1),
    "kimi-k2": ModelConfig(family="kimi_k2", vocab_size=163840, hidden_size=7168, num_layers=61, num_q_heads=64, num_kv_heads=64, head_dim=192, intermediate_size=18432, qk_norm=False, q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128, n_routed_experts=384, n_shared_experts=1, num_experts_per_tok=8, moe_intermediate_size=2048, first_k_dense_replace=1, scoring_func="sigmoid", n_group=1, topk_group=1, norm_topk_prob=True, routed_scaling_factor=2.827, router_bias=True, expert_quant="int4_g32", rope_theta=50000.0, rope_scaling=dict(_YARN_KIMI), rms_eps=1e-5, max_position=131072, num_mtp_layers=1),
}
# the DeepSeek-V2 shapes with block-scaled FP8 e4m3 experts (128x128 scale blocks)
PRESETS["tiny-glm"] = ModelConfig(family="glm_dsa", vocab_size=1024, hidden_size=256, num_layers=3, num_q_heads=4, num_kv_heads=4, head_dim=48, intermediate_size=512, qk_norm=False, q_lora_rank=96,
                                  kv_lora_rank=64, qk_nope_head_dim=32, qk_rope_head_dim=16, v_head_dim=48, n_routed_experts=8, n_shared_experts=1, num_experts_per_tok=2, moe_intermediate_size=128,
                                  first_k_dense_replace=1, scoring_func="sigmoid", n_group=1, topk_group=1, norm_topk_prob=True, routed_scaling_factor=2.5, router_bias=True, rope_theta=10000.0,
                                  rms_eps=1e-5, index_topk=24, index_head_dim=32, index_n_heads=4, num_mtp_layers=1)
PRESETS["small-glm"] = replace(PRESETS["tiny-glm"], vocab_size=4096, hidden_size=1024, num_q_heads=16, num_kv_heads=16, head_dim=256, intermediate_size=2048, q_lora_rank=512, kv_lora_rank=512,
                               qk_nope_head_dim=192, qk_rope_head_dim=64, v_head_dim=256, n_routed_experts=16, num_experts_per_tok=4, moe_intermediate_size=256, index_topk=256, index_head_dim=128,
                               index_n_heads=32, max_position=8192)
# GLM-5 (zai-org/GLM-5): 78 layers, 256 routed experts, MLA with 192 + 64 query dims and 256 value dims, 32-head indexer keeping 2048 keys
PRESETS["glm-5"] = replace(PRESETS["small-glm"], vocab_size=154880, hidden_size=6144, num_layers=78, num_q_heads=64, num_kv_heads=64, intermediate_size=12288, q_lora_rank=2048, n_routed_experts=256,
                           num_experts_per_tok=8, moe_intermediate_size=2048, first_k_dense_replace=3, index_topk=2048, max_position=202752, rope_theta=1e6, expert_quant="fp8_block128")
def _gemma_pattern(n: int) -> tuple:
    return tuple("sliding_attention" if (i + 1) % 6 else "full_attention" for i in range(n))


PRESETS["tiny-gemma4"] = ModelConfig(family="gemma4", vocab_size=1024, hidden_size=256, num_layers=6, num_q_heads=4, num_kv_heads=2, head_dim=64, global_head_dim=128, num_global_kv_heads=1,
                                     attention_k_eq_v=True, intermediate_size=512, sliding_window=32, layer_types=_gemma_pattern(6), rope_theta=1e6, rope_theta_local=1e4,
                                     partial_rotary_factor=0.25, final_logit_softcapping=30.0, hidden_act="gelu_tanh", tie_word_embeddings=True, max_position=4096)
# head dims of the released dense model (256 sliding, 512 global, 5 : 1), two global KV heads of 512 as wide as four local ones of 256
PRESETS["small-gemma4"] = replace(PRESETS["tiny-gemma4"], vocab_size=4096, hidden_size=1024, num_q_heads=8, num_kv_heads=4, head_dim=256, global_head_dim=512, num_global_kv_heads=2,
                                  intermediate_size=2048, sliding_window=128, max_position=8192)
# a 10 B-parameter shape of the line for benchmarks (not a released configuration): 30 sliding + 6 global layers, 16 local
# KV heads of 256 against 4 global KV heads of 512 (the narrower global layers pack their pages at the front of their slab)
PRESETS["gemma4-10b-shape"] = replace(PRESETS["small-gemma4"], vocab_size=262144, hidden_size=4096, num_layers=36, layer_types=_gemma_pattern(36), num_q_heads=32, num_kv_heads=16,
                                      num_global_kv_heads=4, intermediate_size=14336, sliding_window=1024, max_position=131072)


def _k3_pattern(n: int) -> tuple:
    """Full (MLA) attention on every fourth layer and on the last one, KDA elsewhere (pegainfer-k3/src/config.rs:108-114)."""
    return tuple("full_attention" if (i + 1 == n or i % 4 == 3) else "linear_attention" for i in range(n))


PRESETS["tiny-k3"] = ModelConfig(family="kimi_k3", vocab_size=1024, hidden_size=256, num_layers=5, layer_types=_k3_pattern(5), num_q_heads=4, num_kv_heads=4, head_dim=48, gdn_head_dim=32,
                                 gdn_conv_kernel=4, kda_gate_rank=32, intermediate_size=512, qk_norm=False, q_lora_rank=96, kv_lora_rank=64, qk_nope_head_dim=32, qk_rope_head_dim=16,
                                 v_head_dim=32, n_routed_experts=8, n_shared_experts=2, num_experts_per_tok=3, moe_intermediate_size=64, latent_moe_dim=128, first_k_dense_replace=1,
                                 scoring_func="sigmoid", norm_topk_prob=True, router_bias=True, attn_res_block=2, hidden_act="situ", rms_eps=1e-5, max_position=4096)
# head and latent sizes of the released model (KDA heads of 128, MLA 128 + 64 / 128 over a 512-wide latent), few layers and experts
PRESETS["small-k3"] = replace(PRESETS["tiny-k3"], vocab_size=4096, hidden_size=1024, num_layers=6, layer_types=_k3_pattern(6), num_q_heads=16, num_kv_heads=16, head_dim=192, gdn_head_dim=128,
                              kda_gate_rank=128, intermediate_size=2048, q_lora_rank=512, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128, n_routed_experts=16,
                              num_experts_per_tok=4, moe_intermediate_size=256, latent_moe_dim=512, attn_res_block=3, max_position=8192)
# the released text tower (pegainfer-k3/src/config.rs:26-92): 93 layers, 96 heads, 896 routed experts (top 16) in a 3584-wide latent
PRESETS["kimi-k3"] = replace(PRESETS["small-k3"], vocab_size=163840, hidden_size=7168, num_layers=93, layer_types=_k3_pattern(93), num_q_heads=96, num_kv_heads=96, intermediate_size=33792,
                             q_lora_rank=1536, n_routed_experts=896, num_experts_per_tok=16, moe_intermediate_size=3072, latent_moe_dim=3584, attn_res_block=12, max_position=1048576)
# a one-GPU slice of the released shape for benchmarks (not a released configuration): full-width layers (6 KDA + 2 MLA, one dense
# and seven latent-MoE layers), 32 routed experts instead of 896, top 8
PRESETS["k3-8layer-shape"] = replace(PRESETS["kimi-k3"], num_layers=8, layer_types=_k3_pattern(8), n_routed_experts=32, num_experts_per_tok=8, attn_res_block=4, max_position=131072)
def _nemipel(width: int, vocab: int, ff: int, heads: int, kv_heads: int, dim: int, lin_heads: int, lin_dim: int, rank: int, periods: int, lightning_ff: int = 0, **kw) -> ModelConfig:
    """A Nemipel stack of ``periods`` x (lightning, attention, channel-delta); every second attention layer reads the cache
    of the one before it, the lightning layers have no feed-forward unless ``lightning_ff`` gives its width."""
    layers = []
    for n in range(periods):
        own = 3 * n + 1 if n % 2 == 0 else 3 * (n - 1) + 1
        layers.append(LayerSpec(MixerSpec("lightning", lin_heads, lin_dim, lin_dim, decay=tuple(float(f"{1 - 2.0 ** (-1 - 7 * h / max(lin_heads - 1, 1)):.6f}") for h in range(lin_heads))), lightning_ff))
        layers.append(LayerSpec(MixerSpec("attention", heads, dim, dim, kv_heads=kv_heads, scale=dim ** -0.5, softcap=30.0, rot_dims=dim // 2, rot_base=1e4,
                                          kv_from=-1 if own == 3 * n + 1 else own), ff))
        layers.append(LayerSpec(MixerSpec("channel_delta", lin_heads, lin_dim, lin_dim, kv_heads=lin_heads // 2, conv=4, decay_rank=rank, gate_rank=rank), ff))
    base = dict(family="nemipel", vocab_size=vocab, hidden_size=width, num_layers=len(layers), num_q_heads=heads, num_kv_heads=kv_heads, head_dim=dim, intermediate_size=ff, qk_norm=False,
                layer_specs=tuple(layers), postln_alpha=2.0, final_logit_softcapping=20.0, max_position=131072)
    base.update(kw)
    return ModelConfig(**base)


PRESETS["tiny-nemipel"] = _nemipel(96, 256, 160, 4, 2, 32, 4, 16, 12, 2, max_position=4096)
PRESETS["small-nemipel"] = _nemipel(1024, 4096, 2048, 8, 2, 128, 8, 128, 64, 2, max_position=8192)
# layers as wide as those of an 8 B-parameter model, for benchmarks (not a released configuration): 12 lightning, 12
# attention (6 of them with a cache of their own) and 12 channel-delta layers
PRESETS["nemipel-8b-shape"] = _nemipel(4096, 151936, 12288, 32, 8, 128, 32, 128, 128, 12, lightning_ff=12288)
# the Qwen3.5 line at the same sizes: Gated DeltaNet layers in the place of the lightning and channel-delta layers
PRESETS["qwen35-8b-shape"] = replace(PRESETS["small-qwen35"], vocab_size=151936, hidden_size=4096, num_layers=36, num_q_heads=32, num_kv_heads=8, head_dim=128, intermediate_size=12288,
                                     layer_types=("linear_attention", "full_attention", "linear_attention") * 12, partial_rotary_factor=0.5, gdn_num_k_heads=16, gdn_num_v_heads=32, gdn_head_dim=128,
                                     max_position=131072)
def _vekalorn(width: int, vocab: int, heads: int, q_rank: int, kv_rank: int, dim: int, rot: int, vdim: int, window: int, experts: ExpertsSpec, periods: int, **kw) -> ModelConfig:
    """A Vekalorn stack of ``periods`` x (full latent attention with rotation and gate, two windowed layers without
    positions), a mixture of experts in every layer."""
    full = MixerSpec("latent", heads, dim, vdim, scale=(dim + rot) ** -0.5, rot_dims=rot, rot_base=5e4, q_rank=q_rank, kv_rank=kv_rank, out_gate=True, yarn=(16.0, 4096, 32.0, 1.0))
    local = MixerSpec("latent", heads, dim, vdim, scale=dim ** -0.5, q_rank=q_rank, kv_rank=kv_rank, window=window)
    layers = tuple(LayerSpec(m, moe=experts) for _ in range(periods) for m in (full, local, local))
    base = dict(family="vekalorn", vocab_size=vocab, hidden_size=width, num_layers=len(layers), num_q_heads=heads, num_kv_heads=1, head_dim=dim + rot, intermediate_size=experts.ff * experts.top,
                rms_eps=1e-5, qk_norm=False, layer_specs=layers, max_position=65536)
    base.update(kw)
    return ModelConfig(**base)


PRESETS["tiny-vekalorn"] = _vekalorn(88, 256, 3, 40, 48, 24, 8, 32, 20, ExpertsSpec(12, 3, 24, 3, 2), 2, max_position=4096)
PRESETS["small-vekalorn"] = _vekalorn(1024, 4096, 16, 512, 512, 128, 64, 128, 256, ExpertsSpec(16, 4, 512, 4, 2), 2, max_position=8192)
# layers of a mid-size latent-attention mixture of experts, for benchmarks (not a released configuration)
PRESETS["vekalorn-16b-shape"] = _vekalorn(2048, 102400, 16, 1536, 512, 128, 64, 128, 1024, ExpertsSpec(64, 6, 2112, 8, 4), 9)


def _zeripel(width: int, vocab: int, ff: int, heads: int, kv_heads: int, dim: int, kv_rank: int, nope: int, rot: int, vdim: int, rec_heads: int, rec_dim: int, rank: int, experts: ExpertsSpec,
             periods: int, **kw) -> ModelConfig:
    """A Zeripel stack of ``periods`` x (latent attention, latent attention over the same cache, WKV, attention); the first
    layer's feed-forward is dense."""
    latent = MixerSpec("latent", heads, nope, vdim, scale=(nope + rot) ** -0.5, rot_dims=rot, rot_base=1e5, kv_rank=kv_rank, head_gate=True, sink=True)
    wkv = MixerSpec("wkv", rec_heads, rec_dim, rec_dim, decay_rank=rank)
    attn = MixerSpec("attention", heads, dim, dim, kv_heads=kv_heads, scale=dim ** -0.5, head_norm=True, values_are_keys=True, q_temp=(0.1, 4096))
    layers = []
    for n in range(periods):
        layers += [LayerSpec(m, moe=experts) for m in (latent, replace(latent, kv_from=4 * n), wkv, attn)]
    layers[0] = LayerSpec(latent, ff, act="gelu_tanh")
    base = dict(family="zeripel", vocab_size=vocab, hidden_size=width, num_layers=len(layers), num_q_heads=heads, num_kv_heads=kv_heads, head_dim=dim, intermediate_size=ff, rms_eps=1e-6, qk_norm=False,
                layer_specs=tuple(layers), embed_scale=width ** 0.5, bigram=(vocab * 2 - 3, 31, 5), residual_mult=0.5, max_position=65536)
    base.update(kw)
    return ModelConfig(**base)


def _zeripel_experts(experts: int, top: int, ff: int, shared_ff: int, scale: float) -> ExpertsSpec:
    return ExpertsSpec(experts, top, ff, scoring="sigmoid", correction=True, norm=True, scale=scale, act="swiglu", shared_ff=shared_ff)


PRESETS["tiny-zeripel"] = _zeripel(80, 256, 112, 4, 2, 24, 40, 16, 8, 32, 3, 16, 12, _zeripel_experts(10, 2, 24, 40, 2.0), 1, max_position=4096)
PRESETS["small-zeripel"] = _zeripel(1024, 4096, 2048, 16, 4, 128, 512, 128, 64, 128, 8, 128, 64, _zeripel_experts(16, 4, 512, 512, 2.5), 2, max_position=8192)
# layers of a mid-size hybrid mixture of experts, for benchmarks (not a released configuration)
PRESETS["zeripel-16b-shape"] = _zeripel(2048, 102400, 8192, 16, 4, 128, 512, 128, 64, 128, 16, 128, 64, _zeripel_experts(64, 6, 1408, 2816, 2.5), 7)


def alibi_slopes(heads: int) -> tuple:
    """Score lost per position of distance, a geometric row over the heads that ends at 2^-8."""
    return tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads))


def _nonetar_parallel(heads: int, kv_heads: int, dim: int, vdim: int, scale: float, softcap: float, window: int, width: int, blocks: int, conv: int, scales: tuple) -> MixerSpec:
    left = MixerSpec("attention", heads, dim, vdim, kv_heads=kv_heads, scale=scale, softcap=softcap, window=window, head_norm=True, bias=True, head_temp=True, slopes=alibi_slopes(heads))
    return MixerSpec("parallel", 0, 0, 0, parts=(left, MixerSpec("lru", blocks, width // blocks, width // blocks, conv=conv)), part_scales=scales)


def _nonetar_ssd(heads: int, vdim: int, state: int, groups: int, norm_groups: int, conv: int) -> MixerSpec:
    return MixerSpec("ssd", heads, state, vdim, kv_heads=groups, norm_groups=norm_groups, conv=conv)


def _nonetar(width: int, vocab: int, ff: int, streams: int, parallel: MixerSpec, ssd: MixerSpec, periods: int, **kw) -> ModelConfig:
    """A Nonetar stack of ``periods`` x (attention beside a recurrent block, twice, then state-space duality)."""
    layers = tuple(LayerSpec(m, ff, act="xielu") for _ in range(periods) for m in (parallel, parallel, ssd))
    left = parallel.parts[0]
    base = dict(family="nonetar", vocab_size=vocab, hidden_size=width, num_layers=len(layers), num_q_heads=left.heads, num_kv_heads=left.kv_heads, head_dim=left.dim, intermediate_size=ff, rms_eps=1e-6,
                qk_norm=False, layer_specs=layers, streams=streams, logit_scale=0.5, max_position=65536)
    base.update(kw)
    return ModelConfig(**base)


PRESETS["tiny-nonetar"] = _nonetar(72, 256, 104, 3, _nonetar_parallel(4, 2, 24, 32, 0.25, 30.0, 40, 96, 3, 4, (0.9, 0.6)), _nonetar_ssd(6, 16, 24, 3, 2, 4), 1, max_position=4096)
PRESETS["small-nonetar"] = _nonetar(1024, 4096, 4096, 2, _nonetar_parallel(8, 2, 128, 128, 128 ** -0.5, 50.0, 256, 1024, 8, 4, (1.0, 0.5)), _nonetar_ssd(32, 64, 128, 4, 4, 4), 2, max_position=8192)
# layers as wide as those of an 8 B-parameter model, for benchmarks (not a released configuration)
PRESETS["nonetar-8b-shape"] = _nonetar(4096, 102400, 16384, 4, _nonetar_parallel(32, 8, 128, 128, 128 ** -0.5, 50.0, 2048, 4096, 16, 4, (1.0, 0.5)), _nonetar_ssd(128, 64, 128, 8, 8, 4), 10)
PRESETS["small-glm-fp8"] = replace(PRESETS["small-glm"], expert_quant="fp8_block128", dense_quant="fp8_block128")
for _name in ("tiny-dsv2", "small-dsv2", "dsv2-lite"):
    if _name in PRESETS:
        PRESETS[_name + "-fp8"] = replace(PRESETS[_name], expert_quant="fp8_block128")


def preset(name: str, **overrides) -> ModelConfig:
    if name not in PRESETS:
        raise KeyError(f"unknown model preset {name!r}; known: {sorted(PRESETS)}")
    return replace(PRESETS[name], **overrides)


def detect_family(cfg: dict) -> str:
    """Map a ``config.json`` to a model line (exactly one line must claim it)."""
    if cfg.get("architecture") in ("Nemipel", "Vekalorn", "Zeripel", "Nonetar"):
        return cfg["architecture"].lower()
    mt = cfg.get("model_type", "")
    archs = " ".join(cfg.get("architectures", []))
    if mt in ("qwen3",) or "Qwen3ForCausalLM" in archs:
        return "qwen3"
    if mt.startswith("qwen3_5") or mt in ("qwen3_next",) or "Qwen3_5" in archs or "Qwen3Next" in archs:
        return "qwen35"
    if mt == "deepseek_v2" or "DeepseekV2" in archs:
        return "deepseek_v2"
    if mt == "glm_moe_dsa" or "GlmMoeDsa" in archs:
        return "glm_dsa"
    if mt.startswith("gemma4") or "Gemma4" in archs:
        return "gemma4"
    if mt == "kimi_k3" or "KimiK3" in archs or cfg.get("text_config", {}).get("model_type") == "kimi_linear":
        return "kimi_k3"
    if mt in ("kimi_k2", "deepseek_v3", "kimi_k25") or "DeepseekV3" in archs or "Kimi" in archs:
        return "kimi_k2"
    raise ValueError(f"no model line recognises model_type={mt!r} architectures={archs!r}")


def _eos_ids(model_dir: Optional[str], cfg: dict) -> tuple:
    ids = None
    if model_dir:
        p = os.path.join(model_dir, "generation_config.json")
        if os.path.exists(p):
            with open(p) as f:
                ids = json.load(f).get("eos_token_id")
    if ids is None:
        ids = cfg.get("eos_token_id")
    if ids is None:
        return ()
    if isinstance(ids, int):
        ids = [ids]
    return tuple(dict.fromkeys(int(i) for i in ids))


def _k3_from_hf(cfg: dict, top: dict, model_dir: Optional[str]) -> ModelConfig:
    """Text tower of a Kimi-K3 ``config.json`` (keys as pegainfer-k3/src/config.rs:200-330 checks them)."""
    lin = cfg.get("linear_attn_config", {})
    n = cfg["num_hidden_layers"]
    full = lin.get("full_attn_layers")  # one-based in the checkpoint
    types = tuple("full_attention" if (i + 1) in full else "linear_attention" for i in range(n)) if full else _k3_pattern(n)
    for key, want in (("hidden_act", "situ"), ("moe_router_activation_func", "sigmoid")):
        if cfg.get(key, want) != want:
            raise ValueError(f"Kimi-K3 line: {key}={cfg.get(key)!r} is not supported (expected {want!r})")
    if not cfg.get("mla_use_nope", True) or not cfg.get("mla_use_output_gate", True):
        raise ValueError("Kimi-K3 line: MLA layers without positions (mla_use_nope) and with an output gate are the supported form")
    nope, rope = cfg["qk_nope_head_dim"], cfg["qk_rope_head_dim"]
    return ModelConfig(family="kimi_k3", vocab_size=cfg["vocab_size"], hidden_size=cfg["hidden_size"], num_layers=n, layer_types=types, num_q_heads=cfg["num_attention_heads"],
                       num_kv_heads=cfg.get("num_key_value_heads", cfg["num_attention_heads"]), head_dim=nope + rope, gdn_head_dim=lin.get("head_dim", 128),
                       gdn_conv_kernel=lin.get("short_conv_kernel_size", 4), kda_gate_rank=lin.get("gate_rank", lin.get("head_dim", 128)), kda_gate_lower_bound=float(lin.get("gate_lower_bound", -5.0)),
                       intermediate_size=cfg["intermediate_size"], qk_norm=False, q_lora_rank=cfg["q_lora_rank"], kv_lora_rank=cfg["kv_lora_rank"], qk_nope_head_dim=nope, qk_rope_head_dim=rope,
                       v_head_dim=cfg["v_head_dim"], n_routed_experts=cfg["num_experts"], n_shared_experts=cfg.get("num_shared_experts", 0), num_experts_per_tok=cfg["num_experts_per_token"],
                       moe_intermediate_size=cfg["moe_intermediate_size"], latent_moe_dim=cfg["routed_expert_hidden_size"], first_k_dense_replace=cfg.get("first_k_dense_replace", 1),
                       scoring_func="sigmoid", norm_topk_prob=bool(cfg.get("moe_renormalize", True)), routed_scaling_factor=float(cfg.get("routed_scaling_factor", 1.0)), router_bias=True,
                       expert_quant="mxfp4" if "quantization_config" in top or "quantization_config" in cfg else "bf16", attn_res_block=cfg["attn_res_block_size"], hidden_act="situ",
                       rms_eps=cfg.get("rms_norm_eps", 1e-5), max_position=cfg.get("max_position_embeddings", 4096), tie_word_embeddings=bool(top.get("tie_word_embeddings", False)),
                       eos_token_ids=_eos_ids(model_dir, top))


def _nemipel_from_json(cfg: dict, model_dir: Optional[str]) -> ModelConfig:
    """``config.json`` of the Nemipel line: sizes and constants per layer."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        m, kind = entry["mixer"], entry["type"]
        common = dict(kind=kind, heads=m["heads"], dim=m["dim"], vdim=m["vdim"])
        if kind == "attention":
            rot = m.get("rot") or {}
            src = m.get("kv_from")
            spec = MixerSpec(kv_heads=m["kv_heads"], scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0), rot_dims=rot.get("dims", 0), rot_base=float(rot.get("base", 1e4)),
                             kv_from=-1 if src is None else src, **common)
            if src is not None:
                own = layers[src].mixer if 0 <= src < i else None
                if own is None or own.kind != "attention" or own.kv_from >= 0 or (own.kv_heads, own.dim, own.vdim) != (spec.kv_heads, spec.dim, spec.vdim):
                    raise ValueError(f"layer {i}: kv_from={src} is not an earlier attention layer with a cache of the same shape")
        elif kind == "lightning":
            spec = MixerSpec(decay=tuple(float(d) for d in m["decay"]), **common)
        elif kind == "channel_delta":
            spec = MixerSpec(kv_heads=m["kv_heads"], conv=m["conv"], **common)
        else:
            raise ValueError(f"layer {i}: no mixer of type {kind!r}")
        mlp = entry.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: no feed-forward of kind {mlp['kind']!r}")
        layers.append(LayerSpec(spec, mlp["ff"] if mlp else 0))
    attn = [l.mixer for l in layers if l.mixer.kind == "attention"] or [layers[0].mixer]
    return ModelConfig(family="nemipel", vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_layers=len(layers), num_q_heads=attn[0].heads, num_kv_heads=max(attn[0].kv_heads, 1),
                       head_dim=attn[0].dim, intermediate_size=max(l.ff for l in layers), rms_eps=cfg["norm"]["eps"], qk_norm=False, layer_specs=tuple(layers),
                       postln_alpha=float(cfg["postln_alpha"]), final_logit_softcapping=float(cfg.get("logit_softcap") or 0.0), max_position=131072, eos_token_ids=_eos_ids(model_dir, cfg))


def nemipel_to_json(cfg: ModelConfig) -> dict:
    """The ``config.json`` that ``_nemipel_from_json`` reads back."""
    layers = []
    for l in cfg.layer_specs:
        m = l.mixer
        mix = dict(heads=m.heads, dim=m.dim, vdim=m.vdim)
        if m.kind == "attention":
            mix.update(kv_heads=m.kv_heads, scale=m.scale, rot=dict(dims=m.rot_dims, base=m.rot_base))
            if m.softcap:
                mix["softcap"] = m.softcap
            if m.kv_from >= 0:
                mix["kv_from"] = m.kv_from
        elif m.kind == "lightning":
            mix["decay"] = list(m.decay)
        else:
            mix.update(kv_heads=m.kv_heads, conv=m.conv)
        layers.append(dict(type=m.kind, mixer=mix, mlp=dict(kind="dense", ff=l.ff) if l.ff else None))
    out = dict(architecture="Nemipel", vocab=cfg.vocab_size, width=cfg.hidden_size, norm=dict(eps=cfg.rms_eps), postln_alpha=cfg.postln_alpha, layers=layers)
    if cfg.final_logit_softcapping:
        out["logit_softcap"] = cfg.final_logit_softcapping
    if cfg.eos_token_ids:
        out["eos_token_id"] = list(cfg.eos_token_ids)
    return out


# the two mixers of the Vekalorn line by the name config.json gives them: rotated and gated, or without positions and gate
_LATENT_TYPES = {"latent_attention": False, "latent_attention_2": True}


def _vekalorn_from_json(cfg: dict, model_dir: Optional[str]) -> ModelConfig:
    """``config.json`` of the Vekalorn line: sizes and constants per layer."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        m, kind = entry["mixer"], entry["type"]
        if kind not in _LATENT_TYPES:
            raise ValueError(f"layer {i}: no mixer of type {kind!r}")
        rotated = _LATENT_TYPES[kind]
        rot, yarn = (m.get("rot") or {}) if rotated else {}, ()
        if rotated:
            if rot.get("dims", m["rot_dim"]) != m["rot_dim"] or m["rot_dim"] % 2:
                raise ValueError(f"layer {i}: the rotated part has {m['rot_dim']} columns, {rot.get('dims')} are to be rotated")
            if rot.get("scaling"):
                yarn = tuple(rot["scaling"][k] for k in ("factor", "original", "fast", "slow"))
        window = (m.get("mask") or {}).get("size", 0)
        if not rotated and window < 1:
            raise ValueError(f"layer {i}: a window of {window} positions")
        spec = MixerSpec("latent", m["heads"], m["dim"], m["vdim"], scale=float(m["scale"]), rot_dims=m["rot_dim"] if rotated else 0, rot_base=float(rot.get("base", 1e4)), q_rank=m["q_rank"],
                         kv_rank=m["kv_rank"], window=window, out_gate=rotated, yarn=yarn)
        mlp, moe = entry.get("mlp"), None
        if mlp is not None:
            if mlp.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: no feed-forward of kind {mlp['kind']!r}")
            r = mlp["router"]
            g = r.get("groups") or dict(count=1, keep=1)
            moe = ExpertsSpec(r["experts"], r["top"], mlp["expert"]["ff"], g["count"], g["keep"])
            if moe.experts % moe.groups or not 1 <= moe.keep <= moe.groups or not 1 <= moe.top <= moe.experts // moe.groups * moe.keep:
                raise ValueError(f"layer {i}: {moe.top} experts from {moe.keep} of {moe.groups} groups of {moe.experts}")
        layers.append(LayerSpec(spec, moe=moe))
    first = layers[0].mixer
    return ModelConfig(family="vekalorn", vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_layers=len(layers), num_q_heads=first.heads, num_kv_heads=1, head_dim=first.dim + first.rot_dims,
                       intermediate_size=max([l.moe.ff * l.moe.top for l in layers if l.moe] or [0]), rms_eps=cfg["norm"]["eps"], qk_norm=False, layer_specs=tuple(layers), max_position=131072,
                       eos_token_ids=_eos_ids(model_dir, cfg))


def vekalorn_to_json(cfg: ModelConfig) -> dict:
    """The ``config.json`` that ``_vekalorn_from_json`` reads back."""
    layers = []
    for l in cfg.layer_specs:
        m, e = l.mixer, l.moe
        mix = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank, scale=m.scale)
        if m.window:
            mix["mask"] = dict(size=m.window)
        if m.out_gate:
            mix.update(rot_dim=m.rot_dims, rot=dict(dims=m.rot_dims, base=m.rot_base))
            if m.yarn:
                mix["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), m.yarn))
        mlp = dict(kind="moe", expert=dict(ff=e.ff), router=dict(experts=e.experts, top=e.top, groups=dict(count=e.groups, keep=e.keep))) if e else None
        layers.append(dict(type="latent_attention_2" if m.out_gate else "latent_attention", mixer=mix, mlp=mlp))
    out = dict(architecture="Vekalorn", vocab=cfg.vocab_size, width=cfg.hidden_size, norm=dict(eps=cfg.rms_eps), layers=layers)
    if cfg.eos_token_ids:
        out["eos_token_id"] = list(cfg.eos_token_ids)
    return out


def _zeripel_mixer(i: int, kind: str, m: dict, layers: list) -> MixerSpec:
    if kind == "wkv":
        return MixerSpec("wkv", m["heads"], m["dim"], m["dim"])
    if kind == "attention":
        if m.get("vdim", m["dim"]) != m["dim"]:
            raise ValueError(f"layer {i}: values of {m['vdim']} columns, which are keys of {m['dim']}")
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"layer {i}: {m['heads']} query heads over {m['kv_heads']} key heads")
        t = m.get("q_temp")
        if t and (t["every"] != int(t["every"]) or t["every"] < 1):
            raise ValueError(f"layer {i}: the query temperature steps every {t['every']} positions")
        return MixerSpec("attention", m["heads"], m["dim"], m["dim"], kv_heads=m["kv_heads"], scale=float(m["scale"]), head_norm=True, values_are_keys=True,
                         q_temp=(float(t["coef"]), int(t["every"])) if t else ())
    if kind == "latent_attention":
        rot, src = m.get("rot") or {}, m.get("kv_from")
        if rot.get("dims", m["rot_dim"]) != m["rot_dim"] or m["rot_dim"] % 2:
            raise ValueError(f"layer {i}: the rotated part has {m['rot_dim']} columns, {rot.get('dims')} are to be rotated")
        spec = MixerSpec("latent", m["heads"], m["dim"], m["vdim"], scale=float(m["scale"]), rot_dims=m["rot_dim"], rot_base=float(rot.get("base", 1e4)), kv_rank=m["kv_rank"],
                         kv_from=-1 if src is None else src, head_gate=True, sink=True)
        if src is not None:
            own = layers[src].mixer if 0 <= src < i else None
            if own is None or own.kind != "latent" or own.kv_from >= 0 or (own.kv_rank, own.rot_dims, own.rot_base) != (spec.kv_rank, spec.rot_dims, spec.rot_base):
                raise ValueError(f"layer {i}: kv_from={src} is not an earlier latent attention layer with a cache of the same shape and rotation")
        return spec
    raise ValueError(f"layer {i}: no mixer of type {kind!r}")


def _zeripel_from_json(cfg: dict, model_dir: Optional[str]) -> ModelConfig:
    """``config.json`` of the Zeripel line: sizes and constants per layer."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        mixer, mlp = _zeripel_mixer(i, entry["type"], entry["mixer"], layers), entry.get("mlp")
        if mlp is None:
            layers.append(LayerSpec(mixer))
        elif mlp.get("kind", "dense") == "dense":
            layers.append(LayerSpec(mixer, mlp["ff"], act="gelu_tanh"))
        elif mlp["kind"] == "moe":
            r = mlp["router"]
            if not 1 <= r["top"] <= r["experts"]:
                raise ValueError(f"layer {i}: {r['top']} of {r['experts']} experts")
            layers.append(LayerSpec(mixer, moe=_zeripel_experts(r["experts"], r["top"], mlp["expert"]["ff"], (mlp.get("shared") or {}).get("ff", 0), float(r.get("scale", 1.0)))))
        else:
            raise ValueError(f"layer {i}: no feed-forward of kind {mlp['kind']!r}")
    attn = [l.mixer for l in layers if l.mixer.kind == "attention"] or [layers[0].mixer]
    emb = cfg.get("embedding") or {}
    big = emb.get("bigram")
    return ModelConfig(family="zeripel", vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_layers=len(layers), num_q_heads=attn[0].heads, num_kv_heads=max(attn[0].kv_heads, 1), head_dim=attn[0].dim,
                       intermediate_size=max([l.ff for l in layers] + [l.moe.ff * l.moe.top + l.moe.shared_ff for l in layers if l.moe]), rms_eps=cfg["norm"]["eps"], qk_norm=False,
                       layer_specs=tuple(layers), embed_scale=float(emb.get("scale", 1.0)), bigram=(big["buckets"], big["mul_prev"], big["mul_cur"]) if big else (),
                       residual_mult=float(cfg.get("residual_mult", 1.0)), max_position=131072, eos_token_ids=_eos_ids(model_dir, cfg))


def zeripel_to_json(cfg: ModelConfig) -> dict:
    """The ``config.json`` that ``_zeripel_from_json`` reads back."""
    layers = []
    for l in cfg.layer_specs:
        m, e = l.mixer, l.moe
        mix = dict(heads=m.heads, dim=m.dim)
        if m.kind == "attention":
            mix.update(vdim=m.vdim, kv_heads=m.kv_heads, scale=m.scale)
            if m.q_temp:
                mix["q_temp"] = dict(coef=m.q_temp[0], every=m.q_temp[1])
        elif m.kind == "latent":
            mix.update(vdim=m.vdim, rot_dim=m.rot_dims, kv_rank=m.kv_rank, scale=m.scale, rot=dict(dims=m.rot_dims, base=m.rot_base))
            if m.kv_from >= 0:
                mix["kv_from"] = m.kv_from
        mlp = None
        if e:
            mlp = dict(kind="moe", expert=dict(ff=e.ff), router=dict(experts=e.experts, top=e.top, scale=e.scale))
            if e.shared_ff:
                mlp["shared"] = dict(ff=e.shared_ff)
        elif l.ff:
            mlp = dict(kind="dense", ff=l.ff)
        layers.append(dict(type="latent_attention" if m.kind == "latent" else m.kind, mixer=mix, mlp=mlp))
    emb = dict(scale=cfg.embed_scale)
    if cfg.bigram:
        emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), cfg.bigram))
    out = dict(architecture="Zeripel", vocab=cfg.vocab_size, width=cfg.hidden_size, norm=dict(eps=cfg.rms_eps), residual_mult=cfg.residual_mult, embedding=emb, layers=layers)
    if cfg.eos_token_ids:
        out["eos_token_id"] = list(cfg.eos_token_ids)
    return out


def _nonetar_mixer(i: int, kind: str, m: dict) -> MixerSpec:
    if kind == "parallel":
        a, b = m["left"], m["right"]
        window = (a.get("mask") or {}).get("size", 0)
        if a["heads"] % a["kv_heads"]:
            raise ValueError(f"layer {i}: {a['heads']} query heads over {a['kv_heads']} key heads")
        if a.get("mask") and window < 1:
            raise ValueError(f"layer {i}: a window of {window} positions")
        if b["width"] % b["blocks"]:
            raise ValueError(f"layer {i}: {b['width']} channels in {b['blocks']} blocks")
        return _nonetar_parallel(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), float(a.get("softcap") or 0.0), window, b["width"], b["blocks"], b["conv"],
                                 (float(m.get("left_scale", 1.0)), float(m.get("right_scale", 1.0))))
    if kind == "mamba2":
        if m["heads"] % m["groups"] or m["heads"] * m["vdim"] % m["norm_groups"]:
            raise ValueError(f"layer {i}: {m['heads']} heads of {m['vdim']} in {m['groups']} groups, normed in {m['norm_groups']} parts")
        return _nonetar_ssd(m["heads"], m["vdim"], m["state"], m["groups"], m["norm_groups"], m["conv"])
    raise ValueError(f"layer {i}: no mixer of type {kind!r}")


def _nonetar_from_json(cfg: dict, model_dir: Optional[str]) -> ModelConfig:
    """``config.json`` of the Nonetar line: sizes and constants per layer."""
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        mlp = entry.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: no feed-forward of kind {mlp['kind']!r}")
        layers.append(LayerSpec(_nonetar_mixer(i, entry["type"], entry["mixer"]), mlp["ff"] if mlp else 0, act="xielu"))
    flat = [m for l in layers for m in l.mixer.flat()]
    attn = [m for m in flat if m.kind == "attention"] or flat[:1]
    return ModelConfig(family="nonetar", vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_layers=len(layers), num_q_heads=attn[0].heads, num_kv_heads=max(attn[0].kv_heads, 1), head_dim=attn[0].dim,
                       intermediate_size=max(l.ff for l in layers), rms_eps=cfg["norm"]["eps"], qk_norm=False, layer_specs=tuple(layers), streams=cfg.get("streams", 1),
                       logit_scale=float(cfg.get("logit_scale", 1.0)), max_position=131072, eos_token_ids=_eos_ids(model_dir, cfg))


def nonetar_to_json(cfg: ModelConfig) -> dict:
    """The ``config.json`` that ``_nonetar_from_json`` reads back."""
    layers = []
    for l in cfg.layer_specs:
        m = l.mixer
        if m.kind == "parallel":
            a, b = m.parts
            left = dict(heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale)
            if a.softcap:
                left["softcap"] = a.softcap
            if a.window:
                left["mask"] = dict(size=a.window)
            mix = dict(left=left, right=dict(width=b.heads * b.dim, blocks=b.heads, conv=b.conv), left_scale=m.part_scales[0], right_scale=m.part_scales[1])
        else:
            mix = dict(heads=m.heads, vdim=m.vdim, state=m.dim, groups=m.kv_heads, norm_groups=m.norm_groups, conv=m.conv)
        layers.append(dict(type="parallel" if m.kind == "parallel" else "mamba2", mixer=mix, mlp=dict(kind="dense", ff=l.ff) if l.ff else None))
    out = dict(architecture="Nonetar", vocab=cfg.vocab_size, width=cfg.hidden_size, norm=dict(eps=cfg.rms_eps), streams=cfg.streams, logit_scale=cfg.logit_scale, layers=layers)
    if cfg.eos_token_ids:
        out["eos_token_id"] = list(cfg.eos_token_ids)
    return out


def from_hf(cfg: dict, model_dir: Optional[str] = None) -> ModelConfig:
    family = detect_family(cfg)
    top = cfg
    if family == "nemipel":
        return _nemipel_from_json(cfg, model_dir)
    if family == "vekalorn":
        return _vekalorn_from_json(cfg, model_dir)
    if family == "zeripel":
        return _zeripel_from_json(cfg, model_dir)
    if family == "nonetar":
        return _nonetar_from_json(cfg, model_dir)
    if family == "qwen35" and "text_config" in cfg:
        cfg = cfg["text_config"]
    if family == "kimi_k2" and "text_config" in cfg:
        cfg = cfg["text_config"]
    if family == "gemma4" and "text_config" in cfg:
        cfg = cfg["text_config"]
    if family == "kimi_k3":
        return _k3_from_hf(cfg.get("text_config", cfg), top, model_dir)
    common = dict(
        family=family,
        vocab_size=cfg["vocab_size"],
        hidden_size=cfg["hidden_size"],
        num_layers=cfg["num_hidden_layers"],
        num_q_heads=cfg["num_attention_heads"],
        num_kv_heads=cfg.get("num_key_value_heads", cfg["num_attention_heads"]),
        intermediate_size=cfg["intermediate_size"],
        rms_eps=cfg.get("rms_norm_eps", 1e-6),
        max_position=cfg.get("max_position_embeddings", 4096),
        tie_word_embeddings=bool(top.get("tie_word_embeddings", cfg.get("tie_word_embeddings", False))),
        eos_token_ids=_eos_ids(model_dir, top),
    )
    if family == "gemma4":
        for key in ("hidden_size_per_layer_input", "num_kv_shared_layers"):
            if cfg.get(key, 0):
                raise ValueError(f"gemma4: {key}={cfg[key]} (per-layer input embeddings / cross-layer KV sharing of the small variants) is not supported")
        if cfg.get("enable_moe_block"):
            raise ValueError("gemma4: the mixture-of-experts variant is not supported")
        rp = cfg.get("rope_parameters") or {}
        full, local = rp.get("full_attention", {}), rp.get("sliding_attention", {})
        n = cfg["num_hidden_layers"]
        types = cfg.get("layer_types") or ["sliding_attention" if (i + 1) % 6 else "full_attention" for i in range(n)]
        common["tie_word_embeddings"] = bool(top.get("tie_word_embeddings", cfg.get("tie_word_embeddings", True)))
        return ModelConfig(
            head_dim=cfg.get("head_dim", 256),
            global_head_dim=cfg.get("global_head_dim", 512) or cfg.get("head_dim", 256),
            num_global_kv_heads=cfg.get("num_global_key_value_heads") or common["num_kv_heads"],
            attention_k_eq_v=bool(cfg.get("attention_k_eq_v", False)),
            sliding_window=cfg.get("sliding_window", 512),
            layer_types=tuple(types),
            rope_theta=full.get("rope_theta", 1e6),
            partial_rotary_factor=full.get("partial_rotary_factor", 0.25),
            rope_theta_local=local.get("rope_theta", 1e4),
            final_logit_softcapping=cfg.get("final_logit_softcapping") or 0.0,
            hidden_act="gelu_tanh",
            qk_norm=True,
            **common,
        )
    if family == "qwen3":
        return ModelConfig(head_dim=cfg.get("head_dim", cfg["hidden_size"] // cfg["num_attention_heads"]), rope_theta=cfg.get("rope_theta", 1e6), **common)
    if family == "qwen35":
        rp = cfg.get("rope_parameters", {})
        return ModelConfig(
            head_dim=cfg.get("head_dim", 256),
            rope_theta=rp.get("rope_theta", cfg.get("rope_theta", 1e7)),
            partial_rotary_factor=rp.get("partial_rotary_factor", cfg.get("partial_rotary_factor", 0.25)),
            layer_types=tuple(cfg["layer_types"]),
            attn_output_gate=True,
            norm_weight_offset=True,
            gdn_num_k_heads=cfg["linear_num_key_heads"],
            gdn_num_v_heads=cfg["linear_num_value_heads"],
            gdn_head_dim=cfg.get("linear_key_head_dim", 128),
            gdn_conv_kernel=cfg.get("linear_conv_kernel_dim", 4),
            **common,
        )
    mla = dict(
        qk_norm=False,
        q_lora_rank=cfg.get("q_lora_rank") or 0,
        kv_lora_rank=cfg["kv_lora_rank"],
        qk_nope_head_dim=cfg["qk_nope_head_dim"],
        qk_rope_head_dim=cfg["qk_rope_head_dim"],
        v_head_dim=cfg["v_head_dim"],
        head_dim=cfg["qk_nope_head_dim"] + cfg["qk_rope_head_dim"],
        rope_theta=cfg.get("rope_theta") or (cfg.get("rope_parameters") or {}).get("rope_theta", 10000.0),
        rope_scaling=cfg.get("rope_scaling"),
        n_routed_experts=cfg.get("n_routed_experts", 0),
        n_shared_experts=cfg.get("n_shared_experts", 0),
        num_experts_per_tok=cfg.get("num_experts_per_tok", 0),
        moe_intermediate_size=cfg.get("moe_intermediate_size", 0),
        first_k_dense_replace=cfg.get("first_k_dense_replace", 0),
        scoring_func=cfg.get("scoring_func", "softmax"),
        n_group=cfg.get("n_group", 1) or 1,
        topk_group=cfg.get("topk_group", 1) or 1,
        norm_topk_prob=bool(cfg.get("norm_topk_prob", False)),
        routed_scaling_factor=cfg.get("routed_scaling_factor", 1.0),
    )
    q = cfg.get("quantization_config") or top.get("quantization_config") or {}
    quant = "bf16"
    if q.get("quant_method") == "compressed-tensors" or q.get("format") == "pack-quantized":
        quant = "int4_g32"
    elif q.get("quant_method") == "fp8":
        quant = "fp8_block128"
    mla.update(expert_quant=quant)
    if family == "kimi_k2":
        mla.update(router_bias=True, num_mtp_layers=cfg.get("num_nextn_predict_layers", 0))
    if family == "glm_dsa":
        types = cfg.get("mlp_layer_types")
        dense = cfg.get("first_k_dense_replace", 3) if types is None else next((i for i, t in enumerate(types) if t == "sparse"), len(types))
        mla.update(dense_quant="fp8_block128" if quant == "fp8_block128" else "bf16", router_bias=True, scoring_func="sigmoid", first_k_dense_replace=dense, num_mtp_layers=cfg.get("num_nextn_predict_layers", 0),
                   index_topk=cfg.get("index_topk", 2048), index_head_dim=cfg.get("index_head_dim", 128), index_n_heads=cfg.get("index_n_heads", 32))
    return ModelConfig(**common, **mla)


def load_model_config(model_dir: str) -> ModelConfig:
    with open(os.path.join(model_dir, "config.json")) as f:
        return from_hf(json.load(f), model_dir)


@dataclass
class EngineConfig:
    """Serving knobs (one per CLI flag)."""

    model_path: Optional[str] = None
    preset: Optional[str] = None
    served_model_name: Optional[str] = None
    port: int = 8000
    host: str = "127.0.0.1"
    cuda_graph: bool = True
    precapture_graphs: bool = False  # capture every decode bucket at start-up
    dump_graph_dot: Optional[str] = None
    device_ordinal: int = 0
    tp_size: int = 1
    dp_size: int = 1
    ep_size: int = 1
    kv_page_size: int = 16
    num_kv_blocks: Optional[int] = None
    gpu_memory_utilization: float = 0.90
    kv_cache_memory_margin_mib: int = 150
    no_prefix_cache: bool = False
    kv_offload: bool = False
    kv_offload_host_gib: float = 4.0
    kv_offload_l1_disabled: bool = False  # test mode: evict idle GPU blocks before every probe
    kv_offload_disk_dir: Optional[str] = None  # third tier: blocks evicted from host memory go to files here
    kv_offload_disk_gib: float = 0.0
    max_prefill_tokens: int = 1024
    max_decode_batch: int = 256
    max_model_len: Optional[int] = None
    batch_invariant: bool = False
    decode_overlap: bool = False
    run_ahead: bool = True  # greedy graph decode launches the next step before reading this one's tokens
    tune_gc: bool = False  # freeze start-up objects and raise the collector thresholds (utils/runtime.py); the server and the benches turn it on
    decode_sm_pct: int = 50
    decode_sm_split: bool = False  # --decode-sm-pct given: the prefill lane gets its own SM partition (green contexts)
    enable_lora: bool = False
    max_loras: int = 4
    max_lora_rank: int = 64
    lora_modules: tuple = ()
    spec_method: Optional[str] = None  # None | "mtp" | "draft" | "dflash" | "dspark" | "eagle3"
    spec_draft_len: int = 1
    draft_model_path: Optional[str] = None
    comm: str = "fused"  # fused | nccl
    gemm: str = "sm100"  # sm100 | cublas
    seed: int = 0
    dtype: str = "bfloat16"  # activations and cache on the GPU; "float32" on the lines that have 32-bit kernels
    state_slots: Optional[int] = None  # lines with recurrent state: requests that hold state at a time (default: from the decode batch)

    def validate(self) -> None:
        if self.kv_page_size not in (16, 32, 64):
            raise ValueError("--kv-page-size must be 16, 32 or 64")
        if not (0.05 <= self.gpu_memory_utilization <= 0.99):
            raise ValueError("--gpu-memory-utilization must be in [0.05, 0.99]")
        if self.max_prefill_tokens < 1:
            raise ValueError("--max-prefill-tokens must be positive")
        if self.comm not in ("fused", "nccl"):
            raise ValueError("--comm must be fused or nccl")
        if self.gemm not in ("sm100", "cublas"):
            raise ValueError("--gemm must be sm100 or cublas")
        if self.dtype not in ("bfloat16", "float32"):
            raise ValueError("--dtype must be bfloat16 or float32")
        if self.state_slots is not None and self.state_slots < 1:
            raise ValueError("--state-slots must be positive")
        for n in ("tp_size", "dp_size", "ep_size"):
            if getattr(self, n) < 1:
                raise ValueError(f"--{n.replace('_', '-')} must be >= 1")
