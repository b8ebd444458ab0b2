"""Model and engine configuration.

One ``ModelConfig`` describes every supported family; fields that a family does not use
keep their neutral default (``index_topk == 0`` means no DSA indexer, ``moe_latent_size == 0``
means experts work in the hidden size, ``num_kv_heads > 0`` selects GQA instead of MLA).

Reference parity: the reference spreads this over per-model ``config.py`` / planner files and
``batchgen/config/config.py:26-293`` (engine config dataclasses + JSON parser) and identifies
models through ``batchgen/config/model_registry.py:60-117``.  Here a single registry maps model
names (and HF-style ids) to presets.
"""
from __future__ import annotations

import dataclasses
import json
import math
import os
import re
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple


@dataclass(frozen=True)
class MixerSpec:
    """A token mixer of a layer-listed model."""
    kind: str                              # "attention" | "latent_attention" | "general_delta" | "channel_delta" | "mlstm" | "retention" | "hgrn2"
    heads: int
    dim: int                               # query / key width of a head
    kv_heads: int = 0                      # key / value heads of attention, query / key heads of channel_delta (0 = heads)
    vdim: int = 0                          # value width of a head
    scale: float = 1.0                     # attention: factor of the scores
    chunk: int = 0                         # attention: keys are seen inside the query's own chunk of this many positions (0 = all)
    window: int = 0                        # attention: the last so many positions are seen, the query's own among them (0 = all)
    keep_first: int = 0                    # attention with a window: this many first positions of a sequence stay visible
    bias: bool = False                     # attention: biases on the q, k and v projections
    out_bias: bool = False                 # attention: a bias on the output projection
    qk_norm: bool = False                  # attention: RMS norm of every query and key head, weights shared by the heads
    qk_norm_all: bool = False              # attention: RMS norm of all query heads (and of all key heads) at once
    talking: bool = False                  # attention: a [heads, heads] matrix mixes the heads' scores before the softmax
    sink: bool = False                     # attention: one is added to the softmax denominator
    head_sinks: bool = False               # attention: exp of a learned number per head is added to the softmax denominator
    out_gate: bool = False                 # attention: a sigmoid gate per head scales its output
    out_gate_all: bool = False             # attention: a sigmoid gate per element of the heads' outputs
    q_rank: int = 0                        # latent_attention: width of the latent that the queries go through
    kv_rank: int = 0                       # latent_attention: width of the cached latent
    rot_dim: int = 0                       # latent_attention: rotated query / key dimensions beside the ``dim`` unrotated ones
    kv_from: int = -1                      # latent_attention: >= 0: the layer whose cached latents this one reads
    rot_dims: int = 0                      # attention, retention: leading head dimensions with rotary positions
    rot_base: float = 10000.0
    rot_interleaved: bool = False          # pairs (2 i, 2 i + 1) turn together; else (i, i + rot_dims / 2)
    yarn: Tuple[float, ...] = ()           # YaRN frequencies: (factor, original positions, fast turns, slow turns); () = plain ones
    out_scale: float = 1.0                 # factor of the mixer's output
    decay_rank: int = 0                    # general_delta, channel_delta: width of the low-rank decay projection
    gate_rank: int = 0                     # channel_delta: width of the low-rank output-gate projection
    conv: int = 0                          # channel_delta: taps of the short convolutions of q, k and v
    gate_cap: float = 0.0                  # mlstm: soft cap of the gates' pre-activations
    decay: Tuple[float, ...] = ()          # retention: decay per head

    @property
    def recurrent(self) -> bool:
        return self.kind not in ("attention", "latent_attention")

    @property
    def latent(self) -> bool:
        return self.kind == "latent_attention"

    @property
    def qk_heads(self) -> int:
        """Heads of the keys (and, for recurrent mixers, of the queries)."""
        return self.kv_heads or self.heads

    @property
    def dim_p(self) -> int:
        """Head width as stored: padded with zero channels to a multiple of 8 (16-byte bf16 vectors)."""
        return -(-self.dim // 8) * 8

    @property
    def vdim_p(self) -> int:
        return -(-self.vdim // 8) * 8

    @property
    def rank_p(self) -> int:
        """Latent width as stored."""
        return -(-self.kv_rank // 8) * 8

    @property
    def rot_p(self) -> int:
        return -(-self.rot_dim // 8) * 8

    @property
    def kv_row(self) -> int:
        """Elements of a cached token row: keys of every key head, then values; the latent, then the shared rotated key part."""
        if self.latent:
            return self.rank_p + self.rot_p if self.kv_from < 0 else 0
        return 0 if self.recurrent else self.kv_heads * (self.dim_p + self.vdim_p)

    @property
    def state_shape(self) -> Tuple[int, int, int]:
        """fp32 state [head, key channel, value channel]; empty for attention."""
        return (self.heads, self.dim_p, self.vdim_p) if self.recurrent else (0, 0, 0)

    @property
    def state_parts(self) -> Dict[str, Tuple[int, ...]]:
        """Everything a sequence carries from token to token, by name (fp32)."""
        if not self.recurrent:
            return {}
        parts: Dict[str, Tuple[int, ...]] = {"S": self.state_shape}
        if self.kind == "mlstm":
            parts["n"] = (self.heads, self.dim_p)                  # normaliser, decayed and written like a column of S
            parts["m"] = (self.heads,)                             # running maximum of the log gates
        if self.kind == "channel_delta":
            parts["conv"] = (self.conv - 1, self.conv_channels)    # last inputs of the short convolutions, oldest first
        return parts

    @property
    def conv_channels(self) -> int:
        return 2 * self.qk_heads * self.dim_p + self.heads * self.vdim_p

    @property
    def in_columns(self) -> int:
        """fp32 columns a token's projections take (a workspace estimate, padding aside)."""
        qk, v = self.heads * self.dim_p, self.heads * self.vdim_p
        return {"attention": qk + self.kv_heads * (self.dim_p + self.vdim_p) + (v if self.out_gate_all else self.heads),
                # projections, queries, then a token's expanded keys and values (16 bits)
                "latent_attention": 2 * self.q_rank + self.rank_p + 2 * self.heads * (self.dim_p + self.rot_p) + v // 2,
                "hgrn2": 2 * qk + v,
                "general_delta": 6 * qk,
                "channel_delta": 2 * self.conv_channels + 2 * v + qk + self.decay_rank + self.gate_rank + self.heads,
                "mlstm": 2 * qk + 2 * v + 2 * self.heads, "retention": 2 * qk + 2 * v}[self.kind]

    def param_count(self, width: int) -> int:
        qk, v, H = self.heads * self.dim, self.heads * self.vdim, self.heads
        if self.kind == "attention":
            n = width * (H + self.kv_heads) * (self.dim + self.vdim) + (H * H if self.talking else 0)
            n += (H + self.kv_heads) * self.dim + self.kv_heads * self.vdim if self.bias else 0
            n += (width if self.out_bias else 0) + (width * v if self.out_gate_all else 0)
            return n + (2 * self.dim if self.qk_norm else 0) + ((H + self.kv_heads) * self.dim if self.qk_norm_all else 0)
        if self.latent:
            n = width * (self.q_rank + v) + self.q_rank * H * (self.dim + self.rot_dim) + self.kv_rank * (qk + v)
            return n + (width * (self.kv_rank + self.rot_dim) if self.kv_from < 0 else 0)
        if self.kind == "hgrn2":
            return 2 * width * (qk + v)
        if self.kind == "general_delta":
            return width * (6 * qk + self.decay_rank) + self.decay_rank * qk
        if self.kind == "channel_delta":
            return (width * (2 * self.qk_heads * self.dim + 2 * v + H + self.decay_rank + self.gate_rank)
                    + self.decay_rank * qk + self.gate_rank * v)
        return width * (2 * qk + 3 * v + (2 * H if self.kind == "mlstm" else 0))


@dataclass(frozen=True)
class MlpSpec:
    """The feed-forward of one layer of a layer-listed model."""
    kind: str = "none"                     # none | dense | moe
    ff: int = 0                            # dense width, or width of one routed expert
    activation: str = "gelu_tanh"          # gelu_tanh | silu | swiglu_oai (clamped gate and up, sigmoid slope 1.702, up + 1) | relu2 (no gate)
    limit: float = 0.0                     # clamp of swiglu_oai
    experts: int = 0
    top: int = 0
    weight_on_input: bool = False          # the routing weight scales the expert's input instead of its output
    shared_ff: int = 0                     # shared expert (0 = none), same activation
    shared_limit: float = 0.0
    shared_gate: bool = True               # the shared expert's output is scaled by a sigmoid gate per token
    scoring: str = "sigmoid"               # router scores: sigmoid | softmax (over the chosen) | softmax_all (over all experts)
    correction: bool = False               # a bias per expert takes part in the choice, not in the weights
    groups: int = 1                        # experts form this many groups, of which the best ``keep_groups`` take part
    keep_groups: int = 1
    group_score: str = "top2"              # a group counts with the sum of its two best choice scores, or its "max"
    norm_weights: bool = False             # weights are divided by their sum
    router_scale: float = 1.0


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    mlp: MlpSpec = MlpSpec()
    second: Optional[MixerSpec] = None     # a mixer beside the first: sandwich blocks average both RMS-normed outputs, hyper-
                                           # connected blocks add them (``MixerSpec.out_scale``)
    weights_of: int = -1                   # >= 0: the layer whose tensors this one uses, with a cache and state of its own

    @property
    def mixers(self) -> Tuple[MixerSpec, ...]:
        return (self.mixer,) if self.second is None else (self.mixer, self.second)

    @property
    def kv_row(self) -> int:
        return sum(m.kv_row for m in self.mixers)

    def state_parts(self, width: int, canon_taps: int, token_shift: bool = False) -> Dict[str, Tuple[int, ...]]:
        """fp32 state of a sequence in this layer: the mixers' parts (the second mixer's names end in ".1"), with input
        convolutions the last inputs of each sublayer, with a token shift the last input of the mixer."""
        parts = {name + (f".{i}" if i else ""): shape for i, m in enumerate(self.mixers) for name, shape in m.state_parts.items()}
        if canon_taps:
            rows = (canon_taps - 1, -(-width // 4) * 4)
            parts["canon1"] = rows
            if self.mlp.kind != "none":
                parts["canon2"] = rows
        if token_shift:
            parts["shift"] = (1, -(-width // 4) * 4)
        return parts


@dataclass
class ModelConfig:
    name: str = "tiny-deepseek-v3"
    family: str = "deepseek_v3"  # deepseek_v3 | deepseek_v2 | deepseek_v4 | glm5 | kimi_k3 | kimi_k25 | gpt_oss | minimax | mixtral | qwen2_moe | nanurax | pamevik | bolisun | pitudra
    vocab_size: int = 1024
    hidden_size: int = 256
    num_layers: int = 2
    first_k_dense: int = 1
    intermediate_size: int = 512          # dense MLP intermediate
    moe_intermediate_size: int = 128      # routed / shared expert intermediate
    n_routed_experts: int = 8
    n_shared_experts: int = 1
    num_experts_per_tok: int = 2
    n_group: int = 1
    topk_group: int = 1
    routed_scaling_factor: float = 1.0
    norm_topk_prob: bool = True
    scoring_func: str = "sigmoid"          # sigmoid | softmax (over the selected) | softmax_all | sqrtsoftplus
    shared_expert_gate: bool = False       # Qwen2-MoE: the shared expert's output is scaled by sigmoid(x . w_gate)
    moe_latent_size: int = 0               # Kimi-K3 LatentMoE: experts run in this width
    activation: str = "silu"               # silu | swiglu_clamped (GPT-OSS)
    # ---- attention: MLA
    num_heads: int = 4
    q_lora_rank: int = 128
    kv_lora_rank: int = 64
    qk_nope_head_dim: int = 32
    qk_rope_head_dim: int = 16
    v_head_dim: int = 32
    # ---- attention: GQA (used when num_kv_heads > 0)
    num_kv_heads: int = 0
    head_dim: int = 0
    sliding_window: int = 0
    attention_sinks: bool = False
    attention_bias: bool = False           # GQA: q/k/v projections carry a bias (Qwen2)
    # ---- rope
    rope_theta: float = 10000.0
    rope_interleaved: bool = True
    rope_scaling_factor: float = 1.0       # YaRN factor (1 = off)
    rope_original_max_pos: int = 4096
    rope_beta_fast: float = 32.0
    rope_beta_slow: float = 1.0
    rope_mscale: float = 1.0
    rope_mscale_all_dim: float = 0.0
    max_position_embeddings: int = 163840
    rms_eps: float = 1e-6
    # ---- DSA sparse-attention indexer (GLM-5.x / Kimi-K3.1)
    index_n_heads: int = 0
    index_head_dim: int = 0
    index_topk: int = 0
    indexer_full_layers: Tuple[int, ...] = ()   # layers that own an indexer; others reuse
    # ---- KDA linear-attention layers (Kimi-Linear / Kimi-K3): those layers keep a recurrent state per
    # sequence instead of paged KV; the other layers are MLA
    kda_layers: Tuple[int, ...] = ()
    kda_num_heads: int = 0
    kda_head_dim: int = 128
    kda_gate_rank: int = 0                 # width of the low-rank decay-gate projection (0 = head dim)
    # ---- DeepSeek-V4: one latent KV head shared by all query heads (K = V), a sliding window of raw KV plus one
    # pooled entry per ``compress_ratios[layer]`` tokens (0 = window only; 4 = overlapped windows + top-k indexer),
    # grouped low-rank output projection, hyper-connection residual streams, hash-routed first layers
    compress_ratios: Tuple[int, ...] = ()
    compress_rope_theta: float = 0.0
    o_groups: int = 0
    o_lora_rank: int = 0
    hc_mult: int = 0
    hc_sinkhorn_iters: int = 20
    hc_eps: float = 1e-6
    num_hash_layers: int = 0
    swiglu_limit: float = 0.0
    # ---- quantisation of linear / expert weights
    quant: str = "none"                    # none | fp8_block | mxfp4 | int4
    quant_block: int = 128
    # ---- layer-listed models: every layer has its own mixer and feed-forward, with an fp32 residual and scaled embeddings
    layer_specs: Tuple[LayerSpec, ...] = ()
    embed_scale: float = 1.0
    sandwich: bool = False                 # False: mixer and feed-forward read one RMS norm and are added together (parallel
                                           # block); True: one after the other, a norm before and after each
    pre_norm: bool = True                  # sandwich: False: sublayers read the residual itself, only their outputs are normed
    layer_norm: bool = False               # sandwich: norms subtract the mean and have biases (else RMS norms)
    token_shift: bool = False              # sandwich: a mixer reads h + (h' - h) * shift, h' the previous token's h
    side_dim: int = 0                      # sandwich: > 0: after the feed-forward a token's own row of a table per layer, so many
                                           # numbers gated by the residual, is projected, RMS-normed and added
    streams: int = 0                       # > 0: pre-norm blocks (mixer, then feed-forward) around this many residual streams with
                                           # hyper-connections of fixed weights
    canon_taps: int = 0                    # sandwich: every sublayer reads h + conv(h), a causal convolution of this many taps
    checkpoint_dir: str = ""               # directory the config was read from (its .safetensors files are the weights)
    # ---- misc
    eos_token_id: int = 1
    bos_token_id: int = 0
    tie_word_embeddings: bool = False

    # derived ------------------------------------------------------------------
    @property
    def qk_head_dim(self) -> int:
        return self.qk_nope_head_dim + self.qk_rope_head_dim

    @property
    def is_v4(self) -> bool:
        return len(self.compress_ratios) > 0

    @property
    def is_layered(self) -> bool:
        return len(self.layer_specs) > 0

    @property
    def recurrent_layers(self) -> Tuple[int, ...]:
        return tuple(l for l, s in enumerate(self.layer_specs) if any(m.recurrent for m in s.mixers))

    @property
    def has_state(self) -> bool:
        """A live sequence holds a state slot besides (or instead of) paged KV."""
        return self.has_kda or self.is_v4 or len(self.layered_state_parts()) > 0

    def layered_state_parts(self) -> List[Tuple[Tuple[int, str], Tuple[int, ...]]]:
        """((layer, name), shape) of everything a sequence of a layer-listed model carries outside the paged rows."""
        return [((l, name), shape) for l, s in enumerate(self.layer_specs)
                for name, shape in s.state_parts(self.hidden_size, self.canon_taps, self.token_shift).items()]

    def layered_state_floats_per_seq(self) -> int:
        return sum(math.prod(shape) for _, shape in self.layered_state_parts())

    def v4_state_floats_per_seq(self) -> int:
        """fp32 words of per-sequence state of a DeepSeek-V4 model: per layer the window ring, the compressor's
        pending window(s) of projections and gate scores, and the same for the indexer's compressor."""
        n, D, Di, win = 0, self.head_dim, self.index_head_dim, self.sliding_window
        for r in self.compress_ratios:
            n += win * D
            if r:
                c = 2 if r == 4 else 1
                n += 2 * (c * r) * (c * D)
                if r == 4:
                    n += 2 * (2 * r) * (2 * Di)
        return n

    @property
    def kv_cache_dim(self) -> int:
        """Width of one cached latent row (normalised c_kv followed by roped k_pe)."""
        if self.is_v4:
            return self.head_dim
        if self.is_layered:
            return sum(s.kv_row for s in self.layer_specs)
        if self.num_kv_heads > 0:
            return 2 * self.num_kv_heads * self.head_dim
        return self.kv_lora_rank + self.qk_rope_head_dim

    @property
    def is_mla(self) -> bool:
        return self.num_kv_heads == 0 and not self.is_layered

    @property
    def has_dsa(self) -> bool:
        return self.index_topk > 0 and not self.is_v4

    @property
    def expert_hidden(self) -> int:
        return self.moe_latent_size or self.hidden_size

    @property
    def softmax_scale(self) -> float:
        d = self.qk_head_dim if self.is_mla else self.head_dim
        scale = d ** -0.5
        if self.rope_scaling_factor > 1.0 and self.rope_mscale_all_dim:
            m = 0.1 * self.rope_mscale_all_dim * math.log(self.rope_scaling_factor) + 1.0
            scale = scale * m * m
        return scale

    @property
    def has_kda(self) -> bool:
        return len(self.kda_layers) > 0

    def layer_is_kda(self, layer: int) -> bool:
        return layer in self.kda_layers

    @property
    def kda_rank(self) -> int:
        return self.kda_gate_rank or self.kda_head_dim

    def kda_state_bytes_per_seq(self, tp_size: int = 1) -> int:
        """Recurrent state (fp32 [H, D, D]) plus convolution windows (fp32 [3 H D, 3]) of all KDA layers."""
        h, d = self.kda_num_heads // tp_size, self.kda_head_dim
        return len(self.kda_layers) * 4 * (h * d * d + 9 * h * d)

    def is_moe_layer(self, layer: int) -> bool:
        return self.n_routed_experts > 0 and layer >= self.first_k_dense

    def layer_has_indexer(self, layer: int) -> bool:
        if not self.has_dsa:
            return False
        return (not self.indexer_full_layers) or layer in self.indexer_full_layers

    def kv_bytes_per_token(self, kv_dtype_bytes: int = 2) -> int:
        if self.is_v4:
            # paged part only (pooled entries and their index keys); the window and compressor state is per sequence
            b = 0.0
            for r in self.compress_ratios:
                if r:
                    b += self.head_dim * kv_dtype_bytes / r
                    if r == 4:
                        b += self.index_head_dim * kv_dtype_bytes / r
            return int(math.ceil(b))
        if self.is_layered:
            return max(self.kv_cache_dim * kv_dtype_bytes, 1)
        b = (self.num_layers - len(self.kda_layers)) * self.kv_cache_dim * kv_dtype_bytes
        if self.has_dsa:
            n_idx = len(self.indexer_full_layers) or self.num_layers
            b += n_idx * (self.index_head_dim + 4)  # e4m3 keys + fp32 scale per token
        return b

    def param_count(self) -> int:
        h = self.hidden_size
        n = (1 if self.tie_word_embeddings and self.is_layered else 2) * self.vocab_size * h
        if self.is_v4:
            D, Di = self.head_dim, self.index_head_dim
            for l, r in enumerate(self.compress_ratios):
                n += h * self.q_lora_rank + self.q_lora_rank * self.num_heads * D + h * D
                n += self.num_heads * D * self.o_lora_rank + self.o_groups * self.o_lora_rank * h
                if r:
                    c = 2 if r == 4 else 1
                    n += 2 * h * c * D
                    if r == 4:
                        n += self.q_lora_rank * self.index_n_heads * Di + h * self.index_n_heads + 4 * h * Di
                n += 3 * h * self.moe_intermediate_size * (self.n_routed_experts + self.n_shared_experts)
                n += h * self.n_routed_experts + 2 * (2 + self.hc_mult) * self.hc_mult * self.hc_mult * h
            return n
        if self.is_layered:
            for spec in self.layer_specs:
                if spec.weights_of >= 0:
                    continue
                f = spec.mlp
                n += sum(m.param_count(h) for m in spec.mixers)
                n += (2 if f.activation == "relu2" else 3) * h * f.ff * (f.experts if f.kind == "moe" else 1) + h * f.experts + 3 * h * f.shared_ff
            return n + len(self.layer_specs) * self.side_dim * (self.vocab_size + 2 * h)
        for l in range(self.num_layers):
            if self.layer_is_kda(l):
                hd = self.kda_num_heads * self.kda_head_dim
                n += h * (4 * hd + self.kda_num_heads + self.kda_rank) + self.kda_rank * hd + hd * h
            elif self.is_mla:
                n += h * self.q_lora_rank + self.q_lora_rank * self.num_heads * self.qk_head_dim
                n += h * self.kv_cache_dim
                n += self.kv_lora_rank * self.num_heads * (self.qk_nope_head_dim + self.v_head_dim)
                n += self.num_heads * self.v_head_dim * h
            else:
                n += h * (self.num_heads + 2 * self.num_kv_heads) * self.head_dim
                n += self.num_heads * self.head_dim * h
            if self.is_moe_layer(l):
                eh = self.expert_hidden
                n += 3 * eh * self.moe_intermediate_size * (self.n_routed_experts + self.n_shared_experts)
                n += h * self.n_routed_experts
            else:
                n += 3 * h * self.intermediate_size
        return n

    def to_json(self) -> str:
        return json.dumps(dataclasses.asdict(self), indent=1)

    @classmethod
    def from_dict(cls, d: Dict) -> "ModelConfig":
        names = {f.name for f in dataclasses.fields(cls)}
        kw = {k: v for k, v in d.items() if k in names}
        if "kda_layers" in kw:
            kw["kda_layers"] = tuple(kw["kda_layers"])
        if "indexer_full_layers" in kw:
            kw["indexer_full_layers"] = tuple(kw["indexer_full_layers"])
        if "compress_ratios" in kw:
            kw["compress_ratios"] = tuple(kw["compress_ratios"])
        if "layer_specs" in kw:
            def mixer(m):
                return None if m is None else MixerSpec(**{**m, **{k: tuple(m.get(k, ())) for k in ("decay", "yarn")}})
            kw["layer_specs"] = tuple(
                x if isinstance(x, LayerSpec) else LayerSpec(mixer(x["mixer"]), MlpSpec(**x["mlp"]), mixer(x.get("second")),
                                                             x.get("weights_of", -1))
                for x in kw["layer_specs"])
        return cls(**kw)


# ------------------------------------------------------------------ presets
def tiny_deepseek_v3() -> ModelConfig:
    """The CPU fp32 correctness model: 2 layers (dense, MoE), hidden 256, 8 experts top-2."""
    return ModelConfig()


def tiny_glm5() -> ModelConfig:
    return ModelConfig(name="tiny-glm5", family="glm5", num_layers=3, first_k_dense=1,
                       index_n_heads=4, index_head_dim=32, index_topk=16,
                       indexer_full_layers=(0, 2), rope_interleaved=True,
                       routed_scaling_factor=2.5)


def tiny_kimi_k3() -> ModelConfig:
    return ModelConfig(name="tiny-kimi-k3", family="kimi_k3", num_layers=2, first_k_dense=0,
                       n_routed_experts=16, num_experts_per_tok=4, moe_latent_size=128,
                       moe_intermediate_size=64, quant="none")


def tiny_kimi_linear() -> ModelConfig:
    """Three KDA layers to one MLA layer, as in Kimi-Linear; LatentMoE off."""
    return ModelConfig(name="tiny-kimi-linear", family="kimi_k3", num_layers=4, first_k_dense=1,
                       n_routed_experts=8, num_experts_per_tok=2, moe_intermediate_size=64,
                       kda_layers=(0, 1, 2), kda_num_heads=2, kda_head_dim=64, kda_gate_rank=32)


def tiny_kimi_k31() -> ModelConfig:
    """KDA layers plus an MLA layer that carries a DSA indexer (the Kimi-K3.1 arrangement)."""
    import dataclasses
    return dataclasses.replace(tiny_kimi_linear(), name="tiny-kimi-k3.1", index_n_heads=4, index_head_dim=32,
                               index_topk=16, indexer_full_layers=(3,))


def tiny_gpt_oss() -> ModelConfig:
    return ModelConfig(name="tiny-gpt-oss", family="gpt_oss", num_layers=2, first_k_dense=0,
                       num_heads=8, num_kv_heads=2, head_dim=32, sliding_window=16,
                       attention_sinks=True, scoring_func="softmax", n_shared_experts=0,
                       n_routed_experts=8, num_experts_per_tok=2, activation="swiglu_clamped",
                       rope_interleaved=False)


def tiny_minimax() -> ModelConfig:
    """MiniMax-shaped GQA + FP8 MoE at the smallest geometry the GPU kernels tile (head_dim 128, hidden 1024)."""
    return ModelConfig(name="tiny-minimax", family="minimax", vocab_size=4096, hidden_size=1024, num_layers=2,
                       first_k_dense=0, moe_intermediate_size=512, n_routed_experts=16, n_shared_experts=0,
                       num_experts_per_tok=4, num_heads=16, num_kv_heads=4, head_dim=128, rope_interleaved=False,
                       quant="fp8_block")


def tiny_gpt_oss_64() -> ModelConfig:
    """GPT-OSS-shaped GQA (head_dim 64, sinks, sliding window on alternate layers) at kernel-sized geometry."""
    return ModelConfig(name="tiny-gpt-oss-64", family="gpt_oss", vocab_size=4096, hidden_size=1024, num_layers=2,
                       first_k_dense=0, moe_intermediate_size=512, n_routed_experts=16, n_shared_experts=0,
                       num_experts_per_tok=4, num_heads=16, num_kv_heads=4, head_dim=64, sliding_window=128,
                       attention_sinks=True, scoring_func="softmax", activation="swiglu_clamped",
                       rope_interleaved=False)


def tiny_deepseek_v2() -> ModelConfig:
    """DeepSeek-V2 routing at toy size: softmax over all experts, groups ranked by their best expert, weights not
    renormalised, two shared experts."""
    return ModelConfig(name="tiny-deepseek-v2", family="deepseek_v2", num_layers=2, first_k_dense=1,
                       n_routed_experts=16, n_shared_experts=2, num_experts_per_tok=4, n_group=4, topk_group=2,
                       scoring_func="softmax_all", norm_topk_prob=False, routed_scaling_factor=4.0,
                       moe_intermediate_size=64)


def tiny_mixtral() -> ModelConfig:
    return ModelConfig(name="tiny-mixtral", family="mixtral", num_layers=2, first_k_dense=0, num_heads=8,
                       num_kv_heads=2, head_dim=32, scoring_func="softmax", n_shared_experts=0, n_routed_experts=8,
                       num_experts_per_tok=2, rope_interleaved=False, rope_theta=1e6)


def tiny_qwen2_moe() -> ModelConfig:
    """Qwen2-MoE at toy size: biased q/k/v, softmax over all experts without renormalisation, gated shared expert."""
    return ModelConfig(name="tiny-qwen2-moe", family="qwen2_moe", num_layers=2, first_k_dense=0, num_heads=8,
                       num_kv_heads=2, head_dim=32, attention_bias=True, scoring_func="softmax_all",
                       norm_topk_prob=False, n_shared_experts=2, shared_expert_gate=True, n_routed_experts=8,
                       num_experts_per_tok=2, moe_intermediate_size=64, rope_interleaved=False, rope_theta=1e6)


def deepseek_v2_236b() -> ModelConfig:
    """DeepSeek-V2 (236B): the MLA + MoE generation before V3 (reference: batchgen/models/deepseek/deepseekv2/config_v2.json)."""
    return ModelConfig(
        name="deepseek-v2", family="deepseek_v2", vocab_size=102400, hidden_size=5120, num_layers=60,
        first_k_dense=1, intermediate_size=12288, moe_intermediate_size=1536, n_routed_experts=160,
        n_shared_experts=2, num_experts_per_tok=6, n_group=8, topk_group=3, routed_scaling_factor=16.0,
        norm_topk_prob=False, scoring_func="softmax_all", num_heads=128, q_lora_rank=1536, kv_lora_rank=512,
        qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128, rope_theta=10000.0, rope_scaling_factor=40.0,
        rope_original_max_pos=4096, rope_mscale=0.707, rope_mscale_all_dim=0.707, eos_token_id=100001,
        bos_token_id=100000)


def mixtral_8x7b() -> ModelConfig:
    """Mixtral-8x7B (reference: batchgen/models/mixtral/config.py)."""
    return ModelConfig(
        name="mixtral-8x7b", family="mixtral", vocab_size=32000, hidden_size=4096, num_layers=32, first_k_dense=0,
        moe_intermediate_size=14336, n_routed_experts=8, n_shared_experts=0, num_experts_per_tok=2,
        scoring_func="softmax", num_heads=32, num_kv_heads=8, head_dim=128, rope_theta=1e6, rope_interleaved=False,
        max_position_embeddings=32768, rms_eps=1e-5, eos_token_id=2, bos_token_id=1)


def mixtral_8x22b() -> ModelConfig:
    import dataclasses
    return dataclasses.replace(mixtral_8x7b(), name="mixtral-8x22b", hidden_size=6144, num_layers=56,
                               moe_intermediate_size=16384, num_heads=48, max_position_embeddings=65536)


def qwen2_57b_a14b() -> ModelConfig:
    """Qwen2-57B-A14B, the Qwen2-MoE checkpoint family the reference's Qwen initializer serves
    (batchgen/models/Qwen_Initializer.py)."""
    return ModelConfig(
        name="qwen2-57b-a14b", family="qwen2_moe", vocab_size=151936, hidden_size=3584, num_layers=28,
        first_k_dense=0, moe_intermediate_size=2560, n_routed_experts=64, n_shared_experts=8,
        shared_expert_gate=True, num_experts_per_tok=8, scoring_func="softmax_all", norm_topk_prob=False,
        num_heads=28, num_kv_heads=4, head_dim=128, attention_bias=True, rope_theta=1e6, rope_interleaved=False,
        max_position_embeddings=65536, eos_token_id=151643, bos_token_id=151643)


def qwen15_moe_a27b() -> ModelConfig:
    return ModelConfig(
        name="qwen1.5-moe-a2.7b", family="qwen2_moe", vocab_size=151936, hidden_size=2048, num_layers=24,
        first_k_dense=0, moe_intermediate_size=1408, n_routed_experts=60, n_shared_experts=4,
        shared_expert_gate=True, num_experts_per_tok=4, scoring_func="softmax_all", norm_topk_prob=False,
        num_heads=16, num_kv_heads=16, head_dim=128, attention_bias=True, rope_theta=1e6, rope_interleaved=False,
        max_position_embeddings=8192, eos_token_id=151643, bos_token_id=151643)


def tiny_deepseek_v4() -> ModelConfig:
    """DeepSeek-V4 at toy size: a window-only layer, an overlapped ratio-4 layer with its indexer, and a ratio-8
    layer; the first layer routes by token id."""
    return ModelConfig(name="tiny-deepseek-v4", family="deepseek_v4", vocab_size=512, hidden_size=128, num_layers=3,
                       first_k_dense=0, moe_intermediate_size=64, n_routed_experts=8, n_shared_experts=1,
                       num_experts_per_tok=2, scoring_func="sqrtsoftplus", routed_scaling_factor=1.5,
                       num_heads=4, head_dim=64, q_lora_rank=64, qk_rope_head_dim=16, sliding_window=8,
                       compress_ratios=(0, 4, 8), compress_rope_theta=160000.0, rope_scaling_factor=4.0,
                       rope_original_max_pos=64, o_groups=2, o_lora_rank=32, hc_mult=2, hc_sinkhorn_iters=4,
                       num_hash_layers=1, swiglu_limit=10.0, index_n_heads=8, index_head_dim=32, index_topk=4)


def _v4_ratios(head: Tuple[int, ...], n_layers: int) -> Tuple[int, ...]:
    rest = n_layers - len(head)
    return head + tuple(4 if i % 2 == 0 else 128 for i in range(rest))


def deepseek_v4_flash() -> ModelConfig:
    """DeepSeek-V4-Flash (reference: batchgen/models/deepseek/deepseekv4_flash/config.py:36-119)."""
    return ModelConfig(
        name="deepseek-v4-flash", family="deepseek_v4", vocab_size=129280, hidden_size=4096, num_layers=43,
        first_k_dense=0, moe_intermediate_size=2048, n_routed_experts=256, n_shared_experts=1,
        num_experts_per_tok=6, scoring_func="sqrtsoftplus", routed_scaling_factor=1.5, norm_topk_prob=True,
        num_heads=64, head_dim=512, q_lora_rank=1024, qk_rope_head_dim=64, sliding_window=128,
        compress_ratios=_v4_ratios((0, 0), 43), compress_rope_theta=160000.0, rope_theta=10000.0,
        rope_scaling_factor=16.0, rope_original_max_pos=65536, o_groups=8, o_lora_rank=1024, hc_mult=4,
        hc_sinkhorn_iters=20, num_hash_layers=3, swiglu_limit=10.0, index_n_heads=64, index_head_dim=128,
        index_topk=512, max_position_embeddings=1048576, quant="mxfp4", quant_block=32, eos_token_id=1,
        bos_token_id=0)


def deepseek_v4_pro() -> ModelConfig:
    import dataclasses
    return dataclasses.replace(
        deepseek_v4_flash(), name="deepseek-v4-pro", hidden_size=7168, num_layers=61, moe_intermediate_size=3072,
        n_routed_experts=384, routed_scaling_factor=2.5, num_heads=128, q_lora_rank=1536, o_groups=16,
        compress_ratios=_v4_ratios((128, 128), 61), index_topk=1024)


def deepseek_v3_671b() -> ModelConfig:
    return ModelConfig(
        name="deepseek-v3-671b", family="deepseek_v3", vocab_size=129280, hidden_size=7168,
        num_layers=61, first_k_dense=3, intermediate_size=18432, moe_intermediate_size=2048,
        n_routed_experts=256, n_shared_experts=1, num_experts_per_tok=8, n_group=8, topk_group=4,
        routed_scaling_factor=2.5, norm_topk_prob=True, num_heads=128, q_lora_rank=1536,
        kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
        rope_theta=10000.0, rope_scaling_factor=40.0, rope_original_max_pos=4096,
        rope_mscale=1.0, rope_mscale_all_dim=1.0, quant="fp8_block", eos_token_id=1)


def glm5_3() -> ModelConfig:
    full = tuple(sorted(set(list(range(0, 78, 4)) + [77])))[:21]
    return ModelConfig(
        name="glm-5.3-fp8", family="glm5", vocab_size=154880, hidden_size=6144, num_layers=78,
        first_k_dense=3, intermediate_size=12288, moe_intermediate_size=2048,
        n_routed_experts=256, n_shared_experts=1, num_experts_per_tok=8, n_group=1, topk_group=1,
        routed_scaling_factor=2.5, num_heads=64, q_lora_rank=2048, kv_lora_rank=512,
        qk_nope_head_dim=192, qk_rope_head_dim=64, v_head_dim=256, rope_theta=1000000.0,
        rope_interleaved=True, index_n_heads=32, index_head_dim=128, index_topk=2048,
        indexer_full_layers=full, quant="fp8_block", max_position_embeddings=1048576)


def kimi_k3() -> ModelConfig:
    return ModelConfig(
        name="kimi-k3", family="kimi_k3", vocab_size=163840, hidden_size=7168, num_layers=93,
        first_k_dense=1, intermediate_size=18432, moe_intermediate_size=3072,
        n_routed_experts=896, n_shared_experts=1, num_experts_per_tok=16, n_group=1,
        topk_group=1, routed_scaling_factor=2.5, moe_latent_size=3584, num_heads=64,
        q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64,
        v_head_dim=128, quant="mxfp4", quant_block=32)


def kimi_k3_kda() -> ModelConfig:
    """Kimi-K3 with its linear-attention layers: of the 93 layers every fourth (24 in all) is NoPE-MLA,
    the other 69 are KDA (64 heads of 128)."""
    import dataclasses
    mla = set(range(3, 93, 4)) | {92}
    return dataclasses.replace(kimi_k3(), name="kimi-k3-kda", kda_layers=tuple(l for l in range(93) if l not in mla),
                               kda_num_heads=64, kda_head_dim=128)


def kimi_k31() -> ModelConfig:
    """Kimi-K3.1: K3 with KDA layers and a DSA indexer (top-2048, 32 heads of 128) on every MLA layer."""
    import dataclasses
    base = kimi_k3_kda()
    mla = tuple(l for l in range(base.num_layers) if l not in base.kda_layers)
    return dataclasses.replace(base, name="kimi-k3.1", index_n_heads=32, index_head_dim=128, index_topk=2048,
                               indexer_full_layers=mla)


def kimi_linear_48b() -> ModelConfig:
    return ModelConfig(
        name="kimi-linear-48b", family="kimi_k3", vocab_size=163840, hidden_size=2304, num_layers=27,
        first_k_dense=1, intermediate_size=9216, moe_intermediate_size=1024, n_routed_experts=256,
        n_shared_experts=1, num_experts_per_tok=8, routed_scaling_factor=2.446, num_heads=32,
        q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
        kda_layers=tuple(l for l in range(27) if l % 4 != 3), kda_num_heads=32, kda_head_dim=128)


def kimi_k25() -> ModelConfig:
    return ModelConfig(
        name="kimi-k2.5", family="kimi_k25", vocab_size=163840, hidden_size=7168, num_layers=61,
        first_k_dense=1, intermediate_size=18432, moe_intermediate_size=2048,
        n_routed_experts=384, n_shared_experts=1, num_experts_per_tok=8, routed_scaling_factor=2.827,
        num_heads=64, q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128,
        qk_rope_head_dim=64, v_head_dim=128, quant="mxfp4", quant_block=32)


def gpt_oss_120b() -> ModelConfig:
    return ModelConfig(
        name="gpt-oss-120b", family="gpt_oss", vocab_size=201088, hidden_size=2880, num_layers=36,
        first_k_dense=0, moe_intermediate_size=2880, n_routed_experts=128, n_shared_experts=0,
        num_experts_per_tok=4, scoring_func="softmax", num_heads=64, num_kv_heads=8, head_dim=64,
        sliding_window=128, attention_sinks=True, activation="swiglu_clamped",
        rope_theta=150000.0, rope_interleaved=False, rope_scaling_factor=32.0, quant="mxfp4",
        quant_block=32)


def minimax_m25() -> ModelConfig:
    return ModelConfig(
        name="minimax-m2.5", family="minimax", vocab_size=200064, hidden_size=3072, num_layers=62,
        first_k_dense=0, moe_intermediate_size=1536, n_routed_experts=256, n_shared_experts=0,
        num_experts_per_tok=8, num_heads=48, num_kv_heads=8, head_dim=128, rope_interleaved=False,
        quant="fp8_block")


# ------------------------------------------------------------------ Nanurax: layer-listed config.json
def _nanurax_layer(d: Dict, index: int) -> LayerSpec:
    m, kind = d["mixer"], d["type"]
    if kind == "general_delta":
        mixer = MixerSpec(kind, heads=m["heads"], dim=m["dim"], vdim=m["dim"])
    elif kind == "attention":
        mixer = MixerSpec(kind, heads=m["heads"], dim=m["dim"], kv_heads=m.get("kv_heads", m["heads"]),
                          vdim=m.get("vdim", m["dim"]), scale=float(m["scale"]),
                          chunk=int((m.get("mask") or {}).get("size", 0)), talking=True, sink=True)
        if mixer.heads % mixer.kv_heads:
            raise ValueError(f"layer {index}: {mixer.heads} heads do not divide over {mixer.kv_heads} key/value heads")
    else:
        raise ValueError(f"layer {index}: unknown mixer type {kind!r}")
    f = d.get("mlp")
    if not f:
        return LayerSpec(mixer)
    if f["kind"] == "dense":
        return LayerSpec(mixer, MlpSpec("dense", ff=f["ff"]))
    if f["kind"] != "moe":
        raise ValueError(f"layer {index}: unknown feed-forward kind {f['kind']!r}")
    sh = f.get("shared") or {}
    return LayerSpec(mixer, MlpSpec("moe", ff=f["expert"]["ff"], activation="swiglu_oai", limit=float(f["expert"]["limit"]),
                                    experts=f["router"]["experts"], top=f["router"]["top"], weight_on_input=True,
                                    shared_ff=sh.get("ff", 0), shared_limit=float(sh.get("limit", 0.0))))


def nanurax_config(d: Dict, name: str = "nanurax", decay_ranks: Optional[Dict[int, int]] = None) -> ModelConfig:
    """A Nanurax config.json (parsed) as a ``ModelConfig``.  ``decay_ranks``: per recurrent layer the width of its
    low-rank decay projection, which only the checkpoint's tensor shapes tell (default 64)."""
    layers = [_nanurax_layer(x, i) for i, x in enumerate(d["layers"])]
    for i, s in enumerate(layers):
        if s.mixer.recurrent:
            rank = (decay_ranks or {}).get(i, 64)
            layers[i] = dataclasses.replace(s, mixer=dataclasses.replace(s.mixer, decay_rank=rank))
    moe = [s.mlp for s in layers if s.mlp.kind == "moe"]
    att = [s.mixer for s in layers if not s.mixer.recurrent]
    return ModelConfig(
        name=name, family="nanurax", vocab_size=d["vocab"], hidden_size=d["width"], num_layers=len(layers),
        layer_specs=tuple(layers), embed_scale=float(d["embedding"]["scale"]), rms_eps=float(d["norm"]["eps"]),
        # summaries that planners read; the layers themselves are described by ``layer_specs``
        num_heads=max(s.mixer.heads for s in layers), num_kv_heads=max((m.kv_heads for m in att), default=1),
        head_dim=max(s.mixer.dim for s in layers), first_k_dense=0,
        intermediate_size=max((s.mlp.ff for s in layers if s.mlp.kind == "dense"), default=0),
        moe_intermediate_size=max((f.ff for f in moe), default=0), n_routed_experts=max((f.experts for f in moe), default=0),
        num_experts_per_tok=max((f.top for f in moe), default=0), n_shared_experts=int(any(f.shared_ff for f in moe)),
        attention_sinks=bool(att), max_position_embeddings=1 << 30, eos_token_id=-1, bos_token_id=-1)


def _nanurax_dir(path: str, d: Dict) -> ModelConfig:
    from .ckpt.safetensors_dir import checkpoint_shapes
    shapes = checkpoint_shapes(path)
    ranks = {i: shapes[f"l{i}.mix.w1"][0] for i in range(len(d["layers"])) if f"l{i}.mix.w1" in shapes}
    cfg = nanurax_config(d, os.path.basename(os.path.normpath(path)) or "nanurax", ranks)
    cfg.checkpoint_dir = path
    return cfg


# ------------------------------------------------------------------ Pamevik: layer-listed config.json
def _pamevik_layer(d: Dict, index: int, ranks: Tuple[int, int]) -> LayerSpec:
    m, kind = d["mixer"], d["type"]

    def divides(x: MixerSpec) -> MixerSpec:
        if x.heads % x.qk_heads:
            raise ValueError(f"layer {index}: {x.heads} heads do not divide over {x.qk_heads} key heads")
        if x.rot_dims % 2 or x.rot_dims > x.dim:
            raise ValueError(f"layer {index}: {x.rot_dims} rotary dimensions in heads of {x.dim}")
        return x

    def rotary(x: Dict) -> Dict:
        r = x.get("rot")
        return {"rot_dims": int(r["dims"]), "rot_base": float(r["base"])} if r else {}
    second = None
    if kind == "mlstm":
        mixer = MixerSpec(kind, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], gate_cap=float(m["gate_cap"]))
    elif kind == "channel_delta":
        mixer = MixerSpec(kind, heads=m["heads"], dim=m["dim"], kv_heads=m.get("kv_heads", m["heads"]), vdim=m["vdim"],
                          conv=int(m["conv"]), decay_rank=ranks[0], gate_rank=ranks[1])
    elif kind == "parallel":
        a, r = m["left"], m["right"]
        mixer = MixerSpec("attention", heads=a["heads"], dim=a["dim"], kv_heads=a.get("kv_heads", a["heads"]), vdim=a["vdim"],
                          scale=float(a["scale"]), out_gate=True, **rotary(a))
        second = divides(MixerSpec("retention", heads=r["heads"], dim=r["dim"], vdim=r["vdim"],
                                   decay=tuple(float(x) for x in r["decay"]), **rotary(r)))
        if len(second.decay) != second.heads:
            raise ValueError(f"layer {index}: {len(second.decay)} decays for {second.heads} heads")
    else:
        raise ValueError(f"layer {index}: unknown mixer type {kind!r}")
    f = d.get("mlp")
    if f and f["kind"] != "dense":
        raise ValueError(f"layer {index}: unknown feed-forward kind {f['kind']!r}")
    return LayerSpec(divides(mixer), MlpSpec("dense", ff=f["ff"], activation="relu2") if f else MlpSpec(), second)


def pamevik_config(d: Dict, name: str = "pamevik", ranks: Optional[Dict[int, Tuple[int, int]]] = None) -> ModelConfig:
    """A Pamevik config.json (parsed) as a ``ModelConfig``.  ``ranks``: per channel_delta layer the widths of its low-rank
    decay and output-gate projections, which only the checkpoint's tensor shapes tell (default 64)."""
    layers = tuple(_pamevik_layer(x, i, (ranks or {}).get(i, (64, 64))) for i, x in enumerate(d["layers"]))
    att = [m for s in layers for m in s.mixers if not m.recurrent]
    return ModelConfig(
        name=name, family="pamevik", vocab_size=d["vocab"], hidden_size=d["width"], num_layers=len(layers), layer_specs=layers,
        rms_eps=float(d["norm"]["eps"]), sandwich=True, layer_norm=True, canon_taps=int(d["canon"]["taps"]),
        # summaries that planners read; the layers themselves are described by ``layer_specs``
        num_heads=max(m.heads for s in layers for m in s.mixers), num_kv_heads=max((m.kv_heads for m in att), default=1),
        head_dim=max(m.dim for s in layers for m in s.mixers), first_k_dense=0,
        intermediate_size=max(s.mlp.ff for s in layers), moe_intermediate_size=0, n_routed_experts=0, n_shared_experts=0,
        num_experts_per_tok=0, max_position_embeddings=1 << 30, eos_token_id=-1, bos_token_id=-1)


def _pamevik_dir(path: str, d: Dict) -> ModelConfig:
    from .ckpt.safetensors_dir import checkpoint_shapes
    shapes = checkpoint_shapes(path)
    ranks = {i: (shapes[f"l{i}.mix.a1"][0], shapes[f"l{i}.mix.g1"][0]) for i in range(len(d["layers"]))
             if f"l{i}.mix.a1" in shapes and f"l{i}.mix.g1" in shapes}
    cfg = pamevik_config(d, os.path.basename(os.path.normpath(path)) or "pamevik", ranks)
    cfg.checkpoint_dir = path
    return cfg


# ------------------------------------------------------------------ Bolisun: layer-listed config.json
def _bolisun_layer(d: Dict, index: int) -> LayerSpec:
    if d["type"] != "parallel":
        raise ValueError(f"layer {index}: unknown mixer type {d['type']!r}")
    m, f = d["mixer"], d.get("mlp")
    a, r, rot, mask = m["left"], m["right"], m["left"].get("rot") or {}, m["left"].get("mask") or {}
    sc = rot.get("scaling")
    left = MixerSpec(
        "attention", heads=a["heads"], dim=a["dim"], kv_heads=a.get("kv_heads", a["heads"]), vdim=a["vdim"], scale=float(a["scale"]),
        window=int(mask.get("size", 0)), keep_first=int(mask.get("keep_first", 0)), bias=True, out_bias=True, qk_norm=True,
        rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)), rot_interleaved=True,
        yarn=tuple(float(sc[k]) for k in ("factor", "original", "fast", "slow")) if sc else (), out_scale=float(m["left_scale"]))
    right = MixerSpec("retention", heads=r["heads"], dim=r["dim"], vdim=r["vdim"], decay=tuple(float(x) for x in r["decay"]),
                      out_scale=float(m["right_scale"]))
    if left.heads % left.kv_heads:
        raise ValueError(f"layer {index}: {left.heads} heads do not divide over {left.kv_heads} key heads")
    if left.rot_dims % 2 or left.rot_dims > left.dim:
        raise ValueError(f"layer {index}: {left.rot_dims} rotary dimensions in heads of {left.dim}")
    if mask and left.window < 1:
        raise ValueError(f"layer {index}: a window of {left.window} positions")
    if len(right.decay) != right.heads:
        raise ValueError(f"layer {index}: {len(right.decay)} decays for {right.heads} heads")
    mlp = MlpSpec()
    if f and f["kind"] == "dense":
        mlp = MlpSpec("dense", ff=f["ff"], activation="swiglu_oai", limit=float(f["limit"]))
    elif f and f["kind"] == "moe":
        ro = f["router"]
        g = ro.get("groups") or {"count": 1, "keep": 1}
        mlp = MlpSpec("moe", ff=f["expert"]["ff"], activation="silu", experts=ro["experts"], top=ro["top"],
                      shared_ff=(f.get("shared") or {}).get("ff", 0), shared_gate=False, scoring="softmax_all", correction=True,
                      groups=g["count"], keep_groups=g["keep"], group_score="max", norm_weights=True, router_scale=float(ro["scale"]))
        if mlp.experts % mlp.groups or mlp.keep_groups > mlp.groups or mlp.top > mlp.experts // mlp.groups * mlp.keep_groups:
            raise ValueError(f"layer {index}: top {mlp.top} of {mlp.experts} experts in the best {mlp.keep_groups} of {mlp.groups} groups")
    elif f:
        raise ValueError(f"layer {index}: unknown feed-forward kind {f['kind']!r}")
    return LayerSpec(left, mlp, right)


def bolisun_config(d: Dict, name: str = "bolisun") -> ModelConfig:
    """A Bolisun config.json (parsed) as a ``ModelConfig``."""
    layers = []
    for i, x in enumerate(d["layers"]):
        j, seen = i, {i}
        while d["layers"][j].get("weights_of") is not None:
            j = d["layers"][j]["weights_of"]
            if not 0 <= j < len(d["layers"]) or j in seen:
                raise ValueError(f"layer {i}: weights of layer {j}")
            seen.add(j)
        spec = _bolisun_layer({**d["layers"][j], **x}, i)
        if j != i:
            if spec != _bolisun_layer(d["layers"][j], j):
                raise ValueError(f"layer {i} differs from layer {j}, whose weights it uses")
            spec = dataclasses.replace(spec, weights_of=j)
        layers.append(spec)
    moe = [s.mlp for s in layers if s.mlp.kind == "moe"]
    return ModelConfig(
        name=name, family="bolisun", vocab_size=d["vocab"], hidden_size=d["width"], num_layers=len(layers), layer_specs=tuple(layers),
        embed_scale=float(d["embedding"]["scale"]), rms_eps=float(d["norm"]["eps"]), streams=int(d["streams"]), tie_word_embeddings=True,
        # summaries that planners read; the layers themselves are described by ``layer_specs``
        num_heads=max(m.heads for s in layers for m in s.mixers), num_kv_heads=max(s.mixer.kv_heads for s in layers),
        head_dim=max(m.dim for s in layers for m in s.mixers), sliding_window=max(s.mixer.window for s in layers), first_k_dense=0,
        intermediate_size=max((s.mlp.ff for s in layers if s.mlp.kind == "dense"), default=0),
        moe_intermediate_size=max((f.ff for f in moe), default=0), n_routed_experts=max((f.experts for f in moe), default=0),
        num_experts_per_tok=max((f.top for f in moe), default=0), n_shared_experts=int(any(f.shared_ff for f in moe)),
        attention_bias=True, scoring_func="softmax_all", max_position_embeddings=1 << 30, eos_token_id=-1, bos_token_id=-1)


def _bolisun_dir(path: str, d: Dict) -> ModelConfig:
    cfg = bolisun_config(d, os.path.basename(os.path.normpath(path)) or "bolisun")
    cfg.checkpoint_dir = path
    return cfg


# ------------------------------------------------------------------ Pitudra: layer-listed config.json
def _pitudra_layer(d: Dict, index: int, layers: List[Dict]) -> LayerSpec:
    m, kind, f = d["mixer"], d["type"], d.get("mlp")
    window = int((m.get("mask") or {}).get("size", 0))
    if m.get("mask") and window < 1:
        raise ValueError(f"layer {index}: a window of {window} positions")
    if kind == "hgrn2":
        mixer = MixerSpec(kind, heads=m["heads"], dim=m["dim"], vdim=m.get("vdim", m["dim"]))
    elif kind == "attention":
        mixer = MixerSpec(kind, heads=m["heads"], dim=m["dim"], kv_heads=m.get("kv_heads", m["heads"]), vdim=m.get("vdim", m["dim"]),
                          scale=float(m["scale"]), window=window, bias=True, qk_norm_all=True, head_sinks=True, out_gate_all=True)
        if mixer.heads % mixer.kv_heads:
            raise ValueError(f"layer {index}: {mixer.heads} heads do not divide over {mixer.kv_heads} key/value heads")
    elif kind == "latent_attention":
        rot, j = m["rot"], m.get("kv_from")
        mixer = MixerSpec(kind, heads=m["heads"], dim=m["dim"], vdim=m.get("vdim", m["dim"]), scale=float(m["scale"]), window=window, head_sinks=True,
                          q_rank=m["q_rank"], kv_rank=m["kv_rank"], rot_dim=m["rot_dim"], rot_dims=int(rot["dims"]),
                          rot_base=float(rot["base"]), kv_from=-1 if j is None else int(j))
        if mixer.rot_dims != mixer.rot_dim or mixer.rot_dim % 2:
            raise ValueError(f"layer {index}: {mixer.rot_dims} rotary dimensions in a rotated part of {mixer.rot_dim}")
        if j is not None:
            src = layers[j]["mixer"] if 0 <= j < index and layers[j]["type"] == kind else {"kv_from": j}
            if src.get("kv_from") is not None:
                raise ValueError(f"layer {index}: latents of layer {j}, which has none of its own before it")
            if any(src[k] != m[k] for k in ("kv_rank", "rot_dim", "rot")):
                raise ValueError(f"layer {index}: latents of another shape or rotation than those of layer {j}")
    else:
        raise ValueError(f"layer {index}: unknown mixer type {kind!r}")
    if not f:
        return LayerSpec(mixer)
    if f["kind"] != "moe":
        raise ValueError(f"layer {index}: unknown feed-forward kind {f['kind']!r}")
    mlp = MlpSpec("moe", ff=f["expert"]["ff"], activation="relu2", experts=f["router"]["experts"], top=f["router"]["top"], scoring="softmax")
    if not 0 < mlp.top <= mlp.experts:
        raise ValueError(f"layer {index}: top {mlp.top} of {mlp.experts} experts")
    return LayerSpec(mixer, mlp)


def pitudra_config(d: Dict, name: str = "pitudra") -> ModelConfig:
    """A Pitudra config.json (parsed) as a ``ModelConfig``."""
    layers = tuple(_pitudra_layer(x, i, d["layers"]) for i, x in enumerate(d["layers"]))
    moe = [s.mlp for s in layers if s.mlp.kind == "moe"]
    return ModelConfig(
        name=name, family="pitudra", vocab_size=d["vocab"], hidden_size=d["width"], num_layers=len(layers), layer_specs=layers,
        rms_eps=float(d["norm"]["eps"]), sandwich=True, pre_norm=False, layer_norm=True, token_shift=True,
        side_dim=int((d.get("token_side") or {}).get("dim", 0)),
        # summaries that planners read; the layers themselves are described by ``layer_specs``
        num_heads=max(s.mixer.heads for s in layers), num_kv_heads=max((s.mixer.kv_heads for s in layers), default=1) or 1,
        head_dim=max(s.mixer.dim for s in layers), sliding_window=max(s.mixer.window for s in layers), first_k_dense=0,
        intermediate_size=0, moe_intermediate_size=max((f.ff for f in moe), default=0),
        n_routed_experts=max((f.experts for f in moe), default=0), num_experts_per_tok=max((f.top for f in moe), default=0),
        n_shared_experts=0, attention_sinks=any(s.mixer.head_sinks for s in layers), attention_bias=True, scoring_func="softmax",
        max_position_embeddings=1 << 30, eos_token_id=-1, bos_token_id=-1)


def _pitudra_dir(path: str, d: Dict) -> ModelConfig:
    cfg = pitudra_config(d, os.path.basename(os.path.normpath(path)) or "pitudra")
    cfg.checkpoint_dir = path
    return cfg


# config.json "architecture" -> reader of the model directory
_ARCHITECTURES = {"Nanurax": _nanurax_dir, "Pamevik": _pamevik_dir, "Bolisun": _bolisun_dir, "Pitudra": _pitudra_dir}


def load_model_dir(path: str) -> ModelConfig:
    """Config of a model directory (config.json + .safetensors), chosen by the file's ``architecture``."""
    with open(os.path.join(path, "config.json")) as f:
        d = json.load(f)
    arch = d.get("architecture")
    if arch not in _ARCHITECTURES:
        raise KeyError(f"{path}: architecture {arch!r} is not supported from a directory; known: {sorted(_ARCHITECTURES)}")
    return _ARCHITECTURES[arch](path, d)


def tiny_nanurax() -> ModelConfig:
    """One attention layer between two delta-rule layers; dense, mixture and no feed-forward."""
    delta = {"type": "general_delta", "mixer": {"heads": 3, "dim": 24}}
    attn = {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 32, "scale": 0.25,
                                           "mask": {"size": 40}}}
    moe = {"kind": "moe", "expert": {"ff": 40, "limit": 1.25}, "router": {"experts": 6, "top": 2},
           "shared": {"ff": 56, "limit": 0.8}}
    return nanurax_config({
        "vocab": 320, "width": 120, "norm": {"eps": 1e-5}, "embedding": {"scale": 9.0},
        "layers": [dict(delta, mlp={"kind": "dense", "ff": 200}), dict(attn, mlp=moe), dict(delta, mlp=None)]},
        "tiny-nanurax", {0: 12, 2: 12})


def nanurax_bench() -> ModelConfig:
    """Layers of a real model's size: three delta-rule layers to one attention layer, dense and mixture feed-forwards."""
    delta = {"type": "general_delta", "mixer": {"heads": 32, "dim": 128}}
    attn = {"type": "attention", "mixer": {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                           "mask": {"size": 4096}}}
    dense = {"kind": "dense", "ff": 9216}
    moe = {"kind": "moe", "expert": {"ff": 1024, "limit": 7.0}, "router": {"experts": 64, "top": 8},
           "shared": {"ff": 1024, "limit": 7.0}}
    return nanurax_config({
        "vocab": 163840, "width": 2304, "norm": {"eps": 1e-6}, "embedding": {"scale": 48.0},
        "layers": [dict(delta, mlp=dense), dict(delta, mlp=moe), dict(delta, mlp=moe), dict(attn, mlp=moe)]},
        "nanurax-bench")


def tiny_pamevik() -> ModelConfig:
    """One layer of every mixer, with and without a feed-forward."""
    cd = {"type": "channel_delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 40, "conv": 3}}
    ml = {"type": "mlstm", "mixer": {"heads": 3, "dim": 20, "vdim": 32, "gate_cap": 9.0}}
    par = {"type": "parallel", "mixer": {
        "left": {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 24, "scale": 0.2, "rot": {"base": 5000.0, "dims": 16}},
        "right": {"heads": 2, "dim": 16, "vdim": 40, "decay": [0.9, 0.99], "rot": {"base": 800.0, "dims": 16}}}}
    return pamevik_config({
        "vocab": 320, "width": 120, "norm": {"eps": 1e-5}, "canon": {"taps": 3},
        "layers": [dict(cd, mlp={"kind": "dense", "ff": 200}), dict(par, mlp=None), dict(ml, mlp={"kind": "dense", "ff": 88})]},
        "tiny-pamevik", {0: (12, 20)})


def pamevik_bench() -> ModelConfig:
    """Layers of a real model's size: channel-delta, mLSTM, channel-delta and one attention-beside-retention layer.  The
    feed-forward's two matrices hold as many weights as the three of a gated one of width 9216."""
    dense = {"kind": "dense", "ff": 13824}
    cd = {"type": "channel_delta", "mlp": dense, "mixer": {"heads": 32, "kv_heads": 32, "dim": 128, "vdim": 128, "conv": 4}}
    ml = {"type": "mlstm", "mlp": dense, "mixer": {"heads": 32, "dim": 128, "vdim": 128, "gate_cap": 15.0}}
    rot = {"base": 1e6, "dims": 128}
    par = {"type": "parallel", "mlp": dense, "mixer": {
        "left": {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": rot},
        "right": {"heads": 32, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-5 - 7 * i / 31) for i in range(32)], "rot": rot}}}
    return pamevik_config({"vocab": 163840, "width": 2304, "norm": {"eps": 1e-6}, "canon": {"taps": 4},
                           "layers": [cd, ml, dict(cd), par]}, "pamevik-bench", {0: (128, 128), 2: (128, 128)})


def tiny_bolisun() -> ModelConfig:
    """A dense layer, a mixture layer that runs twice, a layer without a feed-forward."""
    def layer(window, keep, mlp):
        return {"type": "parallel", "mlp": mlp, "mixer": {
            "left_scale": 0.7, "right_scale": 1.1,
            "left": {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 24, "scale": 0.2, "mask": {"size": window, "keep_first": keep},
                     "rot": {"base": 9000.0, "dims": 16, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}},
            "right": {"heads": 3, "dim": 16, "vdim": 40, "decay": [0.9, 0.97, 0.995]}}}
    moe = {"kind": "moe", "expert": {"ff": 40}, "shared": {"ff": 56},
           "router": {"experts": 8, "top": 2, "scale": 1.5, "groups": {"count": 4, "keep": 2}}}
    return bolisun_config({
        "vocab": 320, "width": 120, "streams": 3, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
        "layers": [layer(33, 5, {"kind": "dense", "ff": 200, "limit": 2.0}), layer(20, 0, moe), dict(layer(20, 0, moe), weights_of=1),
                   layer(50, 2, None)]}, "tiny-bolisun")


def bolisun_bench() -> ModelConfig:
    """Layers of a real model's size: four layers of windowed attention beside retention, one dense and three mixture
    feed-forwards (64 experts of which 8 run, and a shared one), the last mixture layer with the weights of the one before."""
    dense = {"kind": "dense", "ff": 9216, "limit": 7.0}
    moe = {"kind": "moe", "expert": {"ff": 1024}, "shared": {"ff": 1024},
           "router": {"experts": 64, "top": 8, "scale": 2.5, "groups": {"count": 8, "keep": 4}}}
    par = {"type": "parallel", "mixer": {
        "left_scale": 0.5, "right_scale": 0.5,
        "left": {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 1024, "keep_first": 64},
                 "rot": {"base": 1e6, "dims": 128, "scaling": {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}}},
        "right": {"heads": 32, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-5 - 7 * i / 31) for i in range(32)]}}}
    return bolisun_config({"vocab": 163840, "width": 2304, "streams": 2, "norm": {"eps": 1e-6}, "embedding": {"scale": 48.0},
                           "layers": [dict(par, mlp=dense), dict(par, mlp=moe), dict(par, mlp=moe), dict(par, mlp=moe, weights_of=2)]},
                          "bolisun-bench")


def tiny_pitudra() -> ModelConfig:
    """One layer of every mixer and one that borrows latents; with and without a feed-forward."""
    moe = {"kind": "moe", "expert": {"ff": 40}, "router": {"experts": 6, "top": 2}}
    lat = {"heads": 4, "dim": 24, "rot_dim": 8, "vdim": 16, "q_rank": 40, "kv_rank": 48, "scale": 0.2, "mask": {"size": 50},
           "rot": {"base": 5000.0, "dims": 8}}
    return pitudra_config({
        "vocab": 320, "width": 120, "norm": {"eps": 1e-5}, "token_side": {"dim": 16},
        "layers": [{"type": "hgrn2", "mixer": {"heads": 3, "dim": 16, "vdim": 24}, "mlp": moe},
                   {"type": "latent_attention", "mixer": lat, "mlp": moe},
                   {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 32, "scale": 0.2, "mask": {"size": 33}},
                    "mlp": None},
                   {"type": "latent_attention", "mixer": dict(lat, heads=2, dim=16, vdim=40, kv_from=1, mask={"size": 20}), "mlp": moe}]},
        "tiny-pitudra")


def pitudra_bench() -> ModelConfig:
    """Layers of a real model's size: two HGRN2 layers, one of windowed attention and one of latent attention, each with 64 experts of
    which 8 run.  An expert's two matrices hold as many weights as the three of a gated one of width 1024."""
    moe = {"kind": "moe", "expert": {"ff": 1536}, "router": {"experts": 64, "top": 8}}
    rec = {"type": "hgrn2", "mlp": moe, "mixer": {"heads": 32, "dim": 128, "vdim": 128}}
    att = {"type": "attention", "mlp": moe, "mixer": {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                                      "mask": {"size": 1024}}}
    lat = {"type": "latent_attention", "mlp": moe, "mixer": {
        "heads": 32, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": 1536, "kv_rank": 512, "scale": 192 ** -0.5,
        "mask": {"size": 4096}, "rot": {"base": 1e6, "dims": 64}}}
    return pitudra_config({"vocab": 163840, "width": 2304, "norm": {"eps": 1e-6}, "token_side": {"dim": 128},
                           "layers": [rec, att, dict(rec), lat]}, "pitudra-bench")


_PRESETS = {
    "tiny-pitudra": tiny_pitudra,
    "pitudra-bench": pitudra_bench,
    "tiny-bolisun": tiny_bolisun,
    "bolisun-bench": bolisun_bench,
    "tiny-pamevik": tiny_pamevik,
    "pamevik-bench": pamevik_bench,
    "tiny-nanurax": tiny_nanurax,
    "nanurax-bench": nanurax_bench,
    "tiny-deepseek-v3": tiny_deepseek_v3,
    "tiny-glm5": tiny_glm5,
    "tiny-kimi-k3": tiny_kimi_k3,
    "tiny-kimi-linear": tiny_kimi_linear,
    "tiny-kimi-k3.1": tiny_kimi_k31,
    "kimi-k3.1": kimi_k31,
    "kimi-k3-kda": kimi_k3_kda,
    "kimi-linear-48b": kimi_linear_48b,
    "tiny-gpt-oss": tiny_gpt_oss,
    "tiny-gpt-oss-64": tiny_gpt_oss_64,
    "tiny-minimax": tiny_minimax,
    "tiny-deepseek-v2": tiny_deepseek_v2,
    "tiny-mixtral": tiny_mixtral,
    "tiny-qwen2-moe": tiny_qwen2_moe,
    "tiny-deepseek-v4": tiny_deepseek_v4,
    "deepseek-v4-flash": deepseek_v4_flash,
    "deepseek-v4-pro": deepseek_v4_pro,
    "deepseek-v2": deepseek_v2_236b,
    "mixtral-8x7b": mixtral_8x7b,
    "mixtral-8x22b": mixtral_8x22b,
    "qwen2-57b-a14b": qwen2_57b_a14b,
    "qwen1.5-moe-a2.7b": qwen15_moe_a27b,
    "deepseek-v3-671b": deepseek_v3_671b,
    "deepseek-r1": deepseek_v3_671b,
    "glm-5.3-fp8": glm5_3,
    "kimi-k3": kimi_k3,
    "kimi-k2.5": kimi_k25,
    "gpt-oss-120b": gpt_oss_120b,
    "minimax-m2.5": minimax_m25,
}

# HF-style identity patterns -> preset (the reference matches on substrings of the model id,
# batchgen/config/model_registry.py:63-117).
_PATTERNS = [
    (r"deepseek[-_/]?(ai/)?.*(v3|r1)", "deepseek-v3-671b"),
    (r"deepseek[-_/]?(ai/)?.*v4[-_]?pro", "deepseek-v4-pro"),
    (r"deepseek[-_/]?(ai/)?.*v4", "deepseek-v4-flash"),
    (r"deepseek[-_/]?(ai/)?.*v2", "deepseek-v2"),
    (r"mixtral.*8x22b", "mixtral-8x22b"),
    (r"mixtral", "mixtral-8x7b"),
    (r"qwen1\.5[-_]?moe", "qwen1.5-moe-a2.7b"),
    (r"qwen2?[-_].*(moe|a14b)", "qwen2-57b-a14b"),
    (r"glm[-_]?5", "glm-5.3-fp8"),
    (r"kimi[-_]?linear", "kimi-linear-48b"),
    (r"kimi[-_]?k3\.1", "kimi-k3.1"),
    (r"kimi[-_]?k3[-_]?kda", "kimi-k3-kda"),
    (r"kimi[-_]?k3", "kimi-k3"),
    (r"kimi[-_]?k2", "kimi-k2.5"),
    (r"gpt[-_]?oss", "gpt-oss-120b"),
    (r"minimax", "minimax-m2.5"),
    (r"nanurax", "nanurax-bench"),
    (r"pamevik", "pamevik-bench"),
    (r"bolisun", "bolisun-bench"),
    (r"pitudra", "pitudra-bench"),
]


def list_models() -> List[str]:
    return sorted(_PRESETS)


def get_model_config(name: str, **overrides) -> ModelConfig:
    """Config of a preset, of a Hugging Face style id, or of a model directory (``load_model_dir``)."""
    key = name.lower()
    if key not in _PRESETS and os.path.isfile(os.path.join(name, "config.json")):
        cfg = load_model_dir(name)
        for k, v in overrides.items():
            if not hasattr(cfg, k):
                raise AttributeError(f"ModelConfig has no field {k!r}")
            setattr(cfg, k, v)
        return cfg
    if key not in _PRESETS:
        for pat, preset in _PATTERNS:
            if re.search(pat, key):
                key = preset
                break
        else:
            raise KeyError(f"unknown model {name!r}; known: {list_models()}")
    cfg = _PRESETS[key]()
    for k, v in overrides.items():
        if not hasattr(cfg, k):
            raise AttributeError(f"ModelConfig has no field {k!r}")
        setattr(cfg, k, v)
    return cfg


# ------------------------------------------------------------------ engine config
@dataclass
class EngineConfig:
    """Runtime knobs.  Names follow the reference's server flags where one exists
    (docs/server-flags.md; batchgen/server/server_args.py:168-285)."""
    page_size: int = 64
    kv_dtype: str = "bf16"                      # bf16 | fp8
    gpu_memory_frac: float = 0.9
    num_gpu_pages: int = 0                      # 0 = size from free memory
    host_kv_cache_size_gb: float = 0.0          # CPU-DRAM KV tier
    host_kv_chunk_size: int = 8192
    host_kv_watermark: int = 70
    initial_gpu_page_buffer: int = 32
    extension_gpu_page_buffer: int = 4
    decision_frequency_pages: int = 2
    max_prefill_tokens: int = 131072            # packed micro-batch token cap
    max_decode_batch: int = 512                 # rows per rank in decode
    max_state_slots: int = 0                    # sequences holding recurrent (KDA) state at once; 0 = max_decode_batch
    max_host_state_items: int = 0               # parked recurrent states in host memory; 0 = 4 x the device slots
    max_model_len: int = -1
    enable_cuda_graph: bool = True
    cuda_graph_max_bucket_size: int = 128
    cuda_graph_num_buckets: int = 16
    enable_prefix_cache: bool = False
    adaptive_chunk: bool = False
    adaptive_chunk_min: int = 1024              # bounds, smoothing and head-room of the adaptive host-KV chunk
    adaptive_chunk_max: int = 65536
    adaptive_chunk_ema_alpha: float = 0.1
    adaptive_chunk_multiplier: float = 1.5
    # parallel layout
    world_size: int = 1
    attn_tp_size: int = 1                       # TP degree of attention (1 = DP attention)
    ep_size: int = 1                            # expert parallel degree
    decode_attn_split: str = "heads"            # heads | requests: how a TP group divides the decode attention core
    moe_comm: str = "fused"                     # fused | nccl  (nccl = all_gather/reduce_scatter baseline)
    tp_comm: str = "fused"                      # fused | nccl
    expert_offload_ratio: float = 0.0           # fraction of local experts kept in host DRAM
    weight_ring_slots: int = 4
    seed: int = 0
    host_kv_backend: str = "native"       # "native": node-shared region + asynchronous movers (GPU); "torch": pinned tensor
    deferred_readback: bool = True      # with captured decode graphs: read a step's tokens while the next one runs
    device: str = "cpu"
    dtype: str = "fp32"                         # fp32 (CPU oracle) | bf16 (GPU)

    def validate(self) -> None:
        if self.page_size <= 0 or self.page_size & (self.page_size - 1):
            raise ValueError("page_size must be a power of two")
        if self.world_size % max(self.attn_tp_size, 1):
            raise ValueError("attn_tp_size must divide world_size")
        if self.ep_size not in (1, self.world_size):
            raise ValueError("ep_size must be 1 or world_size")
        if not 0.0 <= self.expert_offload_ratio <= 1.0:
            raise ValueError("expert_offload_ratio must be in [0, 1]")
        if self.decode_attn_split not in ("heads", "requests"):
            raise ValueError("decode_attn_split must be 'heads' or 'requests'")
        if self.kv_dtype not in ("bf16", "fp8", "fp32"):
            raise ValueError(f"unsupported kv dtype {self.kv_dtype}")

    @classmethod
    def from_json(cls, path: str) -> "EngineConfig":
        with open(path) as f:
            d = json.load(f)
        names = {f.name for f in dataclasses.fields(cls)}
        unknown = set(d) - names
        if unknown:
            raise ValueError(f"unknown engine config keys: {sorted(unknown)}")
        cfg = cls(**d)
        cfg.validate()
        return cfg
