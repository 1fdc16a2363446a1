"""Model hyper-parameters, normalised from a Hugging Face ``config.json``.

Covers the dense Llama/Mistral/Qwen2/Qwen3 families, the Qwen2/Qwen3 MoE families, MLA
(DeepSeek/GLM-lite style latent attention) and sliding-window fields. The reference does the
same normalisation in python/minisgl/models/config.py:144-1273.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field, replace
from typing import Any, Dict, List, Optional, Tuple

from ..quant.config import QuantConfig


@dataclass(frozen=True)
class RotaryConfig:
    head_dim: int
    rotary_dim: int
    max_position: int
    base: float
    scaling: Optional[Dict[str, Any]] = None  # llama3 / yarn / linear / dynamic parameters
    interleaved: bool = False                 # GPT-J pairing (x0,x1) instead of NeoX halves

    def key(self) -> Tuple:
        return (
            self.head_dim,
            self.rotary_dim,
            self.max_position,
            self.base,
            json.dumps(self.scaling, sort_keys=True) if self.scaling else None,
            self.interleaved,
        )


def _round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class LatentLayer:
    """One layer whose attention keeps a shared latent per token: ``heads`` query heads of ``dim`` channels, values of
    ``vdim``, a latent of ``kv_rank``; ``window`` 0 = every earlier position is visible; ``kv_from``: the layer whose
    latent is read instead of an own one; ``ff`` 0 = no feed-forward (of this kind). ``rot_dim`` further query channels
    per head score against one rotary key that all heads share and that is cached behind the latent: its first
    ``rotary.rotary_dim`` channels are rotated. ``sink``: a learned logit per head in the softmax denominator;
    ``gate``: a sigmoid gate per head on the output. The ``*_pad`` widths are what the kernels see: zero channels that
    change no dot product."""

    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int = 0
    kv_from: Optional[int] = None
    ff: int = 0
    rot_dim: int = 0
    rotary: Optional[RotaryConfig] = None
    sink: bool = False
    gate: bool = False

    @property
    def dim_pad(self) -> int:
        return _round_up(self.dim + self.rot_dim, 16)

    @property
    def vdim_pad(self) -> int:
        return _round_up(self.vdim, 16)

    @property
    def rank_pad(self) -> int:
        """Pool row: the latent, the shared rotary key, zeros."""
        r = _round_up(self.kv_rank + self.rot_dim, 64)
        return r if r <= 256 or r == 576 else _round_up(r, 256)


@dataclass(frozen=True)
class LinearAttnLayer:
    """One linear-attention layer without a delta rule: per head a ``[dim, vdim]`` state that decays and takes up
    ``k v^T`` of every token. The decay is one number per head (``decay``) or comes from the input, one per key channel:
    ``sigmoid(z) ** (1 / tau)`` with ``z`` a projection of rank ``gate_rank`` plus a bias (``decay`` None). ``act``: silu on
    the projected q, k and v. ``rotary``: rotary positions on q and k. The output is RMS-normed over all heads together
    (``joint_norm``) or per head with one shared weight (none with ``weighted`` False), and gated by ``gate_act`` of a
    projection."""

    heads: int
    dim: int
    vdim: int
    decay: Optional[Tuple[float, ...]] = None
    gate_rank: int = 0
    tau: float = 1.0
    act: bool = False
    q_scale: float = 1.0
    joint_norm: bool = False
    gate_act: str = "silu"
    rotary: Optional[RotaryConfig] = None
    weighted: bool = True

    @property
    def dim_pad(self) -> int:
        return _round_up(self.dim, 16)

    @property
    def vdim_pad(self) -> int:
        return _round_up(self.vdim, 16)


@dataclass(frozen=True)
class HeadLayer:
    """One layer of grouped-query attention with sizes of its own: ``heads`` query heads over ``kv_heads`` key / value
    heads, keys of ``dim`` and values of ``vdim`` channels. A row sees the last ``window`` positions (its own included)
    or, with ``chunk``, the positions of its own block of ``chunk`` that are not ahead of it; 0 = no such limit.
    ``softcap`` c > 0: scores go through ``c tanh(s / c)``. ``joint_norm``: weighted RMS norms over all query heads and
    over all key heads together, ahead of the rotation. ``unit_norm``: every query and key head divided by its root mean
    square after the rotation. ``gate``: a sigmoid gate per output channel. ``kv_from``: the layer whose keys and
    values are read instead of own ones. ``log_bias``: a score loses ``r1 ln(1 + r2 distance)``, with two numbers per
    head. ``zero_sink``: the softmax denominator counts a score of 0 that belongs to no key. ``talk``: every head applies a
    mixture of all heads' weights to its values."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: Optional[RotaryConfig] = None
    window: int = 0
    chunk: int = 0
    softcap: float = 0.0
    joint_norm: bool = False
    unit_norm: bool = False
    gate: bool = False
    kv_from: Optional[int] = None
    log_bias: bool = False
    zero_sink: bool = False
    talk: bool = False

    @property
    def row_pad(self) -> int:
        """Width of a head in the pool and in the kernels (keys, values and queries alike), zeros past its channels."""
        n = max(self.dim, self.vdim)
        return next((p for p in (64, 128, 256) if n <= p), _round_up(n, 256))


@dataclass(frozen=True)
class ScanLayer:
    """A selective state-space mixer (Mamba): ``inner`` channels behind a causal convolution of ``taps``, each with a
    ``state`` vector; step sizes come from a projection of rank ``dt_rank``."""

    inner: int
    state: int
    dt_rank: int
    taps: int

    @property
    def state_pad(self) -> int:
        return _round_up(self.state, 4)

    @property
    def rank_pad(self) -> int:
        return _round_up(self.dt_rank, 16)

    def inner_pad(self, tp: int = 1) -> int:
        """Channels of a rank, in the kernels."""
        return _round_up(self.inner // tp, 16)


@dataclass(frozen=True)
class PairMixer:
    """Two mixers that read the same rows; half the sum of their outputs, each RMS-normed over the width."""

    left: HeadLayer
    right: ScanLayer


@dataclass(frozen=True)
class ExpertSpec:
    """A mixture of ``experts`` feed-forwards of width ``ff`` of which each token uses ``top``, chosen by ``scoring`` among
    the best ``keep`` of ``groups`` groups; ``shared_ff`` > 0: a further one for every token, behind a sigmoid gate with
    ``shared_gated``. Activation: silu-gated, or with ``act`` "clamped" gate and up halves clamped at ``limit``,
    ``g * sigmoid(alpha g) * (u + 1)``. ``on_input``: a chosen expert's weight multiplies what goes into it.
    ``correction``: a number per expert that counts in the choice and not in the weights. ``renorm``: the chosen experts'
    scores are divided by their sum."""

    experts: int
    top: int
    ff: int
    limit: float = 0.0
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    shared_ff: int = 0
    shared_limit: float = 0.0
    alpha: float = 1.702
    act: str = "clamped"
    scoring: str = "softmax"
    on_input: bool = False
    shared_gated: bool = True
    correction: bool = False
    renorm: bool = False


@dataclass(frozen=True)
class LayerSpec:
    """A sequential layer of a model whose layers are listed one by one: a mixer, and a feed-forward that is dense and
    gated (``ff`` > 0), a mixture of experts (``moe``) or absent."""

    mixer: Any                              # LatentLayer | LinearAttnLayer | HeadLayer | PairMixer
    ff: int = 0
    moe: Optional[ExpertSpec] = None


@dataclass(frozen=True)
class ModelConfig:
    num_layers: int
    num_qo_heads: int
    num_kv_heads: int
    head_dim: int
    hidden_size: int
    vocab_size: int
    intermediate_size: int
    rms_norm_eps: float
    rotary_config: RotaryConfig
    hidden_act: str = "silu"
    tie_word_embeddings: bool = False
    model_type: str = "llama"
    architectures: Tuple[str, ...] = ("LlamaForCausalLM",)
    attention_bias: bool = False
    mlp_bias: bool = False
    qk_norm: bool = False
    # mixture of experts
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True
    shared_expert_intermediate_size: int = 0
    shared_expert_gate: bool = False
    decoder_sparse_step: int = 1
    mlp_only_layers: Tuple[int, ...] = ()
    first_k_dense_replace: int = 0
    n_shared_experts: int = 0
    routed_scaling_factor: float = 1.0
    scoring_func: str = "softmax"
    n_group: int = 1
    topk_group: int = 1
    # latent attention
    kv_lora_rank: Optional[int] = None
    q_lora_rank: Optional[int] = None
    qk_nope_head_dim: Optional[int] = None
    qk_rope_head_dim: Optional[int] = None
    v_head_dim: Optional[int] = None
    # gated delta net (linear-attention layers of the Qwen3.5 / Qwen3-Next hybrid family)
    linear_num_key_heads: int = 0
    linear_num_value_heads: int = 0
    linear_key_head_dim: int = 0
    linear_value_head_dim: int = 0
    linear_conv_kernel_dim: int = 4
    # Mamba-2 mixers (Nemotron-H hybrid family): layer_types entries "mamba" / "attention" / "moe" / "mlp"
    mamba_num_heads: int = 0
    mamba_head_dim: int = 0
    ssm_state_size: int = 0
    mamba_n_groups: int = 1
    mamba_conv_bias: bool = True
    mamba_proj_bias: bool = False
    time_step_min: float = 0.0
    moe_latent_size: Optional[int] = None
    mlp_hidden_act: str = "silu"          # "relu2": non-gated squared-ReLU MLPs and experts
    attn_output_gate: bool = False        # q_proj also emits a per-head sigmoid gate of the attention output
    norm_plus_one: bool = False           # RMSNorm weights are stored as (w - 1)
    # layers that keep an attention latent per token, each with its own sizes; a short causal convolution ahead of
    # every sublayer (taps, 0 = none) whose last inputs are per-request state
    latent_layers: Optional[Tuple[Optional[LatentLayer], ...]] = None    # None at a layer that keeps no latent
    input_conv_taps: int = 0
    # models whose layers are described one by one (mixer and feed-forward of different kinds and sizes)
    layer_specs: Optional[Tuple[LayerSpec, ...]] = None
    embedding_multiplier: float = 1.0
    residual_multiplier: float = 1.0        # of a sublayer's output where it joins the residual stream
    depth_average: bool = False             # a layer's input is a weighted sum of the results of all layers before
    # misc
    sliding_window: Optional[int] = None
    layer_types: Optional[Tuple[str, ...]] = None
    final_logit_softcapping: Optional[float] = None
    # Gemma family
    query_pre_attn_scalar: Optional[float] = None   # attention scale = this ** -0.5 (default head_dim)
    rope_local_base_freq: Optional[float] = None    # RoPE base of the sliding-window layers
    # Gemma-4: global layers with their own head width / K/V head count, keys reused as values, the last
    # layers reading the K/V of an earlier layer of their kind, per-layer input embeddings
    global_head_dim: Optional[int] = None
    num_global_kv_heads: Optional[int] = None
    attention_k_eq_v: bool = False
    num_kv_shared_layers: int = 0
    hidden_size_per_layer_input: int = 0
    vocab_size_per_layer_input: int = 0
    use_double_wide_mlp: bool = False
    enable_moe_block: bool = False
    num_nextn_predict_layers: int = 0
    mtp_num_hidden_layers: int = 0            # Qwen3.5 / Qwen3-Next: decoder layers stored under mtp.*
    canvas_length: int = 0                    # block-diffusion models: tokens written per block
    vision: Any = None                        # models.siglip.VisionConfig of a multimodal checkpoint
    # Muse-Glimmer: the two post-norms of a layer have an epsilon of their own, layers whose rotary base is 0
    # have no positional encoding, logits are multiplied before the soft cap, queries are scaled after their norm
    # Laguna: a query-head count per layer and a rotary table of their own for the sliding layers
    attn_head_counts: Optional[Tuple[int, ...]] = None
    sliding_rotary: Optional[RotaryConfig] = None
    post_norm_eps: Optional[float] = None
    layer_rope_theta: Optional[Tuple[float, ...]] = None
    output_multiplier: Optional[float] = None
    qk_scale_factor: Optional[float] = None
    image_bidirectional: bool = True          # the tokens of one image see each other in both directions in the prefill
    pad_token_id: int = 0
    mask_token_id: Optional[int] = None       # absorbing-state diffusion models
    eos_token_ids: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None
    torch_dtype: str = "bfloat16"
    max_position_embeddings: int = 32768
    quant: Optional[QuantConfig] = None
    # EAGLE3 draft head fields
    draft_vocab_size: Optional[int] = None
    eagle_aux_layers: Optional[Tuple[int, ...]] = None

    # ---- derived ----
    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank is not None

    @property
    def latent_widths(self) -> Tuple[int, ...]:
        """Pool row width of every layer that keeps a latent of its own, in layer order."""
        return tuple(s.rank_pad for s in self.latent_layers or () if s is not None and s.kv_from is None)

    def latent_row(self, layer: int) -> int:
        """Index in the latent pool of the layer whose latent ``layer`` reads."""
        specs = self.latent_layers
        owner = layer if specs[layer].kv_from is None else specs[layer].kv_from
        return sum(1 for s in specs[:owner] if s is not None and s.kv_from is None)

    def head_mixer(self, layer: int) -> Optional[HeadLayer]:
        """The attention of a layer whose mixer is or contains one with keys and values per head."""
        m = self.layer_specs[layer].mixer
        m = m.left if isinstance(m, PairMixer) else m
        return m if isinstance(m, HeadLayer) else None

    @property
    def head_layers(self) -> Tuple[HeadLayer, ...]:
        """The attention layers, in layer order, of a model whose layers each have a geometry of their own."""
        mixers = (self.head_mixer(i) for i in range(len(self.layer_specs or ())))
        return tuple(m for m in mixers if m is not None)

    def head_geometry(self, tp: int = 1) -> Tuple[Tuple[int, int], ...]:
        """``(kv heads of a rank, row width)`` of every layer with keys and values of its own, in layer order. Heads whose
        weights are mixed are on every rank."""
        return tuple((m.kv_heads if m.talk else max(m.kv_heads // tp, 1), m.row_pad)
                     for m in self.head_layers if m.kv_from is None)

    def head_row(self, layer: int) -> int:
        """Index in the pool of the layer whose keys and values ``layer`` reads."""
        donor = self.head_mixer(layer).kv_from
        before = (self.head_mixer(i) for i in range(layer if donor is None else donor))
        return sum(1 for m in before if m is not None and m.kv_from is None)

    @property
    def layered(self) -> bool:
        """Described layer by layer, without attention latents: keys and values per head, a geometry per layer."""
        return bool(self.layer_specs) and not self.latent_layers

    @property
    def has_fp32_kernels(self) -> bool:
        """Every kernel the model runs on a GPU has an fp32 form."""
        return bool(self.latent_layers or self.layered)

    @property
    def is_recurrent(self) -> bool:
        """Some layers keep a recurrent state (or a convolution tail) per request besides or instead of K/V pages."""
        return (self.input_conv_taps > 0 or bool(self.linear_layers)
                or bool(self.layer_types) and any(t in ("linear_attention", "mamba") for t in self.layer_types))

    @property
    def linear_layers(self) -> Tuple[Tuple[int, Any], ...]:
        """``(layer, LinearAttnLayer | ScanLayer)`` of the layers with a recurrent state of a model with ``layer_specs``."""
        mixers = ((i, s.mixer.right if isinstance(s.mixer, PairMixer) else s.mixer)
                  for i, s in enumerate(self.layer_specs or ()))
        return tuple((i, m) for i, m in mixers if isinstance(m, (LinearAttnLayer, ScanLayer)))

    def state_row(self, layer: int) -> int:
        """Index of a layer with a recurrent state in the state cache."""
        return sum(1 for i, _ in self.linear_layers if i < layer)

    def state_geometries(self, tp: int = 1) -> Optional[Tuple[Tuple[int, int, int], ...]]:
        """``(heads, rows, cols)`` of every state layer where layers may differ; ``None``: ``recurrent_geometry``."""
        if not self.linear_layers:
            return None
        return tuple((1, m.inner_pad(tp), m.state_pad) if isinstance(m, ScanLayer)
                     else (m.heads // tp, m.dim_pad, m.vdim_pad) for _, m in self.linear_layers)

    def conv_geometries(self, tp: int = 1) -> Optional[Tuple[Tuple[int, int], ...]]:
        """``(channels, taps - 1)`` of the convolution tail of every state layer where layers may differ."""
        if not any(isinstance(m, ScanLayer) for _, m in self.linear_layers):
            return None
        return tuple((m.inner_pad(tp), m.taps - 1) if isinstance(m, ScanLayer) else (0, 0) for _, m in self.linear_layers)

    @property
    def num_linear_layers(self) -> int:
        """Layers with a recurrent state (gated delta net, Mamba-2, input convolutions)."""
        if self.input_conv_taps:
            return self.num_layers
        if self.layer_specs:
            return len(self.linear_layers)
        return sum(1 for t in (self.layer_types or ()) if t in ("linear_attention", "mamba"))

    @property
    def num_kv_layers(self) -> int:
        """Layers that keep K/V pages."""
        if self.latent_layers:
            return len(self.latent_widths)
        if self.layered:
            return len(self.head_geometry())
        if self.model_type == "nemotron_h":
            return sum(1 for t in (self.layer_types or ()) if t == "attention")
        return self.num_layers - self.num_linear_layers - self.num_kv_shared_layers

    @property
    def swa_layers(self) -> Tuple[int, ...]:
        """Decoder layers whose attention only looks at the last ``sliding_window`` positions (of those
        that keep K/V of their own)."""
        if not self.sliding_window or self.is_recurrent:
            return ()
        if self.layer_types:
            own = self.num_layers - self.num_kv_shared_layers
            return tuple(i for i, t in enumerate(self.layer_types[:own]) if t == "sliding_attention")
        return tuple(range(self.num_layers)) if self.model_type == "mistral" else ()

    def kv_donor(self, layer: int) -> Optional[int]:
        """The earlier layer whose K/V ``layer`` reads instead of keeping its own: the last layer of the
        same kind before the shared range (Gemma-4). ``None`` for a layer with K/V of its own."""
        first = self.num_layers - self.num_kv_shared_layers
        if not self.num_kv_shared_layers or layer < first:
            return None
        kind = self.layer_types[layer]
        return max(i for i in range(first) if self.layer_types[i] == kind)

    def attn_geometry(self, layer: int) -> Tuple[int, int]:
        """``(kv heads, head width)`` of a layer's attention."""
        if self.global_head_dim and self.layer_types and self.layer_types[layer] != "sliding_attention":
            heads = self.num_global_kv_heads if (self.attention_k_eq_v and self.num_global_kv_heads) \
                else self.num_kv_heads
            return int(heads), int(self.global_head_dim)
        return self.num_kv_heads, self.head_dim

    @property
    def mixed_kv_geometry(self) -> bool:
        return len({self.attn_geometry(i) for i in range(self.num_kv_layers)}) > 1 if self.global_head_dim else False

    @property
    def recurrent_geometry(self) -> Tuple[int, int, int, int]:
        """``(conv channels, heads, rows, cols)`` of one recurrent layer's state: a convolution window
        over ``conv channels`` inputs and a ``[heads, rows, cols]`` fp32 state matrix per request (``heads`` 0: the window alone)."""
        if self.input_conv_taps:
            return self.hidden_size, 0, 0, 0
        if self.linear_layers:                 # the convolution tails and state matrices of all layers as one row each
            return (sum(c * k for c, k in self.conv_geometries() or ()), 1, 1,
                    sum(h * r * c for h, r, c in self.state_geometries()))
        if self.mamba_num_heads:
            inter = self.mamba_num_heads * self.mamba_head_dim
            return (inter + 2 * self.mamba_n_groups * self.ssm_state_size, self.mamba_num_heads, self.mamba_head_dim,
                    self.ssm_state_size)
        return (2 * self.linear_num_key_heads * self.linear_key_head_dim
                + self.linear_num_value_heads * self.linear_value_head_dim,
                self.linear_num_value_heads, self.linear_key_head_dim, self.linear_value_head_dim)

    @property
    def q_size(self) -> int:
        return self.num_qo_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    def layer_is_moe(self, layer: int) -> bool:
        if not self.is_moe or layer in self.mlp_only_layers:
            return False
        if layer < self.first_k_dense_replace:
            return False
        return (layer + 1) % max(self.decoder_sparse_step, 1) == 0

    def with_quant(self, quant: Optional[QuantConfig]) -> "ModelConfig":
        return replace(self, quant=quant)

    def param_count(self) -> int:
        """Parameter count of the unquantised model (used for memory planning)."""
        h, v = self.hidden_size, self.vocab_size
        attn = h * (self.q_size + 2 * self.kv_size) + self.q_size * h
        total = v * h * (1 if self.tie_word_embeddings else 2)
        for layer in range(self.num_layers):
            total += attn + 2 * h
            if self.layer_is_moe(layer):
                total += self.num_experts * 3 * h * self.moe_intermediate_size + h * self.num_experts
                total += 3 * h * self.shared_expert_intermediate_size
            else:
                total += 3 * h * self.intermediate_size
        return total

    # ---- construction ----
    @staticmethod
    def from_hf(cfg: Any) -> "ModelConfig":
        """Build from a dict, a ``transformers`` config object or a path to ``config.json``."""
        folder = None
        if isinstance(cfg, (str, os.PathLike)):
            path = os.fspath(cfg)
            if os.path.isdir(path):
                folder, path = path, os.path.join(path, "config.json")
            with open(path) as fh:
                cfg = json.load(fh)
        if not isinstance(cfg, dict):
            cfg = cfg.to_dict()
        if cfg.get("architecture") == "Mitilix":
            return _mitilix_config(cfg)
        if cfg.get("architecture") == "Rafodra":
            return _rafodra_config(cfg, folder)
        if cfg.get("architecture") == "Zobelorn":
            return _zobelorn_config(cfg)
        if cfg.get("architecture") == "Ligipel":
            return _ligipel_config(cfg)
        vision = None
        if "text_config" in cfg and isinstance(cfg["text_config"], dict):
            if str(cfg.get("model_type", "")).startswith("gemma3") and cfg.get("vision_config"):
                from .siglip import VisionConfig

                vision = VisionConfig.from_hf(cfg)
            elif str(cfg.get("model_type", "")) in ("gemma4", "diffusion_gemma") and cfg.get("vision_config"):
                from .gemma4_vision import Gemma4VisionConfig

                vision = Gemma4VisionConfig.from_hf(cfg)
            inner = dict(cfg["text_config"])
            for key in ("quantization_config", "architectures", "torch_dtype", "tie_word_embeddings", "canvas_length",
                        "mask_token_id"):
                if key in cfg and key not in inner:
                    inner[key] = cfg[key]
            cfg = inner
        g = cfg.get
        model_type = g("model_type", "llama")
        archs = tuple(g("architectures") or _default_arch(model_type))
        heads = int(g("num_attention_heads"))
        hidden = int(g("hidden_size"))
        head_dim = int(g("head_dim") or hidden // heads)
        kv_heads = int(g("num_key_value_heads") or heads)
        max_pos = int(g("max_position_embeddings", 32768))
        rope_params = g("rope_parameters") or {}
        scaling = g("rope_scaling") or ({k: v for k, v in rope_params.items() if k != "rope_theta"} or None)
        if scaling and scaling.get("rope_type", scaling.get("type", "default")) in ("default", None):
            scaling = None
        theta = float(g("rope_theta") or rope_params.get("rope_theta") or 10000.0)
        partial = float(g("partial_rotary_factor") or rope_params.get("partial_rotary_factor") or 1.0)
        rope_dim = int(g("qk_rope_head_dim") or 0) or int(head_dim * partial)
        rotary = RotaryConfig(
            head_dim=head_dim, rotary_dim=rope_dim, max_position=max_pos, base=theta, scaling=scaling
        )
        eos = g("eos_token_id")
        eos_ids = tuple(eos) if isinstance(eos, (list, tuple)) else (() if eos is None else (int(eos),))
        num_experts = int(g("num_experts") or g("num_local_experts") or g("n_routed_experts") or 0)
        quant = QuantConfig.from_hf(g("quantization_config")) if g("quantization_config") else None
        layer_types = g("layer_types")
        gdn_family = model_type in ("qwen3_5", "qwen3_5_text", "qwen3_5_moe", "qwen3_5_moe_text", "qwen3_next")
        qk_norm = (model_type in ("qwen3", "qwen3_moe", "gemma3", "gemma3_text") or gdn_family
                   or bool(g("use_qk_norm", False)))
        if gdn_family:
            if layer_types is None:
                every = int(g("full_attention_interval") or 4)
                layer_types = ["linear_attention" if (i + 1) % every else "full_attention"
                               for i in range(int(g("num_hidden_layers")))]
            if partial == 1.0 and "partial_rotary_factor" not in cfg and "partial_rotary_factor" not in rope_params:
                rope_dim = head_dim // 4
                rotary = RotaryConfig(head_dim=head_dim, rotary_dim=rope_dim, max_position=max_pos, base=theta,
                                      scaling=scaling)
            if archs and not any(a.startswith("Qwen3_5") or a.startswith("Qwen3Next") for a in archs):
                archs = ("Qwen3_5ForCausalLM",)
        if layer_types is None and model_type in ("gemma3", "gemma3_text") and g("sliding_window_pattern"):
            pat = int(g("sliding_window_pattern"))
            layer_types = ["full_attention" if (i + 1) % pat == 0 else "sliding_attention"
                           for i in range(int(g("num_hidden_layers")))]
        if layer_types is None and model_type == "gemma2":
            layer_types = ["sliding_attention" if i % 2 == 0 else "full_attention"
                           for i in range(int(g("num_hidden_layers")))]
        sliding_rotary = None
        local_theta = g("rope_local_base_freq")
        if local_theta is None and isinstance(rope_params.get("sliding_attention"), dict):
            local_theta = rope_params["sliding_attention"].get("rope_theta")
        muse = model_type in ("muse_glimmer", "muse_glimmer_text")
        if muse:
            cfg = dict(cfg, hidden_act=g("hidden_act") or g("hidden_activation") or "silu")
            g = cfg.get
        gemma4 = model_type in ("gemma4", "gemma4_text", "diffusion_gemma", "diffusion_gemma_text")
        if model_type.startswith("diffusion_gemma") and "attention_k_eq_v" not in cfg:
            # the block-diffusion variant's config does not carry the field; its global layers have no
            # value projection all the same
            cfg = dict(cfg, attention_k_eq_v=True)
            g = cfg.get
        if isinstance(rope_params.get("full_attention"), dict):  # per-layer-type RoPE tables
            full = rope_params["full_attention"]
            theta = float(full.get("rope_theta", theta))
            scaling = {k: v for k, v in full.items() if k != "rope_theta"} or None
            if scaling and scaling.get("rope_type", "default") in ("default", None):
                scaling = None
            g_dim = int(g("global_head_dim") or head_dim) if gemma4 else head_dim
            if full.get("partial_rotary_factor") and not gemma4:
                rope_dim = int(head_dim * float(full["partial_rotary_factor"]))
            rotary = RotaryConfig(head_dim=g_dim, rotary_dim=g_dim if gemma4 else rope_dim, max_position=max_pos,
                                  base=theta, scaling=scaling)
            sub = rope_params.get("sliding_attention")
            if isinstance(sub, dict) and model_type == "laguna":
                sub_scaling = {k: v for k, v in sub.items() if k != "rope_theta"} or None
                if sub_scaling and sub_scaling.get("rope_type", "default") in ("default", None):
                    sub_scaling = None
                sliding_rotary = RotaryConfig(head_dim=head_dim,
                                              rotary_dim=int(head_dim * float(sub.get("partial_rotary_factor") or 1.0)),
                                              max_position=max_pos, base=float(sub.get("rope_theta", theta)),
                                              scaling=sub_scaling)
        if gemma4:
            if layer_types is None:
                layer_types = ["sliding_attention" if (i + 1) % 6 else "full_attention"
                               for i in range(int(g("num_hidden_layers")))]
            layer_types = list(layer_types)
            layer_types[-1] = "full_attention"
            cfg = dict(cfg, hidden_act=g("hidden_activation", "gelu_pytorch_tanh"),
                       num_experts_per_tok=g("top_k_experts"), tie_word_embeddings=g("tie_word_embeddings", True),
                       num_experts=g("num_experts") if g("enable_moe_block") else 0)
            g = cfg.get
            num_experts = int(g("num_experts") or 0)
        if g("kv_lora_rank"):
            # latent attention: the pool holds materialised per-head keys of qk_nope + qk_rope channels;
            # the rotary part is GPT-J interleaved unless the checkpoint says otherwise
            # (where the value head is narrower than that, or the width is not one the attention kernels
            # are built for, keys, queries and values are zero-padded to a common width: DeepSeek-V2/V3's
            # 128 + 64 key channels and 128 value channels are stored 256 wide)
            head_dim = max(int(g("qk_nope_head_dim")) + int(g("qk_rope_head_dim")), int(g("v_head_dim") or 0))
            if head_dim > 64 and head_dim not in (128, 256):
                head_dim = 128 if head_dim < 128 else 256 if head_dim < 256 else head_dim
            kv_heads = heads
            rotary = RotaryConfig(head_dim=head_dim, rotary_dim=int(g("qk_rope_head_dim")), max_position=max_pos,
                                  base=theta, scaling=scaling, interleaved=bool(g("rope_interleave", True)))
            if g("mlp_layer_types") and not g("first_k_dense_replace"):
                dense = [i for i, t in enumerate(g("mlp_layer_types")) if t != "sparse"]
                cfg = dict(cfg, mlp_only_layers=dense)
                g = cfg.get
        attn_bias = bool(g("attention_bias", model_type in ("qwen2", "qwen2_moe")))
        if model_type == "nemotron_h":
            # one mixer per layer: M = Mamba-2, * = attention, E = mixture of experts, - = MLP; no rotary embedding
            pattern = g("hybrid_override_pattern")
            names = {"M": "mamba", "*": "attention", "E": "moe", "-": "mlp"}
            layer_types = list(g("layers_block_type") or g("layer_types") or [names[ch] for ch in (pattern or "")])
            if not layer_types:
                raise ValueError("nemotron_h config without layers_block_type / hybrid_override_pattern")
            rotary = RotaryConfig(head_dim=head_dim, rotary_dim=0, max_position=max_pos, base=theta)
            cfg = dict(cfg, num_hidden_layers=len(layer_types), rms_norm_eps=g("layer_norm_epsilon", g("rms_norm_eps", 1e-5)),
                       shared_expert_intermediate_size=g("moe_shared_expert_intermediate_size") or 0,
                       scoring_func="sigmoid")
            g = cfg.get
        return ModelConfig(
            num_layers=int(g("num_hidden_layers")),
            num_qo_heads=heads,
            num_kv_heads=kv_heads,
            head_dim=head_dim,
            hidden_size=hidden,
            vocab_size=int(g("vocab_size")),
            intermediate_size=int(g("intermediate_size") or 0),
            rms_norm_eps=float(g("rms_norm_eps", 1e-6)),
            rotary_config=rotary,
            hidden_act=g("hidden_act", "silu"),
            tie_word_embeddings=bool(g("tie_word_embeddings", False)),
            model_type=model_type,
            architectures=archs,
            attention_bias=attn_bias,
            mlp_bias=bool(g("mlp_bias", False)),
            qk_norm=qk_norm,
            num_experts=num_experts,
            num_experts_per_tok=int(g("num_experts_per_tok") or 0),
            # Mixtral's experts have the width its config calls intermediate_size
            moe_intermediate_size=int(g("moe_intermediate_size") or (g("intermediate_size") if model_type == "mixtral" else 0) or 0),
            norm_topk_prob=bool(g("norm_topk_prob", True)),
            shared_expert_intermediate_size=int(g("shared_expert_intermediate_size") or 0),
            # a sigmoid gate on the shared expert's output: Qwen2-MoE and the Qwen3.5 / Qwen3-Next MoE blocks
            shared_expert_gate=model_type in ("qwen2_moe", "qwen3_5_moe", "qwen3_5_moe_text", "qwen3_next"),
            decoder_sparse_step=int(g("decoder_sparse_step") or 1),
            mlp_only_layers=tuple(g("mlp_only_layers") or ()),
            first_k_dense_replace=int(g("first_k_dense_replace") or 0),
            n_shared_experts=int(g("n_shared_experts") or 0),
            routed_scaling_factor=float(g("routed_scaling_factor") or 1.0),
            scoring_func=g("scoring_func", "sigmoid" if model_type in ("glm4_moe_lite", "glm4_moe", "deepseek_v3", "laguna")
                           else "softmax"),
            # DeepSeek-V2's plain "greedy" top-k ignores the routing groups its config still lists
            n_group=1 if g("topk_method") == "greedy" else int(g("n_group") or 1),
            topk_group=int(g("topk_group") or 1),
            kv_lora_rank=g("kv_lora_rank"),
            q_lora_rank=g("q_lora_rank"),
            qk_nope_head_dim=g("qk_nope_head_dim"),
            qk_rope_head_dim=g("qk_rope_head_dim"),
            v_head_dim=g("v_head_dim"),
            linear_num_key_heads=int(g("linear_num_key_heads") or 0),
            linear_num_value_heads=int(g("linear_num_value_heads") or 0),
            linear_key_head_dim=int(g("linear_key_head_dim") or 0),
            linear_value_head_dim=int(g("linear_value_head_dim") or 0),
            linear_conv_kernel_dim=int(g("linear_conv_kernel_dim") or g("conv_kernel") or g("mamba_d_conv") or 4),
            mamba_num_heads=int(g("mamba_num_heads") or 0),
            mamba_head_dim=int(g("mamba_head_dim") or 0),
            ssm_state_size=int(g("ssm_state_size") or 0),
            mamba_n_groups=int(g("n_groups") or g("mamba_n_groups") or 1),
            mamba_conv_bias=bool(g("use_conv_bias", g("mamba_conv_bias", True))),
            mamba_proj_bias=bool(g("mamba_proj_bias", g("use_bias", False))),
            time_step_min=float(g("time_step_min") or g("mamba_dt_min") or 0.0) if model_type == "nemotron_h" else 0.0,
            moe_latent_size=g("moe_latent_size"),
            mlp_hidden_act=g("mlp_hidden_act", "silu"),
            attn_output_gate=gdn_family,
            norm_plus_one=gdn_family,
            sliding_window=g("sliding_window") if g("use_sliding_window", True) else None,
            layer_types=tuple(layer_types) if layer_types else None,
            final_logit_softcapping=g("final_logit_softcapping"),
            query_pre_attn_scalar=g("query_pre_attn_scalar"),
            rope_local_base_freq=float(local_theta) if local_theta else None,
            global_head_dim=int(g("global_head_dim") or 0) or None if gemma4 else None,
            num_global_kv_heads=g("num_global_key_value_heads") if gemma4 else None,
            attention_k_eq_v=bool(g("attention_k_eq_v", False)) if gemma4 else False,
            num_kv_shared_layers=int(g("num_kv_shared_layers") or 0) if gemma4 else 0,
            hidden_size_per_layer_input=int(g("hidden_size_per_layer_input") or 0) if gemma4 else 0,
            vocab_size_per_layer_input=int(g("vocab_size_per_layer_input") or 0) if gemma4 else 0,
            use_double_wide_mlp=bool(g("use_double_wide_mlp", False)) if gemma4 else False,
            enable_moe_block=bool(g("enable_moe_block", False)) if gemma4 else False,
            num_nextn_predict_layers=int(g("num_nextn_predict_layers") or 0),
            mtp_num_hidden_layers=int(g("mtp_num_hidden_layers") or 0),
            canvas_length=int(g("canvas_length") or g("block_length") or 0),
            vision=vision,
            attn_head_counts=tuple(int(h) for h in g("num_attention_heads_per_layer")) if g("num_attention_heads_per_layer") else None,
            sliding_rotary=sliding_rotary,
            post_norm_eps=g("post_norm_eps") if muse else None,
            layer_rope_theta=tuple(float(x) for x in g("layer_rope_theta")) if muse and g("layer_rope_theta") else None,
            output_multiplier=g("output_multiplier") if muse else None,
            qk_scale_factor=float(g("qk_scale_factor") or 3.87) if muse else None,
            image_bidirectional=(g("use_bidirectional_attention") == "vision") if gemma4 else True,
            pad_token_id=int(g("pad_token_id") or 0),
            mask_token_id=g("mask_token_id"),
            eos_token_ids=eos_ids,
            bos_token_id=g("bos_token_id"),
            torch_dtype=str(g("torch_dtype") or g("dtype") or "bfloat16").replace("torch.", ""),
            max_position_embeddings=max_pos,
            quant=quant,
            draft_vocab_size=g("draft_vocab_size"),
            eagle_aux_layers=tuple(g("eagle_aux_hidden_state_layer_ids") or ()) or None,
        )


def _mitilix_config(cfg: Dict[str, Any]) -> ModelConfig:
    """``layers`` lists every layer's mixer and feed-forward with sizes of their own."""
    specs = []
    for i, layer in enumerate(cfg["layers"]):
        kind, mix, mlp = layer["type"], layer["mixer"], layer.get("mlp")
        if kind != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        donor = mix.get("kv_from")
        if donor is not None:
            donor = int(donor)
            if not 0 <= donor < i or specs[donor].kv_from is not None or specs[donor].kv_rank != int(mix["kv_rank"]):
                raise ValueError(f"layer {i}: kv_from {donor} names no earlier layer with a latent of this size")
        window = int((mix.get("mask") or {}).get("size") or 0)
        specs.append(LatentLayer(heads=int(mix["heads"]), dim=int(mix["dim"]), vdim=int(mix["vdim"]),
                                 kv_rank=int(mix["kv_rank"]), scale=float(mix["scale"]), window=window, kv_from=donor,
                                 ff=int(mlp["ff"]) if mlp is not None else 0))
    width, max_pos = int(cfg["width"]), int(cfg["max_positions"])
    first = specs[0]
    eos = cfg.get("eos_token_id")
    eos_ids = tuple(eos) if isinstance(eos, (list, tuple)) else (() if eos is None else (int(eos),))
    return ModelConfig(
        num_layers=len(specs), num_qo_heads=first.heads, num_kv_heads=1, head_dim=first.rank_pad, hidden_size=width,
        vocab_size=int(cfg["vocab"]),
        # the widest activations of a step: queries in the latent space and the feed-forward
        intermediate_size=max(max(s.ff, s.heads * s.rank_pad) for s in specs),
        rms_norm_eps=float(cfg["norm"]["eps"]),
        rotary_config=RotaryConfig(head_dim=first.rank_pad, rotary_dim=0, max_position=max_pos, base=10000.0),
        hidden_act="gelu", model_type="mitilix", architectures=("MitilixForCausalLM",),
        latent_layers=tuple(specs), input_conv_taps=int(cfg["canon"]["taps"]),
        linear_conv_kernel_dim=int(cfg["canon"]["taps"]), max_position_embeddings=max_pos, eos_token_ids=eos_ids,
        bos_token_id=cfg.get("bos_token_id"),
    )


def _tensor_rows(folder: Optional[str]) -> Dict[str, int]:
    """First dimension of every tensor of the checkpoint in ``folder`` (sizes its config.json does not give)."""
    import glob
    import struct

    rows: Dict[str, int] = {}
    for path in sorted(glob.glob(os.path.join(folder, "*.safetensors"))) if folder else ():
        with open(path, "rb") as fh:
            header = json.loads(fh.read(struct.unpack("<Q", fh.read(8))[0]))
        rows.update({k: int(v["shape"][0]) for k, v in header.items() if k != "__metadata__" and v["shape"]})
    return rows


def _latent_mixer(i: int, mix: Dict[str, Any], specs: List[LayerSpec], max_pos: int) -> LatentLayer:
    rot_dim, rot = int(mix.get("rot_dim") or 0), mix.get("rot") or {}
    dims = int(rot.get("dims", rot_dim)) if rot_dim else 0
    if rot_dim and not 0 < dims <= rot_dim or dims % 2:
        raise ValueError(f"layer {i}: {dims} rotated of {rot_dim} rotary channels")
    rotary = RotaryConfig(rot_dim, dims, max_pos, float(rot["base"]), interleaved=True) if dims else None
    spec = LatentLayer(heads=int(mix["heads"]), dim=int(mix["dim"]), vdim=int(mix["vdim"]), kv_rank=int(mix["kv_rank"]),
                       scale=float(mix["scale"]), kv_from=None if mix.get("kv_from") is None else int(mix["kv_from"]),
                       rot_dim=rot_dim, rotary=rotary, sink=True, gate=True)
    if spec.kv_from is not None:
        donor = specs[spec.kv_from].mixer if 0 <= spec.kv_from < i else None
        if not (isinstance(donor, LatentLayer) and donor.kv_from is None
                and (donor.kv_rank, donor.rot_dim, donor.rotary) == (spec.kv_rank, rot_dim, rotary)):
            raise ValueError(f"layer {i}: kv_from {spec.kv_from} names no earlier layer with a latent of this size")
    return spec


def _rafodra_config(cfg: Dict[str, Any], folder: Optional[str]) -> ModelConfig:
    """``layers`` lists every layer's mixer and feed-forward with sizes of their own. The rank of a channel-decay gate is
    only in the checkpoint's tensor shapes (``gate_rank`` of the mixer where there is no checkpoint)."""
    rows = _tensor_rows(folder)
    max_pos = int(cfg.get("max_positions") or 131072)      # the design sets no limit: one for tables and buffers
    specs: List[LayerSpec] = []
    for i, layer in enumerate(cfg["layers"]):
        kind, mix, mlp = layer["type"], layer["mixer"], layer.get("mlp")
        if kind == "latent_attention":
            mixer: Any = _latent_mixer(i, mix, specs, max_pos)
        elif kind in ("lightning", "gla"):
            sizes = dict(heads=int(mix["heads"]), dim=int(mix["dim"]), vdim=int(mix["vdim"]))
            if kind == "lightning":
                decay = tuple(float(d) for d in mix["decay"])
                if len(decay) != sizes["heads"]:
                    raise ValueError(f"layer {i}: {len(decay)} decays for {sizes['heads']} heads")
                mixer = LinearAttnLayer(**sizes, decay=decay, act=True, joint_norm=True, gate_act="sigmoid")
            else:
                rank = int(mix.get("gate_rank") or rows.get(f"l{i}.mix.a1") or 0)
                if rank <= 0:
                    raise ValueError(f"layer {i}: the rank of its decay gate is neither in the checkpoint nor given")
                mixer = LinearAttnLayer(**sizes, gate_rank=rank, tau=float(mix["tau"]), q_scale=sizes["dim"] ** -0.5)
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        ff, moe = 0, None
        if mlp is not None and mlp["kind"] == "dense":
            ff = int(mlp["ff"])
        elif mlp is not None and mlp["kind"] == "moe":
            router, groups, shared = mlp["router"], mlp["router"].get("groups") or {}, mlp.get("shared")
            moe = ExpertSpec(
                experts=int(router["experts"]), top=int(router["top"]), ff=int(mlp["expert"]["ff"]),
                limit=float(mlp["expert"]["limit"]), groups=int(groups.get("count", 1)), keep=int(groups.get("keep", 1)),
                scale=float(router.get("scale", 1.0)), shared_ff=int(shared["ff"]) if shared else 0,
                shared_limit=float(shared["limit"]) if shared else 0.0)
            if moe.experts % moe.groups or not 0 < moe.top <= moe.experts // moe.groups * moe.keep:
                raise ValueError(f"layer {i}: {moe.top} of {moe.experts} experts in {moe.groups} groups, {moe.keep} kept")
        elif mlp is not None:
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        specs.append(LayerSpec(mixer, ff, moe))
    eos = cfg.get("eos_token_id")
    eos_ids = tuple(eos) if isinstance(eos, (list, tuple)) else (() if eos is None else (int(eos),))
    return layered_config(specs, width=int(cfg["width"]), vocab=int(cfg["vocab"]), eps=float(cfg["norm"]["eps"]),
                          embedding_multiplier=float(cfg["embedding"]["scale"]), max_positions=max_pos,
                          eos_token_ids=eos_ids, bos_token_id=cfg.get("bos_token_id"))


def layered_config(specs, width: int, vocab: int, eps: float, embedding_multiplier: float = 1.0,
                   max_positions: int = 131072, eos_token_ids: Tuple[int, ...] = (), bos_token_id=None) -> ModelConfig:
    """A Rafodra configuration from its layers."""
    latent = tuple(s.mixer if isinstance(s.mixer, LatentLayer) else None for s in specs)
    first = next((m for m in latent if m is not None), None)
    row = first.rank_pad if first is not None else 64

    def widest(s: LayerSpec) -> int:        # activations of one token
        m = s.mixer
        mix = m.heads * m.rank_pad if isinstance(m, LatentLayer) else m.heads * (2 * m.dim + 2 * m.vdim)
        return max(mix, s.ff, s.moe.top * s.moe.ff + s.moe.shared_ff if s.moe else 0)

    return ModelConfig(
        num_layers=len(specs), num_qo_heads=first.heads if first is not None else specs[0].mixer.heads, num_kv_heads=1,
        head_dim=row, hidden_size=width, vocab_size=vocab, intermediate_size=max(widest(s) for s in specs),
        rms_norm_eps=eps, rotary_config=RotaryConfig(row, 0, max_positions, base=10000.0), model_type="rafodra",
        architectures=("RafodraForCausalLM",), latent_layers=latent, layer_specs=tuple(specs), linear_conv_kernel_dim=1,
        embedding_multiplier=embedding_multiplier, max_position_embeddings=max_positions, eos_token_ids=eos_token_ids,
        bos_token_id=bos_token_id)


def _head_mixer(i: int, kind: str, mix: Dict[str, Any], specs: List[LayerSpec], max_pos: int) -> HeadLayer:
    rot, size = mix.get("rot") or {}, int((mix.get("mask") or {}).get("size") or 0)
    dim, dims = int(mix["dim"]), int(rot.get("dims", 0))
    if dims % 2 or not 0 <= dims <= dim:
        raise ValueError(f"layer {i}: {dims} rotated of {dim} channels")
    windowed, scaling = kind == "attention", rot.get("scaling")
    if scaling and windowed:
        scaling = {"rope_type": "linear", "factor": float(scaling["factor"])}
    elif scaling:
        scaling = {"rope_type": "llama3", "factor": float(scaling["factor"]), "low_freq_factor": float(scaling["low"]),
                   "high_freq_factor": float(scaling["high"]),
                   "original_max_position_embeddings": float(scaling["original"])}
    rotary = RotaryConfig(dim, dims, max_pos, float(rot["base"]), scaling or None, interleaved=not windowed) if dims else None
    spec = HeadLayer(
        heads=int(mix["heads"]), kv_heads=int(mix["kv_heads"]), dim=dim, vdim=int(mix["vdim"]), scale=float(mix["scale"]),
        rotary=rotary, window=size if windowed else 0, chunk=0 if windowed else size,
        softcap=float(mix.get("softcap") or 0.0) if windowed else 0.0, joint_norm=windowed, unit_norm=not windowed,
        gate=windowed, kv_from=None if mix.get("kv_from") is None else int(mix["kv_from"]))
    if spec.heads % spec.kv_heads:
        raise ValueError(f"layer {i}: {spec.heads} query heads over {spec.kv_heads} key / value heads")
    if spec.kv_from is not None:
        donor = specs[spec.kv_from].mixer if 0 <= spec.kv_from < i else None
        if donor is None or donor.kv_from is not None or any(
                getattr(donor, f) != getattr(spec, f)
                for f in ("kv_heads", "dim", "vdim", "rotary", "joint_norm", "unit_norm")):
            raise ValueError(f"layer {i}: kv_from {spec.kv_from} names no earlier layer with keys and values of this kind")
    return spec


def _zobelorn_config(cfg: Dict[str, Any]) -> ModelConfig:
    """``layers`` lists every layer's mixer ("attention": sliding window; "attention_2": chunks) and feed-forward with
    sizes of their own."""
    max_pos = int(cfg.get("max_positions") or 131072)      # the design sets no limit: one for tables and buffers
    specs: List[LayerSpec] = []
    for i, layer in enumerate(cfg["layers"]):
        kind, mix, mlp = layer["type"], layer["mixer"], layer.get("mlp")
        if kind not in ("attention", "attention_2"):
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        mixer = _head_mixer(i, kind, mix, specs, max_pos)
        ff, moe = 0, None
        if mlp is not None and mlp["kind"] == "dense":
            ff = int(mlp["ff"])
        elif mlp is not None and mlp["kind"] == "moe":
            router, shared = mlp["router"], mlp.get("shared")
            moe = ExpertSpec(experts=int(router["experts"]), top=int(router["top"]), ff=int(mlp["expert"]["ff"]),
                             shared_ff=int(shared["ff"]) if shared else 0, act="silu", scoring="sigmoid", on_input=True,
                             shared_gated=False)
            if not 0 < moe.top <= moe.experts:
                raise ValueError(f"layer {i}: {moe.top} of {moe.experts} experts")
        elif mlp is not None:
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        specs.append(LayerSpec(mixer, ff, moe))
    eos = cfg.get("eos_token_id")
    eos_ids = tuple(eos) if isinstance(eos, (list, tuple)) else (() if eos is None else (int(eos),))
    return heads_config(specs, width=int(cfg["width"]), vocab=int(cfg["vocab"]), eps=float(cfg["norm"]["eps"]),
                        embedding_multiplier=float(cfg["embedding"]["scale"]),
                        residual_multiplier=float(cfg["residual_mult"]), max_positions=max_pos, eos_token_ids=eos_ids,
                        bos_token_id=cfg.get("bos_token_id"))


def heads_config(specs, width: int, vocab: int, eps: float, embedding_multiplier: float = 1.0,
                 residual_multiplier: float = 1.0, max_positions: int = 131072, eos_token_ids: Tuple[int, ...] = (),
                 bos_token_id=None) -> ModelConfig:
    """A Zobelorn configuration from its layers."""
    first: HeadLayer = specs[0].mixer

    def widest(s: LayerSpec) -> int:        # activations of one token
        m: HeadLayer = s.mixer
        mix = (2 * m.heads + 2 * m.kv_heads) * m.row_pad
        return max(mix, s.ff, s.moe.top * s.moe.ff + s.moe.shared_ff if s.moe else 0)

    return ModelConfig(
        num_layers=len(specs), num_qo_heads=first.heads, num_kv_heads=first.kv_heads, head_dim=first.row_pad,
        hidden_size=width, vocab_size=vocab, intermediate_size=max(widest(s) for s in specs), rms_norm_eps=eps,
        rotary_config=RotaryConfig(first.row_pad, 0, max_positions, base=10000.0), model_type="zobelorn",
        architectures=("ZobelornForCausalLM",), layer_specs=tuple(specs), embedding_multiplier=embedding_multiplier,
        residual_multiplier=residual_multiplier, max_position_embeddings=max_positions, eos_token_ids=eos_token_ids,
        bos_token_id=bos_token_id)


def _pair_mixer(i: int, mix: Dict[str, Any]) -> PairMixer:
    left, right = mix["left"], mix["right"]
    attn = HeadLayer(heads=int(left["heads"]), kv_heads=int(left["kv_heads"]), dim=int(left["dim"]), vdim=int(left["vdim"]),
                     scale=float(left["scale"]), window=int((left.get("mask") or {}).get("size") or 0), log_bias=True,
                     zero_sink=True, talk=True)
    if attn.heads % attn.kv_heads:
        raise ValueError(f"layer {i}: {attn.heads} query heads over {attn.kv_heads} key / value heads")
    return PairMixer(attn, ScanLayer(inner=int(right["inner"]), state=int(right["state"]), dt_rank=int(right["dt_rank"]),
                                     taps=int(right["conv"])))


def _retention_mixer(i: int, mix: Dict[str, Any], max_pos: int) -> LinearAttnLayer:
    heads, dim, rot = int(mix["heads"]), int(mix["dim"]), mix.get("rot") or {}
    decay, dims = tuple(float(d) for d in mix["decay"]), int(rot.get("dims", 0))
    if len(decay) != heads:
        raise ValueError(f"layer {i}: {len(decay)} decays for {heads} heads")
    if dims % 2 or not 0 <= dims <= dim:
        raise ValueError(f"layer {i}: {dims} rotated of {dim} channels")
    # the checkpoint's half-split pairs become neighbours when the weights are loaded
    rotary = RotaryConfig(dim, dims, max_pos, float(rot["base"]), interleaved=True) if dims else None
    return LinearAttnLayer(heads=heads, dim=dim, vdim=int(mix["vdim"]), decay=decay, q_scale=dim ** -0.5, rotary=rotary,
                           weighted=False)


def _ligipel_config(cfg: Dict[str, Any]) -> ModelConfig:
    """``layers`` lists every layer's mixer ("parallel": attention beside a selective scan; "retention") and feed-forward
    with sizes of their own."""
    max_pos = int(cfg.get("max_positions") or 131072)      # the design sets no limit: one for tables and buffers
    specs: List[LayerSpec] = []
    for i, layer in enumerate(cfg["layers"]):
        kind, mix, mlp = layer["type"], layer["mixer"], layer.get("mlp")
        if kind not in ("parallel", "retention"):
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        mixer = _pair_mixer(i, mix) if kind == "parallel" else _retention_mixer(i, mix, max_pos)
        moe = None
        if mlp is not None:
            if mlp["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            router, shared = mlp["router"], mlp.get("shared")
            moe = ExpertSpec(experts=int(router["experts"]), top=int(router["top"]), ff=int(mlp["expert"]["ff"]),
                             shared_ff=int(shared["ff"]) if shared else 0, act="silu", shared_gated=False, correction=True,
                             renorm=True)
            if not 0 < moe.top <= moe.experts:
                raise ValueError(f"layer {i}: {moe.top} of {moe.experts} experts")
        specs.append(LayerSpec(mixer, 0, moe))
    eos = cfg.get("eos_token_id")
    eos_ids = tuple(eos) if isinstance(eos, (list, tuple)) else (() if eos is None else (int(eos),))
    return pair_config(specs, width=int(cfg["width"]), vocab=int(cfg["vocab"]), eps=float(cfg["norm"]["eps"]),
                       logit_scale=float(cfg.get("logit_scale") or 1.0), logit_softcap=float(cfg.get("logit_softcap") or 0.0),
                       max_positions=max_pos, eos_token_ids=eos_ids, bos_token_id=cfg.get("bos_token_id"))


def pair_config(specs, width: int, vocab: int, eps: float, logit_scale: float = 1.0, logit_softcap: float = 0.0,
                max_positions: int = 131072, eos_token_ids: Tuple[int, ...] = (), bos_token_id=None) -> ModelConfig:
    """A Ligipel configuration from its layers."""
    attn = next((s.mixer.left for s in specs if isinstance(s.mixer, PairMixer)), None)
    row = attn.row_pad if attn is not None else 64

    def widest(s: LayerSpec) -> int:        # activations of one token
        m = s.mixer
        if isinstance(m, PairMixer):
            left, right = m.left, m.right
            mix = ((left.heads + 2 * left.kv_heads) * left.row_pad + left.heads * left.kv_heads * left.row_pad
                   + 6 * right.inner_pad())
        else:
            mix = m.heads * (2 * m.dim + 3 * m.vdim)
        return max(mix, s.moe.top * s.moe.ff + s.moe.shared_ff if s.moe else 0)

    # the results of all layers are kept through a step, in fp32
    kept = 2 * (len(specs) + 1) * width
    return ModelConfig(
        num_layers=len(specs), num_qo_heads=attn.heads if attn is not None else 1,
        num_kv_heads=attn.kv_heads if attn is not None else 1, head_dim=row, hidden_size=width, vocab_size=vocab,
        intermediate_size=max(widest(s) for s in specs) + kept // 2, rms_norm_eps=eps,
        rotary_config=RotaryConfig(row, 0, max_positions, base=10000.0), model_type="ligipel",
        architectures=("LigipelForCausalLM",), layer_specs=tuple(specs), linear_conv_kernel_dim=2, depth_average=True,
        output_multiplier=logit_scale, final_logit_softcapping=logit_softcap or None, max_position_embeddings=max_positions,
        eos_token_ids=eos_token_ids, bos_token_id=bos_token_id)


def _default_arch(model_type: str) -> List[str]:
    return {
        "llama": ["LlamaForCausalLM"],
        "mistral": ["MistralForCausalLM"],
        "mixtral": ["MixtralForCausalLM"],
        "qwen2": ["Qwen2ForCausalLM"],
        "qwen2_moe": ["Qwen2MoeForCausalLM"],
        "qwen3": ["Qwen3ForCausalLM"],
        "qwen3_moe": ["Qwen3MoeForCausalLM"],
        "gemma2": ["Gemma2ForCausalLM"],
        "gemma3": ["Gemma3ForCausalLM"],
        "gemma3_text": ["Gemma3ForCausalLM"],
        "gemma4": ["Gemma4ForCausalLM"],
        "gemma4_text": ["Gemma4ForCausalLM"],
        "laguna": ["LagunaForCausalLM"],
        "muse_glimmer": ["MuseGlimmerForConditionalGeneration"],
        "muse_glimmer_text": ["MuseGlimmerForConditionalGeneration"],
        "diffusion_gemma": ["DiffusionGemmaForBlockDiffusion"],
        "diffusion_gemma_text": ["DiffusionGemmaForBlockDiffusion"],
        "glm4_moe_lite": ["Glm4MoeLiteForCausalLM"],
        "glm4_moe": ["Glm4MoeForCausalLM"],
        "deepseek_v2": ["DeepseekV2ForCausalLM"],
        "deepseek_v3": ["DeepseekV3ForCausalLM"],
        "qwen3_5": ["Qwen3_5ForCausalLM"],
        "qwen3_5_text": ["Qwen3_5ForCausalLM"],
        "qwen3_5_moe": ["Qwen3_5MoeForCausalLM"],
        "qwen3_5_moe_text": ["Qwen3_5MoeForCausalLM"],
        "qwen3_next": ["Qwen3NextForCausalLM"],
        "nemotron_h": ["NemotronHForCausalLM"],
    }.get(model_type, ["LlamaForCausalLM"])


# --------------------------------------------------------------------------------------------
# Named shapes used by the benchmark configurations (random-init, no checkpoint on disk).
# --------------------------------------------------------------------------------------------
def _rot(head_dim: int, theta: float, max_pos: int = 40960) -> RotaryConfig:
    return RotaryConfig(head_dim=head_dim, rotary_dim=head_dim, max_position=max_pos, base=theta)


def tiny_llama_config() -> ModelConfig:
    """2 layers, hidden 256, 4 q / 2 kv heads of 64, SwiGLU 512, vocab 1024 (CPU oracle run)."""
    return ModelConfig(
        num_layers=2, num_qo_heads=4, num_kv_heads=2, head_dim=64, hidden_size=256,
        vocab_size=1024, intermediate_size=512, rms_norm_eps=1e-6,
        rotary_config=_rot(64, 1e6, 4096), model_type="llama", torch_dtype="float32",
        max_position_embeddings=4096,
    )


def qwen3_4b_config(quant: Optional[QuantConfig] = None) -> ModelConfig:
    return ModelConfig(
        num_layers=36, num_qo_heads=32, num_kv_heads=8, head_dim=128, hidden_size=2560,
        vocab_size=151936, intermediate_size=9728, rms_norm_eps=1e-6,
        rotary_config=_rot(128, 1e6), model_type="qwen3",
        architectures=("Qwen3ForCausalLM",), qk_norm=True, tie_word_embeddings=True,
        max_position_embeddings=40960, quant=quant,
    )


def qwen3_8b_config(quant: Optional[QuantConfig] = None) -> ModelConfig:
    return ModelConfig(
        num_layers=36, num_qo_heads=32, num_kv_heads=8, head_dim=128, hidden_size=4096,
        vocab_size=151936, intermediate_size=12288, rms_norm_eps=1e-6,
        rotary_config=_rot(128, 1e6), model_type="qwen3",
        architectures=("Qwen3ForCausalLM",), qk_norm=True, max_position_embeddings=40960,
        quant=quant,
    )


def qwen3_30b_a3b_config(quant: Optional[QuantConfig] = None) -> ModelConfig:
    return ModelConfig(
        num_layers=48, num_qo_heads=32, num_kv_heads=4, head_dim=128, hidden_size=2048,
        vocab_size=151936, intermediate_size=6144, rms_norm_eps=1e-6,
        rotary_config=_rot(128, 1e6), model_type="qwen3_moe",
        architectures=("Qwen3MoeForCausalLM",), qk_norm=True, num_experts=128,
        num_experts_per_tok=8, moe_intermediate_size=768, norm_topk_prob=True,
        max_position_embeddings=40960, quant=quant,
    )


def llama3_70b_config(quant: Optional[QuantConfig] = None) -> ModelConfig:
    return ModelConfig(
        num_layers=80, num_qo_heads=64, num_kv_heads=8, head_dim=128, hidden_size=8192,
        vocab_size=128256, intermediate_size=28672, rms_norm_eps=1e-5,
        rotary_config=_rot(128, 5e5, 8192), model_type="llama",
        architectures=("LlamaForCausalLM",), max_position_embeddings=8192, quant=quant,
    )


NAMED_CONFIGS = {
    "tiny-llama": tiny_llama_config,
    "qwen3-4b": qwen3_4b_config,
    "qwen3-8b": qwen3_8b_config,
    "qwen3-30b-a3b": qwen3_30b_a3b_config,
    "llama3-70b": llama3_70b_config,
}
