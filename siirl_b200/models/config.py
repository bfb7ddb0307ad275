"""Architecture description of the decoder families this framework trains and serves.

The reference takes architectures from HF ``config.json`` through transformers / Megatron converters
(siirl/models/loader.py, siirl/models/mcore/config_converter.py:26-284: dense Llama/Qwen2, Qwen2-MoE, Mixtral,
Qwen3-MoE, Qwen2.5-VL).  Here one dataclass covers them; ``from_hf_config`` reads the same ``config.json`` and
``PRESETS`` holds the shapes used by the benchmark configurations (random-init, no checkpoint needed).
"""
from __future__ import annotations

import json
import os
from dataclasses import asdict, dataclass, field
from typing import Any, Dict, List, Optional


@dataclass
class VisionConfig:
    depth: int = 32
    hidden_size: int = 1280
    num_heads: int = 16
    intermediate_size: int = 3420
    patch_size: int = 14
    temporal_patch_size: int = 2
    in_channels: int = 3
    spatial_merge_size: int = 2
    window_size: int = 112
    fullatt_block_indexes: List[int] = field(default_factory=lambda: [7, 15, 23, 31])
    out_hidden_size: int = 3584


@dataclass
class ViTConfig:
    image_size: int = 448
    patch_size: int = 14
    hidden_size: int = 1024
    num_heads: int = 16
    intermediate_size: int = 4096
    depth: int = 24
    in_channels: int = 3
    class_token: bool = True
    num_register_tokens: int = 0        # DINOv2 "reg4" models
    layer_scale: bool = True            # learnable per-channel scale on both residual branches
    norm_type: str = "layer_norm"       # or "rms_norm" (InternViT-6B)
    qkv_bias: bool = True
    norm_eps: float = 1e-6
    final_norm: bool = False            # timm ViTs end in a LayerNorm; InternVL reads the raw last layer
    select_layer: int = -1              # hidden state handed on: -1 last layer, -2 the one before (Prismatic)
    class_pos_embed: bool = True        # False: positions for the patches only (timm ``no_embed_class``, DINOv2)
    act: str = "gelu"                   # or "gelu_tanh"

    @property
    def num_patches(self) -> int:
        return (self.image_size // self.patch_size) ** 2

    @property
    def num_prefix_tokens(self) -> int:
        return (1 if self.class_token else 0) + self.num_register_tokens


@dataclass
class MoonViTConfig:
    """Kimi-VL's native-resolution vision tower: learnable 2-D position table interpolated to each image's grid,
    rotary positions over (x, y), LayerNorm / GELU blocks, 2 x 2 patch merge into the projector."""
    patch_size: int = 14
    init_pos_emb_height: int = 64
    init_pos_emb_width: int = 64
    hidden_size: int = 1152
    num_heads: int = 16
    intermediate_size: int = 4304
    depth: int = 27
    merge: int = 2
    in_channels: int = 3


@dataclass
class PrismaticConfig:
    """OpenVLA's vision side: a DINOv2 ViT and (fused backbone) a SigLIP ViT over the same image, patch features
    concatenated along the channel axis, then a GELU MLP into the language model width."""
    featurizer: ViTConfig = field(default_factory=lambda: ViTConfig(
        image_size=224, patch_size=14, hidden_size=1024, num_heads=16, intermediate_size=4096, depth=24,
        class_token=True, num_register_tokens=4, layer_scale=True, final_norm=True, select_layer=-2,
        class_pos_embed=False))
    fused_featurizer: Optional[ViTConfig] = field(default_factory=lambda: ViTConfig(
        image_size=224, patch_size=14, hidden_size=1152, num_heads=16, intermediate_size=4304, depth=27,
        class_token=False, layer_scale=False, final_norm=True, select_layer=-2))
    num_images_in_input: int = 1
    timm_model_ids: List[str] = field(default_factory=lambda: ["vit_large_patch14_reg4_dinov2.lvd142m",
                                                                "vit_so400m_patch14_siglip_224"])

    @property
    def vision_dim(self) -> int:
        return self.featurizer.hidden_size + (self.fused_featurizer.hidden_size if self.fused_featurizer else 0)

    @property
    def tokens_per_image(self) -> int:
        return self.featurizer.num_patches


@dataclass
class MixerBranch:
    """One token mixer of a hybrid layer.  ``kind``: "attention" (paged cache, sliding window with kept first tokens or with
    pooled blocks before it, linear or learned distance bias, rotation, query / key norms, soft-capped scores, a sink
    without value, gated heads), "latent_attention" (paged cache of one compressed row per token, from which every head's
    keys and values are expanded), "gated_linear" (matrix state, decay per key channel), "matrix_memory" (stabilised mLSTM)
    or "general_delta" (matrix state, decay and removal rate per key channel)."""
    kind: str = "attention"
    heads: int = 4
    dim: int = 32                   # query / key width of a head
    vdim: int = 32                  # value width of a head
    out_scale: float = 1.0          # factor of this branch in the layer's sum
    # attention
    kv_heads: int = 0
    scale: float = 0.0
    window: int = 0                 # 0: no limit
    keep_first: int = 0
    pool: int = 0                   # tokens per pooled block: whole blocks before the window are seen as their mean; 0: none
    bias_exp: float = 8.0           # slope of head h: 2^(-bias_exp (h + 1) / heads); 0: no bias
    proj_bias: bool = False         # biases on the projections of queries, keys, values and on the output matrix
    qk_norm: str = ""               # "rows": RMS norm with weights over a whole projection, before the rotation;
                                    # "heads": every head over its root mean square, after the rotation;
                                    # "head_weights": every head, with one weight vector for all, before the rotation
    rot_dims: int = 0               # rotated dimensions of a head (first half against second half); 0: no rotation
    rot_base: float = 1e4
    rot_scaling: Optional[Dict[str, Any]] = None     # factor, low, high, original: three-band scaling of frequencies;
                                                     # factor, original, fast, slow: YaRN
    softcap: float = 0.0            # score -> softcap * tanh(score / softcap); 0: none
    sink: bool = False              # one more key with score 0 and no value
    sink_weight: bool = False       # likewise with a learned score per head
    key_values: bool = False        # the values are the keys as projected
    rel_rows: int = 0               # rows of a learned distance table (the checkpoint's tensor shape); 0: none
    rel_max: int = 0                # distance from which its last row is used
    head_gate: bool = False         # heads times the sigmoid of one number each, projected from the mixer's input
    # latent_attention (with ``scale``)
    kv_rank: int = 0                # width of the cached row
    output_gate: bool = False       # heads times the sigmoid of a projection of the mixer's input
    # gated_linear, general_delta
    tau: float = 16.0               # "gated_linear" only
    rank: int = 0                   # width of the decay's low-rank bottleneck (the checkpoint's tensor shape)
    # matrix_memory
    gate_cap: float = 15.0

    @property
    def recurrent(self) -> bool:
        return self.kind in ("gated_linear", "matrix_memory", "general_delta")

    def paged(self) -> Optional[tuple]:
        """(kv heads, key width, value width) of what the branch keeps in the paged cache, or ``None``."""
        if self.kind == "attention":
            return (self.kv_heads, self.dim, self.vdim)
        return (1, self.kv_rank, 0) if self.kind == "latent_attention" else None


@dataclass
class ExpertSpec:
    """Routed feed-forward: experts, of which every token takes the ``top`` best by soft-max score (plus a learned
    correction) among the ``keep`` best of ``groups`` equal groups of neighbours; weights are the scores (over their sum),
    times ``scale``.  The last ``identity`` router outputs stand for the input itself."""
    experts: int = 8
    ff: int = 64
    top: int = 2
    groups: int = 1
    keep: int = 1
    identity: int = 0
    scale: float = 1.0
    shared_ff: int = 0              # width of an expert that takes every token; 0: none
    act: str = "silu"
    gated: bool = True              # act(gate x) * (up x), or act(up x)
    corrected: bool = True          # the choice adds a learned number per output
    renormalize: bool = True        # weights over their sum

    @property
    def outputs(self) -> int:
        return self.experts + self.identity


@dataclass
class HybridLayer:
    branches: List[MixerBranch] = field(default_factory=list)
    ff: int = 0                     # 0: no dense feed-forward
    moe: Optional[ExpertSpec] = None

    @property
    def has_ff(self) -> bool:
        return self.ff > 0 or self.moe is not None


@dataclass
class LayerLoop:
    """Layers ``start .. stop - 1`` run ``times`` times in a row with the same weights; every pass keeps its own cache."""
    start: int = 0
    stop: int = 0
    times: int = 1


@dataclass
class HybridSpec:
    """Decoders whose layers mix attention and recurrences; the residual stream is kept in 32-bit.

    ``arrangement``: "sequential" (mixer, then feed-forward on the updated stream; vector norms, gated feed-forward),
    "parallel" (both read the same stream, ``x += residual_mult * (mixer(norm1 x) + ff(norm2 x))``; norms of one number
    each, plain feed-forward, optionally a sigmoid gate per element on each of the two results), "hyper" (``streams``
    copies of the stream: a sublayer reads a learned sum of them and every copy becomes a learned sum of all copies and
    the sublayer's result; layer norms with biases, plain or routed feed-forward) or "sandwich" (like "sequential" with a
    second norm on every sublayer's result, plain or routed feed-forward, and ``token_side`` columns of a second embedding
    table per layer that enter the stream through a gate after the feed-forward)."""
    layers: List[HybridLayer] = field(default_factory=list)
    embed_scale: float = 1.0
    logit_softcap: float = 0.0      # 0: none
    norm: str = "layer_norm"        # or "rms_norm"
    act: str = "gelu_tanh"          # or "silu", "gelu" (exact), "relu2" (square of relu), "xielu" (two learned numbers)
    arrangement: str = "sequential"
    streams: int = 1                # "hyper"
    token_side: int = 0             # "sandwich": columns per layer of the second embedding table; 0: none
    ff_bias: bool = False           # "sandwich": biases on both matrices of the dense feed-forward
    residual_mult: float = 1.0
    residual_gate: bool = False
    loop: Optional[LayerLoop] = None
    hf_naming: str = "domavik"

    @property
    def attention(self) -> List[MixerBranch]:
        return [b for layer in self.layers for b in layer.branches if b.paged() is not None]

    def runs(self) -> List[tuple]:
        """``(layer, pass)`` in the order of execution; ``pass`` is the number of the pass that begins right before the
        layer, or ``None``."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, None) for i in range(n)]
        if not (0 <= lp.start < lp.stop <= n and lp.times >= 0):
            raise ValueError(f"loop over layers {lp.start} .. {lp.stop} of {n}, {lp.times} times")
        body = range(lp.start, lp.stop)
        out = [(i, None) for i in range(lp.start)]
        for t in range(lp.times):
            out += [(i, t if i == lp.start else None) for i in body]
        return out + [(i, None) for i in range(lp.stop, n)]

    def visible_span(self):
        """(window, keep_first) outside which no layer looks, or ``None`` when some layer sees everything."""
        att = self.attention
        if any(b.window <= 0 for b in att):
            return None
        # a pooled block is made when its last token arrives: its tokens stay until then
        return (max((max(b.window, b.pool) for b in att), default=1), max((b.keep_first for b in att), default=0))

    def pools(self) -> List[int]:
        """Block sizes of the attention layers that keep pooled blocks."""
        return sorted({b.pool for b in self.attention if b.pool > 0})


@dataclass
class DecoderConfig:
    model_type: str = "qwen2"
    vocab_size: int = 1024
    hidden_size: int = 128
    intermediate_size: int = 352
    num_layers: int = 2
    num_heads: int = 4
    num_kv_heads: int = 2
    head_dim: int = 32
    rope_theta: float = 1e4
    rms_norm_eps: float = 1e-6
    max_position_embeddings: int = 32768
    qkv_bias: bool = True           # Qwen2 family
    qk_norm: bool = False           # Qwen3 family
    tie_word_embeddings: bool = False
    mrope_section: Optional[List[int]] = None   # Qwen2-VL multimodal rope (t, h, w halves)
    # checkpoint's rope_scaling of type linear / llama3 / yarn (None: plain rotary frequencies)
    rope_scaling: Optional[Dict[str, Any]] = None
    # mixture of experts (0 experts = dense)
    num_experts: int = 0
    num_experts_per_tok: int = 0
    # expert parallelism (runtime layout, not part of the HF config): this rank hosts experts
    # [ep_rank * num_experts / ep_size, (ep_rank + 1) * num_experts / ep_size)
    ep_size: int = 1
    ep_rank: int = 0
    # LoRA adapters on the four projections of every layer (0: none); runtime option, not part of the HF config
    lora_rank: int = 0
    lora_alpha: float = 16.0
    # fused projections that carry an adapter: subset of ("qkv_proj", "o_proj", "gate_up_proj", "down_proj")
    lora_targets: Optional[tuple] = None
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True
    # shared expert (Qwen2-MoE, DeepSeek-style): a dense SwiGLU MLP every token passes through, added to the routed
    # experts' output; ``shared_expert_gate`` multiplies it by sigmoid(x . g) (Qwen2-MoE)
    shared_expert_intermediate_size: int = 0
    shared_expert_gate: bool = False
    # multi-head latent attention (DeepSeek-V2/V3, Kimi-VL's language model): keys and values are expanded from a
    # ``kv_lora_rank``-wide latent; each head has ``qk_nope_head_dim`` position-free and ``qk_rope_head_dim`` rotary
    # query/key dimensions (the rotary key is shared by all heads) and ``v_head_dim`` value dimensions
    kv_lora_rank: int = 0
    q_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    rope_interleave: bool = True
    # DeepSeek-V3 routing: sigmoid scores, a per-expert selection bias, group-limited top-k, scaled weights; the first
    # ``first_k_dense_replace`` layers keep a dense MLP
    scoring_func: str = "softmax"
    topk_method: str = "greedy"
    n_group: int = 1
    topk_group: int = 1
    routed_scaling_factor: float = 1.0
    first_k_dense_replace: int = 0
    # value head (critic / reward model): one scalar per token instead of the vocabulary head
    value_head: bool = False
    vision: Optional[VisionConfig] = None
    # InternVL family: a plain ViT tower whose 2x2 pixel-shuffled patches pass an MLP projector; ``hf_naming`` picks
    # the checkpoint's parameter names ("hf": transformers' own classes, "internvl_chat": the upstream remote-code
    # layout with ``vision_model / mlp1 / language_model``, whose language model may be InternLM2 with fused ``wqkv``)
    vit: Optional[ViTConfig] = None
    downsample_ratio: float = 0.5
    hf_naming: str = "hf"
    llm_type: str = ""
    # OpenVLA / OpenVLA-OFT: Prismatic vision backbone; actions are the last ``n_action_bins`` ids below
    # ``action_vocab_size`` (the tokenizer's size: the embedding matrix is padded beyond it)
    prismatic: Optional[PrismaticConfig] = None
    moonvit: Optional[MoonViTConfig] = None
    # per-layer mixers of a hybrid decoder (models/hybrid.py); the uniform attention fields above do not apply then
    hybrid: Optional[HybridSpec] = None
    action_vocab_size: int = 0
    n_action_bins: int = 256
    image_token_id: int = 151655
    eos_token_id: int = 2
    pad_token_id: int = 0
    bos_token_id: Optional[int] = None
    initializer_range: float = 0.02

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0

    @property
    def rope_dim(self) -> int:
        """Width the rotary embedding acts on."""
        return self.qk_rope_head_dim if self.is_mla else self.head_dim

    def layer_is_moe(self, layer_idx: int) -> bool:
        return self.is_moe and layer_idx >= self.first_k_dense_replace

    @property
    def q_width(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_width(self) -> int:
        return self.num_kv_heads * self.head_dim

    @property
    def qkv_width(self) -> int:
        return self.q_width + 2 * self.kv_width

    @property
    def logit_softcap(self) -> float:
        return self.hybrid.logit_softcap if self.hybrid is not None else 0.0

    def paged_layers(self) -> List[tuple]:
        """(kv heads, key width, value width) of every layer run that keeps something in the paged cache."""
        if self.hybrid is not None:
            return [b.paged() for i, _ in self.hybrid.runs() for b in self.hybrid.layers[i].branches
                    if b.paged() is not None]
        return [(self.num_kv_heads, self.head_dim, self.head_dim)] * self.num_layers

    def num_parameters(self) -> int:
        if self.hybrid is not None:
            return self._hybrid_parameters()
        H, I, V = self.hidden_size, self.intermediate_size, self.vocab_size
        attn = H * self.qkv_width + (self.qkv_width if self.qkv_bias else 0) + self.q_width * H
        if self.qk_norm:
            attn += 2 * self.head_dim
        if self.is_moe:
            mlp = self.num_experts * 3 * H * self.moe_intermediate_size + self.num_experts * H
            mlp += 3 * H * self.shared_expert_intermediate_size + (H if self.shared_expert_gate else 0)
        else:
            mlp = 3 * H * I
        per_layer = attn + mlp + 2 * H
        head = 0 if self.tie_word_embeddings else (H if self.value_head else V * H)
        return V * H + self.num_layers * per_layer + H + head

    def _hybrid_parameters(self) -> int:
        hy, W = self.hybrid, self.hidden_size
        if hy.arrangement == "hyper":
            return self._hyper_parameters()
        if hy.arrangement == "sandwich":
            return self._sandwich_parameters()
        parallel = hy.arrangement == "parallel"
        norm, ffs = (1, 2) if parallel else (W, 3)
        gate = W * (W + 1) if hy.residual_gate else 0
        n = 2 * self.vocab_size * W + norm
        if hy.loop is not None:
            n += 2 * W * W + hy.loop.times * W
        for layer in hy.layers:
            n += norm + gate + (norm + ffs * W * layer.ff + gate if layer.ff else 0)
            for b in layer.branches:
                hk, hv = b.heads * b.dim, b.heads * b.vdim
                if b.kind == "latent_attention":
                    n += W * (hk + b.kv_rank + hv * (1 + int(b.output_gate))) + b.kv_rank * (1 + hk + hv)
                    continue
                if b.kind == "attention":
                    n += W * (hk + b.kv_heads * (b.dim + b.vdim) + hv)
                    continue
                n += W * (2 * hk + 3 * hv)
                n += (b.rank * (W + hk) + hk + b.vdim) if b.kind == "gated_linear" else 2 * b.heads * (W + 1) + hv
        return n

    def _hyper_parameters(self) -> int:
        hy, W = self.hybrid, self.hidden_size
        conn = 2 * W + hy.streams * (hy.streams + 2)
        n = 2 * self.vocab_size * W + 2 * W
        for layer in hy.layers:
            n += conn * (1 + int(layer.has_ff)) + 2 * W * layer.ff
            for b in layer.branches:
                hk, gk, gv, hv = b.heads * b.dim, b.kv_heads * b.dim, b.kv_heads * b.vdim, b.heads * b.vdim
                n += W * (hk + gk + gv + hv) + (hk + gk + gv + W) * int(b.proj_bias) + (hk + gk) * int(b.qk_norm == "rows")
                n += b.rel_rows * b.heads + W * b.heads * int(b.head_gate)
            if layer.moe is not None:
                e = layer.moe
                n += 3 * W * (e.experts * e.ff + e.shared_ff) + e.outputs * (W + 1)
        return n

    def _sandwich_parameters(self) -> int:
        hy, W, V = self.hybrid, self.hidden_size, self.vocab_size
        side = hy.token_side
        n = V * W * (1 if self.tie_word_embeddings else 2) + W + V * side * len(hy.layers)
        for layer in hy.layers:
            n += 2 * W * (1 + int(layer.has_ff)) + (2 * W * side + W if side else 0)
            n += 2 * W * layer.ff + (layer.ff * int(hy.ff_bias) + W * int(hy.ff_bias) + 2 * int(hy.act == "xielu")
                                     if layer.ff else 0)
            for b in layer.branches:
                hk, gk, hv = b.heads * b.dim, b.kv_heads * b.dim, b.heads * b.vdim
                if b.kind == "attention":
                    n += W * (hk + gk + hv) + (0 if b.key_values else W * b.kv_heads * b.vdim)
                    n += 2 * b.dim * int(b.qk_norm == "head_weights") + b.heads * int(b.sink_weight)
                else:
                    n += 6 * W * hk + b.rank * (W + hk) + 3 * hk
            if layer.moe is not None:
                e = layer.moe
                n += (2 + int(e.gated)) * W * e.experts * e.ff + e.outputs * (W + int(e.corrected))
        return n

    def to_dict(self) -> Dict[str, Any]:
        return asdict(self)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "DecoderConfig":
        """Inverse of ``to_dict`` (checkpoint manifests keep the model configuration in that form); unknown keys of
        a newer version are dropped."""
        import dataclasses

        def build(kind, val):
            if val is None or not isinstance(val, dict):
                return val
            names = {f.name for f in dataclasses.fields(kind)}
            return kind(**{k: v for k, v in val.items() if k in names})
        d = dict(d)
        for key, kind in (("vision", VisionConfig), ("vit", ViTConfig), ("moonvit", MoonViTConfig)):
            d[key] = build(kind, d.get(key))
        pr = d.get("prismatic")
        if isinstance(pr, dict):
            pr = dict(pr)
            pr["featurizer"] = build(ViTConfig, pr.get("featurizer"))
            pr["fused_featurizer"] = build(ViTConfig, pr.get("fused_featurizer"))
            d["prismatic"] = build(PrismaticConfig, pr)
        if isinstance(d.get("hybrid"), dict):
            hy = dict(d["hybrid"])
            hy["layers"] = [build(HybridLayer, dict(x, branches=[build(MixerBranch, b) for b in x["branches"]],
                                                    moe=build(ExpertSpec, x.get("moe")))) for x in hy.get("layers", [])]
            hy["loop"] = build(LayerLoop, hy.get("loop"))
            d["hybrid"] = build(HybridSpec, hy)
        for key in ("lora_targets", "mrope_section"):
            if isinstance(d.get(key), list) and key == "lora_targets":
                d[key] = tuple(d[key])
        names = {f.name for f in dataclasses.fields(cls)}
        return cls(**{k: v for k, v in d.items() if k in names})

    # ---- HF interchange -----------------------------------------------------------------------
    @classmethod
    def from_hf_config(cls, cfg: Dict[str, Any]) -> "DecoderConfig":
        own = {"Domavik": cls._from_domavik_config, "Poralorn": cls._from_poralorn_config,
               "Gumazen": cls._from_gumazen_config, "Rizitar": cls._from_rizitar_config}
        if cfg.get("architecture") in own:
            return own[cfg["architecture"]](cfg)
        text = cfg.get("text_config") or cfg.get("llm_config") or cfg
        mt = cfg.get("model_type", "qwen2")
        if mt in ("llama4", "llama4_text"):
            # same answer as the reference's converter, which lists Llama4ForConditionalGeneration and raises
            # (siirl/models/mcore/config_converter.py:282-284): chunked attention, rope-free layers and the
            # interleaved dense / MoE stack of that family are not built
            raise NotImplementedError("Llama4ForConditionalGeneration is not supported")
        if mt in ("internvl", "internvl_chat"):
            return cls._from_internvl_config(cfg)
        if mt in ("openvla", "prismatic"):
            return cls._from_openvla_config(cfg)
        if mt == "kimi_vl":
            out = cls.from_hf_config(dict(cfg["text_config"], model_type="deepseek_v3"))
            out.model_type = "kimi_vl"
            out.image_token_id = int(cfg.get("media_placeholder_token_id", 163605))
            vc = cfg.get("vision_config", {})
            mk = vc.get("merge_kernel_size", [2, 2])
            out.moonvit = MoonViTConfig(
                patch_size=vc.get("patch_size", 14), init_pos_emb_height=vc.get("init_pos_emb_height", 64),
                init_pos_emb_width=vc.get("init_pos_emb_width", 64), hidden_size=vc.get("hidden_size", 1152),
                num_heads=vc.get("num_attention_heads", 16), intermediate_size=vc.get("intermediate_size", 4304),
                depth=vc.get("num_hidden_layers", 27), merge=int(mk[0] if isinstance(mk, (list, tuple)) else mk))
            return out
        nh = text["num_attention_heads"]
        hd = text.get("head_dim") or text["hidden_size"] // nh
        rope_scaling = text.get("rope_scaling") or cfg.get("rope_scaling") or {}
        out = cls(
            model_type=mt,
            vocab_size=text["vocab_size"],
            hidden_size=text["hidden_size"],
            intermediate_size=text.get("intermediate_size", 0),
            num_layers=text["num_hidden_layers"],
            num_heads=nh,
            num_kv_heads=text.get("num_key_value_heads", nh),
            head_dim=hd,
            rope_theta=float(text.get("rope_theta", 1e4)),
            rms_norm_eps=float(text.get("rms_norm_eps", 1e-6)),
            max_position_embeddings=text.get("max_position_embeddings", 32768),
            qkv_bias=mt.startswith("qwen2") or bool(text.get("attention_bias", False)),
            qk_norm=mt.startswith("qwen3"),
            tie_word_embeddings=bool(cfg.get("tie_word_embeddings", False)),
            mrope_section=rope_scaling.get("mrope_section"),
            rope_scaling=(dict(rope_scaling) if rope_scaling.get("rope_type", rope_scaling.get("type")) in
                          ("linear", "llama3", "yarn") else None),
            num_experts=text.get("num_experts", text.get("num_local_experts", 0)) or 0,
            num_experts_per_tok=text.get("num_experts_per_tok", 0) or 0,
            moe_intermediate_size=text.get("moe_intermediate_size", 0) or 0,
            norm_topk_prob=bool(text.get("norm_topk_prob", True)),
            shared_expert_intermediate_size=text.get("shared_expert_intermediate_size", 0) or 0,
            shared_expert_gate=mt == "qwen2_moe" and bool(text.get("shared_expert_intermediate_size", 0)),
            eos_token_id=(cfg.get("eos_token_id") if isinstance(cfg.get("eos_token_id"), int) else 2) or 2,
            pad_token_id=cfg.get("pad_token_id") or 0,
        )
        if mt in ("deepseek_v3", "deepseek_v2"):
            out.qkv_bias = bool(text.get("attention_bias", False))
            out.kv_lora_rank = int(text.get("kv_lora_rank") or 0)
            out.q_lora_rank = int(text.get("q_lora_rank") or 0)
            out.qk_nope_head_dim = int(text.get("qk_nope_head_dim", 128))
            out.qk_rope_head_dim = int(text.get("qk_rope_head_dim", 64))
            out.v_head_dim = int(text.get("v_head_dim", 128))
            out.rope_interleave = bool(text.get("rope_interleave", True))
            out.head_dim = out.qk_nope_head_dim + out.qk_rope_head_dim
            out.num_experts = int(text.get("n_routed_experts") or 0)
            out.scoring_func = text.get("scoring_func", "sigmoid" if mt == "deepseek_v3" else "softmax")
            out.topk_method = text.get("topk_method", "noaux_tc" if mt == "deepseek_v3" else "greedy")
            out.n_group = int(text.get("n_group") or 1)
            out.topk_group = int(text.get("topk_group") or 1)
            out.routed_scaling_factor = float(text.get("routed_scaling_factor", 1.0))
            out.first_k_dense_replace = int(text.get("first_k_dense_replace", 0))
            out.norm_topk_prob = bool(text.get("norm_topk_prob", True))
            out.shared_expert_intermediate_size = int(text.get("n_shared_experts") or 0) * out.moe_intermediate_size
            out.shared_expert_gate = False
        if mt == "mixtral":
            # Mixtral's experts use the dense intermediate size; its router renormalises the top-k weights
            out.moe_intermediate_size = text.get("intermediate_size", 0)
            out.norm_topk_prob = True
            out.qkv_bias = False
        if mt == "qwen2_moe":
            out.norm_topk_prob = bool(text.get("norm_topk_prob", False))
        if "vision_config" in cfg:
            vc = cfg["vision_config"]
            out.vision = VisionConfig(
                depth=vc.get("depth", 32), hidden_size=vc.get("hidden_size", 1280), num_heads=vc.get("num_heads", 16),
                intermediate_size=vc.get("intermediate_size", 3420), patch_size=vc.get("patch_size", 14),
                temporal_patch_size=vc.get("temporal_patch_size", 2), in_channels=vc.get("in_chans", 3),
                spatial_merge_size=vc.get("spatial_merge_size", 2), window_size=vc.get("window_size", 112),
                fullatt_block_indexes=vc.get("fullatt_block_indexes", [7, 15, 23, 31]),
                out_hidden_size=vc.get("out_hidden_size", text["hidden_size"]))
            out.image_token_id = cfg.get("image_token_id", 151655)
        return out

    @classmethod
    def _from_internvl_config(cls, cfg: Dict[str, Any]) -> "DecoderConfig":
        """``internvl`` (transformers' classes: ``text_config`` + ``vision_config`` with list-valued sizes) and
        ``internvl_chat`` (upstream remote code: ``llm_config`` + ``vision_config``; the language model is InternLM2,
        Qwen2 or Llama)."""
        native = cfg.get("model_type") == "internvl"
        text = dict(cfg.get("text_config") or cfg.get("llm_config") or {})
        llm_type = text.get("model_type", "qwen2")
        base = dict(text)
        base["model_type"] = "qwen2" if llm_type == "qwen2" else "llama"
        if llm_type == "internlm2":
            base["attention_bias"] = bool(text.get("bias", False))
        out = cls.from_hf_config(base)
        out.model_type = "internvl" if native else "internvl_chat"
        out.llm_type = llm_type
        out.hf_naming = "hf" if native else "internvl_chat"
        out.tie_word_embeddings = bool(text.get("tie_word_embeddings", False))
        vc = cfg.get("vision_config", {})

        def one(v, default):
            v = vc.get(v, default)
            return int(v[0]) if isinstance(v, (list, tuple)) else int(v)
        out.vit = ViTConfig(
            image_size=one("image_size", 448), patch_size=one("patch_size", 14), hidden_size=vc.get("hidden_size", 1024),
            num_heads=vc.get("num_attention_heads", 16), intermediate_size=vc.get("intermediate_size", 4096),
            depth=vc.get("num_hidden_layers", 24), class_token=True, layer_scale=True,
            norm_type=vc.get("norm_type", "layer_norm"),
            qkv_bias=bool(vc.get("attention_bias", False) if native else vc.get("qkv_bias", True)),
            norm_eps=float(vc.get("layer_norm_eps", 1e-6)), final_norm=False,
            select_layer=int(cfg.get("vision_feature_layer", cfg.get("select_layer", -1))))
        out.downsample_ratio = float(cfg.get("downsample_ratio", 0.5))
        out.image_token_id = int(cfg.get("image_token_id", cfg.get("img_context_token_id", 151667)))
        return out

    @classmethod
    def _from_openvla_config(cls, cfg: Dict[str, Any]) -> "DecoderConfig":
        """``openvla`` / ``prismatic`` configs (siirl/models/embodied/openvla_oft/configuration_prismatic.py): the
        vision towers are named by their timm ids, the language model is a Llama-2 ``text_config`` whose embedding
        matrix is padded to ``pad_to_multiple_of`` rows."""
        text = dict(cfg.get("text_config") or {})
        text.setdefault("model_type", "llama")
        text.setdefault("vocab_size", 32000)
        for k, v in (("hidden_size", 4096), ("intermediate_size", 11008), ("num_hidden_layers", 32),
                     ("num_attention_heads", 32), ("rms_norm_eps", 1e-6)):
            text.setdefault(k, v)
        mult = int(cfg.get("pad_to_multiple_of", 64))
        tok_vocab = int(text["vocab_size"])
        # a new pad token follows the tokenizer's entries; the matrix is then padded to a multiple of ``mult``
        text["vocab_size"] = (tok_vocab + 1 + mult - 1) // mult * mult if tok_vocab % mult == 0 else tok_vocab
        out = cls.from_hf_config(text)
        out.model_type = "openvla"
        out.llm_type = "llama"
        out.action_vocab_size = tok_vocab if tok_vocab % mult == 0 else int(cfg.get("action_vocab_size", tok_vocab))
        out.n_action_bins = int(cfg.get("n_action_bins", 256))
        out.pad_token_id = int(cfg.get("pad_token_id", 32000))
        out.image_token_id = out.pad_token_id
        out.bos_token_id = int(text.get("bos_token_id", 1))
        ids = list(cfg.get("timm_model_ids") or PrismaticConfig().timm_model_ids)
        sizes = list(cfg.get("image_sizes") or [224, 224])
        towers = [vit_from_timm_id(i, int(s)) for i, s in zip(ids, sizes)]
        if "vit_overrides" in cfg:                   # reduced towers of test checkpoints
            towers = [ViTConfig(**o) for o in cfg["vit_overrides"]]
        fused = bool(cfg.get("use_fused_vision_backbone", len(towers) > 1))
        out.prismatic = PrismaticConfig(featurizer=towers[0], fused_featurizer=towers[1] if fused else None,
                                        num_images_in_input=int(cfg.get("num_images_in_input", 1)), timm_model_ids=ids)
        return out

    @classmethod
    def _from_domavik_config(cls, cfg: Dict[str, Any]) -> "DecoderConfig":
        """Domavik: every layer is either one matrix memory ("mlstm") or window attention beside gated linear attention
        ("parallel"), with an optional gated feed-forward.  The decay's low-rank width is not in the file: it is the
        shape of a tensor, filled in by ``from_pretrained``."""
        def attention(m, scale):
            mask = m["mask"]
            return MixerBranch(kind="attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                               vdim=int(m["vdim"]), scale=float(m["scale"]), window=int(mask["size"]),
                               keep_first=int(mask["keep_first"]), bias_exp=8.0, out_scale=float(scale))

        def gated(m, scale):
            return MixerBranch(kind="gated_linear", heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                               tau=float(m["tau"]), out_scale=float(scale))
        layers = []
        for x in cfg["layers"]:
            m, mlp = x["mixer"], x.get("mlp")
            if x["type"] == "mlstm":
                branches = [MixerBranch(kind="matrix_memory", heads=int(m["heads"]), dim=int(m["dim"]),
                                        vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))]
            elif x["type"] == "parallel":
                branches = [attention(m["left"], m["left_scale"]), gated(m["right"], m["right_scale"])]
            else:
                raise ValueError(f"unknown layer type {x['type']!r}")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            layers.append(HybridLayer(branches=branches, ff=int(mlp["ff"]) if mlp is not None else 0))
        spec = HybridSpec(layers=layers, embed_scale=float(cfg["embedding"]["scale"]),
                          logit_softcap=float(cfg.get("logit_softcap") or 0.0))
        return cls.for_hybrid(spec, vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]),
                              rms_norm_eps=float(cfg["norm"]["eps"]), model_type="domavik",
                              eos_token_id=int(cfg.get("eos_token_id", -1)), pad_token_id=int(cfg.get("pad_token_id", 0)))

    @classmethod
    def for_hybrid(cls, spec: HybridSpec, **kw) -> "DecoderConfig":
        """Configuration around a hybrid spec: the uniform fields that metrics and launchers read are filled from it."""
        att = spec.attention
        b = att[0] if att else (spec.layers[0].branches[0] if spec.layers else MixerBranch())
        return cls(hybrid=spec, num_layers=len(spec.layers), num_heads=b.heads, num_kv_heads=b.kv_heads or b.heads,
                   head_dim=b.dim, intermediate_size=max((x.ff for x in spec.layers), default=0), qkv_bias=False, **kw)

    def _to_domavik_config(self) -> Dict[str, Any]:
        hy = self.hybrid

        def sizes(b, *names):
            return {n: getattr(b, n) for n in ("heads", "dim", "vdim") + names}
        layers = []
        for x in hy.layers:
            b = x.branches[0]
            if b.kind == "matrix_memory":
                t, m = "mlstm", sizes(b, "gate_cap")
            else:
                r = x.branches[1]
                t, m = "parallel", {"left": dict(sizes(b, "kv_heads", "scale"), mask={"size": b.window,
                                                                                      "keep_first": b.keep_first}),
                                    "right": sizes(r, "tau"), "left_scale": b.out_scale, "right_scale": r.out_scale}
            layers.append({"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": x.ff} if x.ff else None})
        d = {"architecture": "Domavik", "vocab": self.vocab_size, "width": self.hidden_size,
             "embedding": {"scale": hy.embed_scale}, "norm": {"eps": self.rms_norm_eps},
             "logit_softcap": hy.logit_softcap, "layers": layers}
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d

    @classmethod
    def _from_poralorn_config(cls, cfg: Dict[str, Any]) -> "DecoderConfig":
        """Poralorn: latent attention without positions beside a plain GELU feed-forward, both gated, and a run of layers
        that is repeated."""
        layers = []
        for x in cfg["layers"]:
            m, mlp = x["mixer"], x.get("mlp")
            if x["type"] != "latent_attention":
                raise ValueError(f"unknown layer type {x['type']!r}")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            layers.append(HybridLayer([MixerBranch(
                kind="latent_attention", heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), output_gate=True)],
                ff=int(mlp["ff"]) if mlp is not None else 0))
        lp = cfg.get("loop")
        spec = HybridSpec(layers=layers, logit_softcap=float(cfg.get("logit_softcap") or 0.0), norm="rms_norm", act="gelu",
                          arrangement="parallel", residual_mult=float(cfg["residual_mult"]), residual_gate=True,
                          loop=LayerLoop(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None,
                          hf_naming="poralorn")
        spec.runs()
        return cls.for_hybrid(spec, vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]),
                              rms_norm_eps=float(cfg["norm"]["eps"]), model_type="poralorn",
                              eos_token_id=int(cfg.get("eos_token_id", -1)), pad_token_id=int(cfg.get("pad_token_id", 0)))

    def _to_poralorn_config(self) -> Dict[str, Any]:
        hy = self.hybrid
        layers = [{"type": "latent_attention",
                   "mixer": {n: getattr(x.branches[0], n) for n in ("heads", "dim", "vdim", "kv_rank", "scale")},
                   "mlp": {"kind": "dense", "ff": x.ff} if x.ff else None} for x in hy.layers]
        d = {"architecture": "Poralorn", "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.rms_norm_eps}, "residual_mult": hy.residual_mult, "logit_softcap": hy.logit_softcap,
             "layers": layers}
        if hy.loop is not None:
            d["loop"] = {"start": hy.loop.start, "stop": hy.loop.stop, "times": hy.loop.times}
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d

    @classmethod
    def _from_gumazen_config(cls, cfg: Dict[str, Any]) -> "DecoderConfig":
        """Gumazen: three kinds of attention in any order, dense or routed feed-forwards, hyper-connections, a run of layers
        that is repeated.  The rows of a distance table are not in the file: they are the shape of a tensor, filled in by
        ``from_pretrained``."""
        kinds = {"attention": dict(qk_norm="heads", sink=True), "attention_3": dict(qk_norm="rows", proj_bias=True),
                 "attention_2": dict(qk_norm="rows", head_gate=True)}
        layers = []
        for x in cfg["layers"]:
            m, mlp = x["mixer"], x.get("mlp")
            if x["type"] not in kinds:
                raise ValueError(f"unknown layer type {x['type']!r}")
            b = MixerBranch(kind="attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                            vdim=int(m["vdim"]), scale=float(m["scale"]), bias_exp=0.0, **kinds[x["type"]])
            if x["type"] == "attention_2":
                b.softcap, b.rel_max = float(m.get("softcap") or 0.0), int(m["bias_max"])
                b.window = int((m.get("mask") or {}).get("size") or 0)
            else:
                rot = m["rot"]
                b.rot_dims, b.rot_base = int(rot["dims"]), float(rot["base"])
                if x["type"] == "attention_3":
                    b.rot_scaling = dict(rot["scaling"]) if rot.get("scaling") else None
            layer = HybridLayer(branches=[b])
            if mlp is not None and mlp["kind"] == "dense":
                layer.ff = int(mlp["ff"])
            elif mlp is not None and mlp["kind"] == "moe":
                r, g = mlp["router"], mlp["router"].get("groups") or {"count": 1, "keep": 1}
                layer.moe = ExpertSpec(experts=int(r["experts"]), ff=int(mlp["expert"]["ff"]), top=int(r["top"]),
                                       groups=int(g["count"]), keep=int(g["keep"]), identity=int(r.get("identity") or 0),
                                       scale=float(r.get("scale", 1.0)),
                                       shared_ff=int(mlp["shared"]["ff"]) if mlp.get("shared") else 0)
            elif mlp is not None:
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            layers.append(layer)
        lp = cfg.get("loop")
        spec = HybridSpec(layers=layers, norm="layer_norm", act="relu2", arrangement="hyper", streams=int(cfg["streams"]),
                          loop=LayerLoop(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None,
                          hf_naming="gumazen")
        spec.runs()
        return cls.for_hybrid(spec, vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]),
                              rms_norm_eps=float(cfg["norm"]["eps"]), model_type="gumazen",
                              eos_token_id=int(cfg.get("eos_token_id", -1)), pad_token_id=int(cfg.get("pad_token_id", 0)))

    def _to_gumazen_config(self) -> Dict[str, Any]:
        hy, layers = self.hybrid, []
        for x in hy.layers:
            b, = x.branches
            m: Dict[str, Any] = {n: getattr(b, n) for n in ("heads", "kv_heads", "dim", "vdim", "scale")}
            if b.head_gate:
                t = "attention_2"
                m.update(softcap=b.softcap, bias_max=b.rel_max, mask={"size": b.window})
            else:
                t = "attention" if b.sink else "attention_3"
                m["rot"] = {"base": b.rot_base, "dims": b.rot_dims}
                if b.rot_scaling:
                    m["rot"]["scaling"] = dict(b.rot_scaling)
            mlp: Optional[Dict[str, Any]] = {"kind": "dense", "ff": x.ff} if x.ff else None
            if x.moe is not None:
                e = x.moe
                mlp = {"kind": "moe", "expert": {"ff": e.ff},
                       "router": {"experts": e.experts, "identity": e.identity, "top": e.top, "scale": e.scale,
                                  "groups": {"count": e.groups, "keep": e.keep}}}
                if e.shared_ff:
                    mlp["shared"] = {"ff": e.shared_ff}
            layers.append({"type": t, "mixer": m, "mlp": mlp})
        d = {"architecture": "Gumazen", "vocab": self.vocab_size, "width": self.hidden_size,
             "norm": {"eps": self.rms_norm_eps}, "streams": hy.streams, "layers": layers}
        if hy.loop is not None:
            d["loop"] = {"start": hy.loop.start, "stop": hy.loop.stop, "times": hy.loop.times}
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d

    @classmethod
    def _from_rizitar_config(cls, cfg: Dict[str, Any]) -> "DecoderConfig":
        """Rizitar: generalized delta rule or windowed attention with pooled blocks in any order, dense or routed
        feed-forwards, norms around every sublayer, a second embedding table per layer.  The low-rank width of the decay is
        not in the file: it is the shape of a tensor, filled in by ``from_pretrained``."""
        layers = []
        for x in cfg["layers"]:
            m, mlp = x["mixer"], x.get("mlp")
            if x["type"] == "general_delta":
                b = MixerBranch(kind="general_delta", heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["dim"]))
            elif x["type"] == "attention":
                if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                    raise ValueError("attention: values that are the keys have their width")
                mask, rot = m.get("mask") or {}, m.get("rot")
                b = MixerBranch(kind="attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                                vdim=int(m["dim"]), scale=float(m["scale"]), window=int(mask.get("size") or 0),
                                pool=int(mask.get("pool") or 0), bias_exp=0.0, qk_norm="head_weights", sink_weight=True,
                                key_values=True)
                if b.pool and not b.window:
                    raise ValueError("attention: pooled blocks need a window")
                if rot:
                    b.rot_dims, b.rot_base = int(rot["dims"]), float(rot["base"])
                    b.rot_scaling = dict(rot["scaling"]) if rot.get("scaling") else None
            else:
                raise ValueError(f"unknown layer type {x['type']!r}")
            layer = HybridLayer(branches=[b])
            if mlp is not None and mlp["kind"] == "dense":
                layer.ff = int(mlp["ff"])
            elif mlp is not None and mlp["kind"] == "moe":
                r = mlp["router"]
                layer.moe = ExpertSpec(experts=int(r["experts"]), ff=int(mlp["expert"]["ff"]), top=int(r["top"]), act="relu2",
                                       gated=False, corrected=False, renormalize=False)
            elif mlp is not None:
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            layers.append(layer)
        spec = HybridSpec(layers=layers, embed_scale=float(cfg["embedding"]["scale"]), norm="rms_norm", act="xielu",
                          arrangement="sandwich", token_side=int((cfg.get("token_side") or {}).get("dim") or 0),
                          ff_bias=True, hf_naming="rizitar")
        return cls.for_hybrid(spec, vocab_size=int(cfg["vocab"]), hidden_size=int(cfg["width"]), tie_word_embeddings=True,
                              rms_norm_eps=float(cfg["norm"]["eps"]), model_type="rizitar",
                              eos_token_id=int(cfg.get("eos_token_id", -1)), pad_token_id=int(cfg.get("pad_token_id", 0)))

    def _to_rizitar_config(self) -> Dict[str, Any]:
        hy, layers = self.hybrid, []
        for x in hy.layers:
            b, = x.branches
            if b.kind == "general_delta":
                m: Dict[str, Any] = {"heads": b.heads, "dim": b.dim}
            else:
                m = {n: getattr(b, n) for n in ("heads", "kv_heads", "dim", "vdim", "scale")}
                if b.window:
                    m["mask"] = {"size": b.window, **({"pool": b.pool} if b.pool else {})}
                if b.rot_dims:
                    m["rot"] = {"base": b.rot_base, "dims": b.rot_dims}
                    if b.rot_scaling:
                        m["rot"]["scaling"] = dict(b.rot_scaling)
            mlp: Optional[Dict[str, Any]] = {"kind": "dense", "ff": x.ff} if x.ff else None
            if x.moe is not None:
                mlp = {"kind": "moe", "expert": {"ff": x.moe.ff}, "router": {"experts": x.moe.experts, "top": x.moe.top}}
            layers.append({"type": b.kind, "mixer": m, "mlp": mlp})
        d = {"architecture": "Rizitar", "vocab": self.vocab_size, "width": self.hidden_size,
             "embedding": {"scale": hy.embed_scale}, "norm": {"eps": self.rms_norm_eps}, "layers": layers}
        if hy.token_side:
            d["token_side"] = {"dim": hy.token_side}
        if self.eos_token_id >= 0:
            d["eos_token_id"] = self.eos_token_id
        return d

    @classmethod
    def from_pretrained(cls, path: str) -> "DecoderConfig":
        with open(os.path.join(os.path.expanduser(path), "config.json")) as f:
            out = cls.from_hf_config(json.load(f))
        if out.hybrid is not None:
            from .hf_io import fill_hybrid_ranks
            fill_hybrid_ranks(out, path)
        return out

    def to_hf_config(self) -> Dict[str, Any]:
        if self.hybrid is not None:
            return {"poralorn": self._to_poralorn_config, "gumazen": self._to_gumazen_config,
                    "rizitar": self._to_rizitar_config}.get(
                self.hybrid.hf_naming, self._to_domavik_config)()
        arch = {"qwen2": "Qwen2ForCausalLM", "qwen3": "Qwen3ForCausalLM", "qwen3_moe": "Qwen3MoeForCausalLM",
                "llama": "LlamaForCausalLM", "qwen2_5_vl": "Qwen2_5_VLForConditionalGeneration",
                "mixtral": "MixtralForCausalLM", "qwen2_moe": "Qwen2MoeForCausalLM",
                "deepseek_v3": "DeepseekV3ForCausalLM"}
        d = {
            "architectures": [arch.get(self.model_type, "Qwen2ForCausalLM")], "model_type": self.model_type,
            "vocab_size": self.vocab_size, "hidden_size": self.hidden_size,
            "intermediate_size": self.intermediate_size, "num_hidden_layers": self.num_layers,
            "num_attention_heads": self.num_heads, "num_key_value_heads": self.num_kv_heads,
            "head_dim": self.head_dim, "rope_theta": self.rope_theta, "rms_norm_eps": self.rms_norm_eps,
            "max_position_embeddings": self.max_position_embeddings,
            "tie_word_embeddings": self.tie_word_embeddings, "hidden_act": "silu", "torch_dtype": "bfloat16",
            "eos_token_id": self.eos_token_id, "pad_token_id": self.pad_token_id,
        }
        if self.is_mla:
            d.update(kv_lora_rank=self.kv_lora_rank, q_lora_rank=self.q_lora_rank or None,
                     qk_nope_head_dim=self.qk_nope_head_dim, qk_rope_head_dim=self.qk_rope_head_dim,
                     v_head_dim=self.v_head_dim, rope_interleave=self.rope_interleave, attention_bias=self.qkv_bias,
                     qk_head_dim=self.qk_nope_head_dim + self.qk_rope_head_dim, head_dim=self.qk_rope_head_dim)
        if self.is_moe and self.model_type in ("deepseek_v3", "kimi_vl"):
            d.update(n_routed_experts=self.num_experts, num_experts_per_tok=self.num_experts_per_tok,
                     moe_intermediate_size=self.moe_intermediate_size, norm_topk_prob=self.norm_topk_prob,
                     n_shared_experts=self.shared_expert_intermediate_size // max(self.moe_intermediate_size, 1),
                     n_group=self.n_group, topk_group=self.topk_group, scoring_func=self.scoring_func,
                     topk_method=self.topk_method, routed_scaling_factor=self.routed_scaling_factor,
                     first_k_dense_replace=self.first_k_dense_replace)
        elif self.is_moe and self.model_type == "mixtral":
            d.update(num_local_experts=self.num_experts, num_experts_per_tok=self.num_experts_per_tok,
                     intermediate_size=self.moe_intermediate_size)
        elif self.is_moe:
            d.update(num_experts=self.num_experts, num_experts_per_tok=self.num_experts_per_tok,
                     moe_intermediate_size=self.moe_intermediate_size, norm_topk_prob=self.norm_topk_prob)
            if self.shared_expert_intermediate_size:
                d["shared_expert_intermediate_size"] = self.shared_expert_intermediate_size
        if self.mrope_section:
            d["rope_scaling"] = {"type": "mrope", "mrope_section": self.mrope_section}
        elif self.rope_scaling:
            d["rope_scaling"] = dict(self.rope_scaling)
        if self.moonvit is not None:
            mv = self.moonvit
            text = dict(d, model_type="deepseek_v3")
            text.pop("architectures", None)
            return {"architectures": ["KimiVLForConditionalGeneration"], "model_type": "kimi_vl", "text_config": text,
                    "vision_config": {"model_type": "moonvit", "patch_size": mv.patch_size,
                                      "init_pos_emb_height": mv.init_pos_emb_height,
                                      "init_pos_emb_width": mv.init_pos_emb_width, "hidden_size": mv.hidden_size,
                                      "num_attention_heads": mv.num_heads, "intermediate_size": mv.intermediate_size,
                                      "num_hidden_layers": mv.depth, "merge_kernel_size": [mv.merge, mv.merge]},
                    "media_placeholder_token_id": self.image_token_id, "torch_dtype": "bfloat16"}
        if self.prismatic is not None:
            pc = self.prismatic
            towers = [pc.featurizer] + ([pc.fused_featurizer] if pc.fused_featurizer else [])
            text = dict(d, model_type="llama", vocab_size=self.action_vocab_size or self.vocab_size)
            text.pop("architectures", None)
            return {"architectures": ["OpenVLAForActionPrediction"], "model_type": "openvla", "text_config": text,
                    "timm_model_ids": pc.timm_model_ids[: len(towers)], "image_sizes": [t.image_size for t in towers],
                    "use_fused_vision_backbone": pc.fused_featurizer is not None,
                    "vit_overrides": [asdict(t) for t in towers], "n_action_bins": self.n_action_bins,
                    "pad_to_multiple_of": 64, "pad_token_id": self.pad_token_id,
                    "num_images_in_input": pc.num_images_in_input, "action_vocab_size": self.action_vocab_size,
                    "torch_dtype": "bfloat16"}
        if self.vit is not None:
            v = self.vit
            text = dict(d, model_type=self.llm_type or "qwen2")
            text.pop("architectures", None)
            vision = {"hidden_size": v.hidden_size, "num_hidden_layers": v.depth, "num_attention_heads": v.num_heads,
                      "intermediate_size": v.intermediate_size, "norm_type": v.norm_type, "layer_norm_eps": v.norm_eps}
            if self.hf_naming == "hf":
                vision.update(image_size=[v.image_size] * 2, patch_size=[v.patch_size] * 2, attention_bias=v.qkv_bias,
                              model_type="internvl_vision")
                return {"architectures": ["InternVLForConditionalGeneration"], "model_type": "internvl",
                        "text_config": text, "vision_config": vision, "image_token_id": self.image_token_id,
                        "downsample_ratio": self.downsample_ratio, "vision_feature_layer": v.select_layer,
                        "tie_word_embeddings": self.tie_word_embeddings, "torch_dtype": "bfloat16"}
            vision.update(image_size=v.image_size, patch_size=v.patch_size, qkv_bias=v.qkv_bias)
            if self.llm_type == "internlm2":
                text["bias"] = self.qkv_bias
            return {"architectures": ["InternVLChatModel"], "model_type": "internvl_chat", "llm_config": text,
                    "vision_config": vision, "img_context_token_id": self.image_token_id,
                    "downsample_ratio": self.downsample_ratio, "select_layer": v.select_layer,
                    "torch_dtype": "bfloat16"}
        return d


def vit_from_timm_id(model_id: str, image_size: int = 224) -> ViTConfig:
    """Shapes of the timm vision transformers the Prismatic backbones name (no timm import: the architectures are
    public and fixed)."""
    if "dinov2" in model_id:
        large = "large" in model_id
        return ViTConfig(image_size=image_size, patch_size=14, hidden_size=1024 if large else 768,
                         num_heads=16 if large else 12, intermediate_size=4096 if large else 3072,
                         depth=24 if large else 12, class_token=True, num_register_tokens=4 if "reg4" in model_id else 0,
                         layer_scale=True, final_norm=True, select_layer=-2, class_pos_embed="reg4" not in model_id)
    if "siglip" in model_id:
        so = "so400m" in model_id
        return ViTConfig(image_size=image_size, patch_size=14 if so else 16, hidden_size=1152 if so else 768,
                         num_heads=16 if so else 12, intermediate_size=4304 if so else 3072, depth=27 if so else 12,
                         class_token=False, layer_scale=False, final_norm=True, select_layer=-2)
    raise ValueError(f"unknown vision backbone {model_id}")


def _domavik(n_layers: int, width: int, ff: int, vocab: int, att: dict, gla: dict, mem: dict, scales=(1.0, 1.0),
             softcap: float = 30.0, embed_scale: float = 1.0, **kw) -> DecoderConfig:
    """Alternating Domavik layers: attention beside gated linear attention, then a matrix memory."""
    layers = []
    for i in range(n_layers):
        if i % 2 == 0:
            br = [MixerBranch(kind="attention", out_scale=scales[0], scale=att["dim"] ** -0.5, **att),
                  MixerBranch(kind="gated_linear", out_scale=scales[1], **gla)]
        else:
            br = [MixerBranch(kind="matrix_memory", **mem)]
        layers.append(HybridLayer(branches=br, ff=ff))
    spec = HybridSpec(layers=layers, embed_scale=embed_scale, logit_softcap=softcap)
    return DecoderConfig.for_hybrid(spec, vocab_size=vocab, hidden_size=width, rms_norm_eps=1e-5, model_type="domavik",
                                    **kw)


def _poralorn(n_layers: int, width: int, ff: int, vocab: int, heads: int, dim: int, vdim: int, kv_rank: int,
              loop: Optional[LayerLoop] = None, softcap: float = 30.0, mult: float = 0.5, **kw) -> DecoderConfig:
    layers = [HybridLayer([MixerBranch(kind="latent_attention", heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank,
                                       scale=dim ** -0.5, output_gate=True)], ff=ff) for _ in range(n_layers)]
    spec = HybridSpec(layers=layers, logit_softcap=softcap, norm="rms_norm", act="gelu", arrangement="parallel",
                      residual_mult=mult, residual_gate=True, loop=loop, hf_naming="poralorn")
    return DecoderConfig.for_hybrid(spec, vocab_size=vocab, hidden_size=width, rms_norm_eps=1e-5, model_type="poralorn",
                                    **kw)


def _gumazen(n_layers: int, width: int, ff: int, vocab: int, heads: int, kv_heads: int, dim: int, window: int,
             moe: ExpertSpec, rot_dims: int, streams: int = 2, loop: Optional[LayerLoop] = None, vdim: int = 0,
             **kw) -> DecoderConfig:
    """Gumazen layers in turn: rotated with biases, rotated with a sink, windowed with a distance table; the first layer
    has a dense feed-forward, the others are routed."""
    base = dict(kind="attention", heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim or dim, scale=dim ** -0.5, bias_exp=0.0)
    kinds = [dict(qk_norm="rows", proj_bias=True, rot_dims=rot_dims, rot_base=1e6,
                  rot_scaling={"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}),
             dict(qk_norm="heads", sink=True, rot_dims=rot_dims, rot_base=5e4),
             dict(qk_norm="rows", head_gate=True, softcap=50.0, rel_rows=32, rel_max=window // 2, window=window)]
    layers = [HybridLayer([MixerBranch(**base, **kinds[i % 3])], ff=0 if i else ff, moe=moe if i else None)
              for i in range(n_layers)]
    spec = HybridSpec(layers=layers, act="relu2", arrangement="hyper", streams=streams, loop=loop, hf_naming="gumazen")
    return DecoderConfig.for_hybrid(spec, vocab_size=vocab, hidden_size=width, rms_norm_eps=1e-5, model_type="gumazen", **kw)


def _rizitar(n_layers: int, width: int, ff: int, vocab: int, att: dict, delta: dict, moe: ExpertSpec, side: int,
             rot_base: float = 1e6, **kw) -> DecoderConfig:
    """Rizitar layers in turn: two delta rules, then attention; the first layer has a dense feed-forward, the others are
    routed."""
    dim = att["dim"]
    base = dict(kind="attention", vdim=dim, scale=dim ** -0.5, bias_exp=0.0, qk_norm="head_weights", sink_weight=True,
                key_values=True, rot_dims=dim, rot_base=rot_base,
                rot_scaling={"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0})
    layers = [HybridLayer([MixerBranch(**base, **att) if i % 3 == 2 else
                           MixerBranch(kind="general_delta", vdim=delta["dim"], **delta)],
                          ff=0 if i else ff, moe=moe if i else None) for i in range(n_layers)]
    spec = HybridSpec(layers=layers, embed_scale=width ** 0.5, norm="rms_norm", act="xielu", arrangement="sandwich",
                      token_side=side, ff_bias=True, hf_naming="rizitar")
    return DecoderConfig.for_hybrid(spec, vocab_size=vocab, hidden_size=width, rms_norm_eps=1e-5, model_type="rizitar",
                                    tie_word_embeddings=True, **kw)


def _plain_experts(experts: int, ff: int, top: int) -> ExpertSpec:
    return ExpertSpec(experts=experts, ff=ff, top=top, act="relu2", gated=False, corrected=False, renormalize=False)


PRESETS: Dict[str, DecoderConfig] = {
    "tiny-rizitar": _rizitar(3, 128, 192, 1024, dict(heads=4, kv_heads=2, dim=32, window=50, pool=12),
                             dict(heads=3, dim=24, rank=8), _plain_experts(6, 40, 2), side=16),
    # layer sizes of decoders with about 1 / 3 billion active parameters (benchmark shapes, random weights)
    "rizitar-a1b": _rizitar(18, 1536, 8960, 152064, dict(heads=12, kv_heads=2, dim=128, window=1024, pool=16),
                            dict(heads=24, dim=64, rank=64), _plain_experts(56, 1152, 6), side=128),
    "rizitar-a3b": _rizitar(18, 2048, 11264, 152064, dict(heads=32, kv_heads=4, dim=128, window=1024, pool=16),
                            dict(heads=32, dim=64, rank=64), _plain_experts(120, 1536, 8), side=256),
    "tiny-gumazen": _gumazen(3, 128, 192, 1024, heads=4, kv_heads=2, dim=32, vdim=24, window=70, rot_dims=16,
                             moe=ExpertSpec(experts=6, ff=40, top=3, groups=2, keep=1, identity=2, scale=1.5, shared_ff=56),
                             loop=LayerLoop(1, 3, 2)),
    # layer sizes of decoders with about 1 / 3 billion active parameters (benchmark shapes, random weights)
    "gumazen-a1b": _gumazen(18, 1536, 8960, 152064, heads=12, kv_heads=2, dim=128, window=1024, rot_dims=64,
                            moe=ExpertSpec(experts=56, ff=768, top=6, groups=8, keep=4, identity=8, scale=2.0,
                                           shared_ff=1536), loop=LayerLoop(3, 9, 2)),
    "gumazen-a3b": _gumazen(18, 2048, 11264, 152064, heads=32, kv_heads=4, dim=128, window=1024, rot_dims=64,
                            moe=ExpertSpec(experts=120, ff=1024, top=8, groups=8, keep=4, identity=8, scale=2.0,
                                           shared_ff=2048), loop=LayerLoop(3, 9, 2)),
    "tiny-poralorn": _poralorn(3, 128, 224, 1024, heads=3, dim=24, vdim=40, kv_rank=48, loop=LayerLoop(1, 2, 3)),
    # layer sizes of a 7B / 1.5B-class decoder (benchmark shapes, random weights)
    "poralorn-7b": _poralorn(28, 3584, 18944, 152064, heads=28, dim=128, vdim=128, kv_rank=512, loop=LayerLoop(2, 6, 2)),
    "poralorn-1.5b": _poralorn(28, 1536, 8960, 152064, heads=12, dim=128, vdim=128, kv_rank=512, loop=LayerLoop(2, 8, 2)),
    "tiny-domavik": _domavik(3, 128, 192, 1024, dict(heads=4, kv_heads=2, dim=32, vdim=24, window=70, keep_first=5),
                             dict(heads=2, dim=16, vdim=32, tau=4.0, rank=8), dict(heads=2, dim=32, vdim=40),
                             scales=(0.9, 0.6)),
    # layer sizes of a 7B / 1.5B-class decoder (benchmark shapes, random weights)
    "domavik-7b": _domavik(28, 3584, 18944, 152064, dict(heads=28, kv_heads=4, dim=128, vdim=128, window=1024,
                                                         keep_first=64),
                           dict(heads=16, dim=64, vdim=128, rank=16), dict(heads=16, dim=128, vdim=128)),
    "domavik-1.5b": _domavik(28, 1536, 8960, 152064, dict(heads=12, kv_heads=2, dim=128, vdim=128, window=1024,
                                                          keep_first=64),
                             dict(heads=8, dim=64, vdim=128, rank=16), dict(heads=8, dim=96, vdim=128)),
    # 2-layer gate model used by the CPU/gloo end-to-end test
    "tiny": DecoderConfig(model_type="qwen2", vocab_size=1024, hidden_size=128, intermediate_size=352, num_layers=2,
                          num_heads=4, num_kv_heads=2, head_dim=32, rope_theta=1e4, eos_token_id=2),
    # small GPU smoke model (head_dim 64 path)
    "tiny-gpu": DecoderConfig(model_type="qwen2", vocab_size=4096, hidden_size=512, intermediate_size=1408,
                              num_layers=2, num_heads=8, num_kv_heads=2, head_dim=64, rope_theta=1e6, eos_token_id=2),
    "qwen2.5-0.5b": DecoderConfig(model_type="qwen2", vocab_size=151936, hidden_size=896, intermediate_size=4864,
                                  num_layers=24, num_heads=14, num_kv_heads=2, head_dim=64, rope_theta=1e6,
                                  tie_word_embeddings=True, eos_token_id=151645, pad_token_id=151643),
    "qwen2.5-7b": DecoderConfig(model_type="qwen2", vocab_size=152064, hidden_size=3584, intermediate_size=18944,
                                num_layers=28, num_heads=28, num_kv_heads=4, head_dim=128, rope_theta=1e6,
                                eos_token_id=151645, pad_token_id=151643),
    "qwen3-30b-a3b": DecoderConfig(model_type="qwen3_moe", vocab_size=151936, hidden_size=2048, intermediate_size=6144,
                                   num_layers=48, num_heads=32, num_kv_heads=4, head_dim=128, rope_theta=1e6,
                                   qkv_bias=False, qk_norm=True, num_experts=128, num_experts_per_tok=8,
                                   moe_intermediate_size=768, eos_token_id=151645, pad_token_id=151643),
    "mixtral-8x7b": DecoderConfig(model_type="mixtral", vocab_size=32000, hidden_size=4096, intermediate_size=14336,
                                  num_layers=32, num_heads=32, num_kv_heads=8, head_dim=128, rope_theta=1e6,
                                  qkv_bias=False, num_experts=8, num_experts_per_tok=2, moe_intermediate_size=14336,
                                  rms_norm_eps=1e-5, eos_token_id=2, pad_token_id=0),
    "qwen1.5-moe-a2.7b": DecoderConfig(model_type="qwen2_moe", vocab_size=151936, hidden_size=2048,
                                       intermediate_size=5632, num_layers=24, num_heads=16, num_kv_heads=16,
                                       head_dim=128, rope_theta=1e6, qkv_bias=True, num_experts=60,
                                       num_experts_per_tok=4, moe_intermediate_size=1408, norm_topk_prob=False,
                                       shared_expert_intermediate_size=5632, shared_expert_gate=True,
                                       eos_token_id=151645, pad_token_id=151643),
    "tiny-mixtral": DecoderConfig(model_type="mixtral", vocab_size=1024, hidden_size=128, intermediate_size=64,
                                  num_layers=2, num_heads=4, num_kv_heads=2, head_dim=32, qkv_bias=False,
                                  num_experts=4, num_experts_per_tok=2, moe_intermediate_size=64),
    "tiny-qwen2-moe": DecoderConfig(model_type="qwen2_moe", vocab_size=1024, hidden_size=128, intermediate_size=352,
                                    num_layers=2, num_heads=4, num_kv_heads=2, head_dim=32, num_experts=8,
                                    num_experts_per_tok=2, moe_intermediate_size=64, norm_topk_prob=False,
                                    shared_expert_intermediate_size=96, shared_expert_gate=True),
    # DeepSeek-V3 (671B, 37B active): MLA + 256 routed / 1 shared experts, 3 dense layers
    "deepseek-v3": DecoderConfig(model_type="deepseek_v3", vocab_size=129280, hidden_size=7168, intermediate_size=18432,
                                 num_layers=61, num_heads=128, num_kv_heads=128, head_dim=192, rope_theta=1e4,
                                 qkv_bias=False, kv_lora_rank=512, q_lora_rank=1536, qk_nope_head_dim=128,
                                 qk_rope_head_dim=64, v_head_dim=128, num_experts=256, num_experts_per_tok=8,
                                 moe_intermediate_size=2048, shared_expert_intermediate_size=2048, n_group=8,
                                 topk_group=4, scoring_func="sigmoid", topk_method="noaux_tc",
                                 routed_scaling_factor=2.5, first_k_dense_replace=3, eos_token_id=1, pad_token_id=0),
    # Moonlight-16B-A3B, the language model of Kimi-VL-A3B
    "moonlight-16b-a3b": DecoderConfig(model_type="deepseek_v3", vocab_size=163840, hidden_size=2048,
                                       intermediate_size=11264, num_layers=27, num_heads=16, num_kv_heads=16,
                                       head_dim=192, rope_theta=5e4, qkv_bias=False, kv_lora_rank=512, q_lora_rank=0,
                                       qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128, num_experts=64,
                                       num_experts_per_tok=6, moe_intermediate_size=1408,
                                       shared_expert_intermediate_size=2816, n_group=1, topk_group=1,
                                       scoring_func="sigmoid", topk_method="noaux_tc", routed_scaling_factor=2.446,
                                       first_k_dense_replace=1, eos_token_id=163585, pad_token_id=163839),
    # Kimi-VL-A3B: MoonViT-SO-400M + Moonlight-16B-A3B
    "kimi-vl-a3b": DecoderConfig(model_type="kimi_vl", vocab_size=163840, hidden_size=2048, intermediate_size=11264,
                                 num_layers=27, num_heads=16, num_kv_heads=16, head_dim=192, rope_theta=8e5,
                                 qkv_bias=False, kv_lora_rank=512, q_lora_rank=0, qk_nope_head_dim=128,
                                 qk_rope_head_dim=64, v_head_dim=128, num_experts=64, num_experts_per_tok=6,
                                 moe_intermediate_size=1408, shared_expert_intermediate_size=2816, n_group=1,
                                 topk_group=1, scoring_func="sigmoid", topk_method="noaux_tc",
                                 routed_scaling_factor=2.446, first_k_dense_replace=1, moonvit=MoonViTConfig(),
                                 image_token_id=163605, eos_token_id=163585, pad_token_id=163839),
    "tiny-kimi-vl": DecoderConfig(model_type="kimi_vl", vocab_size=1024, hidden_size=128, intermediate_size=352,
                                  num_layers=2, num_heads=4, num_kv_heads=4, head_dim=48, qkv_bias=False,
                                  kv_lora_rank=32, q_lora_rank=0, qk_nope_head_dim=32, qk_rope_head_dim=16,
                                  v_head_dim=32, num_experts=8, num_experts_per_tok=2, moe_intermediate_size=64,
                                  shared_expert_intermediate_size=128, scoring_func="sigmoid",
                                  topk_method="noaux_tc", routed_scaling_factor=2.0, first_k_dense_replace=1,
                                  moonvit=MoonViTConfig(init_pos_emb_height=8, init_pos_emb_width=8, hidden_size=64,
                                                        num_heads=2, intermediate_size=128, depth=2),
                                  image_token_id=1000),
    "tiny-deepseek-v3": DecoderConfig(model_type="deepseek_v3", vocab_size=1024, hidden_size=128, intermediate_size=352,
                                      num_layers=3, num_heads=4, num_kv_heads=4, head_dim=48, qkv_bias=False,
                                      kv_lora_rank=32, q_lora_rank=48, qk_nope_head_dim=32, qk_rope_head_dim=16,
                                      v_head_dim=32, num_experts=8, num_experts_per_tok=2, moe_intermediate_size=64,
                                      shared_expert_intermediate_size=64, n_group=2, topk_group=1,
                                      scoring_func="sigmoid", topk_method="noaux_tc", routed_scaling_factor=2.5,
                                      first_k_dense_replace=1),
    "tiny-moe": DecoderConfig(model_type="qwen3_moe", vocab_size=1024, hidden_size=128, intermediate_size=352,
                              num_layers=2, num_heads=4, num_kv_heads=2, head_dim=32, qkv_bias=False, qk_norm=True,
                              num_experts=8, num_experts_per_tok=2, moe_intermediate_size=64),
    "qwen2.5-vl-7b": DecoderConfig(model_type="qwen2_5_vl", vocab_size=152064, hidden_size=3584,
                                   intermediate_size=18944, num_layers=28, num_heads=28, num_kv_heads=4, head_dim=128,
                                   rope_theta=1e6, mrope_section=[16, 24, 24], vision=VisionConfig(),
                                   eos_token_id=151645, pad_token_id=151643),
    "tiny-vl": DecoderConfig(model_type="qwen2_5_vl", vocab_size=1024, hidden_size=128, intermediate_size=352,
                             num_layers=2, num_heads=4, num_kv_heads=2, head_dim=32, mrope_section=[4, 6, 6],
                             vision=VisionConfig(depth=2, hidden_size=64, num_heads=4, intermediate_size=128,
                                                 patch_size=14, window_size=56, fullatt_block_indexes=[1],
                                                 out_hidden_size=128), image_token_id=1000),
    # InternVL2.5-8B: InternViT-300M-448px + InternLM2.5-7B
    "internvl2.5-8b": DecoderConfig(model_type="internvl_chat", llm_type="internlm2", hf_naming="internvl_chat",
                                    vocab_size=92553, hidden_size=4096, intermediate_size=14336, num_layers=32,
                                    num_heads=32, num_kv_heads=8, head_dim=128, rope_theta=1e6, qkv_bias=False,
                                    rms_norm_eps=1e-5, vit=ViTConfig(), image_token_id=92546, eos_token_id=92542,
                                    pad_token_id=2),
    # InternVL3-8B in transformers' layout: InternViT-300M + Qwen2.5-7B
    "internvl3-8b": DecoderConfig(model_type="internvl", llm_type="qwen2", vocab_size=151674, hidden_size=3584,
                                  intermediate_size=18944, num_layers=28, num_heads=28, num_kv_heads=4, head_dim=128,
                                  rope_theta=1e6, vit=ViTConfig(), image_token_id=151667, eos_token_id=151645,
                                  pad_token_id=151643),
    "tiny-internvl": DecoderConfig(model_type="internvl", llm_type="qwen2", vocab_size=1024, hidden_size=128,
                                   intermediate_size=352, num_layers=2, num_heads=4, num_kv_heads=2, head_dim=32,
                                   vit=ViTConfig(image_size=56, patch_size=14, hidden_size=64, num_heads=2,
                                                 intermediate_size=128, depth=2, qkv_bias=False),
                                   image_token_id=1000),
    # OpenVLA-7B / OpenVLA-OFT: DINOv2-L/14 (4 registers) + SigLIP-so400m/14 at 224 px, Llama-2-7B
    "openvla-7b": DecoderConfig(model_type="openvla", llm_type="llama", vocab_size=32064, hidden_size=4096,
                                intermediate_size=11008, num_layers=32, num_heads=32, num_kv_heads=32, head_dim=128,
                                rope_theta=1e4, rms_norm_eps=1e-6, qkv_bias=False, prismatic=PrismaticConfig(),
                                action_vocab_size=32000, image_token_id=32000, pad_token_id=32000, eos_token_id=2,
                                bos_token_id=1, max_position_embeddings=2048),
    "tiny-openvla": DecoderConfig(model_type="openvla", llm_type="llama", vocab_size=1088, hidden_size=128,
                                  intermediate_size=352, num_layers=2, num_heads=4, num_kv_heads=4, head_dim=32,
                                  qkv_bias=False, action_vocab_size=1024, image_token_id=1024, pad_token_id=1024,
                                  bos_token_id=1, prismatic=PrismaticConfig(
                                      featurizer=ViTConfig(image_size=56, patch_size=14, hidden_size=64, num_heads=2,
                                                           intermediate_size=128, depth=3, num_register_tokens=4,
                                                           final_norm=True, select_layer=-2, class_pos_embed=False),
                                      fused_featurizer=ViTConfig(image_size=56, patch_size=14, hidden_size=72,
                                                                 num_heads=2, intermediate_size=96, depth=3,
                                                                 class_token=False, layer_scale=False, final_norm=True,
                                                                 select_layer=-2))),
    "tiny-vl-gpu": DecoderConfig(model_type="qwen2_5_vl", vocab_size=2048, hidden_size=256, intermediate_size=512,
                                 num_layers=2, num_heads=4, num_kv_heads=2, head_dim=64, mrope_section=[8, 12, 12],
                                 vision=VisionConfig(depth=2, hidden_size=128, num_heads=2, intermediate_size=256,
                                                     patch_size=14, window_size=56, fullatt_block_indexes=[1],
                                                     out_hidden_size=256), image_token_id=1500),
}


def get_config(name_or_path: str, overrides: Optional[Dict[str, Any]] = None) -> DecoderConfig:
    """Preset name (``qwen2.5-7b``) or a directory with an HF ``config.json``."""
    import copy
    if name_or_path in PRESETS:
        cfg = copy.deepcopy(PRESETS[name_or_path])
    else:
        cfg = DecoderConfig.from_pretrained(name_or_path)
    for k, v in (overrides or {}).items():
        hf_alias = {"num_hidden_layers": "num_layers", "num_attention_heads": "num_heads",
                    "num_key_value_heads": "num_kv_heads"}
        k = hf_alias.get(k, k)
        if hasattr(cfg, k):
            setattr(cfg, k, v)
    return cfg
