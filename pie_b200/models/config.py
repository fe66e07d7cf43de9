"""Model configuration parsed from a Hugging Face ``config.json``.

Keys consumed mirror the reference's HF config reader
(driver/cuda/src/loader/hf_config.hpp:145-215).
"""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field, asdict
from pathlib import Path
from typing import Optional

from .block_spec import EVERYTHING, LatentSpec, PairSpec, _pad, retodra_config, retodra_shape
from .nukelix import nukelix_config, nukelix_shape
from .vulanex import vulanex_config, vulanex_shape

LLAMA_LIKE = {"llama", "qwen2", "qwen3", "mistral", "phi3"}   # pre-norm decoder blocks with SwiGLU and rotate-half RoPE
# `model_type` strings of checkpoints this build loads (the architecture registry of the loader)
SUPPORTED_MODEL_TYPES = ("llama", "mistral", "qwen2", "qwen3", "phi3", "qwen3_moe", "mixtral", "olmo2", "olmo3", "gpt_oss",
                         "qwen3_5", "qwen3_next", "mamba2_hybrid", "gemma2", "gemma3_text", "gemma3", "qwen2_moe", "qwen2_vl",
                         "qwen2_audio", "puzutar", "retodra", "nukelix", "vulanex")
MAMBA_TYPES = {"mamba2_hybrid"}         # Mamba-2 (state-space) mixers in llama-like blocks, between full-attention layers
GDN_TYPES = {"qwen3_5", "qwen3_next"}   # hybrids: Gated DeltaNet (linear attention) layers between full-attention layers
POST_NORM = {"olmo2", "olmo3"}       # same block with the norms after attention / MLP and q, k norms over all heads
MOE_TYPES = {"qwen3_moe", "mixtral", "gpt_oss", "qwen2_moe"}
# Gemma-2 / Gemma-3: norms before AND after attention and MLP, gains stored as (w - 1), GeGLU, scaled embeddings,
# alternating local / global layers (Gemma-3: a RoPE base of their own for the local ones; Gemma-2: soft-capped logits)
GEMMA_TYPES = {"gemma2", "gemma3_text", "gemma3"}
# configs that name the design under "architecture" instead of "model_type"
ARCHITECTURES = {"Puzutar": "puzutar", "Retodra": "retodra", "Nukelix": "nukelix", "Vulanex": "vulanex"}


def config_model_type(cfg: dict) -> str:
    """The registry name a `config.json` dictionary asks for ("" when it names none)."""
    return cfg.get("model_type") or ARCHITECTURES.get(cfg.get("architecture", ""), "")


@dataclass
class ModelConfig:
    model_type: str = "llama"
    hidden_size: int = 4096
    intermediate_size: int = 14336
    num_hidden_layers: int = 32
    num_attention_heads: int = 32
    num_key_value_heads: int = 8
    head_dim: int = 128
    vocab_size: int = 128256
    max_position_embeddings: int = 131072
    rms_norm_eps: float = 1e-5
    rope_theta: float = 500000.0
    rope_scaling: Optional[dict] = None
    tie_word_embeddings: bool = False
    qk_norm: bool = False           # Qwen3: per-head RMSNorm on q and k
    attention_bias: bool = False    # Qwen2: bias on q/k/v projections
    sliding_window: int = -1
    post_norm: bool = False         # OLMo-2: h += norm(attn(h)); h += norm(mlp(h)); q/k RMSNorm over the whole projection
    layer_types: Optional[list] = None   # per layer "sliding_attention" | "full_attention" (GPT-OSS); None: all alike
    attention_sinks: bool = False   # GPT-OSS: a learned per-head logit in every softmax denominator
    o_bias: bool = False            # bias on the attention output projection
    sandwich_norm: bool = False     # Gemma-2/3: h += norm(attn(norm(h))); h += norm(mlp(norm(h)))
    norm_plus_one: bool = False     # checkpoints store RMSNorm gains as (w - 1); the loader adds the 1
    hidden_act: str = "silu"        # gate activation of the GLU: "silu" | "gelu_tanh"
    embed_scale: float = 1.0        # embeddings are multiplied by this (Gemma: sqrt(hidden_size))
    query_pre_attn_scalar: float = 0.0   # attention scale is this ** -0.5 (0: head_dim)
    attn_softcap: float = 0.0       # scores pass through cap * tanh(s / cap) before the softmax (0: off)
    final_softcap: float = 0.0      # same for the output logits
    rope_local_theta: float = 0.0   # RoPE base of the sliding-window layers, unscaled (0: same table as the others)
    # mixture of experts
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True
    # a dense expert that every token also passes through, scaled by sigmoid(x . shared_gate) (Qwen2-MoE, Qwen3-Next); 0: none
    shared_expert_intermediate_size: int = 0
    moe_style: str = "swiglu"       # "gpt_oss": expert and router biases, clamped (up + 1) * gate * sigmoid(1.702 gate)
    swiglu_limit: float = 7.0
    # Gated DeltaNet layers (layer_types entry "linear_attention"): heads and head sizes of the linear mixer
    linear_num_key_heads: int = 0
    linear_num_value_heads: int = 0
    linear_key_head_dim: int = 0
    linear_value_head_dim: int = 0
    linear_conv_kernel_dim: int = 4
    # Mamba-2 layers (layer_types entry "mamba2"): heads, head size, state size, B / C groups
    mamba_num_heads: int = 0
    mamba_head_dim: int = 0
    ssm_state_size: int = 0
    mamba_n_groups: int = 1
    mamba_norm_grouped: bool = False   # gated RMSNorm per B / C group (Nemotron-H) instead of over the whole inner width (Mamba-2)
    # parallel blocks over a 32-bit residual stream: x += mixer(shifted norm(x)) + ff(norm(x)), then the token input
    latent: Optional[list] = None      # LatentSpec per layer
    ff_sizes: Optional[list] = None    # per layer width of the xIELU feed-forward (0: the layer has none)
    norm_groups: int = 1               # RMSNorm over this many equal parts of the width, each with its own mean square
    token_shift: bool = False          # the mixer reads h + (previous token's h - h) * shift: state of a sequence
    token_side_dim: int = 0            # width of the per-layer token input (0: none)
    # layers described one by one over a 32-bit residual stream: sandwich-normed blocks, (post_norm) blocks that norm their
    # sublayers' outputs only, or (layer_norm) blocks that read the stream through a layer norm and a convolution
    blocks: Optional[list] = None      # BlockSpec per layer
    layer_norm: bool = False
    conv_taps: int = 0                 # taps of the causal convolution added to every sublayer's input (0: none): state of a sequence
    token_pairs: Optional[PairSpec] = None   # embedding rows for (token before, token): state of a sequence
    logit_scale: float = 1.0
    # quantisation of the linear weights: None | "fp8_block" (128x128 weight scales)
    quantization: Optional[str] = None
    dtype: str = "bfloat16"
    name: str = ""

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    def is_linear_layer(self, li: int) -> bool:
        return self.layer_types is not None and self.layer_types[li] == "linear_attention"

    @property
    def linear_layers(self) -> list:
        """Indices of the Gated DeltaNet layers (empty for pure-attention models)."""
        return [li for li in range(self.num_hidden_layers) if self.is_linear_layer(li)]

    def is_mamba_layer(self, li: int) -> bool:
        return self.layer_types is not None and self.layer_types[li] == "mamba2"

    @property
    def mamba_layers(self) -> list:
        return [li for li in range(self.num_hidden_layers) if self.is_mamba_layer(li)]

    @property
    def recurrent_layers(self) -> list:
        """Layers whose state lives in the recurrent-state cache (Gated DeltaNet or Mamba-2)."""
        return [li for li in range(self.num_hidden_layers)
                if self.token_shift or self.blocks is not None or self.is_linear_layer(li) or self.is_mamba_layer(li)]

    @property
    def latent_cache_layers(self) -> list:
        """Layers that write latent rows; the others read the rows of one of these."""
        return [li for li, s in enumerate(self.latent) if s.kv_from is None]

    @property
    def latent_cache_index(self) -> dict:
        """Layer -> index into the first dimension of the latent cache."""
        own = {li: i for i, li in enumerate(self.latent_cache_layers)}
        return {li: own[li if s.kv_from is None else s.kv_from] for li, s in enumerate(self.latent)}

    @property
    def stream32(self) -> bool:
        """The residual stream is 32-bit, and the whole model also runs in true 32-bit on the device."""
        return self.latent is not None or self.blocks is not None

    @property
    def latent_specs(self) -> list:
        """The latent-attention mixers of all layers."""
        return self.latent if self.latent is not None else [b.latent for b in self.blocks or () if b.latent is not None]

    @property
    def kv_layers(self) -> list:
        """(kv heads, head dim) of every layer that has a cache, in order; latent rows count as no head of the row's width. Two
        more numbers where a layer's pages are laid out otherwise: rows per token and head, tokens per mean (0: no means)."""
        def shape(b):
            if b.latent is not None:
                return 0, b.latent.row
            a = b.attention
            planes, pool = getattr(a, "planes", 2), getattr(a, "pool", 0)
            return (a.kv_heads, a.head_dim) if (planes, pool) == (2, 0) else (a.kv_heads, a.head_dim, planes, pool)
        if self.blocks is not None:
            return [shape(b) for b in self.blocks if b.latent is not None or b.attention is not None]
        return [(self.num_key_value_heads, self.head_dim)] * self.num_hidden_layers

    def kv_page_shapes(self, page_size: int) -> list:
        """Shapes of one page in every layer that has a cache: of its rows, and of the means beside them (None: none)."""
        out = []
        for h, d, *laid in self.kv_layers:
            planes, pool = laid or (2, 0)
            out.append(((planes, h, page_size, d) if h else (page_size, d), (2, h, -(-page_size // pool), d) if pool else None))
        return out

    def kv_elems_per_page(self, page_size: int) -> int:
        """Cache elements one page takes over all layers (unsharded)."""
        if self.latent is not None:
            return len(self.latent_cache_layers) * self.latent_row * page_size
        if self.blocks is not None:
            return sum(math.prod(s) for pair in self.kv_page_shapes(page_size) for s in pair if s is not None)
        return self.num_hidden_layers * 2 * self.num_key_value_heads * self.head_dim * page_size

    def slot_layout(self) -> tuple:
        """What a sequence carries in a row of the state cache of layers described one by one, by first element: recurrent
        states by layer, histories of the input convolutions by (layer, half), the token before (None: not kept); the row's
        elements."""
        states, histories, before, at = {}, {}, None, 0
        for li, b in enumerate(self.blocks):
            if b.recurrent is not None:
                states[li], at = at, at + _pad(b.recurrent.state_elems, 4)
        if self.conv_taps > 1:
            for li, b in enumerate(self.blocks):
                for half in ("1", "2") if b.ff is not None else ("1",):
                    histories[li, half], at = at, at + _pad((self.conv_taps - 1) * self.hidden_size, 4)
        if self.token_pairs is not None:
            before, at = at, at + 4
        return states, histories, before, at

    @property
    def latent_row(self) -> int:
        return max(s.row for s in self.latent)

    @property
    def mamba_inner(self) -> int:
        return self.mamba_num_heads * self.mamba_head_dim

    @property
    def mamba_conv_channels(self) -> int:
        """Channels of the short convolution: x, then B and C of every group."""
        return self.mamba_inner + 2 * self.mamba_n_groups * self.ssm_state_size

    @property
    def mamba_in_features(self) -> int:
        """Rows of the input projection: z (gate) | x B C | dt."""
        return self.mamba_inner + self.mamba_conv_channels + self.mamba_num_heads

    @property
    def gdn_conv_channels(self) -> int:
        """Channels of the short convolution: q and k of the key heads, v of the value heads."""
        return 2 * self.linear_num_key_heads * self.linear_key_head_dim + self.linear_num_value_heads * self.linear_value_head_dim

    @property
    def gdn_in_features(self) -> int:
        """Rows of the fused input projection: q | k | v | z (output gate) | b (beta) | a (decay)."""
        return self.gdn_conv_channels + self.linear_num_value_heads * self.linear_value_head_dim + 2 * self.linear_num_value_heads

    def layer_window_left(self, li: int) -> int:
        """Keys left of the query that layer `li` sees (-1: all, or far ones beside a window). HF `sliding_window` counts the
        query itself."""
        if self.latent is not None:
            return self.latent[li].window - 1
        if self.blocks is not None:
            b = self.blocks[li]
            a = b.latent or b.attention
            return 0 if a is None else -1 if a.window == EVERYTHING or getattr(a, "keep_first", 0) or getattr(a, "pool", 0) else a.window - 1
        if not self.sliding_window or self.sliding_window <= 0:
            return -1
        if self.layer_types is not None and self.layer_types[li] != "sliding_attention":
            return -1
        return self.sliding_window - 1

    @property
    def plan_window_left(self) -> int:
        """The window attention plans may be cut to: the widest any layer needs."""
        ws = [self.layer_window_left(li) for li in range(self.num_hidden_layers)]
        return -1 if any(w < 0 for w in ws) or not ws else max(ws)

    @property
    def q_size(self) -> int:
        return self.num_attention_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_key_value_heads * self.head_dim

    def to_dict(self) -> dict:
        return asdict(self)

    @staticmethod
    def from_hf(cfg: dict, name: str = "") -> "ModelConfig":
        mt = config_model_type(cfg) or "llama"
        if mt == "puzutar":
            return _puzutar_config(cfg, name)
        if mt == "retodra":
            return retodra_config(cfg, name)
        if mt == "nukelix":
            return nukelix_config(cfg, name)
        if mt == "vulanex":
            return vulanex_config(cfg, name)
        if mt == "gemma3" and "text_config" in cfg:       # multimodal wrapper: the language model's own section
            cfg = dict(cfg["text_config"], model_type="gemma3_text")
            mt = "gemma3_text"
        if mt == "qwen2_audio" and "text_config" in cfg:       # the language model of Qwen2-Audio is a plain Qwen2
            tc = dict(cfg["text_config"])
            tc.setdefault("tie_word_embeddings", cfg.get("tie_word_embeddings", False))
            cfg, mt = dict(tc, model_type="qwen2"), "qwen2"
        if mt in ("qwen2_vl", "qwen2_vl_text"):
            # the language model of Qwen2-VL is the Qwen2 block; its three-axis rotary positions are not built: tokens
            # take one-dimensional positions (the same thing for text; image rows then differ from the checkpoint's own code)
            tc = dict(cfg.get("text_config") or cfg)
            tc.setdefault("tie_word_embeddings", cfg.get("tie_word_embeddings", False))
            cfg, mt = dict(tc, model_type="qwen2"), "qwen2"
        cfg = _flatten_rope_parameters(dict(cfg))
        gemma = mt in GEMMA_TYPES
        if gemma:
            cfg.setdefault("head_dim", 256)
            cfg.setdefault("tie_word_embeddings", True)
            cfg.setdefault("rms_norm_eps", 1e-6)
            if cfg.get("layer_types") is None:
                # Gemma-2 alternates local / global; Gemma-3 runs `sliding_window_pattern - 1` local layers per global one
                pat = int(cfg.get("sliding_window_pattern") or cfg.get("_sliding_window_pattern") or (2 if mt == "gemma2" else 6))
                cfg["layer_types"] = ["full_attention" if (i + 1) % pat == 0 else "sliding_attention"
                                      for i in range(cfg["num_hidden_layers"])]
        heads = cfg["num_attention_heads"]
        hd = cfg.get("head_dim") or cfg["hidden_size"] // heads
        q = cfg.get("quantization_config") or {}
        quant = None
        if q.get("quant_method") == "fp8" and q.get("weight_block_size"):
            quant = "fp8_block"
        elif _is_fp8_weight_config(q):
            # per-tensor / per-channel fp8 checkpoints (`weight_scale` next to each weight): the loader spreads the scale
            # over the row blocks of the same runtime format; activations are quantised per call, a stored input scale is unused
            quant = "fp8_block"
        return ModelConfig(
            model_type=mt,
            hidden_size=cfg["hidden_size"],
            intermediate_size=cfg.get("intermediate_size", 0),
            num_hidden_layers=cfg["num_hidden_layers"],
            num_attention_heads=heads,
            num_key_value_heads=cfg.get("num_key_value_heads", heads),
            head_dim=hd,
            vocab_size=cfg["vocab_size"],
            max_position_embeddings=cfg.get("max_position_embeddings", 8192),
            rms_norm_eps=cfg.get("rms_norm_eps", 1e-5),
            rope_theta=cfg.get("rope_theta", 10000.0),
            rope_scaling=cfg.get("rope_scaling"),
            tie_word_embeddings=cfg.get("tie_word_embeddings", False),
            qk_norm=mt in ("qwen3", "qwen3_moe", "olmo2", "olmo3", "gemma3_text") or mt in GDN_TYPES or cfg.get("use_qk_norm", False),
            sandwich_norm=gemma, norm_plus_one=gemma,
            hidden_act="gelu_tanh" if gemma or "gelu" in str(cfg.get("hidden_act", "")) else "silu",
            embed_scale=float(cfg["hidden_size"]) ** 0.5 if gemma else 1.0,
            query_pre_attn_scalar=float(cfg.get("query_pre_attn_scalar") or 0.0) if gemma else 0.0,
            attn_softcap=float(cfg.get("attn_logit_softcapping") or 0.0), final_softcap=float(cfg.get("final_logit_softcapping") or 0.0),
            rope_local_theta=float(cfg.get("rope_local_base_freq") or 0.0) if mt == "gemma3_text" else 0.0,
            post_norm=mt in POST_NORM,
            attention_bias=cfg.get("attention_bias", mt in ("qwen2", "gpt_oss", "qwen2_moe")),
            # Qwen2 gates the window on use_sliding_window; Mistral applies it whenever it is set
            sliding_window=(cfg.get("sliding_window") or -1)
            if cfg.get("use_sliding_window", mt in ("mistral", "gpt_oss", "olmo3") or gemma) else -1,
            # OLMo-3 and GPT-OSS alternate sliding-window and full-attention layers
            layer_types=cfg.get("layer_types") if mt in ("gpt_oss", "olmo3") or gemma or mt in GDN_TYPES or mt in MAMBA_TYPES else None,
            mamba_num_heads=cfg.get("mamba_num_heads", 0), mamba_head_dim=cfg.get("mamba_head_dim", 0),
            ssm_state_size=cfg.get("ssm_state_size", 0), mamba_n_groups=cfg.get("mamba_n_groups", 1),
            mamba_norm_grouped=bool(cfg.get("mamba_norm_grouped", False)),
            linear_num_key_heads=cfg.get("linear_num_key_heads", 0), linear_num_value_heads=cfg.get("linear_num_value_heads", 0),
            linear_key_head_dim=cfg.get("linear_key_head_dim", 0), linear_value_head_dim=cfg.get("linear_value_head_dim", 0),
            linear_conv_kernel_dim=cfg.get("linear_conv_kernel_dim", 4),
            attention_sinks=mt == "gpt_oss",
            o_bias=mt == "gpt_oss" and cfg.get("attention_bias", True),
            moe_style="gpt_oss" if mt == "gpt_oss" else "swiglu",
            swiglu_limit=float(cfg.get("swiglu_limit", 7.0)),
            num_experts=cfg.get("num_experts", cfg.get("num_local_experts", 0)) or 0,
            num_experts_per_tok=cfg.get("num_experts_per_tok", 0) or 0,
            # Mixtral has no separate field: its intermediate_size is the expert FFN width
            moe_intermediate_size=cfg.get("moe_intermediate_size", 0)
            or (cfg.get("intermediate_size", 0) if mt in ("mixtral", "gpt_oss") else 0),
            norm_topk_prob=cfg.get("norm_topk_prob", mt != "qwen2_moe"),
            shared_expert_intermediate_size=cfg.get("shared_expert_intermediate_size", 0) or 0,
            quantization=quant,
            dtype=str(cfg.get("torch_dtype") or cfg.get("dtype") or "bfloat16"),      # newer files say `dtype`
            name=name,
        )

    @staticmethod
    def from_path(path) -> "ModelConfig":
        p = Path(path)
        with open(p / "config.json") as f:
            return ModelConfig.from_hf(json.load(f), name=p.name)


def _puzutar_config(cfg: dict, name: str) -> ModelConfig:
    specs, ffs = [], []
    for i, layer in enumerate(cfg["layers"]):
        if layer["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        m, mlp = layer["mixer"], layer.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        rot = m["rot"]
        src = m.get("kv_from")
        s = LatentSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"],
                       window=m["mask"]["size"], scale=float(m["scale"]), rope_base=float(rot["base"]),
                       rot_dims=rot["dims"], kv_from=src)
        if s.rot_dims % 2 or s.rot_dims > s.rot_dim or s.window < 1:
            raise ValueError(f"layer {i}: rotation over {s.rot_dims} of {s.rot_dim} dimensions, window {s.window}")
        if src is not None:
            j = specs[src] if 0 <= src < i else None
            if j is None or j.kv_from is not None or (j.kv_rank, j.rot_dim) != (s.kv_rank, s.rot_dim):
                raise ValueError(f"layer {i}: kv_from {src} is not an earlier layer with a latent of the same sizes")
        specs.append(s)
        ffs.append(int(mlp["ff"]) if mlp else 0)
    if cfg["width"] % cfg["norm"]["groups"]:
        raise ValueError(f"width {cfg['width']} does not split into {cfg['norm']['groups']} norm groups")
    side = cfg.get("token_side") or {}
    return ModelConfig(
        model_type="puzutar", hidden_size=cfg["width"], intermediate_size=max(ffs), num_hidden_layers=len(specs),
        num_attention_heads=max(s.heads for s in specs), num_key_value_heads=1, head_dim=max(s.row for s in specs),
        vocab_size=cfg["vocab"], max_position_embeddings=cfg.get("max_position_embeddings", 131072),
        rms_norm_eps=cfg["norm"]["eps"], tie_word_embeddings=True, hidden_act="xielu", latent=specs, ff_sizes=ffs,
        norm_groups=cfg["norm"]["groups"], token_shift=True, token_side_dim=side.get("dim", 0), dtype="bfloat16", name=name)


def _puzutar_dict(cfg: ModelConfig) -> dict:
    """The `config.json` dictionary `_puzutar_config` reads `cfg` from."""
    layers = []
    for s, ff in zip(cfg.latent, cfg.ff_sizes):
        m = {"heads": s.heads, "dim": s.dim, "rot_dim": s.rot_dim, "vdim": s.vdim, "kv_rank": s.kv_rank, "scale": s.scale,
             "mask": {"size": s.window}, "rot": {"base": s.rope_base, "dims": s.rot_dims}}
        if s.kv_from is not None:
            m["kv_from"] = s.kv_from
        layers.append({"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None})
    return {"architecture": "Puzutar", "width": cfg.hidden_size, "vocab": cfg.vocab_size, "layers": layers,
            "norm": {"eps": cfg.rms_norm_eps, "groups": cfg.norm_groups}, "token_side": {"dim": cfg.token_side_dim}}


def puzutar_shape(layers: int = 32, width: int = 4096, heads: int = 32, dim: int = 96, rot_dim: int = 32, vdim: int = 128,
                  kv_rank: int = 256, window: int = 1024, ff: int = 21504, vocab: int = 128256, groups: int = 8,
                  side: int = 64, share: int = 2) -> dict:
    """config.json dictionary of a uniform model: of every `share` layers in a row the first keeps latents, the
    others read them."""
    spec = []
    for i in range(layers):
        m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=(dim + rot_dim) ** -0.5,
                 mask={"size": window}, rot={"base": 10000.0, "dims": rot_dim})
        if i % share:
            m["kv_from"] = i - i % share
        spec.append({"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff}})
    return {"architecture": "Puzutar", "width": width, "vocab": vocab, "layers": spec, "norm": {"eps": 1e-5, "groups": groups},
            "token_side": {"dim": side}}


def _is_fp8_weight_config(q: dict) -> bool:
    """`quantization_config` of an 8-bit float weight checkpoint without block scales: `fp8` / `fbgemm_fp8`, or
    compressed-tensors groups whose weights are 8-bit floats with a tensor or channel strategy."""
    method = q.get("quant_method")
    if method in ("fp8", "fbgemm_fp8"):
        return True
    if method == "compressed-tensors":
        groups = (q.get("config_groups") or {}).values()
        ws = [g.get("weights") or {} for g in groups]
        return bool(ws) and all(w.get("type") == "float" and w.get("num_bits") == 8 and w.get("strategy") in ("tensor", "channel")
                                for w in ws)
    return False


def _flatten_rope_parameters(cfg: dict) -> dict:
    """Newer `config.json` files carry RoPE settings as `rope_parameters`: one dict (`rope_theta`, `rope_type`,
    scaling fields), or one such dict per layer type. Rewrites them as the older `rope_theta` / `rope_scaling` /
    `rope_local_base_freq` keys, which win when both are present."""
    rp = cfg.get("rope_parameters")
    if not isinstance(rp, dict):
        return cfg
    local = None
    if "full_attention" in rp or "sliding_attention" in rp:
        local = rp.get("sliding_attention")
        rp = rp.get("full_attention") or local or {}
    if "rope_theta" in rp:
        cfg.setdefault("rope_theta", rp["rope_theta"])
    if rp.get("rope_type", "default") != "default" and not cfg.get("rope_scaling"):
        cfg["rope_scaling"] = {k: v for k, v in rp.items() if k != "rope_theta"}
    if local and "rope_theta" in local:
        cfg.setdefault("rope_local_base_freq", local["rope_theta"])
    return cfg


# Architectures named by the benchmark configurations (random-init weights of these shapes).
PRESETS = {
    "tiny-llama": dict(model_type="llama", hidden_size=256, intermediate_size=688, num_hidden_layers=2,
                       num_attention_heads=4, num_key_value_heads=2, head_dim=64, vocab_size=32000,
                       rope_theta=10000.0, rms_norm_eps=1e-5, dtype="float32"),
    "llama-3.1-8b": dict(model_type="llama", hidden_size=4096, intermediate_size=14336,
                         num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=8,
                         head_dim=128, vocab_size=128256, rope_theta=500000.0, rms_norm_eps=1e-5),
    # the 8B shape with a sliding window: what `puzutar-8b` is measured beside
    "llama-8b-window": dict(model_type="mistral", hidden_size=4096, intermediate_size=14336, num_hidden_layers=32,
                            num_attention_heads=32, num_key_value_heads=8, head_dim=128, vocab_size=128256,
                            rope_theta=500000.0, rms_norm_eps=1e-5, sliding_window=1024),
    # Gated DeltaNet and windowed attention with experts, layer about: what `retodra-19b` is measured beside
    "gdn-moe-window-19b": dict(model_type="qwen3_next", hidden_size=4096, intermediate_size=11008, num_hidden_layers=32,
                               num_attention_heads=32, num_key_value_heads=8, head_dim=128, vocab_size=128256, rope_theta=500000.0,
                               rms_norm_eps=1e-5, qk_norm=True, sliding_window=1024,
                               layer_types=["linear_attention", "sliding_attention"] * 16, linear_num_key_heads=16,
                               linear_num_value_heads=32, linear_key_head_dim=128, linear_value_head_dim=128, num_experts=32,
                               num_experts_per_tok=4, moe_intermediate_size=2048),
    # attention over everything and Gated DeltaNet with states of the same size, layer about, feed-forwards widened to the same
    # parameters: what `vulanex-8b` is measured beside
    "gdn-8b": dict(model_type="qwen3_next", hidden_size=4096, intermediate_size=13952, num_hidden_layers=32, num_attention_heads=32,
                   num_key_value_heads=8, head_dim=128, vocab_size=128256, rope_theta=500000.0, rms_norm_eps=1e-5, qk_norm=True,
                   layer_types=["full_attention", "linear_attention"] * 16, linear_num_key_heads=16, linear_num_value_heads=32,
                   linear_key_head_dim=128, linear_value_head_dim=128),
    "qwen3-32b": dict(model_type="qwen3", hidden_size=5120, intermediate_size=25600,
                      num_hidden_layers=64, num_attention_heads=64, num_key_value_heads=8, head_dim=128,
                      vocab_size=151936, rope_theta=1000000.0, rms_norm_eps=1e-6, qk_norm=True),
    "qwen3-32b-fp8": dict(model_type="qwen3", hidden_size=5120, intermediate_size=25600,
                          num_hidden_layers=64, num_attention_heads=64, num_key_value_heads=8,
                          head_dim=128, vocab_size=151936, rope_theta=1000000.0, rms_norm_eps=1e-6,
                          qk_norm=True, quantization="fp8_block"),
    "qwen3-30b-a3b": dict(model_type="qwen3_moe", hidden_size=2048, intermediate_size=6144,
                          num_hidden_layers=48, num_attention_heads=32, num_key_value_heads=4,
                          head_dim=128, vocab_size=151936, rope_theta=1000000.0, rms_norm_eps=1e-6,
                          qk_norm=True, num_experts=128, num_experts_per_tok=8,
                          moe_intermediate_size=768, norm_topk_prob=True),
    "qwen3-0.6b": dict(model_type="qwen3", hidden_size=1024, intermediate_size=3072,
                       num_hidden_layers=28, num_attention_heads=16, num_key_value_heads=8, head_dim=128,
                       vocab_size=151936, rope_theta=1000000.0, rms_norm_eps=1e-6, qk_norm=True,
                       tie_word_embeddings=True),
    "olmo-2-7b": dict(model_type="olmo2", hidden_size=4096, intermediate_size=11008, num_hidden_layers=32,
                      num_attention_heads=32, num_key_value_heads=32, head_dim=128, vocab_size=100352,
                      rope_theta=500000.0, rms_norm_eps=1e-6, qk_norm=True, post_norm=True),
    "tiny-olmo2": dict(model_type="olmo2", hidden_size=256, intermediate_size=688, num_hidden_layers=2,
                       num_attention_heads=4, num_key_value_heads=2, head_dim=64, vocab_size=32000,
                       rope_theta=10000.0, rms_norm_eps=1e-6, qk_norm=True, post_norm=True, dtype="float32"),
    "gpt-oss-20b": dict(model_type="gpt_oss", hidden_size=2880, intermediate_size=2880, num_hidden_layers=24,
                        num_attention_heads=64, num_key_value_heads=8, head_dim=64, vocab_size=201088,
                        rope_theta=150000.0, rms_norm_eps=1e-5, attention_bias=True, o_bias=True, attention_sinks=True,
                        sliding_window=128, layer_types=["sliding_attention", "full_attention"] * 12,
                        num_experts=32, num_experts_per_tok=4, moe_intermediate_size=2880, moe_style="gpt_oss",
                        rope_scaling=dict(rope_type="yarn", factor=32.0, beta_fast=32.0, beta_slow=1.0,
                                          original_max_position_embeddings=4096, truncate=False)),
    "tiny-gpt-oss": dict(model_type="gpt_oss", hidden_size=256, intermediate_size=128, num_hidden_layers=2,
                         num_attention_heads=4, num_key_value_heads=2, head_dim=64, vocab_size=32000,
                         rope_theta=10000.0, rms_norm_eps=1e-5, attention_bias=True, o_bias=True,
                         attention_sinks=True, sliding_window=20, layer_types=["sliding_attention", "full_attention"],
                         num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128, moe_style="gpt_oss",
                         rope_scaling=dict(rope_type="yarn", factor=4.0, beta_fast=32.0, beta_slow=1.0,
                                           original_max_position_embeddings=64, truncate=False), dtype="float32"),
    "tiny-qwen3.5": dict(model_type="qwen3_5", hidden_size=256, intermediate_size=512, num_hidden_layers=4,
                         num_attention_heads=4, num_key_value_heads=2, head_dim=64, vocab_size=32000, qk_norm=True,
                         rope_theta=1e6, layer_types=["linear_attention", "linear_attention", "linear_attention", "full_attention"],
                         linear_num_key_heads=2, linear_num_value_heads=4, linear_key_head_dim=32, linear_value_head_dim=32),
    "tiny-mamba2": dict(model_type="mamba2_hybrid", hidden_size=256, intermediate_size=512, num_hidden_layers=3,
                        num_attention_heads=4, num_key_value_heads=2, head_dim=64, vocab_size=32000,
                        layer_types=["mamba2", "mamba2", "full_attention"], mamba_num_heads=8, mamba_head_dim=32,
                        ssm_state_size=16, mamba_n_groups=2),
    "gemma-3-27b": dict(model_type="gemma3_text", hidden_size=5376, intermediate_size=21504, num_hidden_layers=62,
                        num_attention_heads=32, num_key_value_heads=16, head_dim=128, vocab_size=262208,
                        rope_theta=1e6, rope_scaling=dict(rope_type="linear", factor=8.0), rope_local_theta=10000.0,
                        rms_norm_eps=1e-6, qk_norm=True, sandwich_norm=True, norm_plus_one=True, hidden_act="gelu_tanh",
                        embed_scale=5376 ** 0.5, query_pre_attn_scalar=168.0, sliding_window=1024, tie_word_embeddings=True,
                        layer_types=(["sliding_attention"] * 5 + ["full_attention"]) * 10 + ["sliding_attention"] * 2),
    "tiny-gemma3": dict(model_type="gemma3_text", hidden_size=256, intermediate_size=512, num_hidden_layers=3,
                        num_attention_heads=4, num_key_value_heads=2, head_dim=64, vocab_size=32000, rope_theta=1e6,
                        rope_scaling=dict(rope_type="linear", factor=8.0), rope_local_theta=10000.0, rms_norm_eps=1e-6,
                        qk_norm=True, sandwich_norm=True, norm_plus_one=True, hidden_act="gelu_tanh", embed_scale=16.0,
                        query_pre_attn_scalar=48.0, sliding_window=8, tie_word_embeddings=True,
                        layer_types=["sliding_attention", "sliding_attention", "full_attention"], dtype="float32"),
    "tiny-gemma2": dict(model_type="gemma2", hidden_size=256, intermediate_size=512, num_hidden_layers=2,
                        num_attention_heads=4, num_key_value_heads=2, head_dim=64, vocab_size=32000, rope_theta=10000.0,
                        rms_norm_eps=1e-6, sandwich_norm=True, norm_plus_one=True, hidden_act="gelu_tanh", embed_scale=16.0,
                        query_pre_attn_scalar=48.0, sliding_window=8, tie_word_embeddings=True, attn_softcap=50.0,
                        final_softcap=30.0, layer_types=["sliding_attention", "full_attention"], dtype="float32"),
    "tiny-qwen2-moe": dict(model_type="qwen2_moe", hidden_size=256, intermediate_size=512, num_hidden_layers=2,
                           num_attention_heads=4, num_key_value_heads=2, head_dim=64, vocab_size=32000, rope_theta=10000.0,
                           rms_norm_eps=1e-6, attention_bias=True, num_experts=8, num_experts_per_tok=2,
                           moe_intermediate_size=128, norm_topk_prob=False, shared_expert_intermediate_size=192, dtype="float32"),
    "tiny-qwen3-moe": dict(model_type="qwen3_moe", hidden_size=256, intermediate_size=512,
                           num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, head_dim=64,
                           vocab_size=32000, rope_theta=10000.0, rms_norm_eps=1e-6, qk_norm=True,
                           num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128,
                           dtype="float32"),
}

# presets of designs whose layers are described one by one: reader, shape and the shape's arguments
LAYERED_PRESETS = {
    "puzutar-8b": (_puzutar_config, puzutar_shape, dict()),
    "retodra-19b": (retodra_config, retodra_shape, dict()),
    "nukelix-20b": (nukelix_config, nukelix_shape, dict()),
    # parallel mixers and experts only: what `nukelix-20b` is measured beside (a fifth route for the shared expert)
    "retodra-parallel-20b": (retodra_config, retodra_shape, dict(layers=24, linear_every=0, right_vdim=256, identity=0, top=5)),
    "tiny-puzutar": (_puzutar_config, puzutar_shape, dict(
        layers=3, width=256, heads=2, dim=48, rot_dim=16, vdim=40, kv_rank=64, window=40, ff=384, vocab=32000, groups=2, side=16)),
    "tiny-retodra": (retodra_config, retodra_shape, dict(
        layers=4, width=256, gla_heads=2, gla_dim=48, gla_vdim=64, rank=8, heads=6, kv_heads=2, dim=40, window=50, buckets=12,
        right_heads=3, right_dim=32, right_vdim=40, ff=384, experts=6, identity=2, top=3, expert_ff=96, vocab=32000)),
    "vulanex-8b": (vulanex_config, vulanex_shape, dict()),
    "tiny-vulanex": (vulanex_config, vulanex_shape, dict(
        layers=4, width=256, heads=6, kv_heads=2, dim=40, vdim=56, window=50, pool=12, every=20, right_heads=3, right_dim=32, rank=8, ff=384,
        vocab=32000, buckets=509, taps=3)),
    "tiny-nukelix": (nukelix_config, nukelix_shape, dict(
        layers=4, width=256, heads=6, kv_heads=2, dim=40, window=50, keep_first=3, right_heads=3, right_dim=32, right_vdim=40, lat_heads=4,
        lat_dim=24, rot_dim=8, q_rank=72, kv_rank=48, ff=96, experts=6, top=2, shared=112, vocab=32000)),
}


def preset(name: str, **overrides) -> ModelConfig:
    if name in LAYERED_PRESETS:
        read, build, args = LAYERED_PRESETS[name]
        if "num_hidden_layers" in overrides:
            args = dict(args, layers=overrides.pop("num_hidden_layers"))
        cfg = read(build(**args), name)
        for k, v in overrides.items():
            setattr(cfg, k, v)
        return cfg
    if name not in PRESETS:
        raise KeyError(f"unknown model preset {name!r}; known: {sorted(list(PRESETS) + list(LAYERED_PRESETS))}")
    kw = dict(PRESETS[name])
    kw.update(overrides)
    return ModelConfig(name=name, **kw)
