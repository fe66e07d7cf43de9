"""Descriptions of layers that a configuration lists one by one (blocks over a 32-bit residual stream): each block names
its mixer and its feed-forward, with sizes and constants of its own. The Retodra reader and writer of `config.json` are at
the end, those of Nukelix in `nukelix.py`, those of Vulanex in `vulanex.py`.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Union


EVERYTHING = 1 << 30            # a window no context fills: every earlier token is visible


def _pad(n: int, m: int = 8) -> int:
    return -(-n // m) * m


@dataclass
class RotarySpec:
    """Rotary positions on the first `dims` dimensions: pairs are neighbours (`adjacent`) or half of `dims` apart. `scaling`:
    a `rope_scaling` dictionary (`ops.reference.rope_inv_freq`); "yarn" also multiplies cos and sin."""
    dims: int
    base: float
    adjacent: bool = False
    scaling: Optional[dict] = None

    @property
    def factor(self) -> float:
        s = self.scaling
        return 0.1 * math.log(s["factor"]) + 1.0 if s and s["rope_type"] == "yarn" else 1.0

    def frequencies(self, device="cpu"):
        """Angle per position of every pair, 32-bit [dims / 2]."""
        from ..ops import reference
        return reference.rope_inv_freq(self.dims, self.base, self.scaling, device)


@dataclass
class LatentSpec:
    """Sizes of one latent-attention mixer: per head `dim` unrotated and `rot_dim` rotated query / key dimensions
    (the first `rot_dims` of the latter rotate) and `vdim` value dimensions; keys and values are projections of a
    latent of `kv_rank` numbers per token, which is cached together with one rotated key part shared by all heads.
    A query sees itself and the `window` - 1 tokens before it. `kv_from`: the layer whose cache this one reads.
    `q_rank`: queries are projections of a normed latent of their own. `head_gate`: each head's output is scaled by a
    sigmoid of the mixer's input. The rotation is `RotarySpec`'s."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    window: int
    scale: float
    rope_base: float
    rot_dims: int
    kv_from: Optional[int] = None
    q_rank: Optional[int] = None
    head_gate: bool = False
    rot_adjacent: bool = False
    rot_scaling: Optional[dict] = None

    @property
    def rotary(self) -> RotarySpec:
        return RotarySpec(self.rot_dims, self.rope_base, self.rot_adjacent, self.rot_scaling)

    @property
    def qk_dim(self) -> int:
        return self.dim + self.rot_dim

    @property
    def rank_pad(self) -> int:
        """Columns of the latent inside a cache row: a multiple of 16 (one tensor-core k step)."""
        return _pad(self.kv_rank, 16)

    @property
    def row(self) -> int:
        """Columns of a cache row: latent, then the rotated key part, each padded with zeros."""
        return self.rank_pad + _pad(self.rot_dim, 16)

    @property
    def q_rows(self) -> int:
        return self.heads * self.qk_dim

    @property
    def proj_rows(self) -> int:
        """Rows of the fused query (+ latent and shared key, unless the layer borrows another's cache) projection."""
        return self.q_rows + (self.kv_rank + self.rot_dim if self.kv_from is None else 0)


@dataclass
class GatedLinearSpec:
    """Gated linear attention: a state [dim, vdim] per head whose rows decay by sigmoid(z)^(1 / tau), z a projection of
    rank `rank` (None: the checkpoint tells)."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: Optional[int] = None

    @property
    def qk(self) -> int:
        return self.heads * self.dim

    @property
    def values(self) -> int:
        return self.heads * self.vdim

    @property
    def state_elems(self) -> int:
        return self.heads * self.dim * self.vdim


@dataclass
class LightningSpec:
    """Linear attention with one constant decay per head."""
    heads: int
    dim: int
    vdim: int
    decay: List[float]

    qk = GatedLinearSpec.qk
    values = GatedLinearSpec.values
    state_elems = GatedLinearSpec.state_elems


@dataclass
class BiasedAttentionSpec:
    """Grouped-query attention without rotation: soft-capped scores plus a learned bias per distance bucket (`buckets`
    rows, None: the checkpoint tells; logarithmic up to `bias_max`), over the query itself and the `window` - 1 tokens
    before it."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    scale: float
    softcap: float
    bias_max: int
    buckets: Optional[int] = None

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads

    @property
    def group_pad(self) -> int:
        """Query heads per key / value head the kernels compute: the next power of two (the added ones are zeros)."""
        return 1 << (self.group - 1).bit_length()

    @property
    def head_dim(self) -> int:
        """Columns of a cached key or value and of a query row, zeros past dim / vdim."""
        need = max(self.dim, self.vdim)
        return 64 if need <= 64 else 128 if need <= 128 else -(-need // 128) * 128

    def bucket(self, n: int) -> int:
        """Bias row of the distance n: a row each for the first half, then logarithmic."""
        half = self.buckets // 2
        if n < half:
            return n
        far = math.log(n / half) / math.log(self.bias_max / half) * (self.buckets - half)
        return min(self.buckets - 1, half + math.floor(far + 1e-9))     # a distance on a bucket's edge stays on it


@dataclass
class GroupedAttentionSpec:
    """Grouped-query attention with biased projections, q and k normed over all heads together, rotary positions and one
    sigmoid gate per head. A query sees itself, the `window` - 1 tokens before it and the first `keep_first` tokens. `sink`:
    a score of 0 without a value takes its share of the softmax. `v_mix`: the values are mixed with those of the first layer
    that has the flag."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotarySpec
    window: int = EVERYTHING
    keep_first: int = 0
    sink: bool = False
    v_mix: bool = False

    group = BiasedAttentionSpec.group
    group_pad = BiasedAttentionSpec.group_pad
    head_dim = BiasedAttentionSpec.head_dim


@dataclass
class MatrixMemorySpec:
    """Matrix memory with exponential input and forget gates (the mLSTM of xLSTM): per head a state [dim, vdim], a
    normaliser [dim] and a running maximum of the gates' logarithms; `gate_cap` limits the gates softly."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    qk = GatedLinearSpec.qk
    values = GatedLinearSpec.values

    @property
    def state_elems(self) -> int:
        """The states of all heads, then the normalisers, then the maxima."""
        return self.heads * (self.dim * self.vdim + self.dim + 1)


@dataclass
class PlainAttentionSpec:
    """Grouped-query attention without biases or gates; the rest is optional. `head_norm`: q and k are normed head by head.
    `rot`: rotary positions. `q_temp` (coef, every): the query at position p is multiplied by 1 + coef * ln(floor((p + 1) /
    every) + 1). `shared_kv`: the values are the keys, cached once. A query sees itself, the `window` - 1 tokens before it and,
    with `pool`, the mean key and value of every block of that many tokens wholly before the window. `sink`: a learned score
    per head without a value takes its share of the softmax."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotarySpec] = None
    head_norm: bool = False
    q_temp: Optional[Tuple[float, int]] = None
    shared_kv: bool = False
    window: int = EVERYTHING
    pool: int = 0
    sink: bool = False

    group = BiasedAttentionSpec.group
    group_pad = BiasedAttentionSpec.group_pad
    head_dim = BiasedAttentionSpec.head_dim

    @property
    def planes(self) -> int:
        """Rows a page holds per token and head: a key and a value, or one for both."""
        return 1 if self.shared_kv else 2


@dataclass
class DeltaRuleSpec:
    """Delta rule with a decay and a removal rate per key channel: a state [dim, dim] per head. The decay lies between
    exp(-`bound`) and 1; it is a projection of rank `rank` (None: the checkpoint tells)."""
    heads: int
    dim: int
    rank: Optional[int] = None
    bound: float = math.exp(-0.5)

    qk = GatedLinearSpec.qk

    @property
    def vdim(self) -> int:
        return self.dim

    @property
    def values(self) -> int:
        return self.heads * self.dim

    @property
    def state_elems(self) -> int:
        return self.heads * self.dim * self.dim


@dataclass
class ParallelSpec:
    """Attention and a recurrent mixer side by side on the same input. `out_norms`: each side's output projection is normed
    before the sum."""
    left: Union[BiasedAttentionSpec, GroupedAttentionSpec, PlainAttentionSpec]
    right: Union[LightningSpec, MatrixMemorySpec, DeltaRuleSpec]
    left_scale: float
    right_scale: float
    out_norms: bool = False


@dataclass
class PairSpec:
    """An embedding row for the pair (token before, token): number (before * mul_prev + token * mul_cur) mod buckets, and one
    more row for a sequence's first token."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class DenseSpec:
    """GLU feed-forward of width `ff`; `act`: activation of the gate ("silu" | "gelu_tanh")."""
    ff: int
    act: str = "silu"


@dataclass
class ExpertsSpec:
    """`experts` GLU experts of width `ff` and `identity` more router outputs whose expert returns its input. Scores are a
    softmax plus a correction for the choice, or ("sigmoid") the sigmoid of each output. `weight_input`: an expert's weight
    scales what it reads instead of what it returns. `limit`: clamped GLU, None: SwiGLU. `shared`: width of a SwiGLU expert
    that every token uses (0: none)."""
    experts: int
    identity: int
    top: int
    ff: int
    limit: Optional[float] = None
    score: str = "softmax"
    weight_input: bool = False
    shared: int = 0

    @property
    def outputs(self) -> int:
        return self.experts + self.identity


@dataclass
class BlockSpec:
    mixer: Union[GatedLinearSpec, ParallelSpec, GroupedAttentionSpec, PlainAttentionSpec, LatentSpec]
    ff: Union[DenseSpec, ExpertsSpec, None]

    @property
    def attention(self) -> Union[BiasedAttentionSpec, GroupedAttentionSpec, PlainAttentionSpec, None]:
        """The part of the mixer that keeps keys and values in pages."""
        a = self.mixer.left if isinstance(self.mixer, ParallelSpec) else self.mixer
        return a if isinstance(a, (BiasedAttentionSpec, GroupedAttentionSpec, PlainAttentionSpec)) else None

    @property
    def latent(self) -> Optional[LatentSpec]:
        return self.mixer if isinstance(self.mixer, LatentSpec) else None

    @property
    def recurrent(self) -> Union[GatedLinearSpec, LightningSpec, MatrixMemorySpec, DeltaRuleSpec, None]:
        """The part of the mixer whose state is carried from token to token."""
        r = self.mixer.right if isinstance(self.mixer, ParallelSpec) else self.mixer
        return r if isinstance(r, (GatedLinearSpec, LightningSpec, MatrixMemorySpec, DeltaRuleSpec)) else None


def projection_sizes(mixer) -> Dict[str, int]:
    """Checkpoint name (within the mixer) -> rows of the projections of its input that run as one product, in order."""
    if isinstance(mixer, GatedLinearSpec):
        return {"q": mixer.qk, "k": mixer.qk, "v": mixer.values, "g": mixer.values, "a1": mixer.rank}
    if isinstance(mixer, LatentSpec):
        return {"dq": mixer.q_rank, "dkv": mixer.kv_rank + mixer.rot_dim, "g": mixer.heads}
    if isinstance(mixer, ParallelSpec):
        return {f"{side}.{n}": k for side, part in (("left", mixer.left), ("right", mixer.right)) for n, k in projection_sizes(part).items()}
    if isinstance(mixer, (LightningSpec, MatrixMemorySpec)):
        return {"q": mixer.qk, "k": mixer.qk, "v": mixer.values, "g": mixer.values}
    if isinstance(mixer, DeltaRuleSpec):
        return {"r": mixer.qk, "k": mixer.qk, "v": mixer.values, "g": mixer.values, "a": mixer.qk, "w1": mixer.rank}
    if isinstance(mixer, PlainAttentionSpec):
        rows = {"q": mixer.heads * mixer.dim, "k": mixer.kv_heads * mixer.dim}
        return rows if mixer.shared_kv else {**rows, "v": mixer.kv_heads * mixer.vdim}
    gates = mixer.heads if isinstance(mixer, GroupedAttentionSpec) else mixer.heads * mixer.vdim
    return {"q": mixer.heads * mixer.dim, "k": mixer.kv_heads * mixer.dim, "v": mixer.kv_heads * mixer.vdim, "g": gates}


def projection_columns(mixer) -> Dict[str, Tuple[int, int]]:
    """Name -> (first column, columns) of the mixer's fused input projection; every part starts on a multiple of 8."""
    out, at = {}, 0
    for name, n in projection_sizes(mixer).items():
        out[name] = (at, n)
        at += _pad(n)
    return out


# ------------------------------------------------------------------ Retodra
def _retodra_mixer(i: int, kind: str, m: dict):
    if kind == "gla":
        return GatedLinearSpec(m["heads"], m["dim"], m["vdim"], float(m["tau"]), m.get("rank"))
    if kind != "parallel":
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    a, b = m["left"], m["right"]
    left = BiasedAttentionSpec(a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["mask"]["size"], float(a["scale"]),
                               float(a["softcap"]), a["bias_max"], a.get("buckets"))
    right = LightningSpec(b["heads"], b["dim"], b["vdim"], [float(x) for x in b["decay"]])
    if left.heads % left.kv_heads or left.window < 1 or left.softcap <= 0:
        raise ValueError(f"layer {i}: {left.heads} query heads on {left.kv_heads}, window {left.window}, soft cap {left.softcap}")
    if len(right.decay) != right.heads or not all(0 < x <= 1 for x in right.decay):
        raise ValueError(f"layer {i}: decays {right.decay} for {right.heads} heads")
    return ParallelSpec(left, right, float(m["left_scale"]), float(m["right_scale"]))


def _retodra_ff(i: int, mlp: Optional[dict]):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return DenseSpec(mlp["ff"])
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    r, e = mlp["router"], mlp["expert"]
    s = ExpertsSpec(r["experts"], r.get("identity", 0), r["top"], e["ff"], float(e["limit"]))
    if not 1 <= s.top <= s.outputs:
        raise ValueError(f"layer {i}: {s.top} of {s.outputs} router outputs")
    return s


def retodra_config(cfg: dict, name: str):
    from .config import ModelConfig
    blocks = [BlockSpec(_retodra_mixer(i, x["type"], x["mixer"]), _retodra_ff(i, x.get("mlp"))) for i, x in enumerate(cfg["layers"])]
    att = [b.attention for b in blocks if b.attention is not None]
    ffs = [b.ff.ff for b in blocks if b.ff is not None]
    return ModelConfig(
        model_type="retodra", hidden_size=cfg["width"], intermediate_size=max(ffs, default=0), num_hidden_layers=len(blocks),
        num_attention_heads=max((a.kv_heads * a.group_pad for a in att), default=1),
        num_key_value_heads=max((a.kv_heads for a in att), default=1), head_dim=max((a.head_dim for a in att), default=64),
        vocab_size=cfg["vocab"], max_position_embeddings=cfg.get("max_position_embeddings", 131072),
        rms_norm_eps=cfg["norm"]["eps"], tie_word_embeddings=False, embed_scale=float(cfg["embedding"]["scale"]),
        norm_plus_one=True, sandwich_norm=True, blocks=blocks, dtype="bfloat16", name=name)


def retodra_dict(cfg) -> dict:
    """The `config.json` dictionary `retodra_config` reads `cfg` from."""
    layers = []
    for b in cfg.blocks:
        m = b.mixer
        if isinstance(m, GatedLinearSpec):
            d = {"type": "gla", "mixer": {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau}}
        else:
            a, r = m.left, m.right
            d = {"type": "parallel", "mixer": {
                "left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "mask": {"size": a.window},
                         "scale": a.scale, "softcap": a.softcap, "bias_max": a.bias_max},
                "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay)},
                "left_scale": m.left_scale, "right_scale": m.right_scale}}
        f = b.ff
        if f is None:
            d["mlp"] = None
        elif isinstance(f, DenseSpec):
            d["mlp"] = {"kind": "dense", "ff": f.ff}
        else:
            d["mlp"] = {"kind": "moe", "expert": {"ff": f.ff, "limit": f.limit},
                        "router": {"experts": f.experts, "identity": f.identity, "top": f.top}}
        layers.append(d)
    return {"architecture": "Retodra", "width": cfg.hidden_size, "vocab": cfg.vocab_size, "layers": layers,
            "norm": {"eps": cfg.rms_norm_eps}, "embedding": {"scale": cfg.embed_scale}}


def retodra_shape(layers: int = 32, width: int = 4096, gla_heads: int = 16, gla_dim: int = 128, gla_vdim: int = 256, rank: int = 16,
                  tau: float = 16.0, heads: int = 32, kv_heads: int = 8, dim: int = 128, window: int = 1024, buckets: int = 32,
                  right_heads: int = 16, right_dim: int = 128, right_vdim: int = 128, ff: int = 11008, experts: int = 32,
                  identity: int = 4, top: int = 4, expert_ff: int = 2048, vocab: int = 128256, linear_every: int = 2) -> dict:
    """config.json dictionary of a model of parallel mixers with experts, every `linear_every`-th layer (0: none) gated linear
    attention with a dense feed-forward instead."""
    spec = []
    decay = [math.exp(-2.0 ** (-8.0 * (h + 1) / right_heads)) for h in range(right_heads)]
    for i in range(layers):
        if linear_every and i % linear_every == 0:
            spec.append({"type": "gla", "mixer": {"heads": gla_heads, "dim": gla_dim, "vdim": gla_vdim, "tau": tau, "rank": rank},
                         "mlp": {"kind": "dense", "ff": ff}})
        else:
            left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": window}, "scale": dim ** -0.5,
                    "softcap": 30.0, "bias_max": 2 * window, "buckets": buckets}
            right = {"heads": right_heads, "dim": right_dim, "vdim": right_vdim, "decay": decay}
            spec.append({"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": 0.75, "right_scale": 0.6},
                         "mlp": {"kind": "moe", "expert": {"ff": expert_ff, "limit": 7.0},
                                 "router": {"experts": experts, "identity": identity, "top": top}}})
    return {"architecture": "Retodra", "width": width, "vocab": vocab, "layers": spec, "norm": {"eps": 1e-5},
            "embedding": {"scale": float(width) ** 0.5}}
