"""The Vulanex reader and writer of `config.json`: pre-normed blocks over a 32-bit residual stream that read it through a layer
norm and a short convolution, with attention whose values are its keys, or pooled windowed attention beside a delta rule.
"""
from __future__ import annotations

from .block_spec import BlockSpec, DeltaRuleSpec, DenseSpec, PairSpec, ParallelSpec, PlainAttentionSpec, RotarySpec
from .nukelix import _YARN, _scaling, _scaling_dict


def _grouping(i: int, s: PlainAttentionSpec) -> PlainAttentionSpec:
    if s.kv_heads < 1 or s.heads % s.kv_heads:
        raise ValueError(f"layer {i}: {s.heads} query heads on {s.kv_heads}")
    return s


def _attention(i: int, m: dict) -> PlainAttentionSpec:
    t = m.get("q_temp")
    s = PlainAttentionSpec(m["heads"], m["kv_heads"], m["dim"], m.get("vdim", m["dim"]), float(m["scale"]),
                           q_temp=(float(t["coef"]), int(t["every"])) if t else None, shared_kv=True)
    if s.dim != s.vdim or (s.q_temp and s.q_temp[1] < 1):
        raise ValueError(f"layer {i}: keys of {s.dim} as values of {s.vdim}, query factor {t}")
    return _grouping(i, s)


def _pooled(i: int, m: dict) -> PlainAttentionSpec:
    rot, mask = m["rot"], m["mask"]
    s = PlainAttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]),
                           RotarySpec(rot["dims"], float(rot["base"]), False, _scaling(rot, "yarn", _YARN)), head_norm=True,
                           window=mask["size"], pool=mask["pool"], sink=True)
    if s.window < 1 or s.pool < 1 or s.rot.dims % 2 or s.rot.dims > s.dim:
        raise ValueError(f"layer {i}: window {s.window} beside blocks of {s.pool}, rotation over {s.rot.dims} of {s.dim} dimensions")
    return _grouping(i, s)


def _mixer(i: int, kind: str, m: dict):
    if kind == "attention":
        return _attention(i, m)
    if kind != "parallel":
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    r = m["right"]
    return ParallelSpec(_pooled(i, m["left"]), DeltaRuleSpec(r["heads"], r["dim"], r.get("rank")), 0.5, 0.5, out_norms=True)


def _ff(i: int, mlp):
    if mlp is None:
        return None
    if mlp["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    return DenseSpec(mlp["ff"], "gelu_tanh")


def vulanex_config(cfg: dict, name: str):
    from .config import ModelConfig
    blocks = [BlockSpec(_mixer(i, x["type"], x["mixer"]), _ff(i, x.get("mlp"))) for i, x in enumerate(cfg["layers"])]
    att = [b.attention for b in blocks]
    pair = cfg["embedding"]["bigram"]
    if cfg["canon"]["taps"] < 1 or pair["buckets"] < 1:
        raise ValueError(f"{cfg['canon']['taps']} taps, {pair['buckets']} pair rows")
    return ModelConfig(
        model_type="vulanex", hidden_size=cfg["width"], intermediate_size=max((b.ff.ff for b in blocks if b.ff is not None), default=0),
        num_hidden_layers=len(blocks), num_attention_heads=max(a.kv_heads * a.group_pad for a in att),
        num_key_value_heads=max(a.kv_heads for a in att), head_dim=max(a.head_dim for a in att), vocab_size=cfg["vocab"],
        max_position_embeddings=cfg.get("max_position_embeddings", 131072), rms_norm_eps=cfg["norm"]["eps"], tie_word_embeddings=True,
        hidden_act="gelu_tanh", layer_norm=True, conv_taps=cfg["canon"]["taps"], logit_scale=float(cfg["logit_scale"]),
        token_pairs=PairSpec(pair["buckets"], pair["mul_prev"], pair["mul_cur"]), blocks=blocks, dtype="bfloat16", name=name)


def vulanex_dict(cfg) -> dict:
    """The `config.json` dictionary `vulanex_config` reads `cfg` from."""
    layers = []
    for b in cfg.blocks:
        a = b.attention
        d = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
        if isinstance(b.mixer, ParallelSpec):
            d["rot"] = {"dims": a.rot.dims, "base": a.rot.base, **_scaling_dict(a.rot.scaling, _YARN)}
            d["mask"] = {"size": a.window, "pool": a.pool}
            x = {"type": "parallel", "mixer": {"left": d, "right": {"heads": b.mixer.right.heads, "dim": b.mixer.right.dim}}}
        else:
            if a.q_temp:
                d["q_temp"] = {"coef": a.q_temp[0], "every": a.q_temp[1]}
            x = {"type": "attention", "mixer": d}
        x["mlp"] = None if b.ff is None else {"kind": "dense", "ff": b.ff.ff}
        layers.append(x)
    pair = cfg.token_pairs
    return {"architecture": "Vulanex", "width": cfg.hidden_size, "vocab": cfg.vocab_size, "layers": layers, "norm": {"eps": cfg.rms_norm_eps},
            "canon": {"taps": cfg.conv_taps}, "logit_scale": cfg.logit_scale,
            "embedding": {"bigram": {"buckets": pair.buckets, "mul_prev": pair.mul_prev, "mul_cur": pair.mul_cur}}}


def vulanex_shape(layers: int = 32, width: int = 4096, heads: int = 32, kv_heads: int = 8, dim: int = 128, window: int = 1024, pool: int = 16,
                  every: int = 8192, right_heads: int = 32, right_dim: int = 128, rank: int = 64, ff: int = 11008, vocab: int = 128256,
                  buckets: int = 65537, taps: int = 4, parallel_every: int = 2, vdim: int = 0) -> dict:
    """config.json dictionary of a model whose layers alternate between attention over everything and the two mixers side by
    side (in every `parallel_every`-th layer; 1: in all)."""
    size = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim or dim, "scale": dim ** -0.5}
    att = {**size, "vdim": dim, "q_temp": {"coef": 0.1, "every": every}}
    left = {**size, "mask": {"size": window, "pool": pool},
            "rot": {"dims": dim, "base": 500000.0, "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}
    par = {"left": left, "right": {"heads": right_heads, "dim": right_dim, "rank": rank}}
    spec = [{"type": "parallel", "mixer": par} if (i + 1) % parallel_every == 0 else {"type": "attention", "mixer": att} for i in range(layers)]
    return {"architecture": "Vulanex", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "canon": {"taps": taps}, "logit_scale": 0.5,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": 31, "mul_cur": 17}},
            "layers": [{**x, "mlp": {"kind": "dense", "ff": ff}} for x in spec]}
