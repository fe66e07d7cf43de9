"""The Nukelix reader and writer of `config.json`: blocks that norm each sublayer's output over a 32-bit residual stream,
with grouped attention (windowed, or beside a matrix memory), latent attention, and experts whose weight scales their input.
"""
from __future__ import annotations

from .block_spec import BlockSpec, EVERYTHING, ExpertsSpec, GroupedAttentionSpec, LatentSpec, MatrixMemorySpec, ParallelSpec, RotarySpec

# config.json key -> `rope_scaling` key, by kind of scaling
_WAVELENGTH = {"factor": "factor", "low": "low_freq_factor", "high": "high_freq_factor", "original": "original_max_position_embeddings"}
_YARN = {"factor": "factor", "fast": "beta_fast", "slow": "beta_slow", "original": "original_max_position_embeddings"}


def _scaling(rot: dict, kind: str, keys: dict):
    s = rot.get("scaling")
    return None if s is None else {"rope_type": kind, **{keys[k]: float(s[k]) for k in keys}}


def _scaling_dict(scaling, keys: dict) -> dict:
    return {} if scaling is None else {"scaling": {k: scaling[v] for k, v in keys.items()}}


def _grouped(i: int, m: dict, adjacent: bool, sink: bool) -> GroupedAttentionSpec:
    rot, mask = m["rot"], m.get("mask")
    s = GroupedAttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]),
                             RotarySpec(rot["dims"], float(rot["base"]), adjacent, _scaling(rot, "llama3", _WAVELENGTH)),
                             mask["size"] if mask else EVERYTHING, mask.get("keep_first", 0) if mask else 0, sink, bool(m.get("v_mix")))
    if s.heads % s.kv_heads or s.window < 1 or s.keep_first < 0 or s.rot.dims % 2 or s.rot.dims > s.dim:
        raise ValueError(f"layer {i}: {s.heads} query heads on {s.kv_heads}, window {s.window} after {s.keep_first}, rotation over "
                         f"{s.rot.dims} of {s.dim} dimensions")
    return s


def _mixer(i: int, kind: str, m: dict):
    if kind == "attention":
        return _grouped(i, m, True, True)
    if kind == "parallel":
        r = m["right"]
        right = MatrixMemorySpec(r["heads"], r["dim"], r["vdim"], float(r["gate_cap"]))
        if right.gate_cap <= 0:
            raise ValueError(f"layer {i}: gate cap {right.gate_cap}")
        return ParallelSpec(_grouped(i, m["left"], False, False), right, float(m["left_scale"]), float(m["right_scale"]))
    if kind != "latent_attention":
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    rot = m["rot"]
    s = LatentSpec(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], EVERYTHING, float(m["scale"]), float(rot["base"]),
                   rot["dims"], q_rank=m["q_rank"], head_gate=True, rot_adjacent=True, rot_scaling=_scaling(rot, "yarn", _YARN))
    if s.rot_dims % 2 or s.rot_dims > s.rot_dim:
        raise ValueError(f"layer {i}: rotation over {s.rot_dims} of {s.rot_dim} dimensions")
    return s


def _experts(i: int, mlp):
    if mlp is None:
        return None
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    r, shared = mlp["router"], mlp.get("shared")
    s = ExpertsSpec(r["experts"], 0, r["top"], mlp["expert"]["ff"], None, "sigmoid", True, shared["ff"] if shared else 0)
    if not 1 <= s.top <= s.experts:
        raise ValueError(f"layer {i}: {s.top} of {s.experts} experts")
    return s


def nukelix_config(cfg: dict, name: str):
    from .config import ModelConfig
    blocks = [BlockSpec(_mixer(i, x["type"], x["mixer"]), _experts(i, x.get("mlp"))) for i, x in enumerate(cfg["layers"])]
    att = [b.attention for b in blocks if b.attention is not None]
    lat = [b.latent for b in blocks if b.latent is not None]
    mixed = [a for a in att if a.v_mix]
    if any(a.kv_heads * a.vdim != mixed[0].kv_heads * mixed[0].vdim for a in mixed):
        raise ValueError("layers that mix values have values of unequal sizes")
    return ModelConfig(
        model_type="nukelix", hidden_size=cfg["width"], intermediate_size=max((b.ff.ff for b in blocks if b.ff is not None), default=0),
        num_hidden_layers=len(blocks),
        num_attention_heads=max([a.kv_heads * a.group_pad for a in att] + [s.heads for s in lat]),
        num_key_value_heads=max((a.kv_heads for a in att), default=1),
        head_dim=max([a.head_dim for a in att] + [s.row for s in lat]), vocab_size=cfg["vocab"],
        max_position_embeddings=cfg.get("max_position_embeddings", 131072), rms_norm_eps=cfg["norm"]["eps"], tie_word_embeddings=True,
        post_norm=True, final_softcap=float(cfg.get("logit_softcap") or 0.0), blocks=blocks, dtype="bfloat16", name=name)


def _grouped_dict(a: GroupedAttentionSpec) -> dict:
    d = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
         "rot": {"dims": a.rot.dims, "base": a.rot.base, **_scaling_dict(a.rot.scaling, _WAVELENGTH)}}
    if a.window != EVERYTHING:
        d["mask"] = {"size": a.window, "keep_first": a.keep_first}
    if a.v_mix:
        d["v_mix"] = True
    return d


def nukelix_dict(cfg) -> dict:
    """The `config.json` dictionary `nukelix_config` reads `cfg` from."""
    layers = []
    for b in cfg.blocks:
        m, f = b.mixer, b.ff
        if isinstance(m, ParallelSpec):
            r = m.right
            d = {"type": "parallel", "mixer": {
                "left": _grouped_dict(m.left), "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "gate_cap": r.gate_cap},
                "left_scale": m.left_scale, "right_scale": m.right_scale}}
        elif isinstance(m, LatentSpec):
            d = {"type": "latent_attention", "mixer": {
                "heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
                "scale": m.scale, "rot": {"dims": m.rot_dims, "base": m.rope_base, **_scaling_dict(m.rot_scaling, _YARN)}}}
        else:
            d = {"type": "attention", "mixer": _grouped_dict(m)}
        d["mlp"] = None
        if f is not None:
            d["mlp"] = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            if f.shared:
                d["mlp"]["shared"] = {"ff": f.shared}
        layers.append(d)
    return {"architecture": "Nukelix", "width": cfg.hidden_size, "vocab": cfg.vocab_size, "layers": layers,
            "norm": {"eps": cfg.rms_norm_eps}, "logit_softcap": cfg.final_softcap}


def nukelix_shape(layers: int = 24, width: int = 4096, heads: int = 32, kv_heads: int = 8, dim: int = 128, window: int = 1024,
                  keep_first: int = 4, right_heads: int = 16, right_dim: int = 128, right_vdim: int = 256, lat_heads: int = 32,
                  lat_dim: int = 96, rot_dim: int = 32, q_rank: int = 1536, kv_rank: int = 224, ff: int = 2048, experts: int = 32,
                  top: int = 4, shared: int = 2048, vocab: int = 128256, softcap: float = 30.0) -> dict:
    """config.json dictionary of a model whose layers go round: parallel mixers, latent attention, windowed attention."""
    far = {"dims": dim, "base": 500000.0}
    kinds = [
        ("parallel", {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "rot": far},
                      "right": {"heads": right_heads, "dim": right_dim, "vdim": right_vdim, "gate_cap": 15.0},
                      "left_scale": 1.0, "right_scale": 0.8}),
        ("latent_attention", {"heads": lat_heads, "dim": lat_dim, "rot_dim": rot_dim, "vdim": dim, "q_rank": q_rank, "kv_rank": kv_rank,
                              "scale": (lat_dim + rot_dim) ** -0.5,
                              "rot": {"dims": rot_dim, "base": 500000.0,
                                      "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}),
        ("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "v_mix": True,
                       "mask": {"size": window, "keep_first": keep_first},
                       "rot": {"dims": dim // 2, "base": 10000.0,
                               "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}),
    ]
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}
    return {"architecture": "Nukelix", "width": width, "vocab": vocab, "norm": {"eps": 1e-5}, "logit_softcap": softcap,
            "layers": [{"type": kinds[i % 3][0], "mixer": kinds[i % 3][1], "mlp": mlp} for i in range(layers)]}
