"""Sandwich-normed blocks over a 32-bit residual stream (Retodra): x += ls1 * norm1b(mixer(norm1(x))), then the same with
the feed-forward. Each layer names its mixer - gated linear attention, or windowed attention with a distance bias beside
lightning attention - and a dense or expert feed-forward.

Output norm, layer scale, residual sum and the next input norm are one pass over the stream (`ResidualStream`); the
projections of a mixer are one GEMM, also those of two mixers side by side, whose output projections are one GEMM over
their heads next to each other.
"""
from __future__ import annotations

import torch

from ..ops import latent as lops, linear as lin, linear_reference as lref
from .block_spec import ExpertsSpec, GatedLinearSpec, ParallelSpec
from .config import _pad
from .moe import _buffers


def projection_columns(mixer) -> dict:
    """Name -> (first column, columns) of the mixer's fused input projection; every part starts on a multiple of 8."""
    if isinstance(mixer, GatedLinearSpec):
        sizes = {"q": mixer.qk, "k": mixer.qk, "v": mixer.values, "g": mixer.values, "a1": mixer.rank}
    else:
        a, r = mixer.left, mixer.right
        sizes = {"left.q": a.heads * a.dim, "left.k": a.kv_heads * a.dim, "left.v": a.kv_heads * a.vdim, "left.g": a.heads * a.vdim,
                 "right.q": r.qk, "right.k": r.qk, "right.v": r.values, "right.g": r.values}
    out, at = {}, 0
    for name, n in sizes.items():
        out[name] = (at, n)
        at += _pad(n)
    return out


def prepare_blocks(m) -> None:
    """Derived tensors: 32-bit gains (1 + w, and (1 + w) * layer scale on the way out), bias by distance, decays."""
    cfg = m.cfg
    m.vocab_local = cfg.vocab_size
    with_kv = [li for li, b in enumerate(cfg.blocks) if b.attention is not None]
    m.cache_index = {li: i for i, li in enumerate(with_kv)}
    one_plus = lambda w: (1.0 + w.float()).contiguous()
    m.final_gain = one_plus(m.w["final_norm"])
    for b, lw in zip(cfg.blocks, m.w["layers"]):
        lw["gain1"], lw["gain1b"] = one_plus(lw["ln1"]), one_plus(lw["ln1b"]) * lw["ls1"].float()
        if b.ff is not None:
            if isinstance(b.ff, ExpertsSpec):
                lw["top"] = b.ff.top
            lw["gain2"], lw["gain2b"] = one_plus(lw["ln2"]), one_plus(lw["ln2b"]) * lw["ls2"].float()
        lw["columns"] = projection_columns(b.mixer)
        if isinstance(b.mixer, ParallelSpec):
            lw["bias_table"] = lin.bias_table(lw["rel"], b.mixer.left, m.device)
            lw["head_decay"] = torch.tensor(b.mixer.right.decay, dtype=torch.float32, device=m.device)


def _state(fi, li: int, spec):
    """This layer's columns of the linear-attention state cache [slots, all layers]."""
    at = fi.rs.linear_at[li]
    return fi.rs.linear_state[:, at:at + spec.state_elems]


def gla_mixer(m, h, lw: dict, li: int, fi) -> torch.Tensor:
    s, eps = m.cfg.blocks[li].mixer, m.cfg.rms_norm_eps
    y = m._gemm(h, lw["w_in"])
    col = {k: y[:, a:a + n] for k, (a, n) in lw["columns"].items()}
    logs = lin.decay_logs(col["a1"], lw["a2"], lw["a2_b"], s.tau)
    o = lin.linear_attention(col["q"], col["k"], col["v"], s, fi.rs, _state(fi, li, s), fi.is_decode, log_decay=logs, q_scale=s.dim ** -0.5)
    z = torch.empty(h.shape[0], lw["w_out"].shape[1], dtype=h.dtype, device=h.device)
    lin.gated_norm([(o, lw["o_norm"], col["g"], z, dict(act="silu", norm_cols=s.vdim, eps=eps, scale=1.0))])
    return m._gemm(z, lw["w_out"])


def parallel_mixer(m, h, lw: dict, li: int, fi, cache) -> torch.Tensor:
    s, eps = m.cfg.blocks[li].mixer, m.cfg.rms_norm_eps
    a, r = s.left, s.right
    y = m._gemm(h, lw["w_in"])
    col = {k: y[:, c:c + n] for k, (c, n) in lw["columns"].items()}
    pages = cache[m.cache_index[li]]
    q = lin.biased_rows(col["left.q"], col["left.k"], col["left.v"], lw["q_norm"], lw["k_norm"], fi.slots, pages, a, eps)
    left = lin.biased_attention(q, pages, lw["bias_table"], fi.attn, fi.rs, fi.slots, a)
    right = lin.linear_attention(col["right.q"], col["right.k"], col["right.v"], r, fi.rs, _state(fi, li, r), fi.is_decode,
                                 head_decay=lw["head_decay"], silu=True)
    n, cut = h.shape[0], _pad(a.heads * a.vdim)
    z = torch.empty(n, lw["w_out"].shape[1], dtype=h.dtype, device=h.device)       # gated heads of both, side by side
    lin.gated_norm([(left.view(n, -1), None, col["left.g"], z[:, :cut], dict(act="sigmoid", norm_cols=0, scale=s.left_scale, spec=a)),
                    (right, lw["o_norm"], col["right.g"], z[:, cut:], dict(act="sigmoid", norm_cols=r.values, eps=eps, scale=s.right_scale))])
    return m._gemm(z, lw["w_out"])


def expert_ff(m, h, lw: dict, spec: ExpertsSpec) -> torch.Tensor:
    if h.is_cuda and h.dtype == torch.bfloat16:
        return lin.scored_experts(h, lw["router"], lw["correction"], lw["experts_gate_up"], lw["experts_down"], spec,
                                  _buffers(m, h.shape[0], lw, h.device))
    logits = torch.matmul(h.float(), lw["router"].float().t())
    return lref.experts(h, logits, lw["correction"], lw["experts_gate_up"], lw["experts_down"], spec)


def sandwich_block(m, st, lw: dict, li: int, fi, cache) -> None:
    cfg = m.cfg
    b = cfg.blocks[li]
    h = st.normed(cfg, lw["gain1"], m.dtype)
    st.y = gla_mixer(m, h, lw, li, fi) if isinstance(b.mixer, GatedLinearSpec) else parallel_mixer(m, h, lw, li, fi, cache)
    st.y_norm = lw["gain1b"]
    if b.ff is None:
        return
    h = st.normed(cfg, lw["gain2"], m.dtype)
    if isinstance(b.ff, ExpertsSpec):
        st.y = expert_ff(m, h, lw, b.ff)
    else:
        st.y = m._gemm(m._gemm(h, lw["w_gate_up"], swiglu=True), lw["w_down"])
    st.y_norm = lw["gain2b"]


def final_rows(m, rows) -> torch.Tensor:
    """The model's norm on the rows that need logits."""
    return lops.stream_norm(rows, m.cfg.hidden_size, m.cfg.rms_norm_eps, norm_w=m.final_gain, dtype=m.dtype)[1]
