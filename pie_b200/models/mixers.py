"""Mixers of Nukelix blocks: grouped-query attention with one gate per head, alone (windowed, with kept first tokens, a
softmax sink and values mixed across layers) or beside a matrix memory, and latent attention whose queries pass through a
latent of their own. Mixers of Vulanex blocks: attention whose values are its keys, and windowed attention with means of the
blocks ahead beside a delta rule.

The projections of a mixer's input are one GEMM, also those of two mixers side by side; gates, norms and scales of both
sides are one launch that leaves their heads next to each other for one output GEMM.
"""
from __future__ import annotations

import torch

from ..ops import delta, grouped, linear as lin
from .block_spec import DeltaRuleSpec, GroupedAttentionSpec, LatentSpec, MatrixMemorySpec, ParallelSpec, PlainAttentionSpec
from .config import _pad
from .latent import latent_attend, prepare_latent_layer


def prepare_mixer(m, b, lw: dict, tables: dict) -> None:
    """Derived tensors of a layer with one of these mixers: rotation tables, sink scores, mixing factors."""
    if isinstance(b.mixer, LatentSpec):
        prepare_latent_layer(m, b.mixer, lw, tables)
        return
    a = b.attention
    if isinstance(a, PlainAttentionSpec):
        prepare_plain(m, b, lw, tables)
        return
    key = (a.rot.base, a.rot.dims, str(a.rot.scaling))
    if key not in tables:
        tables[key] = a.rot.frequencies(m.device)
    lw["rope"] = tables[key]
    lw["sink_scores"] = torch.zeros(a.kv_heads * a.group_pad, dtype=torch.float32, device=m.device) if a.sink else None
    lw["mix"] = float(lw["vmix"]) if a.v_mix else 0.0


def prepare_plain(m, b, lw: dict, tables: dict) -> None:
    a = b.attention
    if a.rot is not None:
        key = (a.rot.base, a.rot.dims, str(a.rot.scaling))
        if key not in tables:
            tables[key] = a.rot.frequencies(m.device)
        lw["rope"] = tables[key]
    if a.head_norm:
        lw["q_gain"], lw["k_gain"] = lw["q_norm"].float().contiguous(), lw["k_norm"].float().contiguous()
    lw["sinks"] = None
    if a.sink:                      # per padded head, as natural and as base-2 logarithms
        s = torch.zeros(a.kv_heads, a.group_pad, device=m.device)
        s[:, :a.group] = lw["sink"].view(a.kv_heads, a.group)
        lw["sinks"] = (s.flatten(), s.flatten() * lin.LOG2E)
    if isinstance(b.mixer, ParallelSpec):
        lw["left_gain"] = lw["left_norm"].float() * b.mixer.left_scale
        lw["right_gain"] = lw["right_norm"].float() * b.mixer.right_scale


def attend(m, col: dict, side: str, a: GroupedAttentionSpec, lw: dict, li: int, fi, cache, st):
    """Attention of one layer on its projections (`col`, names after `side`); padded rows [N, kv * group_pad, D]. The first
    layer that mixes values leaves its own in the stream's `values` for the others."""
    pages = cache[m.cache_index[li]]
    first = st.values if a.v_mix else None
    q, kept = grouped.grouped_rows(col[side + "q"], col[side + "k"], col[side + "v"], lw, fi.positions, fi.slots, pages, a,
                                   m.cfg.rms_norm_eps, first, lw["mix"], a.v_mix and first is None)
    if kept is not None:
        st.values = kept
    return grouped.grouped_attention(q, pages, fi.attn, fi.rs, fi.slots, a, lw["sink_scores"])


def gated_attention_mixer(m, h, lw: dict, li: int, fi, cache, st) -> torch.Tensor:
    a, n = m.cfg.blocks[li].mixer, h.shape[0]
    y = m._gemm(h, lw["w_in"])
    col = {k: y[:, c:c + w] for k, (c, w) in lw["columns"].items()}
    o = attend(m, col, "", a, lw, li, fi, cache, st)
    z = torch.empty(n, lw["w_out"].shape[1], dtype=h.dtype, device=h.device)
    lin.gated_norm([(o.view(n, -1), None, col["g"], z, dict(act="sigmoid", norm_cols=0, scale=1.0, spec=a, gate_cols=a.vdim))])
    return m._gemm(z, lw["w_out"])


def memory_mixer(m, h, lw: dict, li: int, fi, cache, st) -> torch.Tensor:
    """Attention and a matrix memory side by side."""
    s, n = m.cfg.blocks[li].mixer, h.shape[0]
    a, r = s.left, s.right
    y = m._gemm(h, lw["w_in"])
    col = {k: y[:, c:c + w] for k, (c, w) in lw["columns"].items()}
    left = attend(m, col, "left.", a, lw, li, fi, cache, st)
    state = fi.rs.state_of(li, r.state_elems)
    decay, key, floor = lin.memory_gates(h, lw["w_gates"], lw["b_gates"], r, fi.rs, state, fi.is_decode)
    right, den = lin.linear_attention(col["right.q"], col["right.k"], col["right.v"], r, fi.rs, state, fi.is_decode,
                                      q_scale=r.dim ** -0.5, gates=(decay, key))
    cut = _pad(a.heads * a.vdim)
    z = torch.empty(n, lw["w_out"].shape[1], dtype=h.dtype, device=h.device)       # gated heads of both, side by side
    lin.gated_norm([(left.view(n, -1), None, col["left.g"], z[:, :cut],
                     dict(act="sigmoid", norm_cols=0, scale=s.left_scale, spec=a, gate_cols=a.vdim)),
                    (right, lw["o_norm"], col["right.g"], z[:, cut:],
                     dict(act="sigmoid", norm_cols=r.vdim, eps=m.cfg.rms_norm_eps, scale=s.right_scale, den=den, floor=floor))])
    return m._gemm(z, lw["w_out"])


def gated_latent_mixer(m, h, lw: dict, li: int, fi, cache, st) -> torch.Tensor:
    s, n = m.cfg.blocks[li].mixer, h.shape[0]
    y = m._gemm(h, lw["w_in"])
    col = {k: y[:, c:c + w] for k, (c, w) in lw["columns"].items()}
    cq = torch.empty(n, lw["w_uq"].shape[1], dtype=h.dtype, device=h.device)
    lin.gated_norm([(col["dq"], lw["q_latent_norm"], None, cq, dict(norm_cols=s.q_rank, cols=s.q_rank, eps=m.cfg.rms_norm_eps, scale=1.0))])
    o = torch.empty(n, _pad(s.heads * s.vdim), dtype=h.dtype, device=h.device)
    latent_attend(m, m._gemm(cq, lw["w_uq"]), col["dkv"], lw, s, fi, cache[m.cache_index[li]], o[:, :s.heads * s.vdim])
    z = torch.empty(n, lw["w_out"].shape[1], dtype=h.dtype, device=h.device)
    lin.gated_norm([(o[:, :s.heads * s.vdim], None, col["g"], z, dict(act="sigmoid", norm_cols=0, scale=1.0, gate_cols=s.vdim))])
    return m._gemm(z, lw["w_out"])


def attend_plain(m, col: dict, side: str, a: PlainAttentionSpec, lw: dict, li: int, fi, cache):
    """Attention of one layer on its projections (`col`, names after `side`); padded rows [N, kv * group_pad, D]."""
    at = m.cache_index[li]
    pages, means = cache[at], cache.means[at]
    q = grouped.head_rows(col[side + "q"], col[side + "k"], col.get(side + "v"), lw, fi.positions, fi.slots, pages, a, m.cfg.rms_norm_eps)
    if a.pool:
        grouped.pool_rows(pages, means, fi.attn, fi.rs, fi.slots, a)
    return grouped.laid_attention(q, pages, means, fi.attn, fi.rs, fi.slots, a, lw["sinks"])


def plain_attention_mixer(m, h, lw: dict, li: int, fi, cache, st) -> None:
    a, n = m.cfg.blocks[li].mixer, h.shape[0]
    y = m._gemm(h, lw["w_in"])
    col = {k: y[:, c:c + w] for k, (c, w) in lw["columns"].items()}
    st.add_product(side_by_side(attend_plain(m, col, "", a, lw, li, fi, cache).view(n, -1), a, lw["w_out"]), lw["w_out"])


def side_by_side(o, a: PlainAttentionSpec, w):
    """The heads of padded rows next to each other, as the product with `w` reads them."""
    if o.shape[1] == w.shape[1] and (a.group, a.vdim) == (a.group_pad, a.head_dim):
        return o
    z = torch.empty(o.shape[0], w.shape[1], dtype=o.dtype, device=o.device)
    lin.gated_norm([(o, None, None, z, dict(norm_cols=0, scale=1.0, spec=a, cols=a.heads * a.vdim))])
    return z


def delta_mixer(m, h, lw: dict, li: int, fi, cache, st) -> None:
    """Attention and a delta rule side by side, each output normed on its own. On the device the delta rule runs on a stream of
    its own beside the attention."""
    s, n, eps = m.cfg.blocks[li].mixer, h.shape[0], m.cfg.rms_norm_eps
    a, r = s.left, s.right
    y = m._gemm(h, lw["w_in"])
    col = {k: y[:, c:c + w] for k, (c, w) in lw["columns"].items()}
    with m.beside() as joined:
        logs = delta.bounded_decay_logs(col["right.w1"], lw["w2"], lw["w0"], r.bound)
        o = delta.delta_rule(col["right.r"], col["right.k"], col["right.v"], col["right.a"], lw["a_bias"], logs, r, fi.rs,
                             fi.rs.state_of(li, r.state_elems), fi.is_decode)
        zr = torch.empty(n, lw["w_right"].shape[1], dtype=h.dtype, device=h.device)
        lin.gated_norm([(o, lw["o_norm"], col["right.g"], zr, dict(act="sigmoid", norm_cols=r.dim, eps=eps, scale=1.0))])
    zl = side_by_side(attend_plain(m, col, "left.", a, lw, li, fi, cache).view(n, -1), a, lw["w_left"])
    joined()
    st.pair = ((m._gemm(zl, lw["w_left"]), lw["left_gain"]), (m._gemm(zr, lw["w_right"]), lw["right_gain"]))


def mixer_of(b):
    """The forward function of a block's mixer, None when it is not one of these."""
    if isinstance(b.mixer, PlainAttentionSpec):
        return plain_attention_mixer
    if isinstance(b.mixer, ParallelSpec) and isinstance(b.mixer.right, DeltaRuleSpec):
        return delta_mixer
    if isinstance(b.mixer, LatentSpec):
        return gated_latent_mixer
    if isinstance(b.mixer, GroupedAttentionSpec):
        return gated_attention_mixer
    return memory_mixer if isinstance(b.mixer, ParallelSpec) and isinstance(b.mixer.right, MatrixMemorySpec) else None
