"""Mixers of Nukelix blocks: grouped-query attention with one gate per head, alone (windowed, with kept first tokens, a
softmax sink and values mixed across layers) or beside a matrix memory, and latent attention whose queries pass through a
latent of their own.

The projections of a mixer's input are one GEMM, also those of two mixers side by side; gates, norms and scales of both
sides are one launch that leaves their heads next to each other for one output GEMM.
"""
from __future__ import annotations

import torch

from ..ops import grouped, linear as lin
from .block_spec import GroupedAttentionSpec, LatentSpec, MatrixMemorySpec, ParallelSpec
from .config import _pad
from .latent import latent_attend, prepare_latent_layer


def prepare_mixer(m, b, lw: dict, tables: dict) -> None:
    """Derived tensors of a layer with one of these mixers: rotation tables, sink scores, mixing factors."""
    if isinstance(b.mixer, LatentSpec):
        prepare_latent_layer(m, b.mixer, lw, tables)
        return
    a = b.attention
    key = (a.rot.base, a.rot.dims, str(a.rot.scaling))
    if key not in tables:
        tables[key] = a.rot.frequencies(m.device)
    lw["rope"] = tables[key]
    lw["sink_scores"] = torch.zeros(a.kv_heads * a.group_pad, dtype=torch.float32, device=m.device) if a.sink else None
    lw["mix"] = float(lw["vmix"]) if a.v_mix else 0.0


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


def mixer_of(b):
    """The forward function of a block's mixer, None when it is not one of these."""
    if isinstance(b.mixer, LatentSpec):
        return gated_latent_mixer
    if isinstance(b.mixer, GroupedAttentionSpec):
        return gated_attention_mixer
    return memory_mixer if isinstance(b.mixer, ParallelSpec) and isinstance(b.mixer.right, MatrixMemorySpec) else None
