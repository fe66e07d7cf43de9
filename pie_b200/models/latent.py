"""Parallel blocks with latent attention over a 32-bit residual stream (Puzutar).

One layer: h = grouped RMSNorm(x), hs = h shifted towards the previous token's h; x += mixer(hs) + ff(h); then the
per-layer token input, x += RMSNorm(W_proj (gelu(W_gate x) * e)). The norm of a layer also finishes the token input of
the layer before (`ResidualStream` carries what is pending), and the products that end both sublayers run as one GEMM over
their inputs side by side.

Latent attention decodes in its absorbed form: with W_uk folded into the query and W_uv applied to the result, keys and
values of every head are the cached rows themselves, so that a step reads one row per token whatever the head count.
Prefill has many queries per key: it projects keys and values out of the visible latents and runs on the tcgen05 kernel.
"""
from __future__ import annotations

import torch

from ..ops import latent as lops
from .config import _pad
from .stream import ResidualStream


def prepare_latent_layer(m, s, lw: dict, tables: dict) -> None:
    """The per-head factors of one mixer in the layout the absorbed products read, its rotation table (shared by `tables`)."""
    key = (s.rope_base, s.rot_dims, str(s.rot_scaling))
    if key not in tables:
        tables[key] = s.rotary.frequencies(m.device)
    lw["rope"] = tables[key]
    # query into the latent: [H, rank, dim]; latent into the value: [H, vdim, rank_pad] (a cached row is padded)
    lw["w_uk_t"] = lw["w_uk"].view(s.heads, s.dim, s.kv_rank).transpose(1, 2).contiguous()
    uv = lw["w_uv"].view(s.heads, s.vdim, s.kv_rank)
    lw["w_uv_p"] = torch.nn.functional.pad(uv, (0, s.rank_pad - s.kv_rank)).contiguous()
    d = lops.projected_width(s)
    if m.device.type == "cuda" and m.dtype == torch.bfloat16 and d:
        # cache row -> (key | value) of every head, D columns each; the rotated key part is copied by a unit block
        w = torch.zeros(s.heads, 2, d, s.row, dtype=m.dtype, device=m.device)
        w[:, 0, :s.dim, :s.kv_rank] = lw["w_uk"].view(s.heads, s.dim, s.kv_rank)
        w[:, 0, s.dim:s.qk_dim, s.rank_pad:s.rank_pad + s.rot_dim] = torch.eye(s.rot_dim, dtype=m.dtype, device=m.device)
        w[:, 1, :s.vdim, :s.kv_rank] = uv
        lw["w_kv_row"] = w.view(-1, s.row)


def prepare_latent(m) -> None:
    """Derived tensors of every layer."""
    cfg, tables = m.cfg, {}
    m.vocab_local = cfg.vocab_size
    m.cache_index = cfg.latent_cache_index
    if m.w["lm_head"].shape == m.w["embed"].shape:
        m.w["lm_head"] = m.w["embed"]                   # tied and unpadded: one copy
    for s, lw in zip(cfg.latent, m.w["layers"]):
        prepare_latent_layer(m, s, lw, tables)


def latent_attend(m, q_in, kv, lw: dict, s, fi, layer_cache, out) -> None:
    """Latent attention with queries q_in [N, >= heads * qk_dim] and the new tokens' rows kv [N, kv_rank + rot_dim] (None: a
    layer that reads another's); the heads' values go to out [N, heads * vdim], which may be a column range."""
    n, page, eps = q_in.shape[0], layer_cache.shape[1], m.cfg.rms_norm_eps
    cache = layer_cache if kv is not None else None
    rows = lambda width, rot, copy: lops.latent_rows(q_in, fi.positions, fi.slots, lw["rope"], lw.get("latent_norm"), cache, s, eps, width,
                                                     rot, copy, kv)
    if "w_kv_row" in lw and not fi.is_decode and fi.attn.mask_bits is None and page % 16 == 0:
        lops.projected_prefill_attention(rows(lops.projected_width(s), s.dim, True), layer_cache, fi.attn, lw["w_kv_row"], s, page,
                                         s.window - 1, out)
        return
    q = rows(s.row, s.rank_pad, False)
    lops.per_head(q_in.as_strided((n, s.heads, s.dim), (q_in.stride(0), s.qk_dim, 1)), lw["w_uk_t"], q[..., :s.kv_rank])
    o = lops.latent_attention(q, layer_cache, fi.attn, fi.rs, fi.slots, s, page, s.window - 1)
    lops.per_head(o, lw["w_uv_p"], out.as_strided((n, s.heads, s.vdim), (out.stride(0), s.vdim, 1)))


def parallel_latent_block(m, st: ResidualStream, lw: dict, li: int, fi, cache) -> None:
    cfg = m.cfg
    s, ff, W, eps = cfg.latent[li], cfg.ff_sizes[li], cfg.hidden_size, cfg.rms_norm_eps
    x, h, hs = lops.stream_norm(st.x, W, eps, st.y, st.y_norm, lw["ln1"], cfg.norm_groups, lw.get("shift"), fi.rs, li)
    n, hv = x.shape[0], s.heads * s.vdim
    cols = lw["w_block_out"].shape[1]
    both = torch.empty(n, cols, dtype=h.dtype, device=h.device)       # attention heads | feed-forward activations
    if _pad(hv) > hv:
        both[:, hv:_pad(hv)] = 0
    qkv = m._gemm(hs if hs is not None else h, lw["w_latent_in"])
    latent_attend(m, qkv, qkv[:, s.q_rows:s.proj_rows] if s.kv_from is None else None, lw, s, fi, cache[m.cache_index[li]], both[:, :hv])
    side = cfg.token_side_dim
    fused = m.gemm_backend == "tcgen05" and h.dtype == torch.bfloat16
    if ff and fused:
        lops.gemm_xielu(h, lw["w_up"], lw["b_up"], lw["act"], both[:, _pad(hv):])
    elif ff:
        act = both[:, _pad(hv):]
        act.copy_(m._gemm(h, lw["w_up"]))
        lops.bias_xielu(act, lw["b_up"], lw["act"])
    if fused:
        st.x, xc = lops.gemm_stream(both, lw["w_block_out"], lw.get("b_down"), x, copy=side > 0)
    else:
        st.x, xc = lops.stream_add(x, m._gemm(both, lw["w_block_out"]), lw.get("b_down"), copy=side > 0)
    st.y = st.y_norm = None
    if side:
        z = lops.split_product(xc, lw["side_gate"]) if fused else m._gemm(xc, lw["side_gate"])
        g = lops.side_gate(z, m.w["side_embed"], fi.tokens, li * side, side)
        if fused and n <= 256:                          # short K, few rows: latency bound
            st.y = torch.empty(n, lw["side_proj"].shape[0], dtype=g.dtype, device=g.device)
            lops.per_head(g[:, None], lw["side_proj"][None], st.y[:, None])
        else:
            st.y = m._gemm(g, lw["side_proj"])
        st.y_norm = lw["side_norm"]


def final_rows(m, rows):
    """The model's norm on the rows that need logits."""
    return lops.stream_norm(rows, m.cfg.hidden_size, m.cfg.rms_norm_eps, norm_w=m.w["final_norm"], groups=m.cfg.norm_groups)[1]
