"""Ops of grouped-query attention with biased projections, norms over all heads together, rotation in part, mixed values, a
window beside kept first tokens, and a softmax sink. CUDA tensors go to `csrc/kernels/attention_gqa.cu` and the paged
attention kernels (bf16 when serving, float32 on the 32-bit path), CPU tensors to the plain statements at the end.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import replace

import torch

from .. import ops
from ._lib import check, fn, ptr, stream_ptr
from .latent import _f32, _struct, f32, i32, p
from .latent_reference import rotate
from .linear import _prefill_tiles

# mirrors of the argument structs in csrc/kernels/attention_gqa.cu
GqaRowsArgs = _struct("GqaRowsArgs", ("q k v q_b k_b v_b q_norm k_norm positions slots inv_freq v_first v_keep q_out cache", p),
                      ("n ld heads kv_heads group group_pad dim vdim D page_size rot_dims adjacent", i32), ("eps mix", f32))
GqaAnyArgs = _struct("GqaAnyArgs", ("q kv out page_indices kv_page_indptr kv_lens qo_indptr tok_req slots mask_bits mask_word_indptr", p),
                     ("n hq hkv D page_size window_left keep_first sink", i32), ("scale", f32))


def grouped_rows(q, k, v, lw: dict, positions, slots, cache, spec, eps: float, v_first=None, mix: float = 0.0, keep_values: bool = False):
    """Queries as padded rows [N, kv * group_pad, D]; keys and values go into the layer's pages. q, k, v: column ranges of
    one projection; `lw`: biases q_b, k_b, v_b, gains q_norm, k_norm and the table `rope`. Values are mixed with `v_first`
    [N, kv * vdim] (32-bit), v + mix (v_first - v). Returns (queries, values in 32-bit if `keep_values`)."""
    n, D = q.shape[0], spec.head_dim
    out = torch.empty(n, spec.kv_heads * spec.group_pad, D, dtype=q.dtype, device=q.device)
    kept = torch.empty(n, spec.kv_heads * spec.vdim, dtype=torch.float32, device=q.device) if keep_values else None
    if not q.is_cuda:
        _rows(q, k, v, lw, positions, slots, cache, spec, eps, v_first, mix, out, kept)
        return out, kept
    a = GqaRowsArgs(q=ptr(q), k=ptr(k), v=ptr(v), q_b=ptr(lw["q_b"]), k_b=ptr(lw["k_b"]), v_b=ptr(lw["v_b"]), q_norm=ptr(lw["q_norm"]),
                    k_norm=ptr(lw["k_norm"]), positions=ptr(positions), slots=ptr(slots), inv_freq=ptr(lw["rope"]), v_first=ptr(v_first),
                    v_keep=ptr(kept), q_out=ptr(out), cache=ptr(cache), n=n, ld=q.stride(0), heads=spec.heads, kv_heads=spec.kv_heads,
                    group=spec.group, group_pad=spec.group_pad, dim=spec.dim, vdim=spec.vdim, D=D, page_size=cache.shape[3],
                    rot_dims=spec.rot.dims, adjacent=1 if spec.rot.adjacent else 0, eps=eps, mix=mix)
    check(fn("pie_gqa_rows")(C.byref(a), _f32(q), stream_ptr()), "gqa_rows")
    return out, kept


def grouped_attention(q, cache, plan, rs, slots, spec, sink_scores=None):
    """Softmax over the visible keys of q [N, kv * group_pad, D], with `sink_scores` [kv * group_pad] (32-bit zeros: a score
    of 0 per head that takes its share) where the mixer has a sink. Same shape out."""
    if not q.is_cuda:
        return _attention(q, cache, plan, spec)
    from ..models.block_spec import EVERYTHING
    n, hq, D = q.shape
    page = cache.shape[3]
    window = -1 if spec.window == EVERYTHING else spec.window - 1
    keep = spec.keep_first if window >= 0 else 0
    if q.dtype == torch.float32 or not fn("pie_gqa_mma_supported")(spec.group_pad, D, page):
        out = torch.empty_like(q)
        a = GqaAnyArgs(q=ptr(q), kv=ptr(cache), out=ptr(out), page_indices=ptr(plan.page_indices), kv_page_indptr=ptr(plan.kv_page_indptr),
                       kv_lens=ptr(plan.kv_lens), qo_indptr=ptr(rs.qo_indptr), tok_req=ptr(rs.tok_req), slots=ptr(slots),
                       mask_bits=ptr(getattr(plan, "mask_bits", None)), mask_word_indptr=ptr(getattr(plan, "mask_word_indptr", None)),
                       n=n, hq=hq, hkv=spec.kv_heads, D=D, page_size=page, window_left=window, keep_first=keep,
                       sink=1 if spec.sink else 0, scale=spec.scale)
        check(fn("pie_gqa_any")(C.byref(a), _f32(q), stream_ptr()), "gqa_any")
        return out
    if isinstance(plan, ops.DecodePlan):
        return ops.paged_decode_attention(q, cache, plan, spec.scale, window_left=window, sinks_log2=sink_scores, keep_first=keep)
    rows = ops.prefill_tile_rows(hq, spec.kv_heads, D, page)
    t = _prefill_tiles(plan, spec.group_pad, rows, q.device)
    tiles = replace(plan, tile_req=t[0], tile_qstart=t[1], num_tiles=t.shape[1], tile_rows=rows)
    return ops.paged_prefill_attention(q, cache, tiles, spec.scale, window_left=window, sinks_log2=sink_scores, keep_first=keep)


# ------------------------------------------------------------------ plain statements
def _rows(q, k, v, lw, positions, slots, cache, spec, eps, v_first, mix, out, kept):
    n, page = q.shape[0], cache.shape[3]

    def normed(x, b, w):
        x = x.float() + b.float()
        return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    turn = lambda x: rotate(x, positions, lw["rope"], spec.rot.adjacent)
    out.zero_()
    out.view(n, spec.kv_heads, spec.group_pad, -1)[:, :, :spec.group, :spec.dim] = \
        turn(normed(q, lw["q_b"], lw["q_norm"]).view(n, spec.heads, spec.dim)).view(n, spec.kv_heads, spec.group, spec.dim).to(q.dtype)
    kn = turn(normed(k, lw["k_b"], lw["k_norm"]).view(n, spec.kv_heads, spec.dim)).to(cache.dtype)
    vn = v.float() + lw["v_b"].float()
    if kept is not None:
        kept.copy_(vn)
    if v_first is not None:
        vn = (1 - mix) * vn + mix * v_first
    vn = vn.view(n, spec.kv_heads, spec.vdim).to(cache.dtype)
    for t, slot in enumerate(slots.tolist()):
        if slot >= 0:
            pg, off = divmod(slot, page)
            cache[pg, 0, :, off, :spec.dim], cache[pg, 1, :, off, :spec.vdim] = kn[t], vn[t]


def _attention(q, cache, batch, spec):
    out = torch.zeros_like(q)
    for r in range(batch.num_requests):
        a, b, n = int(batch.qo_indptr[r]), int(batch.qo_indptr[r + 1]), int(batch.kv_lens[r])
        if a == b:
            continue
        ids = torch.as_tensor(batch.page_indices[batch.kv_page_indptr[r]:batch.kv_page_indptr[r + 1]]).long()
        kv = cache[ids].float()                                   # [pages, 2, hkv, page, D]
        flat = lambda x: x.transpose(0, 1).reshape(kv.shape[2], -1, kv.shape[-1])[:, :n].repeat_interleave(spec.group_pad, 0)
        s = torch.einsum("thd,hjd->htj", q[a:b].float(), flat(kv[:, 0])) * spec.scale
        j = torch.arange(n)[None]
        gap = torch.arange(n - (b - a), n)[:, None] - j
        mask = batch.masks[r] if batch.masks is not None else None
        hide = (gap < 0) if mask is None else ~torch.as_tensor(mask, dtype=torch.bool)
        hide = hide | ((gap >= spec.window) & (j >= spec.keep_first))
        s = s.masked_fill(hide[None], float("-inf"))
        if spec.sink:
            w = torch.softmax(torch.cat([s, torch.zeros_like(s[..., :1])], -1), -1)[..., :-1]
        else:
            w = torch.softmax(s, -1).nan_to_num(0.0)
        out[a:b] = torch.einsum("htj,hjd->thd", w, flat(kv[:, 1])).to(out.dtype)
    return out
