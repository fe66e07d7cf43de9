"""Ops of grouped-query attention with biased projections, norms over all heads together, rotation in part, mixed values, a
window beside kept first tokens, and a softmax sink; of attention whose heads are normed one by one, whose values may be the
keys, and whose window may stand beside means of the blocks ahead of it. CUDA tensors go to
`csrc/kernels/attention_{gqa,pool}.cu` and the paged attention kernels (bf16 when serving, float32 on the 32-bit path), CPU
tensors to the plain statements at the end.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import replace

import numpy as np
import torch

from .. import ops
from ._lib import check, fn, ptr, stream_ptr
from .latent import _f32, _struct, f32, i32, p
from .latent_reference import rotate
from .linear import _prefill_tiles

# mirrors of the argument structs in csrc/kernels/attention_gqa.cu
GqaRowsArgs = _struct("GqaRowsArgs", ("q k v q_b k_b v_b q_norm k_norm positions slots inv_freq v_first v_keep q_out cache", p),
                      ("n ld heads kv_heads group group_pad dim vdim D page_size rot_dims adjacent", i32), ("eps mix", f32))
HeadRowsArgs = _struct("HeadRowsArgs", ("q k v q_norm k_norm positions slots inv_freq q_out cache", p),
                       ("n ld heads kv_heads group group_pad dim vdim D page_size rot_dims temp_every", i32),
                       ("eps rot_factor temp_coef", f32))
GqaAnyArgs = _struct("GqaAnyArgs", ("q kv out sink_scores means page_indices kv_page_indptr kv_lens qo_indptr tok_req slots mask_bits "
                                    "mask_word_indptr", p),
                     ("n hq hkv D page_size window_left keep_first sink planes pool per_page", i32), ("scale", f32))
# mirrors of the argument structs in csrc/kernels/attention_pool.cu
PoolArgs = _struct("PoolArgs", ("cache means page_indices kv_page_indptr kv_lens qo_indptr tok_req slots gathered first seen page_req", p),
                   ("n hkv D page_size pool per_page total", i32))
LaidAttnArgs = _struct("LaidAttnArgs", ("q kv means out sinks_log2 page_indices kv_page_indptr kv_lens qo_indptr tile_req tile_qstart "
                                        "mask_bits mask_word_indptr first item_req item_start item_end req_item_indptr num_items scratch", p),
                       ("n hq hkv D page_size window_left planes pool per_page num_tiles total_pages means_pages max_items num_reqs num_ctas",
                        i32), ("scale", f32))


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
        _attend_any(q, cache, plan, rs, slots, spec, page, out, window_left=window, keep_first=keep, sink=1 if spec.sink else 0, planes=2)
        return out
    if isinstance(plan, ops.DecodePlan):
        return ops.paged_decode_attention(q, cache, plan, spec.scale, window_left=window, sinks_log2=sink_scores, keep_first=keep)
    rows = ops.prefill_tile_rows(hq, spec.kv_heads, D, page)
    t = _prefill_tiles(plan, spec.group_pad, rows, q.device)
    tiles = replace(plan, tile_req=t[0], tile_qstart=t[1], num_tiles=t.shape[1], tile_rows=rows)
    return ops.paged_prefill_attention(q, cache, tiles, spec.scale, window_left=window, sinks_log2=sink_scores, keep_first=keep)


def _attend_any(q, cache, plan, rs, slots, spec, page: int, out, **kw):
    n, hq, D = q.shape
    a = GqaAnyArgs(q=ptr(q), kv=ptr(cache), out=ptr(out), page_indices=ptr(plan.page_indices), kv_page_indptr=ptr(plan.kv_page_indptr),
                   kv_lens=ptr(plan.kv_lens), qo_indptr=ptr(rs.qo_indptr), tok_req=ptr(rs.tok_req), slots=ptr(slots),
                   mask_bits=ptr(getattr(plan, "mask_bits", None)), mask_word_indptr=ptr(getattr(plan, "mask_word_indptr", None)),
                   n=n, hq=hq, hkv=spec.kv_heads, D=D, page_size=page, scale=spec.scale, **kw)
    check(fn("pie_gqa_any")(C.byref(a), _f32(q), stream_ptr()), "gqa_any")


# ------------------------------------------------------------------ heads normed one by one, keys as values, means of blocks
def head_rows(q, k, v, lw: dict, positions, slots, cache, spec, eps: float):
    """Queries as padded rows [N, kv * group_pad, D]; keys and values (`v` None: the values are the keys) go into the layer's
    pages [pages, planes, kv, page, D]. q, k, v: column ranges of one projection. Each as far as the mixer
    (`PlainAttentionSpec`) has it: norm per head (`lw`: q_gain, k_gain, 32-bit), rotation (table `rope`), factor on the query by
    position."""
    n, D = q.shape[0], spec.head_dim
    out = torch.empty(n, spec.kv_heads * spec.group_pad, D, dtype=q.dtype, device=q.device)
    if not q.is_cuda:
        _head_rows(q, k, v, lw, positions, slots, cache, spec, eps, out)
        return out
    rot, (coef, every) = spec.rot, spec.q_temp or (0.0, 0)
    a = HeadRowsArgs(q=ptr(q), k=ptr(k), v=ptr(v), q_norm=ptr(lw.get("q_gain")), k_norm=ptr(lw.get("k_gain")), positions=ptr(positions),
                     slots=ptr(slots), inv_freq=ptr(lw.get("rope")), q_out=ptr(out), cache=ptr(cache), n=n, ld=q.stride(0), heads=spec.heads,
                     kv_heads=spec.kv_heads, group=spec.group, group_pad=spec.group_pad, dim=spec.dim, vdim=spec.vdim, D=D,
                     page_size=cache.shape[3], rot_dims=rot.dims if rot else 0, temp_every=every, eps=eps,
                     rot_factor=rot.factor if rot else 1.0, temp_coef=coef)
    check(fn("pie_head_rows")(C.byref(a), _f32(q), stream_ptr()), "head_rows")
    return out


def pool_rows(cache, means, plan, rs, slots, spec):
    """Means of the keys and of the values of every block of `spec.pool` tokens that the fire's tokens complete, into `means`
    [pages, 2, kv, per page, D] beside the page of the block's last token."""
    if not cache.is_cuda:
        return _pool_rows(cache, means, plan, slots, spec)
    a = PoolArgs(cache=ptr(cache), means=ptr(means), page_indices=ptr(plan.page_indices), kv_page_indptr=ptr(plan.kv_page_indptr),
                 kv_lens=ptr(plan.kv_lens), qo_indptr=ptr(rs.qo_indptr), tok_req=ptr(rs.tok_req), slots=ptr(slots), n=slots.numel(),
                 hkv=spec.kv_heads, D=spec.head_dim, page_size=cache.shape[3], pool=spec.pool, per_page=means.shape[3])
    check(fn("pie_pool_rows")(C.byref(a), _f32(cache), stream_ptr()), "pool_rows")


def _gathered_means(cache, means, plan, spec):
    """The means a prefill's tokens can see in 16-row pages of their own, the last one zeros: (pages, first page per request)."""
    h = plan.host
    key = ("means", spec.window, spec.pool)
    if key not in plan.derived:
        seen = np.maximum(0, np.asarray(h.kv_lens, dtype=np.int64) - spec.window) // spec.pool
        pages = -(-seen // 16)
        first = np.concatenate([[0], np.cumsum(pages)])
        buf = np.concatenate([first[:-1], seen, np.repeat(np.arange(len(pages)), pages), [-1]])
        plan.derived[key] = torch.from_numpy(buf.astype(np.int32)).to(cache.device).split([len(seen), len(seen), int(first[-1]) + 1])
    first, seen, page_req = plan.derived[key]
    total = page_req.numel()
    out = torch.empty(total, 2, spec.kv_heads, 16, spec.head_dim, dtype=cache.dtype, device=cache.device)
    a = PoolArgs(means=ptr(means), page_indices=ptr(plan.page_indices), kv_page_indptr=ptr(plan.kv_page_indptr), gathered=ptr(out),
                 first=ptr(first), seen=ptr(seen), page_req=ptr(page_req), hkv=spec.kv_heads, D=spec.head_dim, page_size=cache.shape[3],
                 pool=spec.pool, per_page=means.shape[3], total=total)
    check(fn("pie_pool_gather")(C.byref(a), stream_ptr()), "pool_gather")
    return out, first


def laid_attention(q, cache, means, plan, rs, slots, spec, sinks=None):
    """Softmax over the visible keys of q [N, kv * group_pad, D] in pages as `PlainAttentionSpec` lays them out: keys that are
    their own values, a window beside the `means` of the blocks ahead of it (None: none), a learned sink score per padded
    head (`sinks`: 32-bit, as natural and as base-2 logarithms). Under a custom mask a mean counts if the mask shows all its
    tokens. Same shape out."""
    if not q.is_cuda:
        return _laid_attention(q, cache, means, plan, spec, sinks[0] if sinks is not None else None)
    from ..models.block_spec import EVERYTHING
    n, hq, D = q.shape
    page, planes = cache.shape[3], cache.shape[1]
    window = -1 if spec.window == EVERYTHING else spec.window - 1
    out = torch.empty_like(q)
    decode = isinstance(plan, ops.DecodePlan)
    per_page = means.shape[3] if means is not None else 0
    masked = getattr(plan, "mask_bits", None) is not None
    if q.dtype == torch.float32 or not fn("pie_gqa_mma_supported")(spec.group_pad, D, page) or (masked and spec.pool):
        _attend_any(q, cache, plan, rs, slots, spec, page, out, window_left=window, planes=planes, means=ptr(means), pool=spec.pool,
                    per_page=per_page, sink_scores=ptr(sinks[0] if sinks is not None else None))
        return out
    a = LaidAttnArgs(q=ptr(q), kv=ptr(cache), out=ptr(out), page_indices=ptr(plan.page_indices), kv_page_indptr=ptr(plan.kv_page_indptr),
                     kv_lens=ptr(plan.kv_lens), n=n, hq=hq, hkv=spec.kv_heads, D=D, page_size=page, window_left=window, planes=planes,
                     pool=spec.pool, per_page=per_page, total_pages=cache.shape[0], scale=spec.scale)
    a.sinks_log2 = ptr(sinks[1] if sinks is not None else None)
    if decode:
        a.means = ptr(means)
        a.item_req, a.item_start, a.item_end = ptr(plan.item_req), ptr(plan.item_start), ptr(plan.item_end)
        a.req_item_indptr, a.num_items, a.scratch = ptr(plan.req_item_indptr), ptr(plan.num_items), ptr(plan.scratch)
        a.max_items, a.num_reqs, a.num_ctas = plan.max_items, plan.num_reqs, plan.num_ctas
        check(fn("pie_laid_decode")(C.byref(a), stream_ptr()), "laid_decode")
        return out
    rows = 64 if ops.prefill_tile_rows(hq, spec.kv_heads, D, page) == 64 else 256
    t = _prefill_tiles(plan, spec.group_pad, rows, q.device)
    a.qo_indptr, a.tile_req, a.tile_qstart, a.num_tiles = ptr(plan.qo_indptr), ptr(t[0]), ptr(t[1]), t.shape[1]
    a.mask_bits, a.mask_word_indptr = ptr(plan.mask_bits), ptr(plan.mask_word_indptr)
    if spec.pool:
        rows_, first = _gathered_means(cache, means, plan, spec)
        a.means, a.first, a.means_pages = ptr(rows_), ptr(first), rows_.shape[0]
    check(fn("pie_laid_prefill")(C.byref(a), rows, ptr(ops.kernel_status(q.device)), stream_ptr()), "laid_prefill")
    return out


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


def _head_rows(q, k, v, lw, positions, slots, cache, spec, eps, out):
    n, page = q.shape[0], cache.shape[3]

    def turned(x, gain):
        x = x.float()
        if gain is not None:
            x = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * gain
        return rotate(x, positions, lw["rope"], False, spec.rot.factor) if spec.rot else x
    qn = turned(q.reshape(n, spec.heads, spec.dim), lw.get("q_gain"))
    if spec.q_temp:
        coef, every = spec.q_temp
        qn = qn * (1 + coef * torch.log((positions + 1).div(every, rounding_mode="floor").float() + 1))[:, None, None]
    out.zero_()
    out.view(n, spec.kv_heads, spec.group_pad, -1)[:, :, :spec.group, :spec.dim] = \
        qn.view(n, spec.kv_heads, spec.group, spec.dim).to(q.dtype)
    kn = turned(k.reshape(n, spec.kv_heads, spec.dim), lw.get("k_gain")).to(cache.dtype)
    for t, slot in enumerate(slots.tolist()):
        if slot >= 0:
            pg, off = divmod(slot, page)
            cache[pg, 0, :, off, :spec.dim] = kn[t]
            if v is not None:
                cache[pg, 1, :, off, :spec.vdim] = v[t].view(spec.kv_heads, spec.vdim).to(cache.dtype)


def _context(cache, batch, r: int):
    """Pages of request r in order, and its keys and values [planes, kv, tokens, D]."""
    ids = torch.as_tensor(batch.page_indices[batch.kv_page_indptr[r]:batch.kv_page_indptr[r + 1]]).long()
    kv = cache[ids].float().permute(1, 2, 0, 3, 4)
    return ids, kv.reshape(*kv.shape[:2], -1, kv.shape[-1])[:, :, :int(batch.kv_lens[r])]


def _mean_place(b: int, pool: int, page: int):
    """(page in the request's table, row among its means) of block b."""
    at = ((b + 1) * pool - 1) // page
    return at, b - at * page // pool


def _pool_rows(cache, means, batch, slots, spec):
    page = cache.shape[3]
    for r in range(batch.num_requests):
        a, b, n = int(batch.qo_indptr[r]), int(batch.qo_indptr[r + 1]), int(batch.kv_lens[r])
        if a == b or int(slots[a]) < 0:
            continue
        ids, kv = _context(cache, batch, r)
        for blk in range((n - (b - a)) // spec.pool, n // spec.pool):
            at, row = _mean_place(blk, spec.pool, page)
            means[ids[at], :, :, row] = kv[:, :, blk * spec.pool:(blk + 1) * spec.pool].mean(2).to(means.dtype)


def _laid_attention(q, cache, means, batch, spec, sinks):
    out, page = torch.zeros_like(q), cache.shape[3]
    for r in range(batch.num_requests):
        a, b, n = int(batch.qo_indptr[r]), int(batch.qo_indptr[r + 1]), int(batch.kv_lens[r])
        if a == b:
            continue
        ids, kv = _context(cache, batch, r)
        pos, j = torch.arange(n - (b - a), n)[:, None], torch.arange(n)[None]
        mask = batch.masks[r] if batch.masks is not None else None
        shown = (j <= pos) if mask is None else torch.as_tensor(mask, dtype=torch.bool)
        see, keys, values = shown & (pos - j < spec.window), kv[0], kv[-1]
        blocks = n // spec.pool if spec.pool else 0
        if blocks:
            places = [_mean_place(i, spec.pool, page) for i in range(blocks)]
            rows = torch.stack([means[ids[at], :, :, row].float() for at, row in places], 2)
            whole = (torch.arange(blocks)[None] + 1) * spec.pool - 1 <= pos - spec.window
            whole = whole & shown[:, :blocks * spec.pool].reshape(b - a, blocks, spec.pool).all(-1)
            keys, values, see = torch.cat([rows[0], keys], 1), torch.cat([rows[1], values], 1), torch.cat([whole, see], 1)
        s = torch.einsum("thd,hjd->htj", q[a:b].float(), keys.repeat_interleave(spec.group_pad, 0)) * spec.scale
        s = s.masked_fill(~see[None], float("-inf"))
        if sinks is not None:
            s = torch.cat([s, sinks[:, None, None].expand(-1, b - a, 1)], -1)
        w = torch.softmax(s, -1).nan_to_num(0.0)[..., :keys.shape[1]]
        out[a:b] = torch.einsum("htj,hjd->thd", w, values.repeat_interleave(spec.group_pad, 0)).to(out.dtype)
    return out
