"""Ops of blocks over a 32-bit residual stream with token shift, latent attention and per-layer token input. CUDA tensors
go to `csrc/kernels/latent*.cu` (bf16 when serving, float32 on the 32-bit path), CPU tensors to :mod:`.latent_reference`.
"""
from __future__ import annotations

import ctypes as C
import os

import numpy as np
import torch

from .. import ops
from . import latent_reference as ref
from ._lib import check, fn, ptr, stream_ptr

p, i32, i64, f32 = C.c_void_p, C.c_int, C.c_long, C.c_float


def _struct(name: str, *fields):
    return type(name, (C.Structure,), {"_fields_": [(n, t) for names, t in fields for n in names.split()]})


# mirrors of the argument structs in csrc/kernels/latent.cu and latent_attn.cu
StreamNormArgs = _struct("StreamNormArgs", ("x y y_norm x_out norm_w shift h hs tok_req qo_indptr slots reset state stage", p),
                         ("n width ldx ldy ldh groups rows_per_block", i32), ("eps", f32))
LatentRowsArgs = _struct("LatentRowsArgs", ("q kv positions slots inv_freq norm_w q_out cache", p),
                         ("n ld ld_kv heads dim rot_dim rot_dims rank rank_pad cache_row copy_nope q_width q_rot q_zero adjacent", i32),
                         ("eps rot_factor", f32))
LatentAttnArgs = _struct("LatentAttnArgs", ("q cache page_indices kv_page_indptr qo_indptr kv_lens tok_req slots mask_bits "
                                            "mask_word_indptr out", p),
                         ("n heads row rank_pad cache_row page_size window_left", i32), ("scale", f32))

LatentMmaArgs = _struct("LatentMmaArgs", ("q cache page_indices kv_page_indptr item_req item_start item_end req_item_indptr "
                                          "cta_items qo_indptr kv_lens mask_bits mask_word_indptr out scratch", p),
                        ("items max_items heads row rank_pad cache_row page_size window_left stages reqs page_shift cache_rows", i32),
                        ("scale_log2", f32))
SmallProductArgs = _struct("SmallProductArgs", ("x w out", p), ("x_tok x_head w_head w_row out_tok out_head", i64),
                           ("n heads m k k_total out_f32", i32))


def _f32(t) -> int:
    return 1 if t.dtype == torch.float32 else 0


def stream_embed(tokens, table, ld: int, scale: float = 1.0):
    """Rows of `table` times `scale` as a 32-bit stream [N, ld] (zeros beyond the table's width)."""
    if not table.is_cuda:
        return ref.stream_embed(tokens, table, ld, scale)
    n, w = tokens.numel(), table.shape[1]
    x = torch.empty(n, ld, dtype=torch.float32, device=table.device)
    check(fn("pie_stream_embed")(ptr(tokens), ptr(table), ptr(x), n, w, ld, table.shape[0], scale, _f32(table),
                                 stream_ptr()), "stream_embed")
    return x


def stream_norm(x, width: int, eps: float, y=None, y_norm=None, norm_w=None, groups: int = 1, shift=None, rs=None, layer: int = 0,
                dtype=None, copy: bool = False):
    """Per token: x += y / rms(y) * y_norm (if y); h = RMSNorm(x) in `groups` parts * norm_w; hs = h + (h of the token
    before - h) * shift. The token before the first one of a portion comes from the sequence's state in `rs`
    (a `driver.recurrent.RecurrentInputs`), which advances. The gains (norm_w, y_norm) are in the activation type or, both,
    in 32-bit; `dtype` then names the activation type. `copy`: h = x in the activation type, without a norm (x itself where
    that is 32-bit). Returns (x, h, hs); what was not asked for is None."""
    dtype = dtype or (norm_w if norm_w is not None else y).dtype
    if not x.is_cuda:
        x, h, hs = ref.stream_norm(x, width, eps, y, y_norm, norm_w, groups, shift, rs, layer, dtype)
        return x, x.to(dtype) if copy else h, hs
    if copy and dtype == torch.float32:
        if y is not None:
            x = stream_norm(x, width, eps, y, y_norm, dtype=dtype)[0]
        return x, x, None
    n, ld = x.shape
    new = lambda dt: torch.empty(n, ld, dtype=dt, device=x.device)
    x_out = new(torch.float32) if y is not None else None
    h = new(dtype) if norm_w is not None or copy else None
    hs = new(dtype) if shift is not None else None
    a = StreamNormArgs(x=ptr(x), y=ptr(y), y_norm=ptr(y_norm), x_out=ptr(x_out), norm_w=ptr(norm_w), shift=ptr(shift), h=ptr(h),
                       hs=ptr(hs), n=n, width=width, ldx=ld, ldy=y.stride(0) if y is not None else 0, ldh=ld, groups=groups,
                       rows_per_block=max(1, min(8, n // 592)), eps=eps)
    gain = norm_w if norm_w is not None else y_norm
    commit, gain_f32 = 0, _f32(gain) if gain is not None else 0
    if shift is not None:
        state = rs.shift_state[layer]
        a.tok_req, a.qo_indptr, a.slots, a.reset = ptr(rs.tok_req), ptr(rs.qo_indptr), ptr(rs.slots), ptr(rs.reset)
        a.state, a.stage = ptr(state), ptr(rs.shift_stage)
        if rs.staged is None:               # portions of two tokens or more leave their last h in the stage
            rs.staged = len(rs.slots_host) if any(b - a > 1 for a, b in zip(rs.qo_host, rs.qo_host[1:])) else 0
        commit = rs.staged
    check(fn("pie_stream_norm")(C.byref(a), 1 if dtype == torch.float32 else 0, gain_f32, commit, stream_ptr()), "stream_norm")
    return (x if x_out is None else x_out), h, hs


def latent_rows(qkv, positions, slots, inv_freq, norm_w, cache, spec, eps: float, q_width: int, q_rot: int, copy_nope: bool, kv=None):
    """Rotate the queries of a projection into rows [N, heads, q_width] (rotated part at column q_rot; with `copy_nope` the
    unrotated part in front of it, else the columns before rank_pad are left for `per_head`), and write the new tokens'
    cache rows: normalised latent, rotated shared key part. They are read from `kv` (latent | key part, may be a column
    range), or from behind the queries. `cache` None: a layer that borrows rows."""
    n = qkv.shape[0]
    q = torch.empty(n, spec.heads, q_width, dtype=qkv.dtype, device=qkv.device)
    if kv is None:
        kv = qkv[:, spec.q_rows:]
    if not qkv.is_cuda:
        return ref.latent_rows(qkv, kv, positions, slots, inv_freq, norm_w, cache, spec, eps, q, q_rot, copy_nope)
    a = LatentRowsArgs(q=ptr(qkv), kv=ptr(kv), positions=ptr(positions), slots=ptr(slots), inv_freq=ptr(inv_freq), norm_w=ptr(norm_w),
                       q_out=ptr(q), cache=ptr(cache), n=n, ld=qkv.stride(0), ld_kv=kv.stride(0), heads=spec.heads, dim=spec.dim,
                       rot_dim=spec.rot_dim, rot_dims=spec.rot_dims, rank=spec.kv_rank, rank_pad=spec.rank_pad,
                       cache_row=cache.shape[-1] if cache is not None else 0, copy_nope=1 if copy_nope else 0, q_width=q_width,
                       q_rot=q_rot, q_zero=q_rot if copy_nope else spec.kv_rank, adjacent=1 if spec.rot_adjacent else 0, eps=eps,
                       rot_factor=spec.rotary.factor)
    check(fn("pie_latent_rows")(C.byref(a), _f32(qkv), stream_ptr()), "latent_rows")
    return q


def per_head(x, w, out):
    """out[:, h, :] = x[:, h, :] @ w[h].T for x [N, H, K] and w [H, M, K]; x and out may be strided views."""
    if not x.is_cuda or x.dtype == torch.float32:
        out.copy_(torch.bmm(x.transpose(0, 1), w.transpose(1, 2)).transpose(0, 1))
        return out
    n, heads, k = x.shape
    a = SmallProductArgs(x=ptr(x), w=ptr(w), out=ptr(out), x_tok=x.stride(0), x_head=x.stride(1), w_head=w.stride(0), w_row=w.stride(1),
                         out_tok=out.stride(0), out_head=out.stride(1), n=n, heads=heads, m=w.shape[1], k=k)
    check(fn("pie_small_product")(C.byref(a), stream_ptr()), "per_head")
    return out


def decode_on_tcgen05(spec, page_size: int) -> bool:
    """Whether bf16 decode of this mixer runs on the tcgen05 kernel (PIE_LATENT_TC=0: never; then mma.sync)."""
    return os.environ.get("PIE_LATENT_TC", "1") != "0" and \
        bool(fn("pie_latent_attn_tc_supported")(spec.row, spec.rank_pad, page_size))


def latent_attention(q, cache, plan, rs, slots, spec, page_size: int, window_left: int):
    """Softmax over the visible cache rows of q [N, heads, row] . row * scale; returns the weighted latents
    [N, heads, rank_pad]. The absorbed form: keys and values of every head are the rows themselves. Decode splits a
    request's keys over the plan's work items."""
    if not q.is_cuda:
        return ref.latent_attention(q, cache, plan, spec, window_left)
    n = q.shape[0]
    out = torch.empty(n, spec.heads, spec.rank_pad, dtype=q.dtype, device=q.device)
    decode = isinstance(plan, ops.DecodePlan)
    tiles = fn("pie_latent_attn_mma_tiles")(spec.heads, spec.row, spec.rank_pad) \
        if q.dtype == torch.bfloat16 and page_size & (page_size - 1) == 0 else 0
    if not tiles:           # 32-bit, or a shape that the tensor-core kernel does not take
        a = LatentAttnArgs(q=ptr(q), cache=ptr(cache), page_indices=ptr(plan.page_indices), kv_page_indptr=ptr(plan.kv_page_indptr),
                           qo_indptr=ptr(rs.qo_indptr), kv_lens=ptr(plan.kv_lens), tok_req=ptr(rs.tok_req), slots=ptr(slots),
                           mask_bits=ptr(getattr(plan, "mask_bits", None)),
                           mask_word_indptr=ptr(getattr(plan, "mask_word_indptr", None)), out=ptr(out), n=n, heads=spec.heads,
                           row=q.shape[2], rank_pad=spec.rank_pad, cache_row=cache.shape[-1], page_size=page_size,
                           window_left=window_left, scale=spec.scale)
        check(fn("pie_latent_attn_warp")(C.byref(a), _f32(q), stream_ptr()), "latent_attn_warp")
        return out
    a = LatentMmaArgs(q=ptr(q), cache=ptr(cache), page_indices=ptr(plan.page_indices), kv_page_indptr=ptr(plan.kv_page_indptr),
                      qo_indptr=ptr(rs.qo_indptr), kv_lens=ptr(plan.kv_lens), out=ptr(out), heads=spec.heads, row=spec.row,
                      rank_pad=spec.rank_pad, cache_row=cache.shape[-1], page_size=page_size, window_left=window_left,
                      reqs=len(rs.slots_host), page_shift=page_size.bit_length() - 1,
                      cache_rows=cache.shape[0] * cache.shape[1], scale_log2=spec.scale * 1.4426950408889634)
    if decode:
        a.item_req, a.item_start, a.item_end = ptr(plan.item_req), ptr(plan.item_start), ptr(plan.item_end)
        a.req_item_indptr, a.cta_items, a.scratch = ptr(plan.req_item_indptr), ptr(plan.cta_items), ptr(plan.scratch)
        a.max_items, ctas = plan.max_items, plan.cta_items.numel() - 1
        if decode_on_tcgen05(spec, page_size):
            check(fn("pie_latent_attn_tc")(C.byref(a), ctas, ptr(ops.kernel_status(q.device)), stream_ptr()), "latent_attn_tc")
            return out
    else:
        key, rows = ("absorbed", spec.heads), 16 * tiles
        if key not in plan.derived:
            tr, tqs = ops.plan_prefill_tiles(plan.host.qo_indptr, 1, max(1, rows // min(spec.heads, rows)), plan.host.kv_lens)
            plan.derived[key] = torch.from_numpy(np.stack([tr, tqs]).astype(np.int32)).to(q.device)
        t = plan.derived[key]
        a.item_req, a.item_start, a.items, a.max_items = ptr(t[0]), ptr(t[1]), t.shape[1], t.shape[1]
        a.mask_bits, a.mask_word_indptr = ptr(plan.mask_bits), ptr(plan.mask_word_indptr)
        ctas = t.shape[1]
    check(fn("pie_latent_attn_mma")(C.byref(a), ctas, stream_ptr()), "latent_attn_mma")
    return out


def projected_width(spec) -> int:
    """Head width of the prefill kernel that takes this mixer's keys and values projected out of the latents; 0: none."""
    need = max(spec.qk_dim, spec.vdim)
    return 0 if need > 128 or spec.vdim % 8 else (64 if need <= 64 else 128)


def _projected_context(plan, window_left: int, page_size: int, device):
    """Rows of the cache that a prefill's tokens can see, in 16-token pieces: (cache pieces to gather, page table of the
    gathered copy, its page indptr, key counts), as one int32 device tensor sliced up. Keys before a request's window
    are left out, so every count is relative to the first piece kept."""
    h = plan.host
    qlens, kv = np.diff(h.qo_indptr), np.asarray(h.kv_lens, dtype=np.int64)
    lo = np.maximum(0, kv - qlens - window_left) // 16
    hi = -(-kv // 16)
    per = page_size // 16
    pieces = [np.asarray(h.page_indices[h.kv_page_indptr[r] + np.arange(lo[r], hi[r]) // per], np.int64) * per + np.arange(lo[r], hi[r]) % per
              for r in range(len(kv))]
    flat = np.concatenate(pieces)
    indptr = np.concatenate([[0], np.cumsum(hi - lo)])
    buf = torch.from_numpy(np.concatenate([flat, np.arange(len(flat)), indptr, kv - lo * 16]).astype(np.int32)).to(device)
    return buf.split([len(flat), len(flat), len(indptr), len(kv)])


def projected_prefill_attention(q, cache, plan, w_kv, spec, page_size: int, window_left: int, out):
    """Prefill attention on keys and values projected from the visible latents for this pass: one GEMM (the shared rotated
    key part passes through it on a unit block) gives [tokens, heads, 2, D], which the tcgen05 kernel reads in place.
    q [N, heads, D] = (unrotated | rotated | zeros); out [N, heads * vdim], may be a column range."""
    key = ("projected", window_left)
    if key not in plan.derived:
        if plan.mask_bits is not None:
            raise ValueError("custom masks index keys of the whole context")
        plan.derived[key] = _projected_context(plan, window_left, page_size, q.device)
    src, table, indptr, kv_lens = plan.derived[key]
    row, d = cache.shape[-1], q.shape[2]
    rows = ops.gather_rows(cache.view(-1, 16 * row), src).view(-1, row)
    kv = ops.gemm(rows[:, :spec.row], w_kv)
    check(fn("pie_projected_prefill_attn_tc")(
        ptr(q), ptr(kv), ptr(table), ptr(indptr), ptr(plan.qo_indptr), ptr(kv_lens), ptr(plan.tile_req), ptr(plan.tile_qstart),
        plan.num_tiles, None, None, ptr(out), q.shape[0], spec.heads, d, rows.shape[0], spec.vdim, out.stride(0), spec.scale,
        window_left, ptr(ops.kernel_status(q.device)), stream_ptr()), "projected_prefill_attn_tc")
    return out


def bias_xielu(y, bias, act):
    """y = xIELU(y + bias) in place; y may be a column range of a wider buffer."""
    if not y.is_cuda:
        return ref.bias_xielu(y, bias, act)
    check(fn("pie_bias_xielu")(ptr(y), y.stride(0), ptr(bias), ptr(act), y.shape[0], y.shape[1], _f32(y), stream_ptr()), "bias_xielu")
    return y


def stream_add(x, d, bias=None, copy: bool = False):
    """(x + d + bias, the same in d's type or None): a sublayer's output joins the 32-bit stream."""
    if not x.is_cuda:
        return ref.stream_add(x, d, bias, copy)
    out = torch.empty_like(x)
    cp = torch.empty_like(d) if copy and d.dtype != torch.float32 else None
    check(fn("pie_stream_add")(ptr(x), ptr(d), ptr(bias), ptr(out), ptr(cp), x.shape[0], x.shape[1], _f32(d), stream_ptr()), "stream_add")
    return out, (out if d.dtype == torch.float32 else cp)


def gemm_xielu(x, w, bias, act, out):
    """out = xIELU(x @ w.T + bias), bf16; bias and activation in the GEMM's epilogue. `out` may be a column range."""
    m, k = x.shape
    ops.ensure_gemm_workspace(x.device)
    check(fn("pie_gemm_bf16_xielu")(ptr(x), ptr(w), ptr(out), ptr(bias), ptr(act), m, w.shape[0], k, x.stride(0), w.stride(0),
                                    out.stride(0), ptr(ops.kernel_status(x.device)), ops.num_sms(x.device), stream_ptr()), "gemm_xielu")
    return out


def gemm_stream(a, w, bias, x, copy: bool = False):
    """x += a @ w.T + bias in place for a 32-bit stream x, in the GEMM's epilogue; returns (x, x in bf16 if `copy`)."""
    m, k = a.shape
    cp = torch.empty(m, w.shape[0], dtype=a.dtype, device=a.device) if copy else None
    ops.ensure_gemm_workspace(a.device)
    check(fn("pie_gemm_bf16_stream")(ptr(a), ptr(w), ptr(bias), ptr(x), ptr(x), x.stride(0), ptr(cp), m, w.shape[0], k, a.stride(0),
                                     w.stride(0), w.shape[0], ptr(ops.kernel_status(a.device)), ops.num_sms(a.device), stream_ptr()),
          "gemm_stream")
    return x, cp


def side_gate(z, table, tokens, col0: int, dim: int):
    """gelu_tanh(z) * table[tokens, col0:col0 + dim], zeros in the padding columns of z. z [N, cols], or 32-bit partial
    products [splits, N, cols] that add up to it."""
    if not z.is_cuda:
        return ref.side_gate(z, table, tokens, col0, dim)
    splits = z.shape[0] if z.dim() == 3 else 1
    n, cols = z.shape[-2:]
    g = torch.empty(n, cols, dtype=table.dtype, device=z.device)
    check(fn("pie_side_gate")(ptr(z), z.stride(-2), z.stride(0), splits, _f32(z), ptr(table), table.stride(0), ptr(tokens), ptr(g), cols,
                              dim, col0, table.shape[0], n, _f32(table), stream_ptr()), "side_gate")
    return g


def split_product(x, w):
    """x @ w.T for a narrow w [M, K], bf16 in, as 32-bit partial products [splits, N, M] over ranges of K (the reader adds
    them up): enough CTAs for a product with few output tiles and a long K."""
    n, k = x.shape
    m = w.shape[0]
    tiles = -(-n // 64) * -(-m // 64)
    splits = max(1, min(16, k // 256, 4 * ops.num_sms(x.device) // tiles))
    per = -(-(-(-k // splits)) // 64) * 64
    splits = -(-k // per)
    z = torch.empty(splits, n, m, dtype=torch.float32, device=x.device)
    a = SmallProductArgs(x=ptr(x), w=ptr(w), out=ptr(z), x_tok=x.stride(0), x_head=per, w_head=per, w_row=w.stride(0), out_tok=m,
                         out_head=n * m, n=n, heads=splits, m=m, k=per, k_total=k, out_f32=1)
    check(fn("pie_small_product")(C.byref(a), stream_ptr()), "split_product")
    return z
