"""Ops of linear-attention mixers (a decaying state per head), of windowed attention with a learned distance bias, and of
experts with identity outputs. CUDA tensors go to `csrc/kernels/{linear_attn,attention_bias,moe}.cu` (bf16 when serving,
float32 on the 32-bit path), CPU tensors to :mod:`.linear_reference`.
"""
from __future__ import annotations

import ctypes as C
import math

import numpy as np
import torch

from .. import ops
from . import linear_reference as ref
from ._lib import check, fn, ptr, stream_ptr
from .latent import _f32, _struct, f32, i32, i64, p

LOG2E = 1.4426950408889634
GUARD = 64              # entries before and after a bias row that the kernels may touch for hidden keys

# mirrors of the argument structs in csrc/kernels/linear_attn.cu and attention_bias.cu
LinAttnArgs = _struct("LinAttnArgs", ("q k v log_decay head_decay tok_decay tok_input den out state qo_indptr slots reset chunk_req "
                                      "chunk_start req_chunks u piece_decay", p), ("slot_stride", i64),
                      ("n ld reqs heads dim vdim silu chunks", i32), ("q_scale", f32))
MemoryGatesArgs = _struct("MemoryGatesArgs", ("z bias qo_indptr slots reset m decay input floor", p), ("slot_stride split_stride", i64),
                          ("n reqs heads ldz splits", i32), ("cap", f32))
GatedNormPart = _struct("GatedNormPart", ("x w gate dst den floor", p),
                        ("x_f32 ldx head_cols head_ld group group_pad norm_cols w_cols ldg gate_cols ldd cols dst_cols act", i32),
                        ("eps scale", f32))
BiasedRowsArgs = _struct("BiasedRowsArgs", ("q k v q_norm k_norm slots q_out cache", p),
                         ("n ld heads kv_heads group group_pad dim vdim D page_size", i32), ("eps", f32))
BiasedAttnArgs = _struct("BiasedAttnArgs", ("q kv out bias page_indices kv_page_indptr kv_lens qo_indptr tok_req slots tile_req tile_qstart "
                                            "mask_bits mask_word_indptr item_req item_start item_end req_item_indptr num_items scratch", p),
                         ("n hq hkv D page_size bias_pitch window_left num_tiles total_pages max_items num_reqs num_ctas", i32),
                         ("scale softcap", f32))


class GatedNormArgs(C.Structure):
    _fields_ = [("part", GatedNormPart * 2), ("n", i32)]


# ------------------------------------------------------------------ linear attention
def decay_logs(x, a2, bias, tau: float):
    """Logarithm of sigmoid(x @ a2.T + bias) ^ (1 / tau), 32-bit [N, channels]: base 2 on the device, natural on the CPU
    (`linear_attention` takes the same). x may be a column range."""
    if not x.is_cuda:
        return ref.decay_logs(x, a2, bias, tau)
    n, rank = x.shape
    out = torch.empty(n, a2.shape[0], dtype=torch.float32, device=x.device)
    check(fn("pie_linear_decay")(ptr(x), x.stride(0), ptr(a2), ptr(bias), ptr(out), n, a2.shape[0], rank, 1.0 / tau, 0, _f32(x), stream_ptr()),
          "linear_decay")
    return out


def chunk_pieces(rs, device, size: int):
    """Pieces of `size` tokens of a fire's portions for a chunked form: (request, first row) of every piece and the pieces of
    every request, as device tensors; kept with the fire's recurrent inputs."""
    if size not in rs.pieces:
        qo = np.asarray(rs.qo_host, dtype=np.int64)
        per = -(-np.diff(qo) // size)
        req = np.repeat(np.arange(len(per)), per)
        indptr = np.concatenate([[0], np.cumsum(per)])
        start = qo[req] + (np.arange(len(req)) - indptr[req]) * size
        buf = torch.from_numpy(np.concatenate([req, start, indptr]).astype(np.int32)).to(device)
        rs.pieces[size] = buf.split([len(req), len(req), len(indptr)])
    return rs.pieces[size]


def memory_gates(h, w, bias, spec, rs, state, decode: bool):
    """Exponential gates of a matrix memory (`MatrixMemorySpec`) on the mixer's input h: (decay, key factor) [heads, N] as
    base-2 logarithms for `linear_attention`, and exp(-m_t). The running maxima m are the last numbers of `state`, this layer's
    columns of the state cache, and advance. w: rows of the input gates, then of the forget gates; bias 32-bit."""
    from .latent import split_product
    n, heads = h.shape[0], spec.heads
    m = state[:, spec.state_elems - heads:]
    if not h.is_cuda:
        return ref.memory_gates(torch.matmul(h.float(), w.float().t()) + bias, spec, rs, m)
    z = split_product(h, w) if h.dtype == torch.bfloat16 else torch.matmul(h, w.t())[None]
    out = torch.empty(3, heads, n, dtype=torch.float32, device=h.device)
    a = MemoryGatesArgs(z=ptr(z), bias=ptr(bias), qo_indptr=ptr(rs.qo_indptr), slots=ptr(rs.slots), reset=ptr(rs.reset),
                        m=ptr(m), decay=ptr(out[0]), input=ptr(out[1]), floor=ptr(out[2]), slot_stride=state.stride(0),
                        split_stride=z.stride(0), n=n, reqs=len(rs.slots_host), heads=heads, ldz=z.stride(1), splits=z.shape[0], cap=spec.gate_cap)
    check(fn("pie_memory_gates")(C.byref(a), 1 if decode else 0, stream_ptr()), "memory_gates")
    return out[0], out[1], out[2]


def linear_attention(q, k, v, spec, rs, state, decode: bool, log_decay=None, head_decay=None, silu: bool = False, q_scale: float = 1.0,
                     gates=None):
    """o [N, heads * vdim] in 32-bit of S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t over the ragged batch `rs`.
    q, k, v: column ranges [N, heads * dim (vdim)] of one projection. The decay is per key channel (`log_decay`), per head
    (`head_decay` [heads] 32-bit), or per head and token with a factor on the key (`gates`: both as base-2 logarithms
    [heads, N]; the state then ends in a normaliser, n_t = a_t n_(t-1) + k_t, and (o, n_t . q_t [heads, N]) is returned).
    `state`: this layer's columns of the state cache [slots, all layers]."""
    n, h, d, e = q.shape[0], spec.heads, spec.dim, spec.vdim
    if not q.is_cuda and gates is not None:
        o, den = ref.normalised_linear_attention(q.reshape(n, h, d), k.reshape(n, h, d), v.reshape(n, h, e), *gates, state, rs, q_scale)
        return o.view(n, h * e), den
    if not q.is_cuda:
        ld = log_decay.view(n, h, d) if log_decay is not None else None
        return ref.linear_attention(q.reshape(n, h, d), k.reshape(n, h, d), v.reshape(n, h, e), ld, head_decay,
                                    state.view(state.shape[0], h, d, e), rs, silu, q_scale).view(n, h * e)
    out = torch.empty(n, h * e, dtype=torch.float32, device=q.device)
    den = torch.empty(h, n, dtype=torch.float32, device=q.device) if gates is not None else None
    tok_decay, tok_input = gates if gates is not None else (None, None)
    a = LinAttnArgs(q=ptr(q), k=ptr(k), v=ptr(v), log_decay=ptr(log_decay), head_decay=ptr(head_decay), tok_decay=ptr(tok_decay),
                    tok_input=ptr(tok_input), den=ptr(den), out=ptr(out), state=ptr(state),
                    qo_indptr=ptr(rs.qo_indptr), slots=ptr(rs.slots), reset=ptr(rs.reset), slot_stride=state.stride(0), n=n, ld=q.stride(0),
                    reqs=len(rs.slots_host), heads=h, dim=d, vdim=e, silu=1 if silu else 0, q_scale=q_scale)
    if decode or q.dtype == torch.float32 or not fn("pie_linear_attn_chunk_supported")(d):
        check(fn("pie_linear_attn_serial")(C.byref(a), _f32(q), stream_ptr()), "linear_attn_serial")
        return out if den is None else (out, den)
    req, start, indptr = chunk_pieces(rs, q.device, fn("pie_linear_attn_chunk_tokens")())
    c = req.numel()
    u = torch.empty(c, h * d * (e + (den is not None)), dtype=torch.float32, device=q.device)
    dec = torch.empty(c, h, d, dtype=torch.float32, device=q.device)
    a.chunk_req, a.chunk_start, a.req_chunks, a.u, a.piece_decay, a.chunks = ptr(req), ptr(start), ptr(indptr), ptr(u), ptr(dec), c
    check(fn("pie_linear_attn_chunked")(C.byref(a), stream_ptr()), "linear_attn_chunked")
    return out if den is None else (out, den)


def gated_norm(parts):
    """Outputs of one mixer or of two side by side: for each part (x, w, gate, dst, kw) dst = RMSNorm(x) * w * act(gate) *
    scale. kw: act "silu" | "sigmoid", norm_cols (columns per mean square, 0: no norm), eps, scale; for attention outputs in
    padded rows `spec` (an attention spec); `cols` of the output where the gate (None: none) has one number per `gate_cols`
    of them; den and floor [groups of norm_cols, N]: the norm is that of x / (max(|den|, floor) + 1e-6). dst may be a column
    range; the columns after the output's are set to zero."""
    if not parts[0][0].is_cuda:
        for x, w, gate, dst, kw in parts:
            s = kw.get("spec")
            if s is not None:
                x = x.view(x.shape[0], s.kv_heads, s.group_pad, s.head_dim)[:, :, :s.group, :s.vdim].reshape(x.shape[0], -1)
            y = ref.gated_norm(x.float(), w, gate, kw.get("act"), kw["scale"], kw["norm_cols"], kw.get("eps", 0.0), kw.get("gate_cols", 1),
                               kw.get("den"), kw.get("floor"))
            dst[:, :y.shape[1]] = y.to(dst.dtype)
            dst[:, y.shape[1]:] = 0
        return
    a = GatedNormArgs()
    a.n = parts[0][0].shape[0]
    for i, (x, w, gate, dst, kw) in enumerate(parts):
        s, gc = kw.get("spec"), kw.get("gate_cols", 1)
        cols = gate.shape[1] * gc if gate is not None else kw["cols"]
        a.part[i] = GatedNormPart(
            x=ptr(x), w=ptr(w), gate=ptr(gate), dst=ptr(dst), den=ptr(kw.get("den")), floor=ptr(kw.get("floor")), x_f32=_f32(x),
            ldx=x.stride(0), head_cols=s.vdim if s else cols, head_ld=s.head_dim if s else cols, group=s.group if s else 1,
            group_pad=s.group_pad if s else 1, norm_cols=kw["norm_cols"], w_cols=w.numel() if w is not None else 1,
            ldg=gate.stride(0) if gate is not None else 0, gate_cols=gc, ldd=dst.stride(0), cols=cols, dst_cols=dst.shape[1],
            act=1 if kw.get("act") == "silu" else 0, eps=kw.get("eps", 0.0), scale=kw["scale"])
    check(fn("pie_gated_norm")(C.byref(a), len(parts), _f32(parts[0][3]), stream_ptr()), "gated_norm")


# ------------------------------------------------------------------ attention with a distance bias
def bias_table(rel, spec, device):
    """`rel` [buckets, heads] spread over the distances of the window. CPU: [kv * group_pad, window]. Device: rows of
    GUARD entries like distance 0, the window, at least GUARD entries more, in units of log2."""
    rows = torch.tensor([spec.bucket(n) for n in range(spec.window)], dtype=torch.long)
    t = torch.zeros(spec.kv_heads, spec.group_pad, spec.window)
    t[:, :spec.group] = rel.detach().float().cpu()[rows].t().reshape(spec.kv_heads, spec.group, spec.window)
    t = t.reshape(-1, spec.window)
    if torch.device(device).type != "cuda":
        return t
    # a pitch of 8 (mod 32) words keeps the heads of a group on different shared-memory banks
    pitch = spec.window + 2 * GUARD
    pitch += (8 - pitch) % 32
    full = torch.zeros(t.shape[0], pitch)
    full[:, :GUARD] = t[:, :1]
    full[:, GUARD:GUARD + spec.window] = t
    full[:, GUARD + spec.window:] = t[:, -1:]
    return (full * LOG2E).to(device)


def biased_rows(q, k, v, q_norm, k_norm, slots, cache, spec, eps: float):
    """Queries normed over the whole projection as padded rows [N, kv * group_pad, D]; normed keys and the values are
    written into the layer's pages. q, k, v: column ranges of one projection."""
    if not q.is_cuda:
        return ref.biased_rows(q, k, v, q_norm, k_norm, slots, cache, spec, eps)
    n, D = q.shape[0], spec.head_dim
    out = torch.empty(n, spec.kv_heads * spec.group_pad, D, dtype=q.dtype, device=q.device)
    a = BiasedRowsArgs(q=ptr(q), k=ptr(k), v=ptr(v), q_norm=ptr(q_norm), k_norm=ptr(k_norm), slots=ptr(slots), q_out=ptr(out),
                       cache=ptr(cache), n=n, ld=q.stride(0), heads=spec.heads, kv_heads=spec.kv_heads, group=spec.group,
                       group_pad=spec.group_pad, dim=spec.dim, vdim=spec.vdim, D=D, page_size=cache.shape[3], eps=eps)
    check(fn("pie_biased_rows")(C.byref(a), _f32(q), stream_ptr()), "biased_rows")
    return out


def _prefill_tiles(plan, group: int, rows: int, device):
    key = ("tiles", group, rows)
    if key not in plan.derived:
        tr, tq = ops.plan_prefill_tiles(plan.host.qo_indptr, group, rows, plan.host.kv_lens)
        plan.derived[key] = torch.from_numpy(np.stack([tr, tq]).astype(np.int32)).to(device)
    return plan.derived[key]


def biased_attention(q, cache, bias, plan, rs, slots, spec):
    """softmax(cap * tanh(q.k * scale / cap) + bias[distance]) v over the window, [N, kv * group_pad, D]; `bias` from
    `bias_table`."""
    if not q.is_cuda:
        return ref.biased_attention(q, cache, bias, plan, spec)
    n, hq, D = q.shape
    page = cache.shape[3]
    out = torch.empty_like(q)
    a = BiasedAttnArgs(q=ptr(q), kv=ptr(cache), out=ptr(out), bias=ptr(bias), page_indices=ptr(plan.page_indices),
                       kv_page_indptr=ptr(plan.kv_page_indptr), kv_lens=ptr(plan.kv_lens), n=n, hq=hq, hkv=spec.kv_heads, D=D, page_size=page,
                       bias_pitch=bias.shape[1], window_left=spec.window - 1, scale=spec.scale, softcap=spec.softcap)
    decode = isinstance(plan, ops.DecodePlan)
    if not decode:
        a.mask_bits, a.mask_word_indptr = ptr(plan.mask_bits), ptr(plan.mask_word_indptr)
    if q.dtype == torch.float32 or not fn("pie_biased_mma_supported")(spec.group_pad, D):
        a.qo_indptr, a.tok_req, a.slots = ptr(rs.qo_indptr), ptr(rs.tok_req), ptr(slots)
        check(fn("pie_biased_any")(C.byref(a), _f32(q), stream_ptr()), "biased_any")
    elif decode:
        a.item_req, a.item_start, a.item_end = ptr(plan.item_req), ptr(plan.item_start), ptr(plan.item_end)
        a.req_item_indptr, a.num_items, a.scratch = ptr(plan.req_item_indptr), ptr(plan.num_items), ptr(plan.scratch)
        a.max_items, a.num_reqs, a.num_ctas = plan.max_items, plan.num_reqs, plan.num_ctas
        check(fn("pie_biased_decode")(C.byref(a), stream_ptr()), "biased_decode")
    else:
        rows = 256 if page == 16 and D <= 128 else 64
        t = _prefill_tiles(plan, spec.group_pad, rows, q.device)
        a.qo_indptr, a.tile_req, a.tile_qstart = ptr(plan.qo_indptr), ptr(t[0]), ptr(t[1])
        a.num_tiles, a.total_pages = t.shape[1], cache.shape[0]
        check(fn("pie_biased_prefill")(C.byref(a), rows, ptr(ops.kernel_status(q.device)), stream_ptr()), "biased_prefill")
    return out


# ------------------------------------------------------------------ experts
def sigmoid_experts(x, router, gate_up, down, spec, buf, shared=None):
    """SwiGLU experts chosen by the sigmoid of the router's outputs (32-bit), whose weight scales what they read; `shared`
    [N, W] is added. bf16 on the grouped tcgen05 GEMMs (static shapes, no host synchronisation); `buf`: ops.MoeBuffers."""
    from .latent import split_product
    n = x.shape[0]
    z = split_product(x, router)
    check(fn("pie_moe_route_sigmoid")(ptr(z), z.shape[0], z.stride(0), spec.experts, n, spec.experts, spec.top, ptr(buf.ids), ptr(buf.w),
                                      ptr(buf.pos), ptr(buf.counts), stream_ptr()), "moe_route_sigmoid")
    mt = ops.moe_max_mtiles(n, spec.top, spec.experts)
    ops.moe_align(buf, mt)
    ops.moe_permute(x, buf, weighted=True)
    ops.grouped_gemm(buf.xs, gate_up, buf.tile_expert, buf.act, mt, ops.EPI_SWIGLU)
    ops.grouped_gemm(buf.act, down, buf.tile_expert, buf.ys, mt, ops.EPI_STORE)
    return ops.moe_combine(buf, n, shared, weighted=False)


def scored_experts(x, router, correction, gate_up, down, spec, buf):
    """Experts chosen by softmax score + correction and weighted by the score, identity experts included. bf16 on the
    grouped tcgen05 GEMMs (static shapes, no host synchronisation); `buf`: ops.MoeBuffers."""
    from .latent import split_product
    n = x.shape[0]
    z = split_product(x, router)
    splits, _, e = z.shape
    dev = x.device
    check(fn("pie_moe_route_scored")(ptr(z), splits, z.stride(0), e, n, e, spec.top, spec.experts, ptr(correction), ptr(buf.ids), ptr(buf.w),
                                     ptr(buf.pos), ptr(buf.counts), stream_ptr()), "moe_route_scored")
    mt = ops.moe_max_mtiles(n, spec.top, spec.experts)
    ops.moe_align(buf, mt)
    ops.moe_permute(x, buf)
    ne, n2, k = gate_up.shape
    check(fn("pie_grouped_gemm_clamp_glu")(ptr(buf.xs), ptr(gate_up), ptr(buf.act), ptr(buf.tile_expert), mt, ne, n2, k, buf.xs.stride(0),
                                           buf.act.stride(0), spec.limit, ptr(ops.kernel_status(dev)), ops.num_sms(dev), stream_ptr()),
          "grouped_gemm_clamp_glu")
    ops.grouped_gemm(buf.act, down, buf.tile_expert, buf.ys, mt, ops.EPI_STORE)
    out = torch.empty(n, buf.H, dtype=x.dtype, device=dev)
    check(fn("pie_moe_combine_identity")(ptr(buf.ys), ptr(buf.slot_of), ptr(buf.w), ptr(x), x.stride(0), n, buf.H, spec.top, ptr(out),
                                         out.stride(0), stream_ptr()), "moe_combine_identity")
    return out
