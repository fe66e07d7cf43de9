"""Ops of delta-rule mixers: decays between a bound and 1, and the recurrence with a decay and a removal rate per key channel.
CUDA tensors go to `csrc/kernels/{delta_rule,linear_attn}.cu` (bf16 when serving, float32 on the 32-bit path), CPU tensors to the
plain statements at the end.
"""
from __future__ import annotations

import ctypes as C
import math

import torch

from ._lib import check, fn, ptr, stream_ptr
from .latent import _f32, _struct, i32, i64, p
from .linear import chunk_pieces

# mirror of the argument struct in csrc/kernels/delta_rule.cu
DeltaArgs = _struct("DeltaArgs", ("r k v a a_bias log_decay out state qo_indptr slots reset chunk_req chunk_start req_chunks pieces", p),
                    ("slot_stride", i64), ("n ld reqs heads dim chunks", i32))
LOG2E = 1.4426950408889634


def bounded_decay_logs(x, w2, w0, bound: float):
    """Base-2 logarithms of exp(-bound * sigmoid(w2 tanh(x) + w0)), 32-bit [N, channels]. x may be a column range."""
    if not x.is_cuda:
        return -LOG2E * bound * torch.sigmoid(torch.tanh(x.float()) @ w2.float().t() + w0.float())
    n, rank = x.shape
    out = torch.empty(n, w2.shape[0], dtype=torch.float32, device=x.device)
    check(fn("pie_linear_decay")(ptr(x), x.stride(0), ptr(w2), ptr(w0), ptr(out), n, w2.shape[0], rank, bound, 1, _f32(x), stream_ptr()),
          "bounded_decay")
    return out


def delta_rule(r, k, v, a, a_bias, log_decay, spec, rs, state, decode: bool):
    """o [N, heads * dim] in 32-bit of S_t = diag(w_t) S_(t-1) - (a_t * u_t) (u_t^T S_(t-1)) + k_t v_t^T, o_t = S_t^T r_t over the
    ragged batch `rs`; u is k divided by sqrt(sum k^2 + 1e-6), the removal rate sigmoid(a + a_bias). r, k, v, a: column
    ranges [N, heads * dim] of one projection; `log_decay` from `bounded_decay_logs`; `state`: this layer's columns of the
    state cache [slots, all layers]."""
    if not r.is_cuda:
        return _delta_rule(r, k, v, a, a_bias, log_decay, spec, rs, state)
    n = r.shape[0]
    out = torch.empty(n, spec.values, dtype=torch.float32, device=r.device)
    args = DeltaArgs(r=ptr(r), k=ptr(k), v=ptr(v), a=ptr(a), a_bias=ptr(a_bias), log_decay=ptr(log_decay), out=ptr(out), state=ptr(state),
                     qo_indptr=ptr(rs.qo_indptr), slots=ptr(rs.slots), reset=ptr(rs.reset), slot_stride=state.stride(0), n=n, ld=r.stride(0),
                     reqs=len(rs.slots_host), heads=spec.heads, dim=spec.dim)
    size = fn("pie_delta_piece_bytes")(spec.dim) if not decode and r.dtype == torch.bfloat16 else 0
    if size:
        req, start, indptr = chunk_pieces(rs, r.device, fn("pie_delta_piece_tokens")())
        pieces = torch.empty(req.numel() * spec.heads * size, dtype=torch.uint8, device=r.device)
        args.chunk_req, args.chunk_start, args.req_chunks, args.pieces, args.chunks = ptr(req), ptr(start), ptr(indptr), ptr(pieces), req.numel()
        check(fn("pie_delta_chunked")(C.byref(args), stream_ptr()), "delta_chunked")
        return out
    name = "delta_step" if decode else "delta_portions"
    check(fn("pie_" + name)(C.byref(args), _f32(r), stream_ptr()), name)
    return out


# ------------------------------------------------------------------ plain statement
def _delta_rule(r, k, v, a, a_bias, log_decay, spec, rs, state):
    n, h, d = r.shape[0], spec.heads, spec.dim
    split = lambda x: x.float().reshape(n, h, d)
    rate = torch.sigmoid(split(a) + a_bias.view(h, d))
    r, k, v, w = split(r), split(k), split(v), torch.exp(split(log_decay) * math.log(2))
    u = k / torch.sqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
    out = torch.zeros(n, h, d)
    for q, (i, j) in enumerate(zip(rs.qo_host, rs.qo_host[1:])):
        slot = rs.slots_host[q]
        if slot < 0 or i == j:
            continue
        s = torch.zeros(h, d, d) if rs.reset_host[q] else state[slot].reshape(h, d, d).clone()
        for t in range(i, j):
            gone = torch.einsum("hd,hde->he", u[t], s)
            s = w[t][..., None] * s - (rate[t] * u[t])[..., None] * gone[:, None] + k[t][..., None] * v[t][:, None]
            out[t] = torch.einsum("hde,hd->he", s, r[t])
        state[slot] = s.flatten()
    return out.view(n, h * d)
