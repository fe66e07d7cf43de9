"""Ops of blocks that read their 32-bit residual stream through a layer norm and a short causal convolution over time, and of
embeddings with a row for the pair (token before, token). CUDA tensors go to `csrc/kernels/stream_conv.cu` (bf16 when serving,
float32 on the 32-bit path), CPU tensors to the plain statements at the end.
"""
from __future__ import annotations

import ctypes as C

import torch

from ._lib import check, fn, ptr, stream_ptr
from .latent import _struct, f32, i32, i64, p

# mirrors of the argument structs in csrc/kernels/stream_conv.cu
PairEmbedArgs = _struct("PairEmbedArgs", ("tokens table pairs x tok_req qo_indptr slots reset state", p),
                        ("slot_stride buckets mul_prev mul_cur", i64), ("n reqs width ldx vocab", i32))
ConvNormArgs = _struct("ConvNormArgs", ("x x_out y0 y1 y0_norm y1_norm w b conv h tok_req qo_indptr slots reset state stage stats", p),
                       ("slot_stride", i64), ("n width ldx ldy ldh taps rows_per_block", i32), ("eps", f32))

MANY_ROWS = 512         # from here on statistics and convolution are two launches


def pair_embed(tokens, table, pairs, spec, ld: int, rs):
    """Rows of `table` plus rows of `pairs` (`PairSpec`) as a 32-bit stream [N, ld], zeros beyond the tables' width. The token
    before a portion's first comes from the sequence's state, which advances."""
    if not table.is_cuda:
        return _pair_embed(tokens, table, pairs, spec, ld, rs)
    n, w = tokens.numel(), table.shape[1]
    x = torch.empty(n, ld, dtype=torch.float32, device=table.device)
    state = rs.token_before
    a = PairEmbedArgs(tokens=ptr(tokens), table=ptr(table), pairs=ptr(pairs), x=ptr(x), tok_req=ptr(rs.tok_req), qo_indptr=ptr(rs.qo_indptr),
                      slots=ptr(rs.slots), reset=ptr(rs.reset), state=ptr(state), slot_stride=state.stride(0), buckets=spec.buckets,
                      mul_prev=spec.mul_prev, mul_cur=spec.mul_cur, n=n, reqs=len(rs.slots_host), width=w, ldx=ld, vocab=table.shape[0])
    check(fn("pie_pair_embed")(C.byref(a), 1 if table.dtype == torch.float32 else 0, 1 if rs.has_portions else 0, stream_ptr()), "pair_embed")
    return x


def conv_norm(x, width: int, eps: float, pending=(), w=None, b=None, conv=None, history=None, rs=None, dtype=None):
    """Per token: x += y / rms(y) * gain for each pending (y, gain); h = LayerNorm(x) * w + b; h <- sum of conv[j] * (h of
    taps - 1 - j tokens before). Gains, w, b and conv [taps, width] are 32-bit; `conv` has the current token's factor last.
    `history`: the convolution's columns of the state cache [slots, all], the last taps - 1 h of a sequence, which advance.
    Returns (x, h in `dtype`); h is None without w. The rows of x and h are padded alike."""
    if not x.is_cuda:
        return _conv_norm(x, width, eps, pending, w, b, conv, history, rs, dtype)
    n, ld = x.shape
    x_out = torch.empty_like(x) if pending else None
    h = torch.empty(n, ld, dtype=dtype, device=x.device) if w is not None else None
    taps = conv.shape[0] if conv is not None else 0
    a = ConvNormArgs(x=ptr(x), x_out=ptr(x_out), w=ptr(w), b=ptr(b), conv=ptr(conv), h=ptr(h), n=n, width=width, ldx=ld, ldh=ld,
                     taps=taps, rows_per_block=16 if n >= MANY_ROWS else 1, eps=eps)
    if n >= MANY_ROWS:
        stats = torch.empty(n, 2, dtype=torch.float32, device=x.device)
        a.stats = ptr(stats)
    if pending:
        if any(y.stride(0) != pending[0][0].stride(0) for y, _ in pending):
            raise ValueError("pending outputs of unequal pitch")
        a.y0, a.y0_norm, a.ldy = ptr(pending[0][0]), ptr(pending[0][1]), pending[0][0].stride(0)
        if len(pending) > 1:
            a.y1, a.y1_norm = ptr(pending[1][0]), ptr(pending[1][1])
    commit = 0
    if taps > 1:
        a.tok_req, a.qo_indptr, a.slots, a.reset = ptr(rs.tok_req), ptr(rs.qo_indptr), ptr(rs.slots), ptr(rs.reset)
        a.state, a.slot_stride = ptr(history), history.stride(0)
        if rs.has_portions:
            commit, a.stage = len(rs.slots_host), ptr(rs.conv_stage)
    act = dtype if dtype is not None else pending[0][0].dtype
    check(fn("pie_conv_norm")(C.byref(a), 1 if act == torch.float32 else 0, commit, stream_ptr()), "conv_norm")
    return (x if x_out is None else x_out), h


# ------------------------------------------------------------------ plain statements
def _pair_embed(tokens, table, pairs, spec, ld, rs):
    ids, prev = tokens.tolist(), []
    state = rs.token_before
    for r, (a, b) in enumerate(zip(rs.qo_host, rs.qo_host[1:])):
        slot = rs.slots_host[r]
        if a == b:
            continue
        prev += [None if rs.reset_host[r] or slot < 0 else int(state[slot]), *ids[a:b - 1]]
        if slot >= 0:
            state[slot] = ids[b - 1]
    rows = [spec.buckets if q is None else (q * spec.mul_prev + t * spec.mul_cur) % spec.buckets for q, t in zip(prev, ids)]
    x = torch.zeros(len(ids), ld)
    x[:, :table.shape[1]] = table[tokens.long()].float() + pairs[torch.tensor(rows, dtype=torch.long)].float()
    return x


def _conv_norm(x, width, eps, pending, w, b, conv, history, rs, dtype):
    x = x.clone()
    for y, gain in pending:
        y = y[:, :width].float()
        x[:, :width] += y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps) * gain
    if w is None:
        return x, None
    f = x[:, :width]
    f = f - f.mean(-1, keepdim=True)
    h = f / torch.sqrt(f.pow(2).mean(-1, keepdim=True) + eps) * w + b
    if conv is not None:
        back, out = conv.shape[0] - 1, torch.zeros_like(h)
        for r, (i, j) in enumerate(zip(rs.qo_host, rs.qo_host[1:])):
            slot = rs.slots_host[r]
            if i == j:
                continue
            before = torch.zeros(back, width)
            if back and slot >= 0 and not rs.reset_host[r]:
                before = history[slot].view(back, width).clone()
            seq = torch.cat([before, h[i:j]])
            for t in range(back + 1):
                out[i:j] += conv[t] * seq[t:t + j - i]
            if back and slot >= 0:
                history[slot] = seq[j - i:].reshape(-1)
        h = out
    full = torch.zeros(x.shape, dtype=dtype)
    full[:, :width] = h.to(dtype)
    return x, full
