"""PyTorch statements of the ops in :mod:`.linear`: what they compute on CPU tensors."""
from __future__ import annotations

import math

import torch


def _silu(x):
    return x * torch.sigmoid(x)


def decay_logs(x, a2, bias, tau: float):
    z = x.float() @ a2.float().t() + bias.float()
    return torch.nn.functional.logsigmoid(z) / tau


def linear_attention(q, k, v, log_decay, head_decay, state, rs, silu: bool, q_scale: float):
    """q, k [N, H, K], v [N, H, V]; natural-log decays [N, H, K] or factors [H]; state [slots, H, K, V] advances."""
    q, k, v = q.float(), k.float(), v.float()
    if silu:
        q, k, v = _silu(q), _silu(k), _silu(v)
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2])
    for r, (a, b) in enumerate(zip(rs.qo_host, rs.qo_host[1:])):
        slot = rs.slots_host[r]
        if slot < 0 or a == b:
            continue
        s = torch.zeros_like(state[slot]) if rs.reset_host[r] else state[slot].clone()
        for t in range(a, b):
            g = log_decay[t].exp()[..., None] if log_decay is not None else head_decay[:, None, None]
            s = g * s + k[t][..., None] * v[t][:, None]
            out[t] = torch.einsum("hkv,hk->hv", s, q[t] * q_scale)
        state[slot] = s
    return out


def memory_gates(z, spec, rs, m):
    """z [N, 2 * heads] biased gate inputs; m [slots, heads] the running maxima, which advance."""
    n, h = z.shape[0], spec.heads
    z = spec.gate_cap * torch.tanh(z / spec.gate_cap)
    i, f = z[:, :h], torch.nn.functional.logsigmoid(z[:, h:])
    decay, key, floor = torch.zeros(n, h), torch.zeros(n, h), torch.zeros(n, h)
    for r, (a, b) in enumerate(zip(rs.qo_host, rs.qo_host[1:])):
        slot = rs.slots_host[r]
        if slot < 0 or a == b:
            continue
        x = torch.zeros(h) if rs.reset_host[r] else m[slot].clone()
        for t in range(a, b):
            new = torch.maximum(f[t] + x, i[t])
            decay[t], key[t], floor[t] = f[t] + x - new, i[t] - new, torch.exp(-new)
            x = new
        m[slot] = x
    return decay.t() / math.log(2), key.t() / math.log(2), floor.t()


def normalised_linear_attention(q, k, v, decay, key, state, rs, q_scale: float):
    """q, k [N, H, K], v [N, H, V]; base-2 logarithms [H, N]; state [slots, H * K * V + H * K + ..] advances. Returns
    (S_t^T q_t, n_t . q_t [H, N])."""
    q, k, v = q.float() * q_scale, k.float(), v.float()
    n, h, d, e = q.shape[0], q.shape[1], q.shape[2], v.shape[2]
    out, den = torch.zeros(n, h, e), torch.zeros(n, h)
    for r, (a, b) in enumerate(zip(rs.qo_host, rs.qo_host[1:])):
        slot = rs.slots_host[r]
        if slot < 0 or a == b:
            continue
        s, c = state[slot, :h * d * e].view(h, d, e).clone(), state[slot, h * d * e:h * d * (e + 1)].view(h, d).clone()
        if rs.reset_host[r]:
            s, c = torch.zeros_like(s), torch.zeros_like(c)
        for t in range(a, b):
            g, kt = torch.exp2(decay[:, t])[:, None], k[t] * torch.exp2(key[:, t])[:, None]
            s = g[..., None] * s + kt[..., None] * v[t][:, None]
            c = g * c + kt
            out[t], den[t] = torch.einsum("hkv,hk->hv", s, q[t]), (c * q[t]).sum(-1)
        state[slot, :h * d * e], state[slot, h * d * e:h * d * (e + 1)] = s.flatten(), c.flatten()
    return out, den.t()


def gated_norm(x, w, gate, act, scale: float, norm_cols: int, eps: float, gate_cols: int = 1, den=None, floor=None):
    """x [N, C] fp32: RMSNorm over runs of norm_cols columns (0: none) * w, times act(gate) * scale; a gate number serves
    gate_cols columns. den, floor: x / (max(|den|, floor) + 1e-6) is normed, one of each per run."""
    n, c = x.shape
    if norm_cols:
        x = x.view(n, -1, norm_cols)
        if den is not None:
            x = x / (torch.maximum(den.abs(), floor) + 1e-6).t()[..., None]
        x = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
        x = (x * w.float().view(-1, norm_cols)).reshape(n, c)
    if gate is None:
        return x * scale
    gate = gate.float().repeat_interleave(gate_cols, -1)
    g = torch.sigmoid(gate)
    return x * (g * gate if act == "silu" else g) * scale


def biased_rows(q, k, v, q_norm, k_norm, slots, cache, spec, eps: float):
    """Normed queries in padded rows [N, kv * group_pad, D]; keys and values into the pages."""
    n, D, page = q.shape[0], spec.head_dim, cache.shape[3]
    rms = lambda x, w: (x.float() / torch.sqrt(x.float().pow(2).mean(-1, keepdim=True) + eps) * w.float())
    out = torch.zeros(n, spec.kv_heads, spec.group_pad, D, dtype=q.dtype)
    out[:, :, :spec.group, :spec.dim] = rms(q, q_norm).view(n, spec.kv_heads, spec.group, spec.dim).to(q.dtype)
    kn = rms(k, k_norm).view(n, spec.kv_heads, spec.dim).to(cache.dtype)
    vn = v.reshape(n, spec.kv_heads, spec.vdim).to(cache.dtype)
    for t, slot in enumerate(slots.tolist()):
        if slot >= 0:
            pg, off = divmod(slot, page)
            cache[pg, 0, :, off, :spec.dim], cache[pg, 1, :, off, :spec.vdim] = kn[t], vn[t]
    return out.view(n, spec.kv_heads * spec.group_pad, D)


def biased_attention(q, cache, bias, batch, spec):
    """Windowed attention with soft-capped scores and `bias` [kv * group_pad, window] by distance; q and the result are
    [N, kv * group_pad, D]."""
    out = torch.zeros_like(q)
    page, gp = cache.shape[3], spec.group_pad
    for r in range(batch.num_requests):
        a, b, n = int(batch.qo_indptr[r]), int(batch.qo_indptr[r + 1]), int(batch.kv_lens[r])
        if a == b:
            continue
        ids = torch.as_tensor(batch.page_indices[batch.kv_page_indptr[r]:batch.kv_page_indptr[r + 1]]).long()
        kv = cache[ids].float()                                   # [pages, 2, hkv, page, D]
        kk = kv[:, 0].transpose(0, 1).reshape(kv.shape[2], -1, kv.shape[-1])[:, :n].repeat_interleave(gp, 0)
        vv = kv[:, 1].transpose(0, 1).reshape(kv.shape[2], -1, kv.shape[-1])[:, :n].repeat_interleave(gp, 0)
        s = torch.einsum("thd,hjd->htj", q[a:b].float(), kk) * spec.scale
        s = spec.softcap * torch.tanh(s / spec.softcap)
        gap = torch.arange(n - (b - a), n)[:, None] - torch.arange(n)[None]
        s = s + bias[:, gap.clamp(0, spec.window - 1)]
        hide = gap >= spec.window
        mask = batch.masks[r] if batch.masks is not None else None
        hide = hide | (gap < 0 if mask is None else ~torch.as_tensor(mask, dtype=torch.bool))
        p = torch.softmax(s.masked_fill(hide[None], float("-inf")), -1).nan_to_num(0.0)
        out[a:b] = torch.einsum("htj,hjd->thd", p, vv).to(out.dtype)
    return out


def experts(x, logits, correction, gate_up, down, spec):
    """Weighted sum of the chosen experts' outputs; gate_up [E, 2 F, W] holds interleaved gate and up rows."""
    s = torch.softmax(logits.float(), -1)
    ids = torch.topk(s + correction, spec.top, -1).indices
    weight = torch.zeros_like(s).scatter(1, ids, torch.gather(s, 1, ids))
    gu = torch.einsum("nw,efw->enf", x, gate_up)
    g, u = gu[..., 0::2].float().clamp(max=spec.limit), gu[..., 1::2].float().clamp(-spec.limit, spec.limit)
    y = torch.bmm((g * torch.sigmoid(1.702 * g) * (u + 1)).to(x.dtype), down.transpose(1, 2))
    out = torch.einsum("enw,ne->nw", y.float(), weight[:, :spec.experts])
    return (out + weight[:, spec.experts:].sum(-1, keepdim=True) * x.float()).to(x.dtype)


def sigmoid_experts(x, logits, gate_up, down, spec):
    """Sum of the chosen experts' outputs on x times the expert's score; gate_up [E, 2 F, W] holds interleaved gate and up
    rows. An expert that was not chosen reads zeros and returns zeros."""
    ids = torch.topk(logits.float(), spec.top, -1).indices
    weight = torch.zeros_like(logits, dtype=torch.float32).scatter(1, ids, torch.sigmoid(torch.gather(logits.float(), 1, ids)))
    xs = (x.float()[None] * weight.t()[..., None]).to(x.dtype)
    gu = torch.bmm(xs, gate_up.transpose(1, 2))
    y = torch.bmm((_silu(gu[..., 0::2].float()) * gu[..., 1::2].float()).to(x.dtype), down.transpose(1, 2))
    return y.float().sum(0).to(x.dtype)
