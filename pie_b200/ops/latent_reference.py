"""Plain PyTorch statements of the ops in :mod:`.latent` (the CPU path of the engine)."""
from __future__ import annotations

import torch


def stream_embed(tokens, table, ld, scale=1.0):
    x = torch.zeros(tokens.numel(), ld, dtype=torch.float32)
    x[:, :table.shape[1]] = table[tokens.long()].float() * scale
    return x


def stream_norm(x, width, eps, y, y_norm, norm_w, groups, shift, rs, layer, dtype):
    x = x.clone()
    if y is not None:
        yf = y[:, :width].float()
        x[:, :width] += yf * torch.rsqrt(yf.pow(2).mean(-1, keepdim=True) + eps) * y_norm.float()
    h = hs = None
    if norm_w is not None:
        g = x[:, :width].reshape(x.shape[0], groups, width // groups)
        hf = (g * torch.rsqrt(g.pow(2).mean(-1, keepdim=True) + eps)).reshape(x.shape[0], width) * norm_w.float()
        h = torch.zeros(x.shape, dtype=dtype)
        h[:, :width] = hf.to(dtype)
        if shift is not None:
            prev = torch.zeros_like(hf)
            prev[1:] = hf[:-1]
            state = rs.shift_state[layer]
            for r, (a, b) in enumerate(zip(rs.qo_host[:-1], rs.qo_host[1:])):
                if b == a:
                    continue
                slot = rs.slots_host[r]
                prev[a] = 0 if rs.reset_host[r] or slot < 0 else state[slot]
                if slot >= 0:
                    state[slot] = hf[b - 1]
            hs = torch.zeros(x.shape, dtype=dtype)
            hs[:, :width] = (hf + (prev - hf) * shift.float()).to(dtype)
    return x, h, hs


def rotate(x, positions, inv_freq, adjacent=False, factor=1.0):
    """The first 2 * len(inv_freq) columns of x [N, ..., D] turned; halves of a pair adjacent or half the width apart."""
    half = inv_freq.numel()
    ang = positions.float()[:, None] * inv_freq.float()[None, :]
    ang = ang.reshape(ang.shape[0], *([1] * (x.dim() - 2)), half)
    c, s = ang.cos() * factor, ang.sin() * factor
    r, rest = x[..., :2 * half].float(), x[..., 2 * half:].float()
    u, v = (r[..., 0::2], r[..., 1::2]) if adjacent else (r[..., :half], r[..., half:])
    a, b = u * c - v * s, v * c + u * s
    return torch.cat([torch.stack([a, b], -1).flatten(-2) if adjacent else torch.cat([a, b], -1), rest], -1)


def latent_rows(qkv, kv, positions, slots, inv_freq, norm_w, cache, spec, eps, q, q_rot, copy_nope):
    n, qk = qkv.shape[0], spec.qk_dim
    src = qkv[:, :spec.q_rows].reshape(n, spec.heads, qk)
    q.zero_()
    if copy_nope:
        q[..., :spec.dim] = src[..., :spec.dim]
    q[..., q_rot:q_rot + spec.rot_dim] = rotate(src[..., spec.dim:], positions, inv_freq, spec.rot_adjacent, spec.rotary.factor).to(q.dtype)
    if cache is not None:
        c = kv[:, :spec.kv_rank].float()
        c = c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
        kr = rotate(kv[:, spec.kv_rank:spec.kv_rank + spec.rot_dim], positions, inv_freq, spec.rot_adjacent, spec.rotary.factor)
        keep = slots >= 0
        rows = cache.view(-1, cache.shape[-1])
        sl = slots[keep].long()
        rows[sl] = 0
        rows[sl, :spec.kv_rank] = c[keep].to(cache.dtype)
        rows[sl, spec.rank_pad:spec.rank_pad + spec.rot_dim] = kr[keep].to(cache.dtype)
    return q


def latent_attention(q, cache, batch, spec, window_left):
    out = torch.zeros(q.shape[0], spec.heads, spec.rank_pad, dtype=q.dtype)
    width = q.shape[2]
    for r in range(len(batch.kv_lens)):
        q0, q1, kl = int(batch.qo_indptr[r]), int(batch.qo_indptr[r + 1]), int(batch.kv_lens[r])
        if q1 == q0:
            continue
        pages = torch.as_tensor(batch.page_indices[int(batch.kv_page_indptr[r]):int(batch.kv_page_indptr[r + 1])]).long()
        k = cache[pages].reshape(-1, cache.shape[-1])[:kl, :width].float()
        s = torch.einsum("qhd,kd->hqk", q[q0:q1].float(), k) * spec.scale
        gap = torch.arange(kl - (q1 - q0), kl)[:, None] - torch.arange(kl)[None, :]
        allow = gap >= 0
        if batch.masks is not None and batch.masks[r] is not None:
            allow = torch.as_tensor(batch.masks[r])[:, :kl].bool()
        allow = allow & (gap <= window_left)
        pr = torch.softmax(s.masked_fill(~allow[None], float("-inf")), -1)
        pr = torch.nan_to_num(pr)           # a row that sees nothing gives zeros
        out[q0:q1] = torch.einsum("hqk,kd->qhd", pr, k[:, :spec.rank_pad]).to(q.dtype)
    return out


def xielu(z, act):
    a = torch.nn.functional.softplus(act[0].float())
    b = 0.5 + torch.nn.functional.softplus(act[1].float())
    neg = z.clamp(max=0)
    return torch.where(z > 0, a * z * z, b * (torch.expm1(neg) - neg)) + 0.5 * z


def bias_xielu(y, bias, act):
    y.copy_(xielu(y.float() + bias.float(), act).to(y.dtype))
    return y


def stream_add(x, d, bias, copy):
    out = x + d.float()
    if bias is not None:
        out = out + bias.float()
    return out, out.to(d.dtype)


def side_gate(z, table, tokens, col0, dim):
    g = torch.zeros_like(z)
    e = table[tokens.long(), col0:col0 + dim].float()
    g[:, :dim] = (torch.nn.functional.gelu(z[:, :dim].float(), approximate="tanh") * e).to(z.dtype)
    return g
