"""Plain, slow statement of the Retodra design: whole sequences from position 0, float32 (or float64), one function per
mechanism, no cache, no batching, no chunks. It shares no code with the package; the tests compare the framework's
kernels, cache, state and scheduler with it."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_about_one(x, w, eps):
    """RMS norm whose gain is stored as the distance from one."""
    return rms(x, eps) * (1 + w)


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def log_sigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-abs(z)))


def decayed_state(q, k, v, decay, keep=None):
    """o_t = S_t^T q_t with S_t = diag(decay_t) S_(t-1) + k_t v_t^T from S = 0. q, k, decay [T, H, K]; v [T, H, V].
    `keep` (a list) collects S after every token."""
    t, heads, dim = k.shape
    s = torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype)
    out = torch.zeros(t, heads, v.shape[-1], dtype=q.dtype)
    for i in range(t):
        s = decay[i][:, :, None] * s + k[i][:, :, None] * v[i][:, None, :]
        out[i] = (s * q[i][:, :, None]).sum(1)
        if keep is not None:
            keep.append(s)
    return out


def channel_decay(h, a1, a2, b, tau):
    """sigmoid(z)^(1 / tau) of a low-rank projection z of h."""
    return torch.exp(log_sigmoid((h @ a1.t()) @ a2.t() + b) / tau)


def gla(h, w, m, eps):
    """Gated linear attention; w holds the mixer's tensors by their short names."""
    t, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].t()).view(t, heads, dim) / math.sqrt(dim)
    k = (h @ w["k"].t()).view(t, heads, dim)
    v = (h @ w["v"].t()).view(t, heads, vdim)
    a = channel_decay(h, w["a1"], w["a2"], w["a2.b"], m["tau"]).view(t, heads, dim)
    o = rms(decayed_state(q, k, v, a), eps) * w["norm"]
    return (o.reshape(t, heads * vdim) * silu(h @ w["g"].t())) @ w["o"].t()


def lightning(h, w, m, eps):
    """Linear attention with a constant decay per head, one norm over all heads together and a sigmoid gate."""
    t, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].t()).view(t, heads, dim)
    k = silu(h @ w["k"].t()).view(t, heads, dim)
    v = silu(h @ w["v"].t()).view(t, heads, vdim)
    a = torch.tensor(m["decay"], dtype=h.dtype)[None, :, None].expand(t, heads, dim)
    o = rms(decayed_state(q, k, v, a).reshape(t, heads * vdim), eps) * w["norm"]
    return (o * sigmoid(h @ w["g"].t())) @ w["o"].t()


def distance_bucket(n, buckets, far):
    """Row of the bias table for a distance: one row each for the near half, then logarithmic up to `far`."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (buckets - half) + 1e-9))


def distance_bias(t, table, far):
    """[H, T, T] bias of query i on key j <= i."""
    rows = torch.tensor([distance_bucket(n, table.shape[0], far) for n in range(t)])
    gap = (torch.arange(t)[:, None] - torch.arange(t)[None, :]).clamp(min=0)
    return table[rows][gap].permute(2, 0, 1)


def softcap(s, cap):
    return cap * torch.tanh(s / cap)


def windowed_softmax(scores, window):
    """Softmax over the keys 0 <= i - j < window of scores [..., T, T]."""
    t = scores.shape[-1]
    gap = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return torch.softmax(scores.masked_fill((gap < 0) | (gap >= window), float("-inf")), -1)


def biased_attention(h, w, m, eps):
    """Grouped-query attention in a window: q, k normed over the whole projection, soft-capped scores, then the distance
    bias; a sigmoid gate ahead of the output projection."""
    t, heads, kv, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w["q"].t(), eps) * w["q.norm"]).view(t, heads, dim)
    k = (rms(h @ w["k"].t(), eps) * w["k.norm"]).view(t, kv, dim)
    v = (h @ w["v"].t()).view(t, kv, vdim)
    k, v = k.repeat_interleave(heads // kv, 1), v.repeat_interleave(heads // kv, 1)
    s = softcap(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], m["softcap"]) + distance_bias(t, w["rel"], m["bias_max"])
    o = torch.einsum("hij,jhd->ihd", windowed_softmax(s, m["mask"]["size"]), v).reshape(t, heads * vdim)
    return (o * sigmoid(h @ w["g"].t())) @ w["o"].t()


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def parallel(h, w, m, eps):
    return m["left_scale"] * biased_attention(h, sub(w, "left."), m["left"], eps) \
        + m["right_scale"] * lightning(h, sub(w, "right."), m["right"], eps)


def dense_ff(h, w):
    return (silu(h @ w["gate"].t()) * (h @ w["up"].t())) @ w["down"].t()


def clamped_expert(h, w, limit):
    g = torch.clamp(h @ w["gate"].t(), max=limit)
    u = torch.clamp(h @ w["up"].t(), -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w["down"].t()


def identity_expert(h):
    return h


def route(h, router, correction, top):
    """(ids, weights) [T, top]: chosen by score + correction, weighted by the score itself."""
    s = torch.softmax(h @ router.t(), -1)
    ids = torch.argsort(-(s + correction), dim=-1, stable=True)[:, :top]
    return ids, torch.gather(s, 1, ids)


def moe(h, w, mlp):
    r = mlp["router"]
    ids, weights = route(h, w["router"], w["correction"], r["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(ids[t].tolist(), weights[t]):
            y = identity_expert(h[t]) if e >= r["experts"] else clamped_expert(h[t], sub(w, f"e{e}."), mlp["expert"]["limit"])
            out[t] += c * y
    return out


def forward(cfg, w, tokens, dtype=torch.float32, trace=None):
    """Logits [T, vocab] of one sequence. `cfg` is the config.json dictionary, `w` its tensors by name; `trace` (a list)
    collects the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, spec in enumerate(cfg["layers"]):
        lw = sub(w, f"l{i}.")
        mix = {"gla": gla, "parallel": parallel}[spec["type"]]
        y = mix(norm_about_one(x, lw["norm1"], eps), sub(lw, "mix."), spec["mixer"], eps)
        x = x + norm_about_one(y, lw["norm1b"], eps) * lw["ls1"]
        mlp = spec.get("mlp")
        if mlp:
            h = norm_about_one(x, lw["norm2"], eps)
            y = moe(h, sub(lw, "mlp."), mlp) if mlp["kind"] == "moe" else dense_ff(h, sub(lw, "mlp."))
            x = x + norm_about_one(y, lw["norm2b"], eps) * lw["ls2"]
        if trace is not None:
            trace.append(x)
    return norm_about_one(x, w["final.norm"], eps) @ w["head"].t()
