"""Plain, slow statement of the Puzutar block: whole sequences from position 0, float32 (or float64), one
function per mechanism, no cache, no batching. It shares no code with the package; the tests compare the
framework's kernels, cache and scheduler with it."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x, w, groups, eps):
    """Each of `groups` equal consecutive parts is divided by its own root mean square."""
    n = x.shape[-1] // groups
    return torch.cat([rms(x[..., g * n:(g + 1) * n], eps) for g in range(groups)], -1) * w


def token_shift(h, mix):
    """h_t + (h_{t-1} - h_t) * mix; the token before the first one is all zeros."""
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)
    return h + (prev - h) * mix


def rotate(x, pos, base):
    """Rotate-half rotation of the whole last dimension; x [T, ..., d], pos [T]."""
    d = x.shape[-1]
    i = torch.arange(d // 2, dtype=torch.float64)
    ang = (pos.double()[:, None] * base ** (-2.0 * i / d)).to(x.dtype)
    ang = ang.reshape(ang.shape[0], *([1] * (x.dim() - 2)), d // 2)
    u, v = x[..., :d // 2], x[..., d // 2:]
    return torch.cat([u * ang.cos() - v * ang.sin(), v * ang.cos() + u * ang.sin()], -1)


def latent_rows(h, w_dkv, norm_w, rank, base, eps):
    """What a layer keeps per token: the normalised latent and the rotated key part all heads share."""
    y = h @ w_dkv.t()
    return rms(y[:, :rank], eps) * norm_w, rotate(y[:, rank:], torch.arange(h.shape[0]), base)


def windowed_softmax(scores, window):
    """Softmax over the keys 0 <= i - j < window of scores [T, T]."""
    t = scores.shape[0]
    gap = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return torch.softmax(scores.masked_fill((gap < 0) | (gap >= window), float("-inf")), -1)


def latent_attention(h, c, k_rot, w_q, w_uk, w_uv, w_o, heads, dim, vdim, base, scale, window):
    q = (h @ w_q.t()).reshape(h.shape[0], heads, -1)
    pos = torch.arange(h.shape[0])
    out = []
    for n in range(heads):
        k = c @ w_uk[n * dim:(n + 1) * dim].t()
        v = c @ w_uv[n * vdim:(n + 1) * vdim].t()
        s = (q[:, n, :dim] @ k.t() + rotate(q[:, n, dim:], pos, base) @ k_rot.t()) * scale
        out.append(windowed_softmax(s, window) @ v)
    return torch.cat(out, -1) @ w_o.t()


def softplus(z):
    return torch.log1p(torch.exp(-abs(z))) + torch.clamp(z, min=0)


def xielu(z, p, q):
    a, b = softplus(p), 0.5 + softplus(q)
    neg = torch.clamp(z, max=0)
    return torch.where(z > 0, a * z * z, b * (torch.expm1(neg) - neg)) + 0.5 * z


def dense_ff(h, up, up_b, down, down_b, act):
    return xielu(h @ up.t() + up_b, act[0], act[1]) @ down.t() + down_b


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def token_side(x, e, gate, proj, norm_w, eps):
    return x + rms((gelu_tanh(x @ gate.t()) * e) @ proj.t(), eps) * norm_w


def forward(cfg, w, tokens, dtype=torch.float32, trace=None):
    """Logits [T, vocab] of one sequence. `cfg` is the config.json dictionary, `w` its tensors by name;
    `trace` (a list) collects the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    side = cfg["token_side"]["dim"]
    x = w["embed"][tokens]
    kept = {}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        h = grouped_norm(x, w[p + "norm1"], groups, eps)
        hs = token_shift(h, w[p + "shift"])
        if m.get("kv_from") is None:
            kept[i] = latent_rows(hs, w[p + "mix.dkv"], w[p + "mix.dkv.norm"], m["kv_rank"], m["rot"]["base"], eps)
        c, kr = kept[i if m.get("kv_from") is None else m["kv_from"]]
        y = latent_attention(hs, c, kr, w[p + "mix.q"], w[p + "mix.uk"], w[p + "mix.uv"], w[p + "mix.o"], m["heads"],
                             m["dim"], m["vdim"], m["rot"]["base"], m["scale"], m["mask"]["size"])
        if spec.get("mlp"):
            y = y + dense_ff(h, w[p + "mlp.up"], w[p + "mlp.up.b"], w[p + "mlp.down"], w[p + "mlp.down.b"], w[p + "mlp.act"])
        x = x + y
        x = token_side(x, w["side.embed"][tokens, i * side:(i + 1) * side], w[p + "side.gate"], w[p + "side.proj"],
                       w[p + "side.norm"], eps)
        if trace is not None:
            trace.append(x)
    return grouped_norm(x, w["final.norm"], groups, eps) @ w["embed"].t()
