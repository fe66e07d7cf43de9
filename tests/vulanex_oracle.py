"""Plain, slow statement of the Vulanex design: whole sequences from position 0, float32 (or float64), one function per
mechanism, no cache, no batching, no chunks. It shares no code with the package; the tests compare the framework's
kernels, cache, state and scheduler with it."""
import math

import torch


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


# ------------------------------------------------------------------ embedding, input convolution
def embedding(tokens, embed, bigram, mul_prev, mul_cur, buckets):
    """Token rows plus a row for the pair (token before, token); the first token's pair has a row of its own."""
    out, prev = [], None
    for t in tokens:
        row = buckets if prev is None else (prev * mul_prev + t * mul_cur) % buckets
        out.append(embed[t] + bigram[row])
        prev = t
    return torch.stack(out)


def input_convolution(h, w):
    """h [T, W] plus its causal convolution over time with w [W, taps], channel by channel."""
    t, taps = h.shape[0], w.shape[1]
    out = h.clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < t:
            out[back:] += w[:, j] * h[:t - back]
    return out


# ------------------------------------------------------------------ rotation
def stretched_frequencies(rot):
    """Angle per position of every pair and the factor on cos and sin: pairs that turn often over the original length are
    left alone, slow ones slowed down, a ramp over the pair's index between."""
    n, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if s is None:
        return torch.tensor(f, dtype=torch.float64), 1.0

    def at(turns):
        return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), n - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * ramp + x * (1 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1


def rotated(x, freq, factor=1.0, positions=None):
    """x [T, H, D] with its first 2 * len(freq) columns turned; the halves of a pair are len(freq) columns apart."""
    t, half = x.shape[0], len(freq)
    pos = torch.arange(t) if positions is None else torch.as_tensor(positions)
    a = (pos.double()[:, None] * freq)[:, None]
    c, s = (a.cos() * factor).to(x.dtype), (a.sin() * factor).to(x.dtype)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


# ------------------------------------------------------------------ attention
def query_factor(positions, coef, every):
    return 1 + coef * torch.log(torch.floor((positions + 1) / every) + 1)


def heads_of(h, w, n):
    return (h @ w.t()).view(h.shape[0], n, -1)


def warm_attention(h, w, m):
    """Grouped attention whose values are its keys, without positions but for a factor on the query."""
    t, g = h.shape[0], m["heads"] // m["kv_heads"]
    q, k = heads_of(h, w["q"], m["heads"]), heads_of(h, w["k"], m["kv_heads"]).repeat_interleave(g, 1)
    if m.get("q_temp"):
        q = q * query_factor(torch.arange(t).to(h.dtype), **m["q_temp"])[:, None, None]
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    s = s.masked_fill(torch.arange(t)[None] > torch.arange(t)[:, None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), k).reshape(t, -1) @ w["o"].t()


def block_means(x, pool):
    """Mean of every whole run of `pool` rows."""
    n = x.shape[0] // pool
    return x[:n * pool].view(n, pool, *x.shape[1:]).mean(1)


def seen_tokens(t, size):
    i, j = torch.arange(t)[:, None], torch.arange(t)[None]
    return (j <= i) & (i - j < size)


def seen_blocks(t, size, pool):
    """A block counts once its last token lies before the window."""
    i, b = torch.arange(t)[:, None], torch.arange(t // pool)[None]
    return b * pool + pool - 1 <= i - size


def weights_with_sink(scores, see, sink):
    """Softmax of scores [H, T, keys] over the seen ones, the denominator with one more exponential per head."""
    s = scores.masked_fill(~see, float("-inf"))
    top = torch.maximum(s.amax(-1, keepdim=True), sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def pooled_attention(h, w, m, eps):
    """Rotated and normed heads, a window of tokens beside one mean key and value for every block ahead of it."""
    t, g = h.shape[0], m["heads"] // m["kv_heads"]
    freq, factor = stretched_frequencies(m["rot"])
    q = rotated(rms(heads_of(h, w["q"], m["heads"]), eps) * w["q.norm"], freq, factor)
    k = rotated(rms(heads_of(h, w["k"], m["kv_heads"]), eps) * w["k.norm"], freq, factor)
    v = heads_of(h, w["v"], m["kv_heads"])
    size, pool = m["mask"]["size"], m["mask"]["pool"]
    keys = torch.cat([k, block_means(k, pool)]).repeat_interleave(g, 1)
    values = torch.cat([v, block_means(v, pool)]).repeat_interleave(g, 1)
    see = torch.cat([seen_tokens(t, size), seen_blocks(t, size, pool)], 1)
    p = weights_with_sink(torch.einsum("ihd,jhd->hij", q, keys) * m["scale"], see, w["sink"])
    return torch.einsum("hij,jhd->ihd", p, values).reshape(t, -1) @ w["o"].t()


# ------------------------------------------------------------------ delta rule
def decays(h, w):
    return torch.exp(-math.exp(-0.5) * sigmoid(torch.tanh(h @ w["w1"].t()) @ w["w2"].t() + w["w0"]))


def removal_rates(h, w):
    return sigmoid(h @ w["a"].t() + w["a.b"])


def unit(k):
    return k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)


def delta_rule(r, k, v, decay, rate, state=None):
    """r, k, v, decay, rate [T, H, D]. Returns (outputs [T, H, D], last state [H, D, D])."""
    t, n, d = r.shape
    s = torch.zeros(n, d, d, dtype=r.dtype) if state is None else state.clone()
    u, out = unit(k), []
    for i in range(t):
        old = torch.einsum("hd,hde->he", u[i], s)
        s = decay[i][..., None] * s - (rate[i] * u[i])[..., None] * old[:, None] + k[i][..., None] * v[i][:, None]
        out.append(torch.einsum("hde,hd->he", s, r[i]))
    return torch.stack(out), s


def delta_mixer(h, w, m, eps):
    t, n = h.shape[0], m["heads"]
    split = lambda x: x.view(t, n, -1)
    o, _ = delta_rule(split(h @ w["r"].t()), split(h @ w["k"].t()), split(h @ w["v"].t()), split(decays(h, w)), split(removal_rates(h, w)))
    return (rms(o, eps).reshape(t, -1) * w["norm"] * sigmoid(h @ w["g"].t())) @ w["o"].t()


def side_by_side(h, w, m, eps):
    left = pooled_attention(h, sub(w, "left."), m["left"], eps)
    right = delta_mixer(h, sub(w, "right."), m["right"], eps)
    return (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"]) / 2


def gated_ff(h, w):
    return (gelu_tanh(h @ w["gate"].t()) * (h @ w["up"].t())) @ w["down"].t()


# ------------------------------------------------------------------ the whole
def forward(cfg, tensors, tokens, dtype=torch.float32, layers=None):
    """Logits [T, vocab]; `layers`: a list that takes the residual stream after every layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = embedding(tokens, w["embed"], w["bigram"], **cfg["embedding"]["bigram"])
    for i, spec in enumerate(cfg["layers"]):
        lw = sub(w, f"l{i}.")
        h = input_convolution(layer_norm(x, lw["norm1"], lw["norm1.b"], eps), lw["canon1"])
        mw = sub(lw, "mix.")
        x = x + (warm_attention(h, mw, spec["mixer"]) if spec["type"] == "attention" else side_by_side(h, mw, spec["mixer"], eps))
        if spec["mlp"] is not None:
            h = input_convolution(layer_norm(x, lw["norm2"], lw["norm2.b"], eps), lw["canon2"])
            x = x + gated_ff(h, sub(lw, "mlp."))
        if layers is not None:
            layers.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].t() * cfg["logit_scale"]
