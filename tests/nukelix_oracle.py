"""Plain, slow statement of the Nukelix design: whole sequences from position 0, float32 (or float64), one function per
mechanism, no cache, no batching, no chunks. It shares no code with the package; the tests compare the framework's
kernels, cache, state and scheduler with it."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gained_norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-abs(z)))


def soft_limit(z, cap):
    return cap * torch.tanh(z / cap)


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


# ------------------------------------------------------------------ rotation
def frequencies(rot):
    """Angle per position of every rotated pair, unscaled."""
    return torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)], dtype=torch.float64)


def stretched_by_wavelength(f, factor, low, high, original):
    """Long waves are slowed down by `factor`, short ones left alone, those between in proportion."""
    out = []
    for x in f.tolist():
        wave = 2 * math.pi / x
        if wave < original / high:
            out.append(x)
        elif wave > original / low:
            out.append(x / factor)
        else:
            share = (original / wave - low) / (high - low)
            out.append((1 - share) * x / factor + share * x)
    return torch.tensor(out, dtype=torch.float64)


def stretched_by_index(f, rot, factor, original, fast, slow):
    """Pairs that turn more than `fast` times over the original length are left alone, those below `slow` turns slowed
    down by `factor`, a ramp over the pair's index between. Returns the frequencies and the factor on cos and sin."""
    def at(turns):
        return rot["dims"] * math.log(original / (2 * math.pi * turns)) / (2 * math.log(rot["base"]))
    lo, hi = max(math.floor(at(fast)), 0), min(math.ceil(at(slow)), rot["dims"] - 1)
    ramp = torch.tensor([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))], dtype=torch.float64)
    return f / factor * ramp + f * (1 - ramp), 0.1 * math.log(factor) + 1


def rotated(x, freq, adjacent, factor=1.0, positions=None):
    """x [T, ..., D] with its first 2 * len(freq) columns turned by position * frequency; the two halves of a pair are
    neighbours (`adjacent`) or half the rotated width apart."""
    t, half = x.shape[0], len(freq)
    pos = torch.arange(t) if positions is None else torch.as_tensor(positions)
    a = (pos.double()[:, None] * freq).reshape(t, *([1] * (x.dim() - 2)), half)
    c, s = (a.cos() * factor).to(x.dtype), (a.sin() * factor).to(x.dtype)
    out = x.clone()
    for i in range(half):
        p, q = (2 * i, 2 * i + 1) if adjacent else (i, i + half)
        u, v = x[..., p], x[..., q]
        out[..., p] = u * c[..., i] - v * s[..., i]
        out[..., q] = v * c[..., i] + u * s[..., i]
    return out


# ------------------------------------------------------------------ attention
def visible(t, window=None, keep_first=0):
    """[T, T]: query i sees key j."""
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    if window is None:
        return j <= i
    return (j <= i) & ((i - j < window) | (j < keep_first))


def weights_over_keys(scores, see, sink):
    """Softmax of scores [..., T, T] over the seen keys; with a sink, a further score of 0 takes its share."""
    s = scores.masked_fill(~see, float("-inf"))
    m = s.amax(-1, keepdim=True)
    if sink:
        m = m.clamp(min=0)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + (torch.exp(-m) if sink else 0))


def projected_heads(h, w, m, eps, name):
    """One biased projection, normed over all its rows where it is a query or a key, split into heads."""
    y = h @ w[name].t() + w[name + ".b"]
    if name != "v":
        y = gained_norm(y, w[name + ".norm"], eps)
    return y.view(h.shape[0], m["heads"] if name == "q" else m["kv_heads"], -1)


def mixed_values(v, first, lam):
    return (1 - lam) * v + lam * first


def head_gate(o, h, g):
    """o [T, H, V] times one sigmoid per head of a projection of the mixer's input."""
    return o * sigmoid(h @ g.t())[..., None]


def grouped_attention(h, w, m, eps, adjacent, sink, first_values=None, keep=None):
    """Grouped-query attention. `keep` (a list) collects the values as attended to."""
    t, groups = h.shape[0], m["heads"] // m["kv_heads"]
    rot = m["rot"]
    f, s = frequencies(rot), rot.get("scaling")
    if s:
        f = stretched_by_wavelength(f, s["factor"], s["low"], s["high"], s["original"])
    q = rotated(projected_heads(h, w, m, eps, "q"), f, adjacent)
    k = rotated(projected_heads(h, w, m, eps, "k"), f, adjacent)
    v = projected_heads(h, w, m, eps, "v")
    if first_values is not None:
        v = mixed_values(v, first_values, w["vmix"])
    if keep is not None:
        keep.append(v)
    k, v = k.repeat_interleave(groups, 1), v.repeat_interleave(groups, 1)
    mask = m.get("mask")
    see = visible(t, mask["size"], mask["keep_first"]) if mask else visible(t)
    p = weights_over_keys(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], see, sink)
    o = head_gate(torch.einsum("hij,jhd->ihd", p, v), h, w["g"])
    return o.reshape(t, -1) @ w["o"].t()


def latent_attention(h, w, m, eps):
    t, H, d, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    rot, s = m["rot"], m["rot"].get("scaling")
    f, factor = frequencies(rot), 1.0
    if s:
        f, factor = stretched_by_index(f, rot, s["factor"], s["original"], s["fast"], s["slow"])
    q = (gained_norm(h @ w["dq"].t(), w["dq.norm"], eps) @ w["uq"].t()).view(t, H, d + r)
    q_plain, q_rot = q[..., :d], rotated(q[..., d:], f, True, factor)
    low = h @ w["dkv"].t()
    c = gained_norm(low[:, :m["kv_rank"]], w["dkv.norm"], eps)
    k_rot = rotated(low[:, m["kv_rank"]:], f, True, factor)
    k_plain, v = (c @ w["uk"].t()).view(t, H, d), (c @ w["uv"].t()).view(t, H, m["vdim"])
    score = (torch.einsum("ihd,jhd->hij", q_plain, k_plain) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    o = head_gate(torch.einsum("hij,jhd->ihd", weights_over_keys(score, visible(t), False), v), h, w["g"])
    return o.reshape(t, -1) @ w["o"].t()


# ------------------------------------------------------------------ matrix memory
def log_gates(h, w, cap):
    """Logarithms of the input and forget gates, [T, H] each."""
    i = soft_limit(h @ w["i"].t() + w["i.b"], cap)
    f = log_sigmoid(soft_limit(h @ w["f"].t() + w["f.b"], cap))
    return i, f


def matrix_memory(q, k, v, i, f, state=None):
    """q, k [T, H, K], v [T, H, V], gates [T, H]; returns o [T, H, V] and the state (S, n, m) after the last token."""
    t, H, K = k.shape
    if state is None:
        state = (q.new_zeros(H, K, v.shape[-1]), q.new_zeros(H, K), q.new_zeros(H))
    s, n, m = state
    out = []
    for x in range(t):
        new = torch.maximum(f[x] + m, i[x])
        keep, add = torch.exp(f[x] + m - new), torch.exp(i[x] - new)
        s = keep[:, None, None] * s + add[:, None, None] * k[x][:, :, None] * v[x][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[x]
        m = new
        size = torch.maximum((n * q[x]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append((s * q[x][:, :, None]).sum(1) / size[:, None])
    return torch.stack(out) if out else v, (s, n, m)


def memory_mixer(h, w, m, eps):
    t, H = h.shape[0], m["heads"]
    q = (h @ w["q"].t()).view(t, H, m["dim"]) * m["dim"] ** -0.5
    k, v = (h @ w["k"].t()).view(t, H, m["dim"]), (h @ w["v"].t()).view(t, H, m["vdim"])
    i, f = log_gates(h, w, m["gate_cap"])
    o = rms(matrix_memory(q, k, v, i, f)[0], eps).reshape(t, -1) * w["norm"]
    return (o * sigmoid(h @ w["g"].t())) @ w["o"].t()


def parallel(h, w, m, eps):
    return m["left_scale"] * grouped_attention(h, sub(w, "left."), m["left"], eps, False, False) \
        + m["right_scale"] * memory_mixer(h, sub(w, "right."), m["right"], eps)


# ------------------------------------------------------------------ experts
def expert(h, w):
    return (silu(h @ w["gate"].t()) * (h @ w["up"].t())) @ w["down"].t()


def route(h, router, top):
    """(ids, weights) [T, top] by sigmoid score, the weights not summing to one."""
    s = sigmoid(h @ router.t())
    ids = torch.argsort(-s, dim=-1, stable=True)[:, :top]
    return ids, torch.gather(s, 1, ids)


def weighted_expert(h, c, w):
    """The weight scales what goes into the expert."""
    return expert(c * h, w)


def experts(h, w, mlp):
    ids, weights = route(h, w["router"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, j = (ids == e).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += weighted_expert(h[rows], weights[rows, j][:, None], sub(w, f"e{e}."))
    if mlp.get("shared"):
        out = out + expert(h, sub(w, "shared."))
    return out


# ------------------------------------------------------------------ model
def forward(cfg, w, tokens, dtype=torch.float32, trace=None):
    """Logits [T, vocab] of one sequence. `cfg` is the config.json dictionary, `w` its tensors by name; `trace` (a list)
    collects the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    first = None
    for i, spec in enumerate(cfg["layers"]):
        lw, m = sub(w, f"l{i}."), spec["mixer"]
        mw = sub(lw, "mix.")
        if spec["type"] == "parallel":
            y = parallel(x, mw, m, eps)
        elif spec["type"] == "latent_attention":
            y = latent_attention(x, mw, m, eps)
        else:
            kept = []
            y = grouped_attention(x, mw, m, eps, True, True, first if m.get("v_mix") else None, kept)
            if m.get("v_mix") and first is None:
                first = kept[0]
        x = x + gained_norm(y, lw["norm1"], eps)
        if spec.get("mlp"):
            x = x + gained_norm(experts(x, sub(lw, "mlp."), spec["mlp"]), lw["norm2"], eps)
        if trace is not None:
            trace.append(x)
    return soft_limit(gained_norm(x, w["final.norm"], eps) @ w["embed"].t(), cfg["logit_softcap"])
