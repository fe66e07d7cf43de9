"""Blocks over a 32-bit residual stream whose layers are described one by one, each with a mixer and a dense or expert
feed-forward of its own. Sandwich-normed (Retodra): x += ls1 * norm1b(mixer(norm1(x))), then the same with the feed-forward,
mixers gated linear attention, or windowed attention with a distance bias beside lightning attention. Normed on the way out
only (Nukelix): x += norm1(mixer(x)), mixers in `mixers.py`. Read through a layer norm and a convolution (Vulanex): x +=
mixer(conv(norm1(x))), whose sublayers end in a product that accumulates into the stream.

Output norm, layer scale, residual sum and the next input norm are one pass over the stream (`ResidualStream`); the
projections of a mixer are one GEMM, also those of two mixers side by side, whose output projections are one GEMM over
their heads next to each other.
"""
from __future__ import annotations

import torch

from ..ops import latent as lops, linear as lin, linear_reference as lref, stream_conv as conv
from .block_spec import BiasedAttentionSpec, ExpertsSpec, GatedLinearSpec, projection_columns
from .config import _pad
from .mixers import mixer_of, prepare_mixer
from .moe import _buffers


def prepare_blocks(m) -> None:
    """Derived tensors: 32-bit gains (with what a design adds to them: 1, the layer scale on the way out), bias by distance,
    decays, and those of `mixers.py`."""
    cfg, tables = m.cfg, {}
    m.vocab_local = cfg.vocab_size
    with_cache = [li for li, b in enumerate(cfg.blocks) if b.latent is not None or b.attention is not None]
    m.cache_index = {li: i for i, li in enumerate(with_cache)}
    if cfg.tie_word_embeddings and m.w["lm_head"].shape == m.w["embed"].shape:
        m.w["lm_head"] = m.w["embed"]                   # tied and unpadded: one copy
    gain = lambda w: (1.0 + w.float() if cfg.norm_plus_one else w.float()).contiguous()
    m.final_gain = gain(m.w["final_norm"])
    if cfg.layer_norm:              # the factor on the logits goes into the norm ahead of their product
        m.final_gain, m.final_offset = m.final_gain * cfg.logit_scale, m.w["final_norm_b"].float() * cfg.logit_scale
    for b, lw in zip(cfg.blocks, m.w["layers"]):
        for h in ("1", "2") if b.ff is not None else ("1",):
            if cfg.layer_norm:
                lw["gain" + h], lw["offset" + h] = lw["ln" + h].float().contiguous(), lw[f"ln{h}_b"].float().contiguous()
                if cfg.conv_taps:   # [taps, width], the input itself counted in
                    taps = lw["conv" + h].float().t().contiguous()
                    taps[-1] += 1.0
                    lw["taps" + h] = taps
                continue
            lw[f"gain{h}b"] = gain(lw[f"ln{h}b"])
            if not cfg.post_norm:
                lw["gain" + h] = gain(lw["ln" + h])
                lw[f"gain{h}b"] *= lw["ls" + h].float()
        if isinstance(b.ff, ExpertsSpec):
            lw["top"] = b.ff.top
        lw["columns"] = projection_columns(b.mixer)
        if mixer_of(b) is not None:
            prepare_mixer(m, b, lw, tables)
        elif isinstance(b.attention, BiasedAttentionSpec):
            lw["bias_table"] = lin.bias_table(lw["rel"], b.mixer.left, m.device)
            lw["head_decay"] = torch.tensor(b.mixer.right.decay, dtype=torch.float32, device=m.device)


def gla_mixer(m, h, lw: dict, li: int, fi, cache, st) -> torch.Tensor:
    s, eps = m.cfg.blocks[li].mixer, m.cfg.rms_norm_eps
    y = m._gemm(h, lw["w_in"])
    col = {k: y[:, a:a + n] for k, (a, n) in lw["columns"].items()}
    logs = lin.decay_logs(col["a1"], lw["a2"], lw["a2_b"], s.tau)
    o = lin.linear_attention(col["q"], col["k"], col["v"], s, fi.rs, fi.rs.state_of(li, s.state_elems), fi.is_decode, log_decay=logs,
                             q_scale=s.dim ** -0.5)
    z = torch.empty(h.shape[0], lw["w_out"].shape[1], dtype=h.dtype, device=h.device)
    lin.gated_norm([(o, lw["o_norm"], col["g"], z, dict(act="silu", norm_cols=s.vdim, eps=eps, scale=1.0))])
    return m._gemm(z, lw["w_out"])


def parallel_mixer(m, h, lw: dict, li: int, fi, cache, st) -> torch.Tensor:
    s, eps = m.cfg.blocks[li].mixer, m.cfg.rms_norm_eps
    a, r = s.left, s.right
    y = m._gemm(h, lw["w_in"])
    col = {k: y[:, c:c + n] for k, (c, n) in lw["columns"].items()}
    pages = cache[m.cache_index[li]]
    q = lin.biased_rows(col["left.q"], col["left.k"], col["left.v"], lw["q_norm"], lw["k_norm"], fi.slots, pages, a, eps)
    left = lin.biased_attention(q, pages, lw["bias_table"], fi.attn, fi.rs, fi.slots, a)
    right = lin.linear_attention(col["right.q"], col["right.k"], col["right.v"], r, fi.rs, fi.rs.state_of(li, r.state_elems), fi.is_decode,
                                 head_decay=lw["head_decay"], silu=True)
    n, cut = h.shape[0], _pad(a.heads * a.vdim)
    z = torch.empty(n, lw["w_out"].shape[1], dtype=h.dtype, device=h.device)       # gated heads of both, side by side
    lin.gated_norm([(left.view(n, -1), None, col["left.g"], z[:, :cut], dict(act="sigmoid", norm_cols=0, scale=s.left_scale, spec=a)),
                    (right, lw["o_norm"], col["right.g"], z[:, cut:], dict(act="sigmoid", norm_cols=r.values, eps=eps, scale=s.right_scale))])
    return m._gemm(z, lw["w_out"])


def expert_ff(m, h, lw: dict, spec: ExpertsSpec) -> torch.Tensor:
    gate_up, down = lw["experts_gate_up"], lw["experts_down"]
    shared = m._gemm(m._gemm(h, lw["shared_gate_up"], swiglu=True), lw["shared_down"]) if spec.shared else None
    if h.is_cuda and h.dtype == torch.bfloat16:
        buf = _buffers(m, h.shape[0], lw, h.device)
        if spec.score == "sigmoid":
            return lin.sigmoid_experts(h, lw["router"], gate_up, down, spec, buf, shared)
        return lin.scored_experts(h, lw["router"], lw["correction"], gate_up, down, spec, buf)
    logits = torch.matmul(h.float(), lw["router"].float().t())
    if spec.score == "sigmoid":
        y = lref.sigmoid_experts(h, logits, gate_up, down, spec)
        return y if shared is None else y + shared
    return lref.experts(h, logits, lw["correction"], gate_up, down, spec)


def block(m, st, lw: dict, li: int, fi, cache) -> None:
    cfg = m.cfg
    b = cfg.blocks[li]
    if cfg.layer_norm:
        mixer_of(b)(m, st.convolved(cfg, lw, "1", li, fi.rs, m.dtype), lw, li, fi, cache, st)
        if b.ff is not None:
            h = st.convolved(cfg, lw, "2", li, fi.rs, m.dtype)
            st.add_product(m._gemm(h, lw["w_gate_up"], glu=b.ff.act), lw["w_down"])
        return
    read = lambda half: st.plain(cfg, m.dtype) if cfg.post_norm else st.normed(cfg, lw["gain" + half], m.dtype)
    mixer = mixer_of(b) or (gla_mixer if isinstance(b.mixer, GatedLinearSpec) else parallel_mixer)
    st.y = mixer(m, read("1"), lw, li, fi, cache, st)
    st.y_norm = lw["gain1b"]
    if b.ff is None:
        return
    h = read("2")
    if isinstance(b.ff, ExpertsSpec):
        st.y = expert_ff(m, h, lw, b.ff)
    else:
        st.y = m._gemm(m._gemm(h, lw["w_gate_up"], swiglu=True), lw["w_down"])
    st.y_norm = lw["gain2b"]


def final_rows(m, rows) -> torch.Tensor:
    """The model's norm on the rows that need logits."""
    if m.cfg.layer_norm:
        return conv.conv_norm(rows, m.cfg.hidden_size, m.cfg.rms_norm_eps, w=m.final_gain, b=m.final_offset, dtype=m.dtype)[1]
    return lops.stream_norm(rows, m.cfg.hidden_size, m.cfg.rms_norm_eps, norm_w=m.final_gain, dtype=m.dtype)[1]
