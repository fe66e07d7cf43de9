"""Kernels of the Vulanex design and the like kernels of the designs beside it, each alone at the sizes of `vulanex-8b`: delta
rule beside Gated DeltaNet, attention on its own keys, pooled windows, rows, norms, decays, feed-forward. CUDA events, a buffer
larger than the L2 written between iterations. Prints time and the fraction of the slower roof (copy bandwidth and bf16 GEMM
throughput given on the command line).

    python -m pie_b200.bench.delta_bench [--hbm 6452.8] [--tflops 1664.6] [--only <part of a name>]
"""
from __future__ import annotations

import argparse

import numpy as np
import torch

from .. import ops
from ..models.block_spec import EVERYTHING, BiasedAttentionSpec, GroupedAttentionSpec, RotarySpec
from ..models.config import preset
from ..ops import delta, grouped, latent as lops, linear as lin, stream_conv as conv
from .latent_attn_bench import _decode_plan
from .linear_bench import BF16, Bench, _rs

LENGTHS = (("decode 64", [1] * 64), ("decode 256", [1] * 256), ("prompt 1 x 2048", [2048]), ("prompts 4 x 2048", [2048] * 4),
           ("prompt 1 x 8192", [8192]))


def mixers(b: Bench, cfg, nb) -> None:
    s = cfg.blocks[1].mixer.right
    hk, hv, dk, dv = nb.linear_num_key_heads, nb.linear_num_value_heads, nb.linear_key_head_dim, nb.linear_value_head_dim
    chans = nb.gdn_conv_channels
    bias, w2 = torch.zeros(s.qk, device="cuda"), torch.randn(s.qk, s.rank, **BF16) * s.rank ** -0.5
    for label, lens in LENGTHS:
        r, n, decode = len(lens), sum(lens), max(lens) == 1
        qo = np.concatenate([[0], np.cumsum(lens)]).tolist()
        x, w1 = torch.randn(n, 4 * s.qk, **BF16), torch.randn(n, s.rank, **BF16)
        q, k, v, a = x.split(s.qk, 1)
        logs = delta.bounded_decay_logs(w1, w2, bias.bfloat16(), s.bound)
        state, rs = torch.zeros(r, s.state_elems, device="cuda"), _rs(qo, r)
        moved = 2.0 * x.numel() + 4.0 * logs.numel() + 4.0 * n * s.values + 8.0 * r * s.state_elems
        b.run(f"delta rule, {label}", lambda: delta.delta_rule(q, k, v, a, bias, logs, s, rs, state, decode), moved, 6.0 * n * s.state_elems)
        b.run(f"bounded decays, {label}", lambda: delta.bounded_decay_logs(w1, w2, bias.bfloat16(), s.bound),
              2.0 * w1.numel() + 4.0 * logs.numel(), 2.0 * logs.numel() * s.rank)
        b.run(f"  channel decays of rank 16, {label}", lambda: lin.decay_logs(w1[:, :16], w2[:, :16].contiguous(), bias.bfloat16(), 16.0),
              2.0 * 16 * n + 4.0 * logs.numel(), 2.0 * logs.numel() * 16)
        mix = torch.randn(n, nb.gdn_in_features, **BF16)
        lw = {"gdn_conv": torch.randn(chans, 4, **BF16), "gdn_A_log": torch.zeros(hv, device="cuda"),
              "gdn_dt_bias": torch.zeros(hv, device="cuda"), "gdn_norm": torch.ones(dv, **BF16)}
        rs.conv_state, rs.rec_state = torch.zeros(1, r, chans, 3, device="cuda"), torch.zeros(1, r, hv, dk, dv, device="cuda")
        rs.scratch = torch.empty(n, chans, device="cuda")
        b.run(f"  Gated DeltaNet mixer (conv, norm, gate), {label}", lambda: ops.gdn_mixer(mix, lw, nb, rs, 0),
              2.0 * mix.numel() + 2.0 * n * hv * dv + 8.0 * r * hv * dk * dv, 6.0 * n * hv * dk * dv)


def attention(b: Bench, cfg) -> None:
    own, win = cfg.blocks[0].mixer, cfg.blocks[1].mixer.left
    D, hq, hkv, w = own.head_dim, own.heads, own.kv_heads, win.window
    sinks = (torch.zeros(hq, device="cuda"), torch.zeros(hq, device="cuda"))
    seen = lambda i: min(i + 1, w) + max(0, i + 1 - w) // win.pool
    for r in (16, 64, 256):
        n = 2049
        kv, items = np.full(r, n, np.int64), r + 296 * 8
        scratch = torch.empty(ops.decode_scratch_floats(items, hq, D), device="cuda")
        plan, pages = _decode_plan(kv, hkv, 0, items, scratch, "cuda", False)
        cut, _ = _decode_plan(kv, hkv, w, items, scratch, "cuda", False)
        cache, q = torch.randn(pages + 1, 2, hkv, 16, D, **BF16), torch.randn(r, hq, D, **BF16)
        keys, means = cache[:, :1].contiguous(), torch.randn(pages + 1, 2, hkv, -(-16 // win.pool), D, **BF16)
        rs, slots = _rs(list(range(r + 1)), r), torch.zeros(r, dtype=torch.int32, device="cuda")
        moved = lambda k, planes=2: r * k * 2.0 * hkv * D * planes + 4.0 * q.numel()
        b.run(f"attention on its own keys, decode {r} x {n}", lambda: grouped.laid_attention(q, keys, None, plan, rs, slots, own), moved(n, 1))
        b.run(f"  attention on keys and values, decode {r} x {n}",
              lambda: ops.paged_decode_attention(q, cache, plan, D ** -0.5, window_left=-1), moved(n))
        b.run(f"pooled window, decode {r} x {n}", lambda: grouped.laid_attention(q, cache, means, plan, rs, slots, win, sinks), moved(seen(n - 1)))
        b.run(f"  window on its own plan, decode {r} x {n}",
              lambda: ops.paged_decode_attention(q, cache, cut, D ** -0.5, window_left=w - 1, sinks_log2=sinks[1]), moved(w))
        b.run(f"means of completed blocks, decode {r} x {n}", lambda: grouped.pool_rows(cache, means, plan, rs, slots, win), 0.0)
    for r, n in ((1, 2048), (4, 2048), (1, 8192)):
        per, tot = n // 16, r * n
        batch = ops.AttnBatch(np.arange(r + 1, dtype=np.int32) * n, np.arange(r + 1, dtype=np.int32) * per,
                              np.random.default_rng(0).permutation(r * per).astype(np.int32), np.full(r, n, np.int32), None, -1)
        plan = ops.build_prefill_plan(batch, own.group, 16, "cuda", 256)
        plan.host = batch
        rs, slots = _rs((np.arange(r + 1) * n).tolist(), r), torch.zeros(tot, dtype=torch.int32, device="cuda")
        cache, q = torch.randn(r * per + 1, 2, hkv, 16, D, **BF16), torch.randn(tot, hq, D, **BF16)
        keys, means = cache[:, :1].contiguous(), torch.randn(r * per + 1, 2, hkv, -(-16 // win.pool), D, **BF16)
        flops = lambda f: 4.0 * r * sum(f(i) for i in range(n)) * hq * D
        moved = lambda planes=2: 4.0 * q.numel() + 2.0 * tot * hkv * D * planes
        b.run(f"attention on its own keys, prompts {r} x {n}", lambda: grouped.laid_attention(q, keys, None, plan, rs, slots, own), moved(1),
              flops(lambda i: i + 1))
        b.run(f"  attention on keys and values, prompts {r} x {n}", lambda: ops.paged_prefill_attention(q, cache, plan, D ** -0.5), moved(),
              flops(lambda i: i + 1))
        b.run(f"pooled window, prompts {r} x {n}", lambda: grouped.laid_attention(q, cache, means, plan, rs, slots, win, sinks), moved(), flops(seen))
        b.run(f"  window, prompts {r} x {n}", lambda: ops.paged_prefill_attention(q, cache, plan, D ** -0.5, window_left=w - 1, sinks_log2=sinks[1]),
              moved(), flops(lambda i: min(i + 1, w)))
        b.run(f"means of completed blocks, prompts {r} x {n}", lambda: grouped.pool_rows(cache, means, plan, rs, slots, win),
              4.0 * tot * hkv * D * (1 + 1 / win.pool))


def rows(b: Bench, cfg) -> None:
    own, m, W = cfg.blocks[0].mixer, cfg.blocks[1].mixer, cfg.hidden_size
    a, s = m.left, m.right
    nq, nk = a.heads * a.dim, a.kv_heads * a.dim
    biased = BiasedAttentionSpec(a.heads, a.kv_heads, a.dim, a.vdim, 1024, 1.0, 30.0, 2048, 32)
    all_heads = GroupedAttentionSpec(a.heads, a.kv_heads, a.dim, a.vdim, 1.0, RotarySpec(a.dim, 1e4))
    for n in (64, 256, 8192):
        y = torch.randn(n, nq + 2 * nk, **BF16)
        q, k, v = y[:, :nq], y[:, nq:nq + nk], y[:, nq + nk:]
        cache = torch.zeros(n // 16 + 1, 2, a.kv_heads, 16, a.head_dim, **BF16)
        keys = torch.zeros(n // 16 + 1, 1, a.kv_heads, 16, a.head_dim, **BF16)
        at = torch.arange(n, dtype=torch.int32, device="cuda")
        gain = torch.ones(a.dim, device="cuda")
        lw = {"q_gain": gain, "k_gain": gain, "rope": a.rot.frequencies("cuda")}
        b.run(f"norm per head + rotation + KV write, {n} rows", lambda: grouped.head_rows(q, k, v, lw, at, at, cache, a, 1e-5), 4.0 * y.numel())
        b.run(f"query factor + key write, {n} rows", lambda: grouped.head_rows(q, k, None, {}, at, at, keys, own, 1e-5), 4.0 * (nq + nk) * n)
        gl = {"q_b": torch.zeros(nq, **BF16), "k_b": torch.zeros(nk, **BF16), "v_b": torch.zeros(nk, **BF16), "q_norm": torch.ones(nq, **BF16),
              "k_norm": torch.ones(nk, **BF16), "rope": lw["rope"]}
        b.run(f"  bias + norm + rotation + KV write, {n} rows", lambda: grouped.grouped_rows(q, k, v, gl, at, at, cache, all_heads, 1e-5),
              4.0 * y.numel())
        b.run(f"  norm over the projection + KV write, {n} rows",
              lambda: lin.biased_rows(q, k, v, gl["q_norm"], gl["k_norm"], at, cache, biased, 1e-5), 4.0 * y.numel())
        x, yl, yr, g32 = torch.randn(n, W, device="cuda"), torch.randn(n, W, **BF16), torch.randn(n, W, **BF16), torch.ones(W, device="cuda")
        lens = [1] * n if n <= 256 else [2048] * (n // 2048)
        rs = _rs(np.concatenate([[0], np.cumsum(lens)]).tolist(), len(lens))
        taps, back = torch.randn(cfg.conv_taps, W, device="cuda"), (cfg.conv_taps - 1) * W
        hist = torch.zeros(len(lens), back, device="cuda")
        rs.conv_stage = torch.empty(len(lens), back, device="cuda")
        carried = 8.0 * hist.numel()
        b.run(f"layer norm + convolution, {n} rows", lambda: conv.conv_norm(x, W, 1e-5, (), g32, g32, taps, hist, rs, torch.bfloat16),
              6.0 * x.numel() + carried)
        b.run(f"two normed outputs + layer norm + convolution, {n} rows",
              lambda: conv.conv_norm(x, W, 1e-5, ((yl, g32), (yr, g32)), g32, g32, taps, hist, rs, torch.bfloat16), 14.0 * x.numel() + carried)
        shift, rs.shift_state, rs.shift_stage = torch.rand(W, **BF16), torch.zeros(1, len(lens), W, device="cuda"), rs.conv_stage
        b.run(f"  output norm + residual + norm + token shift, {n} rows",
              lambda: lops.stream_norm(x, W, 1e-5, yl, shift, shift, shift=shift, rs=rs), 14.0 * x.numel() + 8.0 * len(lens) * W)
        b.run(f"  output norm + residual + next norm, {n} rows",
              lambda: lops.stream_norm(x, W, 1e-5, yl, g32, g32, dtype=torch.bfloat16), 12.0 * x.numel())
        o, g, z, wn = torch.randn(n, s.values, device="cuda"), torch.randn(n, s.values, **BF16), torch.empty(n, s.values, **BF16), \
            torch.ones(s.values, **BF16)
        b.run(f"norm per head + gate, {n} rows",
              lambda: lin.gated_norm([(o, wn, g, z, dict(act="sigmoid", norm_cols=s.dim, eps=1e-5, scale=1.0))]), 8.0 * o.numel())
        h, ff = torch.randn(n, W, **BF16), cfg.blocks[0].ff.ff
        gu, dn = torch.randn(2 * ff, W, **BF16) * 0.02, torch.randn(W, ff, **BF16) * 0.02
        act = torch.randn(n, ff, **BF16)
        b.run(f"gate and up with GELU, {n} rows", lambda: ops.gemm(h, gu, epilogue=ops.EPI_GEGLU), 2.0 * (gu.numel() + h.numel() + act.numel()),
              2.0 * n * gu.numel())
        b.run(f"  gate and up with SiLU, {n} rows", lambda: ops.gemm(h, gu, epilogue=ops.EPI_SWIGLU), 2.0 * (gu.numel() + h.numel() + act.numel()),
              2.0 * n * gu.numel())
        b.run(f"down into the stream, {n} rows", lambda: lops.gemm_stream(act, dn, None, x), 2.0 * (dn.numel() + act.numel()) + 8.0 * x.numel(),
              2.0 * n * dn.numel())
        b.run(f"  down with residual, {n} rows", lambda: ops.gemm(act, dn, residual=h, epilogue=ops.EPI_RESIDUAL),
              2.0 * (dn.numel() + act.numel()) + 4.0 * x.numel(), 2.0 * n * dn.numel())
        rs2, pair = _rs(np.concatenate([[0], np.cumsum(lens)]).tolist(), len(lens)), cfg.token_pairs
        rs2.linear_state, rs2.token_at = torch.zeros(len(lens), 4, device="cuda"), 0
        table, pairs = torch.randn(4096, W, **BF16), torch.randn(pair.buckets + 1, W, **BF16)
        ids = torch.randint(0, 4096, (n,), dtype=torch.int32, device="cuda")
        b.run(f"token and pair rows, {n} rows", lambda: conv.pair_embed(ids, table, pairs, pair, W, rs2), 8.0 * n * W)
        b.run(f"  token rows, {n} rows", lambda: lops.stream_embed(ids, table, W), 6.0 * n * W)


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--hbm", type=float, default=6452.8, help="copy bandwidth, GB/s")
    ap.add_argument("--tflops", type=float, default=1664.6, help="bf16 GEMM throughput")
    ap.add_argument("--only", default="", help="part of a line's name")
    a = ap.parse_args(argv)
    b, cfg = Bench(a.hbm, a.tflops, a.only), preset("vulanex-8b", num_hidden_layers=2)
    assert cfg.blocks[0].mixer.window == EVERYTHING
    torch.manual_seed(0)
    ops.ensure_gemm_workspace("cuda:0")
    mixers(b, cfg, preset("gdn-8b"))
    attention(b, cfg)
    rows(b, cfg)
    ops.check_kernel_status()


if __name__ == "__main__":
    main()
