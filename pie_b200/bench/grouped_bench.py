"""Kernels of the Nukelix design and the like kernels of the designs beside it, each alone at the sizes of `nukelix-20b`:
matrix memory beside lightning attention, grouped and latent attention, rows, gates, norms, experts and logits. CUDA events,
a buffer larger than the L2 written between iterations. Prints time and the fraction of the slower roof (copy bandwidth and
bf16 GEMM throughput given on the command line).

    python -m pie_b200.bench.grouped_bench [--hbm 6452.8] [--tflops 1664.6] [--only <part of a name>]
"""
from __future__ import annotations

import argparse

import numpy as np
import torch

from .. import ops
from ..models.block_spec import BiasedAttentionSpec, ExpertsSpec, LightningSpec
from ..models.config import preset
from ..ops import grouped, latent as lops, linear as lin
from .latent_attn_bench import _decode_plan
from .linear_bench import BF16, Bench, _rs


def memory(b: Bench, cfg) -> None:
    s = cfg.blocks[0].mixer.right
    other = LightningSpec(s.heads, s.dim, s.vdim, [0.99] * s.heads)
    for label, lens in (("decode 64", [1] * 64), ("decode 256", [1] * 256), ("prompt 1 x 2048", [2048]), ("prompts 4 x 2048", [2048] * 4),
                        ("prompt 1 x 8192", [8192])):
        r, n, decode = len(lens), sum(lens), max(lens) == 1
        rs = _rs(np.concatenate([[0], np.cumsum(lens)]).tolist(), r)
        x = torch.randn(n, 2 * s.qk + s.values, **BF16)
        q, k, v = x[:, :s.qk], x[:, s.qk:2 * s.qk], x[:, 2 * s.qk:]
        h, w = torch.randn(n, cfg.hidden_size, **BF16), torch.randn(2 * s.heads, cfg.hidden_size, **BF16) * 0.02
        bias = torch.full((2 * s.heads,), 2.0, device="cuda")
        state = torch.zeros(r, s.state_elems, device="cuda")
        gates = lin.memory_gates(h, w, bias, s, rs, state, decode)[:2]
        b.run(f"exponential gates, {label}", lambda: lin.memory_gates(h, w, bias, s, rs, state, decode), 2.0 * h.numel() + 12.0 * n * s.heads,
              2.0 * h.numel() * 2 * s.heads)
        for name, spec, kw in (("matrix memory", s, dict(gates=gates)),
                               ("  lightning attention", other, dict(head_decay=torch.full((s.heads,), 0.99, device="cuda"), silu=True))):
            st = torch.zeros(r, -(-spec.state_elems // 4) * 4, device="cuda")[:, :spec.state_elems]
            moved = 2.0 * x.numel() + 4.0 * n * s.values + 8.0 * r * spec.state_elems
            b.run(f"{name}, {label}", lambda: lin.linear_attention(q, k, v, spec, rs, st, decode, q_scale=s.dim ** -0.5, **kw), moved,
                  4.0 * n * s.heads * s.dim * s.vdim)


def attention(b: Bench, cfg) -> None:
    full, win, lat = cfg.blocks[0].mixer.left, cfg.blocks[2].mixer, cfg.blocks[1].mixer
    D, hq, w = full.head_dim, full.heads, win.window
    zeros = torch.zeros(hq, device="cuda")
    for r in (16, 64, 256):
        kv, items = np.full(r, 2049, np.int64), r + 296 * 8
        scratch = torch.empty(ops.decode_scratch_floats(items, hq, max(D, lat.row)), device="cuda")
        even, pages = _decode_plan(kv, full.kv_heads, 0, items, scratch, "cuda", True)
        even.num_ctas = 2 * ops.num_sms()
        own, _ = _decode_plan(kv, full.kv_heads, 0, items, scratch, "cuda", False)
        cut, _ = _decode_plan(kv, full.kv_heads, w, items, scratch, "cuda", False)
        cache, q = torch.randn(pages + 1, 2, full.kv_heads, 16, D, **BF16), torch.randn(r, hq, D, **BF16)
        rs, slots = _rs(list(range(r + 1)), r), torch.zeros(r, dtype=torch.int32, device="cuda")
        moved = lambda keys: r * keys * 2.0 * full.kv_heads * D * 2 + 4.0 * q.numel()
        b.run(f"grouped attention, decode {r} x 2049", lambda: grouped.grouped_attention(q, cache, even, rs, slots, full), moved(2049))
        b.run(f"  plain attention on its own plan, decode {r} x 2049",
              lambda: ops.paged_decode_attention(q, cache, own, D ** -0.5, window_left=-1), moved(2049))
        b.run(f"windowed attention with kept tokens, decode {r} x 2049",
              lambda: grouped.grouped_attention(q, cache, even, rs, slots, win, zeros), moved(w + win.keep_first))
        b.run(f"  windowed attention on its own plan, decode {r} x 2049",
              lambda: ops.paged_decode_attention(q, cache, cut, D ** -0.5, window_left=w - 1), moved(w))
        lc, lq = torch.randn(pages + 1, 16, lat.row, **BF16), torch.randn(r, lat.heads, lat.row, **BF16)
        b.run(f"latent attention, decode {r} x 2049", lambda: lops.latent_attention(lq, lc, even, rs, slots, lat, 16, lat.window - 1),
              r * 2049 * lat.row * 2.0 + 2.0 * lq.numel() * 2)
    for r, n in ((1, 2048), (4, 2048), (1, 8192)):
        per, tot = n // 16, r * n
        batch = ops.AttnBatch(np.arange(r + 1, dtype=np.int32) * n, np.arange(r + 1, dtype=np.int32) * per,
                              np.random.default_rng(0).permutation(r * per).astype(np.int32), np.full(r, n, np.int32), None, -1)
        plan = ops.build_prefill_plan(batch, full.group, 16, "cuda", 256)
        plan.host = batch
        cache, q = torch.randn(r * per + 1, 2, full.kv_heads, 16, D, **BF16), torch.randn(tot, hq, D, **BF16)
        flops = lambda seen: 4.0 * r * sum(min(i + 1, seen) for i in range(n)) * hq * D
        moved = 4.0 * q.numel() + 4.0 * tot * full.kv_heads * D
        b.run(f"grouped attention, prompts {r} x {n}", lambda: grouped.grouped_attention(q, cache, plan, None, None, full), moved, flops(n))
        b.run(f"windowed attention with kept tokens, prompts {r} x {n}",
              lambda: grouped.grouped_attention(q, cache, plan, None, None, win, zeros), moved, flops(w + win.keep_first))
        b.run(f"  windowed attention, prompts {r} x {n}", lambda: ops.paged_prefill_attention(q, cache, plan, D ** -0.5, window_left=w - 1),
              moved, flops(w))


def rows(b: Bench, cfg) -> None:
    m, lat, W = cfg.blocks[0].mixer, cfg.blocks[1].mixer, cfg.hidden_size
    a, s = m.left, m.right
    nq, nk = a.heads * a.dim, a.kv_heads * a.dim
    biased = BiasedAttentionSpec(a.heads, a.kv_heads, a.dim, a.vdim, 1024, 1.0, 30.0, 2048, 32)
    for n in (64, 256, 8192):
        y = torch.randn(n, nq + 2 * nk, **BF16)
        q, k, v = y[:, :nq], y[:, nq:nq + nk], y[:, nq + nk:]
        cache = torch.zeros(n // 16 + 1, 2, a.kv_heads, 16, a.head_dim, **BF16)
        at = torch.arange(n, dtype=torch.int32, device="cuda")
        lw = {"q_b": torch.zeros(nq, **BF16), "k_b": torch.zeros(nk, **BF16), "v_b": torch.zeros(nk, **BF16), "q_norm": torch.ones(nq, **BF16),
              "k_norm": torch.ones(nk, **BF16), "rope": a.rot.frequencies("cuda")}
        first = torch.randn(n, nk, device="cuda")
        b.run(f"bias + norm + rotation + mixed values + KV write, {n} rows",
              lambda: grouped.grouped_rows(q, k, v, lw, at, at, cache, a, 1e-5, first, 0.4), 4.0 * y.numel() + 4.0 * first.numel())
        b.run(f"  norm over the projection + KV write, {n} rows",
              lambda: lin.biased_rows(q, k, v, lw["q_norm"], lw["k_norm"], at, cache, biased, 1e-5), 4.0 * y.numel())
        o1, g1, z1 = torch.randn(n, nq, **BF16), torch.randn(n, a.heads, **BF16), torch.empty(n, nq + s.values, **BF16)
        e1, o2, g2 = torch.randn(n, nq, **BF16), torch.randn(n, s.values, device="cuda"), torch.randn(n, s.values, **BF16)
        w2, den = torch.ones(s.values, **BF16), torch.ones(s.heads, n, device="cuda")
        right = lambda **kw: (o2, w2, g2, z1[:, nq:], dict(act="sigmoid", eps=1e-5, scale=1.0, **kw))
        b.run(f"gates of both mixers, {n} rows", lambda: lin.gated_norm([
            (o1, None, g1, z1[:, :nq], dict(act="sigmoid", norm_cols=0, scale=1.0, spec=a, gate_cols=a.vdim)),
            right(norm_cols=s.vdim, den=den, floor=den)]), 4.0 * o1.numel() + 8.0 * o2.numel())
        b.run(f"  elementwise gates of both mixers, {n} rows", lambda: lin.gated_norm([
            (o1, None, e1, z1[:, :nq], dict(act="sigmoid", norm_cols=0, scale=1.0, spec=a)), right(norm_cols=s.values)]),
            6.0 * o1.numel() + 8.0 * o2.numel())
        x, yy, gain = torch.randn(n, W, device="cuda"), torch.randn(n, W, **BF16), torch.ones(W, device="cuda")
        b.run(f"output norm + residual + copy, {n} rows",
              lambda: lops.stream_norm(x, W, 1e-5, yy, gain, dtype=torch.bfloat16, copy=True), 12.0 * x.numel())
        b.run(f"  output norm + residual + next norm, {n} rows",
              lambda: lops.stream_norm(x, W, 1e-5, yy, gain, gain, dtype=torch.bfloat16), 12.0 * x.numel())
        dq, cq = torch.randn(n, lat.q_rank, **BF16), torch.empty(n, lat.q_rank, **BF16)
        b.run(f"norm of the query latent, {n} rows", lambda: lin.gated_norm([
            (dq, torch.ones(lat.q_rank, **BF16), None, cq, dict(norm_cols=lat.q_rank, cols=lat.q_rank, eps=1e-5, scale=1.0))]), 4.0 * dq.numel())
        b.run(f"  RMS norm, {n} rows", lambda: ops.rmsnorm(yy, torch.ones(W, **BF16), 1e-5), 4.0 * yy.numel())
        lq, kv = torch.randn(n, lat.q_rows, **BF16), torch.randn(n, lat.kv_rank + lat.rot_dim, **BF16)
        lc, nw, table = torch.zeros(n // 16 + 1, 16, lat.row, **BF16), torch.ones(lat.kv_rank, **BF16), lat.rotary.frequencies("cuda")
        b.run(f"latent rows, {n} rows", lambda: lops.latent_rows(lq, at, at, table, nw, lc, lat, 1e-5, lops.projected_width(lat), lat.dim, True, kv),
              4.0 * lq.numel() + 4.0 * kv.numel())
        f, h = cfg.blocks[0].ff, torch.randn(n, W, **BF16)
        gu, dn = torch.randn(f.experts, 2 * f.ff, W, **BF16), torch.randn(f.experts, W, f.ff, **BF16)
        router = torch.randn(f.experts, W, **BF16) * W ** -0.5
        buf, buf2 = ops.MoeBuffers(n, W, f.ff, f.experts, f.top, "cuda"), ops.MoeBuffers(n, W, f.ff, f.experts, f.top, "cuda")
        wb, flops = 2.0 * (gu.numel() + dn.numel()), 6.0 * n * f.top * f.ff * W
        shared, scored = torch.randn(n, W, **BF16), ExpertsSpec(f.experts, 0, f.top, f.ff, 7.0)
        b.run(f"experts that read weighted inputs, {n} rows", lambda: lin.sigmoid_experts(h, router, gu, dn, f, buf, shared),
              wb + 6.0 * h.numel(), flops)
        b.run(f"  scored experts, {n} rows",
              lambda: lin.scored_experts(h, router, torch.zeros(f.experts, device="cuda"), gu, dn, scored, buf2), wb + 4.0 * h.numel(), flops)
        if n <= 256:
            logits = torch.randn(n, cfg.vocab_size, **BF16)
            b.run(f"soft cap of the logits, {n} rows", lambda: ops.softcap_(logits, cfg.final_softcap), 4.0 * logits.numel())


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--hbm", type=float, default=6452.8, help="copy bandwidth, GB/s")
    ap.add_argument("--tflops", type=float, default=1664.6, help="bf16 GEMM throughput")
    ap.add_argument("--only", default="", help="part of a line's name")
    a = ap.parse_args(argv)
    b, cfg = Bench(a.hbm, a.tflops, a.only), preset("nukelix-20b", num_hidden_layers=3)
    torch.manual_seed(0)
    ops.ensure_gemm_workspace("cuda:0")
    for part in (memory, attention, rows):
        part(b, cfg)
    ops.check_kernel_status()


if __name__ == "__main__":
    main()
