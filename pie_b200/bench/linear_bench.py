"""Kernels of the Retodra design and of its neighbour model (`bench.py --config 8`), each alone: linear mixers, windowed
attention, rows, gates, norms and experts at the sizes of `retodra-19b`. CUDA events, a buffer larger than the L2 written
between iterations. Prints time and the fraction of the slower roof (copy bandwidth and bf16 GEMM throughput given on the
command line).

    python -m pie_b200.bench.linear_bench [--hbm 6538.9] [--tflops 1608.3] [--only <part of a name>]
"""
from __future__ import annotations

import argparse

import numpy as np
import torch

from .. import ops
from ..driver.recurrent import RecurrentInputs
from ..models.config import preset
from ..ops import latent as lops, linear as lin
from .latent_attn_bench import _decode_plan, _time

BF16 = dict(dtype=torch.bfloat16, device="cuda")


def _rs(qo, slots: int) -> RecurrentInputs:
    t = lambda a: torch.from_numpy(np.asarray(a, np.int32)).cuda()
    r = len(qo) - 1
    return RecurrentInputs(t(qo), t(np.repeat(np.arange(r), np.diff(qo))), t(np.arange(r)), t(np.zeros(r)), list(qo), list(range(r)),
                           [0] * r, None, None, {})


class Bench:
    def __init__(self, hbm: float, tflops: float, only: str):
        self.hbm, self.tflops, self.only = hbm * 1e9, tflops * 1e12, only
        self.flush = torch.empty(64 << 20, dtype=torch.float32, device="cuda")

    def run(self, name: str, fn, nbytes: float, flops: float = 0.0) -> None:
        if self.only in name:
            s, roof = _time(fn, self.flush), max(nbytes / self.hbm, flops / self.tflops)
            print(f"{name:64s} {s * 1e6:9.1f} us   {nbytes / 1e6:8.1f} MB {flops / 1e9:8.1f} GFLOP   {roof / s:5.2f} of roof", flush=True)


def linear_mixers(b: Bench, cfg, nb) -> None:
    gla, right = cfg.blocks[0].mixer, cfg.blocks[1].mixer.right
    hk, hv = nb.linear_num_key_heads, nb.linear_num_value_heads
    dk, dv, chans = nb.linear_key_head_dim, nb.linear_value_head_dim, nb.gdn_conv_channels
    for label, lens in (("decode 64", [1] * 64), ("decode 256", [1] * 256), ("prompt 1 x 2048", [2048]), ("prompts 4 x 2048", [2048] * 4),
                        ("prompt 1 x 8192", [8192])):
        r, n, decode = len(lens), sum(lens), max(lens) == 1
        qo = np.concatenate([[0], np.cumsum(lens)]).tolist()
        for name, s, chan in (("gated linear attention", gla, True), ("lightning attention", right, False)):
            x = torch.randn(n, 2 * s.qk + s.values, **BF16)
            q, k, v = x[:, :s.qk], x[:, s.qk:2 * s.qk], x[:, 2 * s.qk:]
            logs = -torch.rand(n, s.qk, device="cuda") * 0.1 if chan else None
            dec = None if chan else torch.full((s.heads,), 0.99, device="cuda")
            state, rs = torch.zeros(r, s.state_elems, device="cuda"), _rs(qo, r)
            moved = 2.0 * x.numel() + (4.0 * n * s.qk if chan else 0) + 4.0 * n * s.values + 8.0 * r * s.state_elems
            # recurrent form: 2 multiply-adds per state element and token for the update, 1 for the output
            b.run(f"{name}, {label}", lambda: lin.linear_attention(q, k, v, s, rs, state, decode, logs, dec, not chan), moved,
                  4.0 * n * s.state_elems)
        if decode or n <= 2048 * 4:
            mix = torch.randn(n, nb.gdn_in_features, **BF16)
            lw = {"gdn_conv": torch.randn(chans, 4, **BF16), "gdn_A_log": torch.zeros(hv, device="cuda"),
                  "gdn_dt_bias": torch.zeros(hv, device="cuda"), "gdn_norm": torch.ones(dv, **BF16)}
            rs = _rs(qo, r)
            rs.conv_state, rs.rec_state = torch.zeros(1, r, chans, 3, device="cuda"), torch.zeros(1, r, hv, dk, dv, device="cuda")
            rs.scratch = torch.empty(n, chans, device="cuda")
            b.run(f"  Gated DeltaNet mixer (conv, norm, gate), {label}", lambda: ops.gdn_mixer(mix, lw, nb, rs, 0),
                  2.0 * mix.numel() + 2.0 * n * hv * dv + 8.0 * r * hv * dk * dv, 4.0 * n * hv * dk * dv)


def attention(b: Bench, cfg, nb) -> None:
    a = cfg.blocks[1].attention
    D, hq, w = a.head_dim, a.heads, a.window
    bias = lin.bias_table(torch.randn(a.buckets, a.heads), a, "cuda")
    for r in (64, 256):
        kv, items = np.full(r, 2049, np.int64), r + 296 * 8
        scratch = torch.empty(ops.decode_scratch_floats(items, hq, D), device="cuda")
        plan, pages = _decode_plan(kv, a.kv_heads, w, items, scratch, "cuda", False)
        cache, q = torch.randn(pages + 1, 2, a.kv_heads, 16, D, **BF16), torch.randn(r, hq, D, **BF16)
        rs, slots = _rs(list(range(r + 1)), r), torch.zeros(r, dtype=torch.int32, device="cuda")
        moved = r * w * 2.0 * a.kv_heads * D * 2 + 4.0 * q.numel()
        b.run(f"biased attention, decode {r} x 2049", lambda: lin.biased_attention(q, cache, bias, plan, rs, slots, a), moved)
        b.run(f"  plain attention, decode {r} x 2049", lambda: ops.paged_decode_attention(q, cache, plan, D ** -0.5), moved)
    for r, n in ((1, 2048), (4, 2048), (1, 8192)):
        per, tot = n // 16, r * n
        batch = ops.AttnBatch(np.arange(r + 1, dtype=np.int32) * n, np.arange(r + 1, dtype=np.int32) * per,
                              np.random.default_rng(0).permutation(r * per).astype(np.int32), np.full(r, n, np.int32), None, w - 1)
        plan = ops.build_prefill_plan(batch, a.group, 16, "cuda", 256)
        plan.host = batch
        cache, q = torch.randn(r * per + 1, 2, a.kv_heads, 16, D, **BF16), torch.randn(tot, hq, D, **BF16)
        seen = r * sum(min(i + 1, w) for i in range(n))
        moved, flops = 4.0 * q.numel() + 4.0 * tot * a.kv_heads * D, 4.0 * seen * hq * D
        b.run(f"biased attention, prompts {r} x {n}", lambda: lin.biased_attention(q, cache, bias, plan, None, None, a), moved, flops)
        b.run(f"  plain attention, prompts {r} x {n}", lambda: ops.paged_prefill_attention(q, cache, plan, D ** -0.5), moved, flops)
        b.run(f"  soft-capped attention, prompts {r} x {n}",
              lambda: ops.paged_prefill_attention(q, cache, plan, D ** -0.5, softcap=a.softcap), moved, flops)


def rows(b: Bench, cfg, nb) -> None:
    gla, m = cfg.blocks[0].mixer, cfg.blocks[1].mixer
    a, s, W = m.left, m.right, cfg.hidden_size
    for n in (64, 8192):
        nq, nk = a.heads * a.dim, a.kv_heads * a.dim
        y = torch.randn(n, nq + 2 * nk, **BF16)
        cache = torch.zeros(n // 16 + 1, 2, a.kv_heads, 16, a.head_dim, **BF16)
        slots, pos = torch.arange(n, dtype=torch.int32, device="cuda"), torch.arange(n, dtype=torch.int32, device="cuda")
        gq, gk, g = torch.ones(nq, **BF16), torch.ones(nk, **BF16), torch.ones(a.dim, **BF16)
        b.run(f"norm over the projection + KV write, {n} rows",
              lambda: lin.biased_rows(y[:, :nq], y[:, nq:nq + nk], y[:, nq + nk:], gq, gk, slots, cache, a, 1e-5), 4.0 * y.numel())
        inv = torch.ones(a.dim // 2, device="cuda")
        b.run(f"  head norms + rotation + KV write, {n} rows",
              lambda: ops.qk_norm_rope_kvwrite(y, pos, slots, inv, g, g, cache, a.heads, a.kv_heads, a.dim, 16, 1e-5), 4.0 * y.numel())
        o, gate, z = torch.randn(n, gla.values, device="cuda"), torch.randn(n, gla.values, **BF16), torch.empty(n, gla.values, **BF16)
        w = torch.ones(gla.vdim, **BF16)
        b.run(f"head norm + SiLU gate, {n} rows", lambda: lin.gated_norm([(o, w, gate, z, dict(
            act="silu", norm_cols=gla.vdim, eps=1e-5, scale=1.0))]), 8.0 * o.numel())
        o1, g1, z1 = torch.randn(n, nq, **BF16), torch.randn(n, nq, **BF16), torch.empty(n, nq + s.values, **BF16)
        o2, g2, w2 = torch.randn(n, s.values, device="cuda"), torch.randn(n, s.values, **BF16), torch.ones(s.values, **BF16)
        b.run(f"gates of both mixers, {n} rows", lambda: lin.gated_norm([
            (o1, None, g1, z1[:, :nq], dict(act="sigmoid", norm_cols=0, scale=1.0, spec=a)),
            (o2, w2, g2, z1[:, nq:], dict(act="sigmoid", norm_cols=s.values, eps=1e-5, scale=1.0))]), 6.0 * o1.numel() + 8.0 * o2.numel())
        a1, a2, ab = torch.randn(n, 16, **BF16), torch.randn(gla.qk, 16, **BF16), torch.randn(gla.qk, **BF16)
        b.run(f"channel decays, {n} rows", lambda: lin.decay_logs(a1, a2, ab, 16.0), 4.0 * n * gla.qk)
        x, yy, gain = torch.randn(n, W, device="cuda"), torch.randn(n, W, **BF16), torch.ones(W, device="cuda")
        b.run(f"output norm + residual + next norm, {n} rows",
              lambda: lops.stream_norm(x, W, 1e-5, yy, gain, gain, dtype=torch.bfloat16), 12.0 * x.numel())
        h = torch.randn(n, W, **BF16)
        b.run(f"  RMS norm, {n} rows", lambda: ops.rmsnorm(h, torch.ones(W, **BF16), 1e-5), 4.0 * h.numel())
        f = cfg.blocks[1].ff
        gu, dn = torch.randn(f.experts, 2 * f.ff, W, **BF16), torch.randn(f.experts, W, f.ff, **BF16)
        router, corr = torch.randn(f.outputs, W, **BF16) * W ** -0.5, torch.zeros(f.outputs, device="cuda")
        buf, buf2 = ops.MoeBuffers(n, W, f.ff, f.experts, f.top, "cuda"), ops.MoeBuffers(n, W, f.ff, f.experts, f.top, "cuda")
        wb, flops = 2.0 * (gu.numel() + dn.numel()), 6.0 * n * f.top * f.ff * W
        real = f.experts / f.outputs
        b.run(f"experts with identity outputs, {n} rows", lambda: lin.scored_experts(h, router, corr, gu, dn, f, buf),
              wb + 4.0 * h.numel(), flops * real)
        logits = torch.randn(n, f.experts, **BF16)
        b.run(f"  SwiGLU experts, {n} rows", lambda: ops.moe_experts(h, logits, gu, dn, f.top, True, buf2), wb + 4.0 * h.numel(), flops)


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--hbm", type=float, default=6538.9, help="copy bandwidth, GB/s")
    ap.add_argument("--tflops", type=float, default=1608.3, help="bf16 GEMM throughput")
    ap.add_argument("--only", default="", help="part of a line's name")
    a = ap.parse_args(argv)
    b, cfg, nb = Bench(a.hbm, a.tflops, a.only), preset("retodra-19b", num_hidden_layers=2), preset("gdn-moe-window-19b", num_hidden_layers=2)
    torch.manual_seed(0)
    ops.ensure_gemm_workspace("cuda:0")
    for part in (linear_mixers, attention, rows):
        part(b, cfg, nb)
    ops.check_kernel_status()


if __name__ == "__main__":
    main()
