"""Attention kernels of the Puzutar design and of its neighbour model, each alone: decode over paged caches and prefill of
whole prompts, CUDA events, a buffer larger than the L2 written between iterations. Prints achieved bandwidth or FLOP/s and
the fraction of the slower roof (copy bandwidth and bf16 GEMM throughput given on the command line).

    python -m pie_b200.bench.latent_attn_bench [--hbm 6538.9] [--tflops 1608.3]
"""
from __future__ import annotations

import argparse

import numpy as np
import torch

from .. import ops
from ..models.config import LatentSpec
from ..ops import latent as lops


def _time(fn, flush, n: int = 12, warm: int = 4) -> float:
    ev = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(n)]
    for i in range(warm + n):
        flush.zero_()
        if i >= warm:
            ev[i - warm][0].record()
        fn()
        if i >= warm:
            ev[i - warm][1].record()
    torch.cuda.synchronize()
    return float(np.median([a.elapsed_time(b) for a, b in ev])) * 1e-3


class _Rows:
    """The part of a recurrent input the attention ops read."""

    def __init__(self, qo, dev):
        t = lambda a: torch.from_numpy(np.asarray(a, np.int32)).to(dev)
        self.qo_indptr, self.slots_host = t(qo), list(range(len(qo) - 1))
        self.tok_req = t(np.repeat(np.arange(len(qo) - 1), np.diff(qo)))


def _decode_plan(kv, hkv, window, max_items, scratch, dev, even):
    r = len(kv)
    t = lambda a: torch.from_numpy(np.ascontiguousarray(a, np.int32)).to(dev)
    per = -(-int(kv.max()) // 16)
    ctas, ci = ops.num_sms(dev) * (1 if even else 2), None
    if even:
        ir, st, en, ip, ci = ops.plan_even_items(kv, ctas, max_items, window - 1)
        ci = t(ci)
    else:
        ir, st, en, ip = ops.plan_decode_items(kv, hkv, ctas, max_items, window_left=window - 1)
    ids = np.random.default_rng(0).permutation(r * per)
    return ops.DecodePlan(page_indices=t(ids), kv_page_indptr=t(np.arange(r + 1) * per), item_req=t(ir),
                          item_start=t(st), item_end=t(en), req_item_indptr=t(ip), num_items=t([len(ir)]), scratch=scratch,
                          max_items=max_items, num_reqs=r, num_ctas=ctas, page_size=16, window_left=window - 1, kv_lens=t(kv),
                          cta_items=ci), r * per


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--hbm", type=float, default=6538.9, help="copy bandwidth, GB/s")
    ap.add_argument("--tflops", type=float, default=1608.3)
    ap.add_argument("--window", type=int, default=1024)
    a = ap.parse_args(argv)
    dev, w = torch.device("cuda:0"), a.window
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    s = LatentSpec(heads=32, dim=96, rot_dim=32, vdim=128, kv_rank=256, window=w, scale=128 ** -0.5, rope_base=1e4, rot_dims=32)
    bf = dict(dtype=torch.bfloat16, device=dev)

    def report(what, sec, byts, flops):
        roof = max(byts / a.hbm / 1e9, flops / a.tflops / 1e12)
        print(f"{what:58s} {sec * 1e6:9.1f} us  {byts / sec / 1e12:6.2f} TB/s  {flops / sec / 1e12:7.1f} TFLOP/s  {roof / sec:5.2f} of roof")

    for r in (64, 256, 512):
        kv = np.full(r, 2049)
        seen = r * min(w, 2049)
        max_items = r + 8 * 296
        scratch = torch.empty(ops.decode_scratch_floats(max_items, 32, 288), dtype=torch.float32, device=dev)
        plan, pages = _decode_plan(kv, 1, w, max_items, scratch, dev, True)
        cache = torch.randn(pages + 1, 16, s.row, **bf)
        q = torch.randn(r, 32, s.row, **bf)
        rows = _Rows(np.arange(r + 1), dev)
        slots = torch.zeros(r, dtype=torch.int32, device=dev)
        sec = _time(lambda: lops.latent_attention(q, cache, plan, rows, slots, s, 16, w - 1), flush)
        report(f"latent decode, {r} requests, window {w} of 2049", sec, seen * s.row * 2 + r * 32 * (s.row + 256) * 2,
               2.0 * seen * 32 * (s.row + s.rank_pad))
        plan, pages = _decode_plan(kv, 8, w, max_items, scratch, dev, False)
        kvc = torch.randn(pages + 1, 2, 8, 16, 128, **bf)
        q = torch.randn(r, 32, 128, **bf)
        sec = _time(lambda: ops.paged_decode_attention(q, kvc, plan, 128 ** -0.5), flush)
        report(f"grouped-query decode, {r} requests, window {w} of 2049", sec, seen * 4096 + r * 32 * 256 * 2, 2.0 * seen * 32 * 256)
    for n_req, n in ((4, 2048), (1, 8192)):
        pairs = n_req * sum(min(i + 1, w) for i in range(n))
        qo = np.arange(n_req + 1) * n
        kv = np.full(n_req, n)
        tr, tq = ops.plan_prefill_tiles(qo, 1, 256, kv)
        t = lambda x: torch.from_numpy(np.ascontiguousarray(x, np.int32)).to(dev)
        per = n // 16
        ptr_, idx = np.arange(n_req + 1) * per, np.arange(n_req * per)
        plan = ops.PrefillPlan(t(idx), t(ptr_), t(qo), t(kv), t(tr), t(tq), len(tr), 16, window_left=w - 1, tile_rows=256,
                               host=ops.AttnBatch(qo, ptr_, idx, kv))
        cache = torch.randn(n_req * per + 1, 16, s.row, **bf)
        q = torch.randn(n_req * n, 32, 128, **bf)
        w_kv = torch.randn(32 * 2 * 128, s.row, **bf) * 0.06
        out = torch.empty(n_req * n, 32 * 128, **bf)
        kvb = n_req * n * 32 * 256 * 2
        sec = _time(lambda: ops.gemm(cache[:-1].view(-1, s.row), w_kv), flush)
        report(f"  of it the projection, {n_req} x {n}", sec, n_req * n * s.row * 2 + kvb, 2.0 * n_req * n * 32 * 256 * s.row)
        sec = _time(lambda: lops.projected_prefill_attention(q, cache, plan, w_kv, s, 16, w - 1, out), flush)
        report(f"latent prefill with its projection, {n_req} x {n}", sec, n_req * n * (32 * 256 * 2 + s.row * 2) + 2 * kvb,
               pairs * 32 * 4.0 * 128 + 2.0 * n_req * n * 32 * 256 * s.row)
        tr, tq = ops.plan_prefill_tiles(qo, 4, 256, kv)
        plan = ops.PrefillPlan(t(idx), t(ptr_), t(qo), t(kv), t(tr), t(tq), len(tr), 16, window_left=w - 1, tile_rows=256)
        kvc = torch.randn(n_req * per + 1, 2, 8, 16, 128, **bf)
        sec = _time(lambda: ops.paged_prefill_attention(q, kvc, plan, 128 ** -0.5), flush)
        report(f"grouped-query prefill, {n_req} x {n}", sec, n_req * n * (32 * 256 * 2 + 4096), pairs * 32 * 4.0 * 128)


if __name__ == "__main__":
    main()
