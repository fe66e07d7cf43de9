"""Prefill and decode throughput of a design beside the closest other model of equal size, random weights, bf16.

    python bench.py --config 7 [--layers 32]    Puzutar beside the Llama-8B shape with a sliding window
    python bench.py --config 8 [--layers 32]    Retodra beside Gated DeltaNet and windowed attention with experts
    python bench.py --config 9 [--layers 24]    Nukelix beside Retodra's parallel mixers with experts
    python bench.py --config 10 [--layers 32]   Vulanex beside Gated DeltaNet and attention

Both models of a pair have the same width, heads, window, vocabulary and feed-forward sizes (configs 8 and 9: also the same
states of the linear mixers, experts and routes per token; a shared expert counts as a route; config 10: the same states, and
feed-forwards that make up for the parameters of a second mixer). Device-timed with CUDA
events after warm-up. Decode replays the captured step over contexts of `--context` tokens; the weights read per step
exceed the L2. Prefill runs whole prompts as one batch. One JSON line.
"""
from __future__ import annotations

import argparse
import gc
import json

import numpy as np

PAIRS = {7: ("puzutar-8b", "llama-8b-window"), 8: ("retodra-19b", "gdn-moe-window-19b"),
         9: ("nukelix-20b", "retodra-parallel-20b"), 10: ("vulanex-8b", "gdn-8b")}
DECODE_ROWS = (16, 64, 256)
PREFILL = ((1, 2048), (4, 2048), (1, 8192))


def _driver(name: str, layers: int, max_tokens: int, rows: int, pages: int):
    import torch
    from ..driver.executor import TorchDriver
    from ..models.config import preset
    cfg = preset(name, **({"num_hidden_layers": layers} if layers else {}))
    drv = TorchDriver(cfg, "cuda", page_size=16, num_pages=pages, max_requests=rows, max_tokens=max_tokens,
                      rs_slots=rows if cfg.recurrent_layers else 0)
    torch.manual_seed(0)
    for t in drv.kv.parts:
        t.normal_(0.0, 0.5)
    return cfg, drv


def _items(cfg, rows: int, start: int, count: int, sampler, seed: int = 0):
    """`rows` requests that each bring `count` tokens after `start` cached ones, in pages of their own."""
    from ..runtime.scheduler import PendingRequest
    rng = np.random.default_rng(seed)
    per = -(-(start + count) // 16)
    return [PendingRequest(i, rng.integers(0, cfg.vocab_size, count).tolist(), list(range(start, start + count)),
                           list(range(i * per, (i + 1) * per)), start, [(count - 1, sampler)],
                           rs_slot=i if cfg.recurrent_layers else -1, rs_reset=0 if start else 1) for i in range(rows)]


def _timed(fn, warmup: int, steps: int) -> float:
    """Milliseconds per call."""
    import torch
    for _ in range(warmup):
        fn()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(steps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


def measure(name: str, layers: int, context: int, steps: int, warmup: int) -> dict:
    import torch
    from .. import ops
    from ..driver.schema import SamplerKind, SamplerSpec
    from ..runtime.scheduler import fold
    rows = max(DECODE_ROWS)
    cfg, drv = _driver(name, layers, max(n * m for n, m in PREFILL), rows, rows * (-(-(context + 16) // 16)))
    sampler = SamplerSpec(SamplerKind.MULTINOMIAL, temperature=0.0)
    out = {"model": cfg.name, "layers": cfg.num_hidden_layers, "decode": {}, "prefill": {}}
    for r in DECODE_ROWS:
        st = drv.stage_decode(fold(_items(cfg, r, context, 1, sampler), 16))
        ms = _timed(lambda: drv.replay_staged(st, False), warmup, steps)
        out["decode"][f"{r}x{context}"] = {"ms_per_step": round(ms, 4), "tokens_per_s": round(r / ms * 1e3)}
    for r, n in PREFILL:
        req = fold(_items(cfg, r, 0, n, sampler), 16)
        ms = _timed(lambda: drv.fire_batch(req), 3, max(4, steps // 8))
        out["prefill"][f"{r}x{n}"] = {"ms": round(ms, 3), "tokens_per_s": round(r * n / ms * 1e3)}
    ops.check_kernel_status(drv.device)
    del drv
    gc.collect()
    torch.cuda.empty_cache()
    return out


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--steps", type=int, default=32)
    ap.add_argument("--warmup", type=int, default=4)
    ap.add_argument("--layers", type=int, default=0)
    ap.add_argument("--context", type=int, default=2048)
    ap.add_argument("--config", type=int, default=7, choices=sorted(PAIRS))
    ap.add_argument("--only", default="", help="one of the two models")
    a = ap.parse_args(argv)
    from . import harness
    clk = harness.ClockSampler(0).start()
    runs = [measure(m, a.layers, a.context, a.steps, max(3, a.warmup)) for m in PAIRS[a.config] if not a.only or a.only == m]
    clocks = clk.stop()
    line = {"config": a.config, "metric": "decode and prefill tokens/s of two models of equal size", "unit": "tokens/s", "n_gpus": 1,
            "dtype": "bf16", "data": "synthetic random tokens and cache contents, random-init weights", "runs": runs,
            "l2": "weights and cache per step exceed the 126 MB L2; no flush needed", "clocks": clocks}
    print(json.dumps(line), flush=True)


if __name__ == "__main__":
    main()
