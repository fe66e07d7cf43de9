"""Trace replay: given token ids go through a model step by step, as one batch per step, and chosen logits are written.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one JSON line ``{"step": 4, "entries": [{"id": "q7", "tokens": [812, 9], "want": [1]}], "end": ["q3"]}``: the next
tokens of each request and the places among them whose logits are wanted; requests in `end` are finished after the
step and give back what they hold. The logits of a step go to ``DIR/<step>.f32`` (little-endian 32-bit floats,
[wanted, vocab]), and ``done <step>`` is printed. Nothing is sampled.

The steps run on what serves generation: contexts of the context manager (pages, recurrent-state slots), `fold`, and
`TorchDriver.fire_batch`, over a pool of N tokens' pages and four state slots.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Dict, List

import numpy as np

PAGE_SIZE = 16
MAX_LIVE = 4           # live requests, hence state slots
EXIT_UNSUPPORTED = 3   # this model has no path in the asked number format


class Replay:
    """A driver with its page and slot pools, stepped by hand."""

    def __init__(self, driver, page_size: int = PAGE_SIZE):
        from ..driver.schema import SamplerKind, SamplerSpec
        from .context import ContextManager
        from .pagestore import PageStore
        self.driver, self.page_size = driver, page_size
        caps = driver.capabilities()
        self.contexts = ContextManager("trace", page_size, [PageStore(caps.total_pages)], lambda d, req: driver.copy(req),
                                       rs_slots=[caps.rs_cache_slots], rs_copy_fn=lambda d, src, dst: driver.copy_rs(src, dst))
        self.ids: Dict[str, int] = {}
        self._raw = SamplerSpec(SamplerKind.RAW_LOGITS)

    def step(self, entries: List[dict], end: List[str] = ()) -> np.ndarray:
        """Run one batch; returns the wanted logits [wanted, vocab] in the order of the entries."""
        from .scheduler import PendingRequest, fold
        cm, items = self.contexts, []
        for e in entries:
            if e["id"] not in self.ids:
                self.ids[e["id"]] = cm.create("trace", 0)
            cid, toks = self.ids[e["id"]], e["tokens"]
            have = cm.kv_len(cid)
            held = (cm.committed_page_count(cid) + cm.working_page_count(cid)) * self.page_size
            need = -(-(have + len(toks) - held) // self.page_size)
            if need > 0:
                cm.reserve_working_pages(cid, need)
            pin = cm.pin(cid, len(toks))
            if cm.take_pending_replay(cid):
                raise RuntimeError(f"request {e['id']} lost its state")
            items.append(PendingRequest(cid, toks, list(range(have, have + len(toks))), pin.pages, pin.kv_len,
                                        [(int(i), self._raw) for i in e.get("want", ())], rs_slot=pin.rs_slot, rs_reset=pin.rs_reset))
        try:
            resp = self.driver.fire_batch(fold(items, self.page_size)) if items else None
        finally:
            for it in items:
                cm.unpin(it.context_id)
        for it in items:
            cm.append_working_tokens(it.context_id, it.tokens, it.positions)
            full = cm.working_page_token_count(it.context_id) // self.page_size
            if full:
                cm.commit_working_pages(it.context_id, full)
        for name in end:
            cm.destroy(self.ids.pop(name))
        rows = [np.frombuffer(s.logits, dtype=np.float32) for s in resp.slots] if resp is not None else []
        return np.stack(rows) if rows else np.zeros((0, 0), np.float32)


def make_driver(model_dir, dtype: str, max_tokens: int, device: str = "cuda"):
    """The driver that serves `model_dir`, with a pool of `max_tokens` tokens' pages."""
    import torch
    from ..driver.executor import TorchDriver
    from ..models import loader
    if dtype == "float32":
        torch.backends.cuda.matmul.allow_tf32 = False
    cfg, weights = loader.load_checkpoint(model_dir, device, dtype=dtype)
    pages = -(-max_tokens // PAGE_SIZE)
    return TorchDriver(cfg, device, weights=weights, num_pages=pages, page_size=PAGE_SIZE, max_requests=MAX_LIVE,
                       max_tokens=max(max_tokens, 64), rs_slots=MAX_LIVE if cfg.recurrent_layers else 0, compute_dtype=dtype)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--device", default="cuda")
    args = ap.parse_args(argv)
    if args.device.startswith("cuda"):
        from .. import _build
        from ..models.config import ModelConfig
        from ..ops import _lib
        _lib.use_library(_build.kernels_for(ModelConfig.from_path(args.model)))
    try:
        driver = make_driver(args.model, args.dtype, args.max_tokens, args.device)
    except NotImplementedError as e:
        print(f"trace_run: {e}", file=sys.stderr)
        return EXIT_UNSUPPORTED
    replay, out = Replay(driver), Path(args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        rows = replay.step(s["entries"], s.get("end", ()))
        if rows.size:
            rows.astype("<f4").tofile(out / f"{s['step']}.f32")
        print(f"done {s['step']}", flush=True)
    return 0
