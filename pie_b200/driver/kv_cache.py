"""Paged KV cache and its host swap pool.

Device layout: one tensor ``[layers, pages, 2, kv_heads_local, page_size, head_dim]`` so that a
(page, head) K or V block is a contiguous run (bulk copies, tensor-core tiles) and a page of
every layer can be copied with one kernel launch. Page id ``num_pages`` (one extra page at
the end) is a scratch page that padded graph-bucket requests point at.

Reference counterparts: driver/cuda/src/kv_cache.hpp:1-202 (per-layer K/V page pools),
driver/cuda/src/swap_pool.hpp:25-84 (pinned host mirror, D2H/H2D/D2D/H2H page copies).
"""
from __future__ import annotations

import numpy as np
import torch

from .. import ops
from .schema import CopyDir, CopyRequest


class LayerPages:
    """Pages of layers with unequal shapes: one tensor [pages + 1, 2, kv heads, page, D] (keys that are the values: 1 in place of
    2; latent rows: [pages + 1, page, row]) per layer that has a cache. `means` [pages + 1, 2, kv heads, blocks, D]: of those
    that keep the mean key and value of every block of tokens, with the page of the block's last one (else None)."""

    def __init__(self, layers, means):
        self.layers, self.means = layers, means

    def __getitem__(self, i: int):
        return self.layers[i]


class KVCache:
    def __init__(self, layers: int, num_pages: int, kv_heads: int, page_size: int, head_dim: int,
                 dtype, device, swap_pages: int = 0, kv_dtype: str = "auto", latent: bool = False,
                 layer_shapes=None):
        """kv_dtype "auto": pages in the activation dtype. "fp8_e4m3": one byte per element plus one
        fp32 scale per (token, KV head) row in `scale` [layers, pages + 1, 2, kv_heads, page_size]
        (written by the RoPE + KV-write kernel, read by decode attention; prefill attention works on
        pages expanded to bf16 for the batch). Counterpart of the reference's per-token-head fp8 format
        (driver/cuda/src/kv_cache_format.hpp, kernels/kv_paged.cu:188-325).

        `latent`: pages of latent attention, one row of `head_dim` elements per token (latent, then the rotated key part
        that all heads share) in ``[layers, pages + 1, page_size, row]``; `layers` counts the layers that write rows.

        `layer_shapes`: shapes of a page in every layer that has a cache (`ModelConfig.kv_page_shapes`), where a model's layers
        differ (`data` is then a `LayerPages`; it may be empty)."""
        if page_size % 16:
            raise ValueError("kv page size must be a multiple of 16")
        if kv_dtype not in ("auto", "bf16", "fp8_e4m3"):
            raise ValueError(f"unknown kv_dtype {kv_dtype!r} (auto | bf16 | fp8_e4m3)")
        self.kv_dtype = kv_dtype
        self.scale = None
        if kv_dtype == "fp8_e4m3":
            if torch.device(device).type != "cuda":
                raise NotImplementedError("fp8 KV pages need the CUDA kernels")
            dtype = torch.uint8
            self.scale = torch.zeros(layers, num_pages + 1, 2, kv_heads, page_size, dtype=torch.float32, device=device)
        self.layers, self.num_pages, self.kv_heads = layers, num_pages, kv_heads
        self.page_size, self.head_dim, self.dtype = page_size, head_dim, dtype
        self.device = torch.device(device)
        if layer_shapes is not None:
            shapes = [(1, rows) for rows, _ in layer_shapes] + [(1, means) for _, means in layer_shapes if means is not None]
        else:
            shapes = [(layers, (page_size, head_dim) if latent else (2, kv_heads, page_size, head_dim))]
        # zero-filled: unwritten slots are multiplied by p == 0 in attention and must be finite
        self.parts = [torch.zeros(n, num_pages + 1, *shape, dtype=dtype, device=self.device) for n, shape in shapes]
        if layer_shapes is None:
            self.data = self.parts[0]
        else:
            means = iter(self.parts[len(layer_shapes):])
            self.data = LayerPages([t[0] for t in self.parts[:len(layer_shapes)]],
                                   [next(means)[0] if m is not None else None for _, m in layer_shapes])
        self.pad_page = num_pages
        self.swap_pages = swap_pages
        self.host = None
        if swap_pages > 0:
            self.host = [torch.zeros(n, swap_pages, *shape, dtype=dtype, pin_memory=self.device.type == "cuda") for n, shape in shapes]
        self._copy_stream = torch.cuda.Stream(self.device) if self.device.type == "cuda" else None

    @property
    def page_bytes_all_layers(self) -> int:
        return sum(t[:, 0].numel() * t.element_size() for t in self.parts)

    @staticmethod
    def bytes_per_page(layers, kv_heads, page_size, head_dim, elem_size=2) -> int:
        return layers * 2 * kv_heads * page_size * head_dim * elem_size

    def copy(self, req: CopyRequest) -> None:
        """Execute a page copy on every layer. D2D runs on the compute stream (it orders with
        forward passes that read the pages); swaps run on a side stream and are awaited."""
        src = np.ascontiguousarray(req.srcs, dtype=np.int32)
        dst = np.ascontiguousarray(req.dsts, dtype=np.int32)
        if len(src) == 0:
            return
        if req.direction == CopyDir.D2D:
            s = torch.from_numpy(src).to(self.device)
            d = torch.from_numpy(dst).to(self.device)
            for t in self.parts:
                ops.copy_pages(t, s, d)
            if self.scale is not None:
                ops.copy_pages(self.scale, s, d)
            return
        if self.scale is not None:
            raise NotImplementedError("host swap of fp8 KV pages")
        if self.host is None:
            raise RuntimeError("no swap pool configured")
        if req.direction == CopyDir.H2H:
            for h in self.host:
                h[:, torch.from_numpy(dst).long()] = h[:, torch.from_numpy(src).long()]
            return
        if self._copy_stream is None:
            for t, h in zip(self.parts, self.host):
                for s, d in zip(src.tolist(), dst.tolist()):
                    if req.direction == CopyDir.D2H:
                        h[:, d] = t[:, s]
                    else:
                        t[:, d] = h[:, s]
            return
        cur = torch.cuda.current_stream(self.device)
        self._copy_stream.wait_stream(cur)
        with torch.cuda.stream(self._copy_stream):
            for t, h in zip(self.parts, self.host):
                for s, d in zip(src.tolist(), dst.tolist()):
                    if req.direction == CopyDir.D2H:
                        h[:, d].copy_(t[:, s], non_blocking=True)
                    else:
                        t[:, d].copy_(h[:, s], non_blocking=True)
        if req.direction == CopyDir.H2D:
            cur.wait_stream(self._copy_stream)
        else:
            self._copy_stream.synchronize()
