"""Recurrent-state cache of the Gated DeltaNet and Mamba-2 layers and of token-shifted blocks: per (recurrent layer,
slot) the tail of the short convolution's inputs and the fp32 state (delta-rule state [heads, dk, dv], or state-space
state [heads, head_dim, state]), or the previous token's normalised input (token shift, [width] fp32). Linear-attention
mixers of layers described one by one (any head sizes) keep [heads, dim, vdim] fp32 each (a matrix memory also [heads, dim]
and [heads]), all layers of a slot in one row, with the last inputs of their input convolutions ([taps - 1, width] fp32 for
each sublayer) and the token before where the embedding wants it (`ModelConfig.slot_layout`).
A slot belongs to one resident context; the runtime's
slot pool (`runtime/rs_cache.py`) hands slots out, tells the driver when a slot must start from zero
(`rs_reset`) and asks for a slot copy when a context forks.

Counterpart of driver/cuda/src/recurrent_state_cache.hpp:1-40 (slabs per layer and slot, slot D2D copy).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from functools import cached_property
from typing import Dict, List, Optional

import numpy as np
import torch

from ..models.config import ModelConfig


@dataclass
class RecurrentInputs:
    """What the mixer of every linear layer needs for one fire."""
    qo_indptr: torch.Tensor        # int32 [R + 1] on the device
    tok_req: torch.Tensor          # int32 [N] request of every token row
    slots: torch.Tensor            # int32 [R]
    reset: torch.Tensor            # int32 [R] 1 = start this request's state from zero
    qo_host: List[int]
    slots_host: List[int]
    reset_host: List[int]
    conv_state: Optional[torch.Tensor]       # [L, S, C, K - 1] fp32
    rec_state: Optional[torch.Tensor]        # [L, S, Hv, dk, dv] fp32
    layer_index: Dict[int, int]    # model layer -> index into the first dimension of the caches
    scratch: Optional[torch.Tensor] = None   # [N, C] fp32 convolution output (device path)
    shift_state: Optional[torch.Tensor] = None   # [L, S, W] fp32 previous token's input (token shift)
    shift_stage: Optional[torch.Tensor] = None   # [R, W] fp32: a portion's last input until its readers are done
    linear_state: Optional[torch.Tensor] = None  # [S, elements] fp32: the states of all linear-attention layers of a slot
    linear_at: Optional[Dict[int, int]] = None   # model layer -> its first element in a row of `linear_state`
    history_at: Optional[dict] = None            # (model layer, half) -> first element of its convolution's history
    history_elems: int = 0                       # numbers of one history
    token_at: Optional[int] = None               # element that holds the token before, as an integer
    conv_stage: Optional[torch.Tensor] = None    # [R, taps - 1, W] fp32: the new history of portions until its readers are done
    pieces: dict = field(default_factory=dict)   # piece size -> the portions cut for a chunked form (`ops.linear.chunk_pieces`)
    staged: Optional[int] = None   # requests the stage is committed for (0: none of this fire's portions uses it)

    def state_of(self, li: int, elems: int) -> torch.Tensor:
        """Layer `li`'s columns of the linear-attention state cache [slots, all layers]."""
        at = self.linear_at[li]
        return self.linear_state[:, at:at + elems]

    def history_of(self, li: int, half: str) -> Optional[torch.Tensor]:
        """Columns of the state cache with the history of an input convolution (None: it reaches no further back)."""
        if not self.history_at:
            return None
        at = self.history_at[li, half]
        return self.linear_state[:, at:at + self.history_elems]

    @property
    def token_before(self) -> torch.Tensor:
        """int32 [slots] (strided): the token each sequence ended with."""
        return self.linear_state[:, self.token_at].view(torch.int32)

    @cached_property
    def has_portions(self) -> bool:
        """Whether some request of the fire brings more than one token."""
        return any(b - a > 1 for a, b in zip(self.qo_host, self.qo_host[1:]))


class RecurrentStateCache:
    def __init__(self, cfg: ModelConfig, num_slots: int, device):
        self.cfg, self.num_slots, self.device = cfg, num_slots, torch.device(device)
        lin = cfg.recurrent_layers
        if cfg.linear_layers and cfg.mamba_layers:
            raise NotImplementedError("Gated DeltaNet and Mamba-2 layers in one model")
        self.layer_index = {li: i for i, li in enumerate(lin)}
        self.conv_state = self.rec_state = self.shift_state = self.linear_state = None
        self.linear_at: Optional[Dict[int, int]] = None
        self.conv_channels = 0
        self.carried: dict = {}
        if cfg.blocks is not None:
            self.linear_at, histories, before, at = cfg.slot_layout()
            self.carried = dict(history_at=histories, history_elems=max(0, cfg.conv_taps - 1) * cfg.hidden_size, token_at=before)
            self.linear_state = torch.zeros(num_slots, max(at, 4), dtype=torch.float32, device=self.device)
            return
        if cfg.token_shift:
            if cfg.mamba_layers or cfg.linear_layers:
                raise NotImplementedError("token shift beside Gated DeltaNet or Mamba-2 layers")
            self.shift_state = torch.zeros(len(lin), num_slots, cfg.hidden_size, dtype=torch.float32, device=self.device)
            return
        if cfg.mamba_layers:       # [heads, head_dim, state] per slot, convolution over x | B | C
            c, k = cfg.mamba_conv_channels, 4
            hv, dk, dv = cfg.mamba_num_heads, cfg.mamba_head_dim, cfg.ssm_state_size
        else:
            c, k = cfg.gdn_conv_channels, cfg.linear_conv_kernel_dim
            hv, dk, dv = cfg.linear_num_value_heads, cfg.linear_key_head_dim, cfg.linear_value_head_dim
        self.conv_channels = c
        self.conv_state = torch.zeros(len(lin), num_slots, c, k - 1, dtype=torch.float32, device=self.device)
        self.rec_state = torch.zeros(len(lin), num_slots, hv, dk, dv, dtype=torch.float32, device=self.device)

    @property
    def buffers(self) -> List[torch.Tensor]:
        linear = self.linear_state[None] if self.linear_state is not None else None
        return [b for b in (self.conv_state, self.rec_state, self.shift_state, linear) if b is not None]

    @property
    def bytes_per_slot(self) -> int:
        return sum(b[:, 0].numel() for b in self.buffers) * 4

    def device_scratch(self, n: int, r: int) -> dict:
        """Device scratch of a fire of n tokens in r requests."""
        if self.device.type == "cuda" and self.carried.get("history_at") and n > r:
            return {"conv_stage": torch.empty(max(r, 1), self.carried["history_elems"], dtype=torch.float32, device=self.device)}
        if self.device.type != "cuda" or self.linear_state is not None:
            return {}
        if self.shift_state is not None:
            return {"shift_stage": torch.empty(max(r, 1), self.cfg.hidden_size, dtype=torch.float32, device=self.device)}
        return {"scratch": torch.empty(max(n, 1), self.conv_channels, dtype=torch.float32, device=self.device)}

    def inputs(self, qo_indptr, rs_slots, rs_reset) -> RecurrentInputs:
        qo = np.ascontiguousarray(qo_indptr, dtype=np.int32)
        r = len(qo) - 1
        if rs_slots is None or len(rs_slots) != r:
            raise ValueError("this model has recurrent layers: every request needs a recurrent-state slot")
        slots = np.ascontiguousarray(rs_slots, dtype=np.int32)
        if len(slots) and (slots.min() < 0 or slots.max() >= self.num_slots):
            raise ValueError(f"recurrent-state slot outside 0..{self.num_slots - 1}")
        if len(set(slots.tolist())) != len(slots):
            raise ValueError("two requests of one fire share a recurrent-state slot")
        reset = np.ascontiguousarray(rs_reset if rs_reset is not None else np.zeros(r, np.int32), dtype=np.int32)
        tok_req = np.repeat(np.arange(r, dtype=np.int32), np.diff(qo))
        dev = self.device
        t = lambda a: torch.from_numpy(a).to(dev)
        return RecurrentInputs(t(qo), t(tok_req), t(slots), t(reset), qo.tolist(), slots.tolist(), reset.tolist(),
                               self.conv_state, self.rec_state, self.layer_index, shift_state=self.shift_state,
                               linear_state=self.linear_state, linear_at=self.linear_at, **self.carried, **self.device_scratch(int(qo[-1]), r))

    def copy_slot(self, src: int, dst: int) -> None:
        """dst <- src in every layer (a forked context continues from its parent's state)."""
        if src == dst:
            return
        if self.device.type != "cuda":
            for buf in self.buffers:
                buf[:, dst].copy_(buf[:, src])
            return
        from .. import ops
        for buf in self.buffers:
            ops.gdn_copy_slot(buf, src, dst)
