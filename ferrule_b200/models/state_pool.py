"""Recurrent-state pool: what a sequence carries from token to token beside its paged cache.

Kinds of plane: per run of a recurrent layer the fp32 state (a matrix per head of a delta mixer, [inner, state] of a selective
scan) and the last inputs of the short convolutions, and per run of a layer with an input convolution the last rows of the
32-bit residual stream it read, or of a token shift the last normalised row.  Such a plane is indexed by slot (the engine's logical sequence slot) and buffer: every slot has `buffers`
copies and one of them is committed.  A step reads the committed copy and writes the next one, and only the commit of its
transaction makes that one current - a step that fails or is rolled back leaves nothing to undo.  With decode
look-ahead a step may already run before its predecessor has been published, so three buffers are in rotation: the
committed one, the one the unpublished step wrote, the one the step launched ahead writes.

A sequence starts from zeros: its first step reads index -1 and no memory has to be cleared.

Layers that see mean keys and values of whole blocks of tokens keep them here too: `pooled[run]` holds per slot one cache row for
every block a sequence can have, in order.  A row is written by the step that appends its block's last token, and again
whenever that token is appended again; a query only sees blocks whose last token is older.  So there is one buffer.
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from .layered_config import DeltaMixer, LayeredConfig, Mamba2Mixer, MambaMixer


class RecurrentStatePool:
    def __init__(self, cfg: LayeredConfig, n_slots: int, device, dtype=torch.bfloat16, buffers: int = 3,
                 max_tokens: int = 0):
        if buffers < 2:
            raise ValueError("a slot needs at least two buffers")
        self.n_slots, self.buffers = n_slots, buffers
        self.n_states = n_slots * buffers
        self.state: Dict[int, torch.Tensor] = {}
        self.tail: Dict[int, torch.Tensor] = {}
        self.canon: Dict[int, torch.Tensor] = {}
        self.shift: Dict[int, torch.Tensor] = {}
        self.pooled: Dict[int, torch.Tensor] = {}
        plane = lambda *shape, dt=torch.float32: torch.zeros(self.n_states, *shape, dtype=dt, device=device)
        for i, layer in enumerate(cfg.runs):
            m = cfg.layers[layer].mixer
            if isinstance(m, DeltaMixer):
                self.state[i] = plane(m.heads, m.dim, m.vdim)
                self.tail[i] = plane(max(m.taps - 1, 1), m.channels, dt=dtype)
            elif isinstance(m, MambaMixer):
                self.state[i] = plane(m.state, m.inner_pad)
                self.tail[i] = plane(max(m.taps - 1, 1), m.inner_pad, dt=dtype)
            elif isinstance(m, Mamba2Mixer):
                self.state[i] = plane(m.heads, m.state, m.vdim)
                self.tail[i] = plane(max(m.taps - 1, 1), m.channels, dt=dtype)
            elif getattr(m, "pool", 0):
                self.pooled[i] = torch.zeros(n_slots, max_tokens // m.pool + 1, cfg.plane_dim(layer), dtype=dtype, device=device)
            if cfg.token_shift:
                self.shift[i] = plane(cfg.width_pad)
            if cfg.canon_taps:
                self.canon[i] = plane(max(cfg.canon_taps - 1, 1), cfg.width_pad)
        self.current: List[int] = [-1] * n_slots         # committed buffer of every slot, -1: none yet

    @property
    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for d in (self.state, self.tail, self.canon, self.shift, self.pooled)
                   for t in d.values())

    def bind(self, slot: int, fresh: bool, ahead: bool = False) -> Tuple[int, int]:
        """(state index to read, state index to write) of the slot's next step.  `fresh`: the sequence starts with
        this step.  `ahead`: the step after the one that is still unpublished (its result is read)."""
        if not 0 <= slot < self.n_slots:
            raise ValueError(f"state slot {slot} outside the pool of {self.n_slots}")
        cur = -1 if fresh else self.current[slot]
        nxt = (cur + 1) % self.buffers
        if ahead:
            cur, nxt = nxt, (nxt + 1) % self.buffers
        elif not fresh and cur < 0:
            raise RuntimeError(f"state slot {slot} holds no state to continue from")
        base = slot * self.buffers
        return (base + cur if cur >= 0 else -1), base + nxt

    def commit(self, slot: int, written: int) -> None:
        if not 0 <= slot < self.n_slots or written // self.buffers != slot:
            raise ValueError(f"state index {written} does not belong to slot {slot}")
        self.current[slot] = written % self.buffers

    def release(self, slot: int) -> None:
        """The slot's sequence is gone; the next one starts from zeros."""
        self.current[slot] = -1
