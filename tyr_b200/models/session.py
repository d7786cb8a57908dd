"""Decoding sessions of the hybrid models: a batch of sequences that advance together, with the per-layer K/V stores and linear
states and the CUDA-graph decode step.

A model's session supplies ``_prefill`` (whole prompts) and ``_device_step`` (one token per row, positions in ``pos_t``, no host
reads); the bookkeeping of lengths, the capture of the step and the release of finished rows live here."""
from __future__ import annotations

import os
from typing import List, Optional, Sequence

import torch

from .common import KVCache, LinearState


class HybridSession:
    name = "hybrid"

    def __init__(self, batch: int, max_len: int, device):
        if max_len <= 0:
            raise ValueError(f"{self.name} cache capacity must be positive")
        self.batch, self.max_len, self.device = batch, max_len, device
        self.pos = 0                                       # tokens of the longest row
        self.lengths: List[int] = [0] * batch
        self.kv: List[Optional[KVCache]] = []
        self.lin: List[Optional[LinearState]] = []
        self.pos_t: Optional[torch.Tensor] = None
        self._graph = None

    # -- hooks -----------------------------------------------------------------------------------------------------
    def hidden(self, ids: torch.Tensor, lengths: Optional[Sequence[int]] = None) -> torch.Tensor:
        """Run whole prompts [B, S] (right-padded to the longest when ``lengths`` differ) through a fresh session; the final
        normed hidden states [B, S, h]."""
        raise NotImplementedError

    def head(self, h: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    def device_step_supported(self) -> bool:
        return False

    def graph_supported(self) -> bool:
        """The step may be replayed from a CUDA graph (default: whenever it runs with device-side positions)."""
        return os.environ.get("TYR_DECODE_GRAPH", "1") != "0"

    def _device_step(self, tok: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    # -- shared ----------------------------------------------------------------------------------------------------
    def state_bytes(self) -> int:
        return sum(c.nbytes() for c in (*self.kv, *self.lin) if c is not None)

    def _positions(self) -> torch.Tensor:
        return torch.full((1,), self.pos, dtype=torch.int32, device=self.device)

    def _check_room(self, n: int) -> None:
        if self.pos + n > self.max_len:
            raise ValueError(f"{self.name} cache overflow")

    def _advance(self, lengths: Sequence[int]) -> None:
        self.lengths = [a + b for a, b in zip(self.lengths, lengths)]
        self.pos = max(self.lengths)
        for c in self.kv:
            if c is not None:
                c.length = self.pos

    def _advance_host(self) -> None:
        self._advance([1] * self.batch)

    @torch.no_grad()
    def prefill(self, ids: torch.Tensor, lengths: Optional[Sequence[int]] = None) -> torch.Tensor:
        """Logits [B, V] after each row's last prompt token."""
        h = self.hidden(ids, lengths)
        if lengths is None or len(set(lengths)) == 1 and lengths[0] == ids.shape[1]:
            return self.head(h[:, -1])
        last = torch.tensor([n - 1 for n in lengths], device=h.device)
        return self.head(h[torch.arange(h.shape[0], device=h.device), last])

    @torch.no_grad()
    def step(self, tok: torch.Tensor) -> torch.Tensor:
        """One token per row -> logits [B, V]."""
        tok = tok.reshape(-1)
        if self.pos == 0 or not self.device_step_supported():
            return self.head(self.hidden(tok.reshape(-1, 1))[:, -1])
        self._check_room(1)
        if self.pos_t is None:
            self.pos_t = self._positions()
        if not self.graph_supported():
            out = self._device_step(tok)
        else:
            if self._graph is None:
                from ..utils.graph import GraphedStep
                state = [self.pos_t] + [t for s in self.lin if s is not None for t in s.tensors()]
                self._graph = GraphedStep(self._device_step, (tok.clone(),), advancing_state=state)
            out = self._graph(tok)
        self._advance_host()
        return out

    @torch.no_grad()
    def retain(self, rows: Sequence[int]) -> None:
        """Keep these rows (in this order) and give back what the others hold; the session goes on with the smaller batch."""
        rows = list(rows)
        if rows == list(range(self.batch)):
            return
        self._graph = None
        idx = torch.tensor(rows, device=self.device)
        for c in (*self.kv, *self.lin):
            if c is not None:
                c.retain(idx)
        if self.pos_t is not None and self.pos_t.numel() == self.batch:
            self.pos_t = self.pos_t.index_select(0, idx)
        self.lengths = [self.lengths[r] for r in rows]
        self.batch, self.pos = len(rows), max(self.lengths, default=0)
