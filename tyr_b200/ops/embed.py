"""Embedding kernels (csrc/embed.cu): table gradient from rows sorted by token id; scaled rows with sinusoidal positions."""
from __future__ import annotations

import ctypes
import math
from typing import Optional, Tuple

import torch

from .._native import register_signatures
from ._common import check, cur_stream, err_word, lib, ptr


@register_signatures
def _sigs(lib_):
    P, I, L = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong
    fn = getattr(lib_, "tyr_embed_grad_sorted", None)
    if fn is not None:
        fn.argtypes = [P, P, P, P, I, I, L, I, P]
        fn.restype = I
    fn = getattr(lib_, "tyr_embed_positions", None)
    if fn is not None:
        fn.argtypes = [P, P, P, P, P, I, I, I, I, ctypes.c_float, I, P, P]
        fn.restype = I


def sort_tokens(idx: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """(sorted ids, order) of a flat int64 token vector; one sort serves every table indexed by the same tokens."""
    sorted_ids, order = torch.sort(idx.reshape(-1))
    return sorted_ids.contiguous(), order.contiguous()


def embedding_grad_(grad_table: torch.Tensor, dy: torch.Tensor, idx: torch.Tensor, sorted_ids=None, order=None) -> None:
    """grad_table[idx[n]] += dy[n] (fp32 table [V, d], dy [N, d]).  bf16 rows on the GPU go through the sorted
    segment-sum kernel; everything else through ``index_add_``."""
    flat = dy.reshape(-1, dy.shape[-1])
    if (flat.is_cuda and flat.dtype == torch.bfloat16 and grad_table.dtype == torch.float32 and grad_table.is_contiguous()
            and flat.shape[1] % 8 == 0 and flat.stride(1) == 1 and flat.stride(0) % 8 == 0 and flat.data_ptr() % 16 == 0
            and hasattr(lib(), "tyr_embed_grad_sorted")):
        if sorted_ids is None or order is None:
            sorted_ids, order = sort_tokens(idx)
        N, d = flat.shape
        check(lib().tyr_embed_grad_sorted(ptr(flat), ptr(order), ptr(sorted_ids), ptr(grad_table), N, d, flat.stride(0),
                                          grad_table.shape[0], cur_stream(flat.device)), "embed_grad_sorted")
        return
    grad_table.index_add_(0, idx.reshape(-1), flat.to(grad_table.dtype))


def position_turns(width: int, base: float = 10000.0, device="cpu") -> torch.Tensor:
    """Frequencies of the sinusoidal position vector over 2 pi, in double: channel pair i turns ``base^(-2i / width) / 2 pi`` per position."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    return (base ** (-2.0 * i / width) / (2.0 * math.pi)).to(device)


def embed_positions(ids: torch.Tensor, table: torch.Tensor, turns: Optional[torch.Tensor], scale: float, pos: Optional[torch.Tensor] = None,
                    out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """fp32 [B, S, D]: ``table[ids] * scale`` plus the sinusoidal vector of each position (channel 2i the sine, 2i + 1 the cosine; nothing
    without ``turns``), into ``out`` when given.
    ``pos``: int32 [B] positions of single tokens (S == 1); without it positions count from 0 in every row."""
    B, S = ids.shape
    V, D = table.shape
    if not ids.is_cuda:
        x = torch.nn.functional.embedding(ids, table).float() * scale
        if turns is None:
            return x if out is None else out.copy_(x)
        p = (torch.arange(S)[None] if pos is None else pos[:, None]).double()
        angle = 2.0 * math.pi * torch.frac(p[..., None] * turns)
        vec = torch.stack([torch.sin(angle), torch.cos(angle)], -1).flatten(-2)[..., :D].float()
        return x + vec if out is None else out.copy_(x + vec)
    assert ids.dtype == torch.int64 and table.is_contiguous() and (turns is None or (turns.dtype == torch.float64 and turns.numel() == (D + 1) // 2))
    assert pos is None or (S == 1 and pos.dtype == torch.int32 and pos.numel() == B)
    x = torch.empty((B, S, D), dtype=torch.float32, device=ids.device) if out is None else out
    assert x.dtype == torch.float32 and x.shape == (B, S, D) and x.is_contiguous()
    kind = {torch.bfloat16: 0, torch.float32: 1}[table.dtype]
    check(lib().tyr_embed_positions(ptr(ids.contiguous()), ptr(table), ptr(turns), ptr(pos), ptr(x), B, S, D, V, scale, kind, ptr(err_word(ids.device)),
                                    cur_stream(ids.device)), "embed_positions")
    return x
