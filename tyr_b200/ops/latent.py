"""Pieces of latent attention (csrc/latent.cu): norms of the query and key/value latents, the rotated key part all heads share, the store
of both, and the rotation of the queries.  Plain PyTorch computes the same off the GPU."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from .._native import register_signatures
from ._common import check, cur_stream, lib, ptr, row_stride

_KIND = {torch.bfloat16: 0, torch.float32: 1}


@register_signatures
def _sigs(lib_):
    P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
    for name, args in (("tyr_latent_norm_store", [P, L, P, P, P, P, L, P, P, P, P] + [I] * 9 + [F, I, P]),
                       ("tyr_rotate_heads", [P, P, P, P, ctypes.POINTER(L)] + [I] * 7 + [P])):
        fn = getattr(lib_, name, None)
        if fn is not None:
            fn.argtypes, fn.restype = args, I


def rotate(x: torch.Tensor, turns: torch.Tensor, p: torch.Tensor) -> torch.Tensor:
    """x: [B, S, ..., d] in fp32; the channel pairs (2i, 2i + 1) turn by ``turns[i]`` turns per position p [B, S]; the rest passes."""
    n = turns.numel()
    angle = 2.0 * torch.pi * torch.frac(p.double()[..., None] * turns)
    shape = (*p.shape, *(1,) * (x.dim() - 3), n)
    c, s = torch.cos(angle).float().reshape(shape), torch.sin(angle).float().reshape(shape)
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., 2 * n:]], -1)


def _positions(B, S, pos):
    p = torch.arange(S)[None].expand(B, S)
    return p if pos is None else p + pos[:, None].long()


def latent_norm_store(y: torch.Tensor, q_w: torch.Tensor, kv_w: torch.Tensor, turns: torch.Tensor, rot: int, eps: float, *, q_width: int, width: int,
                      store=None, pos: Optional[torch.Tensor] = None, lens: Optional[torch.Tensor] = None, want_rows: bool = True):
    """y: [B, S, >= q_rank + rank + rot] rows (query latent | key/value latent | rotated part).  Returns (RMS-normed query latent
    [B, S, q_width], rows [B, S, width] of normed latent | rotated part | zeros); channels of the first past q_rank are zero.  ``store``
    (a shared ``KVCache`` with one head) receives the rows of the first ``lens[b]`` tokens at positions ``pos[b]`` + s (a ring store: its
    last ``cap``)."""
    B, S, _ = y.shape
    nq, nk = q_w.numel(), kv_w.numel()
    new = torch.zeros if q_width != nq else torch.empty
    cq = new((B, S, q_width), dtype=y.dtype, device=y.device)
    if not y.is_cuda:
        yf = y.float()
        norm = lambda t, w: t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w
        cq[..., :nq] = norm(yf[..., :nq], q_w).to(y.dtype)
        rows = torch.cat([norm(yf[..., nq:nq + nk], kv_w), rotate(yf[..., nq + nk:nq + nk + rot], turns, _positions(B, S, pos))], -1).to(y.dtype)
        rows = torch.nn.functional.pad(rows, (0, width - nk - rot))
        if store is not None:
            for b in range(B):
                n, p0 = S if lens is None else int(lens[b]), 0 if pos is None else int(pos[b])
                s0 = max(0, n - store.cap) if store.ring else 0
                at = torch.arange(p0 + s0, p0 + n)
                store.k[b, 0, at % store.cap if store.ring else at] = rows[b, s0:n]
        return cq, rows
    rows = torch.empty((B, S, width), dtype=y.dtype, device=y.device) if want_rows else None
    assert store is None or (store.k.shape[1] == 1 and store.k.shape[3] == width and store.k.is_contiguous() and store.k.dtype == y.dtype)
    check(lib().tyr_latent_norm_store(ptr(y), row_stride(y), ptr(q_w), ptr(kv_w), ptr(turns), ptr(cq), q_width, ptr(rows),
                                      ptr(store.k) if store is not None else None, ptr(pos), ptr(lens), B, S, nq, nk, rot, 2 * turns.numel(), width,
                                      store.cap if store is not None else 0, 1 if store is not None and store.ring else 0, eps, _KIND[y.dtype],
                                      cur_stream(y.device)), "latent_norm_store")
    return cq, rows


def rotate_heads(x: torch.Tensor, turns: torch.Tensor, pos: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x: [B, S, H, rot] (a view of head rows): its channel pairs turned by position (counted from 0, or from ``pos[b]``), in place or into
    ``out`` [B, S, H, >= rot], whose channels past rot become zero."""
    B, S, H, rot = x.shape
    y = x if out is None else out
    if not x.is_cuda:
        r = rotate(x.float(), turns, _positions(B, S, pos)).to(x.dtype)
        y[..., :rot] = r
        y[..., rot:] = 0
        return y
    assert x.stride(3) == y.stride(3) == 1 and y.dtype == x.dtype and turns.dtype == torch.float64
    st = (ctypes.c_longlong * 6)(*x.stride()[:3], *y.stride()[:3])
    check(lib().tyr_rotate_heads(ptr(x), ptr(y), ptr(turns), ptr(pos), st, B, S, H, rot, 2 * turns.numel(), y.shape[3], _KIND[x.dtype],
                                 cur_stream(x.device)), "rotate_heads")
    return y
