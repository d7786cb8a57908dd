"""Linear attention with one decay per head (csrc/lightning.cu):  S <- decay S + k v^T,  o = S^T q, fp32 state and read-out.  Prompts take
activated q, k and v; single tokens take them before SiLU.  Plain PyTorch computes the same off the GPU."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from .._native import register_signatures
from ._common import check, cur_stream, lib, ptr

_KIND = {torch.bfloat16: 0, torch.float32: 1}


@register_signatures
def _sigs(lib_):
    P, I, L = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong
    for name, args in (("tyr_lightning_recurrent", [P] * 7 + [ctypes.POINTER(L)] + [I] * 7 + [P]),
                       ("tyr_lightning_chunk", [P] * 7 + [ctypes.POINTER(L)] + [I] * 5 + [P]),
                       ("tyr_lightning_step", [P] * 6 + [ctypes.POINTER(L)] + [I] * 6 + [P])):
        fn = getattr(lib_, name, None)
        if fn is not None:
            fn.argtypes, fn.restype = args, I


def _plain(q, k, v, decay, state, lens, silu):
    B, S, H, _ = q.shape
    act = lambda t: torch.nn.functional.silu(t.float()).to(t.dtype).float() if silu else t.float()
    q, k, v = act(q), act(k), act(v)
    out = torch.zeros(B, S, H, v.shape[3])
    d = decay.float()[:, None, None]
    low = (decay - decay.float().double()).float()[:, None, None]
    for b in range(B):
        s = state[b]
        for t in range(S if lens is None else int(lens[b])):
            s = d * s + (low * s + k[b, t][:, :, None] * v[b, t][:, None, :])
            out[b, t] = torch.einsum("hdv,hd->hv", s, q[b, t])
        state[b] = s
    return out


def _strides(q, k, v):
    return (ctypes.c_longlong * 9)(*[t.stride(i) for t in (q, k, v) for i in range(3)])


def recurrent(q, k, v, decay: torch.Tensor, state: torch.Tensor, lens: Optional[torch.Tensor] = None, silu: bool = False) -> torch.Tensor:
    """q, k: [B, S, H, dk], v: [B, S, H, dv] (views with contiguous channels; ``silu``: before their activation), decay double [H];
    ``state`` fp32 [B, H, dk, dv] is advanced IN PLACE over the first ``lens[b]`` tokens of row b; the read-out fp32 [B, S, H, dv] is
    zero past them."""
    B, S, H, dk = q.shape
    dv = v.shape[3]
    if not q.is_cuda:
        return _plain(q, k, v, decay, state, lens, silu)
    assert state.dtype == torch.float32 and state.is_contiguous() and decay.dtype == torch.float64
    assert q.stride(3) == k.stride(3) == v.stride(3) == 1 and q.dtype == k.dtype == v.dtype
    out = torch.empty((B, S, H, dv), dtype=torch.float32, device=q.device)
    check(lib().tyr_lightning_recurrent(ptr(q), ptr(k), ptr(v), ptr(decay), ptr(state), ptr(out), ptr(lens), _strides(q, k, v), B, S, H, dk, dv,
                                        1 if silu else 0, _KIND[q.dtype], cur_stream(q.device)), "lightning_recurrent")
    return out


def chunk_supported(q, k, v) -> bool:
    """bf16, key size up to 128, sizes and strides multiples of 8, 16-byte aligned rows."""
    ok = lambda t: t.stride(3) == 1 and all(x % 8 == 0 for x in t.stride()[:3]) and t.data_ptr() % 16 == 0 and t.shape[3] % 8 == 0
    return q.is_cuda and q.dtype == k.dtype == v.dtype == torch.bfloat16 and q.shape[3] <= 128 and ok(q) and ok(k) and ok(v)


def prefill(q, k, v, decay: torch.Tensor, state: torch.Tensor, lens: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Fresh prompts of activated q, k, v: :func:`recurrent` from a zero state.  The tensor-core chunk form where it applies."""
    if not chunk_supported(q, k, v):
        state.zero_()
        return recurrent(q, k, v, decay, state, lens)
    B, S, H, dk = q.shape
    dv = v.shape[3]
    assert state.dtype == torch.float32 and state.is_contiguous() and decay.dtype == torch.float64
    out = torch.empty((B, S, H, dv), dtype=torch.float32, device=q.device)
    check(lib().tyr_lightning_chunk(ptr(q), ptr(k), ptr(v), ptr(decay), ptr(state), ptr(out), ptr(lens), _strides(q, k, v), B, S, H, dk, dv,
                                    cur_stream(q.device)), "lightning_chunk")
    return out


def step(q, k, v, decay: torch.Tensor, state: torch.Tensor) -> torch.Tensor:
    """One token per row, before SiLU: q, k [B, 1, H, dk], v [B, 1, H, dv]; ``state`` advanced in place, fp32 read-out [B, 1, H, dv]."""
    B, _, H, dk = q.shape
    dv = v.shape[3]
    if not q.is_cuda or dv % 4 or dk > 4096:
        return recurrent(q, k, v, decay, state, silu=True)
    assert state.dtype == torch.float32 and state.is_contiguous() and decay.dtype == torch.float64
    assert q.stride(3) == k.stride(3) == v.stride(3) == 1 and q.dtype == k.dtype == v.dtype
    out = torch.empty((B, 1, H, dv), dtype=torch.float32, device=q.device)
    check(lib().tyr_lightning_step(ptr(q), ptr(k), ptr(v), ptr(decay), ptr(state), ptr(out), _strides(q, k, v), B, H, dk, dv, 1, _KIND[q.dtype],
                                   cur_stream(q.device)), "lightning_step")
    return out
