"""Decode-sized linear layers (1..32 rows) on the weight-streaming kernel (csrc/skinny_gemm.cu)."""
from __future__ import annotations

import ctypes
import os
from typing import Optional

import torch

from .._native import register_signatures
from ._common import check, cur_stream, lib, ptr

MAX_ROWS = 32
_workspaces = {}


def _workspace(device, M: int, N: int) -> torch.Tensor:
    """fp32 [M * N] scratch of the split reduction; zero between calls (the finishing kernel re-zeroes what it read)."""
    key = (device.index, M * N)
    ws = _workspaces.get(key)
    if ws is None:
        ws = _workspaces[key] = torch.zeros(M * N, dtype=torch.float32, device=device)
    return ws


@register_signatures
def _sigs(lib_):
    P, I, L = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong
    fn = getattr(lib_, "tyr_skinny_gemm_bf16", None)
    if fn is not None:
        fn.argtypes = [P, P, P, P, P, L, L, L, I, I, I, P]
        fn.restype = I
        lib_.tyr_skinny_gemm_splits.argtypes = [I, I]
        lib_.tyr_skinny_gemm_splits.restype = I
    F = ctypes.c_float
    for name, args in (("tyr_skinny_gemm_act_bf16", [P, P, P, P, P, L, L, L, I, I, I, I, F, F, P]),
                       ("tyr_skinny_heads_bf16", [P, P, P, L, L, L, L, L, L, I, I, I, I, P]),
                       ("tyr_skinny_gelu_mul_bf16", [P, P, P, P, P, L, L, L, L, I, I, I, P])):
        fn = getattr(lib_, name, None)
        if fn is not None:
            fn.argtypes, fn.restype = args, I
    fn = getattr(lib_, "tyr_skinny_swiglu_bf16", None)
    if fn is not None:
        fn.argtypes = [P, P, P, P, L, L, L, I, I, I, P]
        fn.restype = I


LINEAR_MAX_ROWS = 16     # plain products above this many rows go to the library GEMM (measured 2.5x faster at 32 rows)


def supported(x2: torch.Tensor, w: torch.Tensor, max_rows: int = LINEAR_MAX_ROWS) -> bool:
    M, K = x2.shape
    # 9..16 rows with a long contraction leave too few loads in flight per warp; the library GEMM is faster there
    return (x2.is_cuda and x2.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and 1 <= M <= min(max_rows, MAX_ROWS) and (M <= 8 or K <= 8192) and K >= 32 and K % 32 == 0
            and x2.stride(1) == 1 and w.stride(1) == 1 and x2.stride(0) % 8 == 0 and w.stride(0) % 8 == 0
            and x2.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


def skinny_linear(x2: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x2: [M <= 32, K] bf16, w: [N, K] bf16 (rows may be strided) -> [M, N] bf16 with fp32 accumulation; ``out`` (rows may be
    strided, e.g. a window of a symmetric-heap buffer) receives the result when given."""
    M, K = x2.shape
    N = w.shape[0]
    if not x2.is_cuda:
        y = x2.float() @ w.float().T
        y = (y if bias is None else y + bias.float()).to(x2.dtype)
        if out is not None:
            out.copy_(y)
            return out
        return y
    y = torch.empty((M, N), dtype=torch.bfloat16, device=x2.device) if out is None else out
    assert y.shape == (M, N) and y.dtype == torch.bfloat16 and y.stride(1) == 1
    b = None if bias is None else bias.to(torch.bfloat16).contiguous()
    ws = _workspace(x2.device, M, N) if lib().tyr_skinny_gemm_splits(N, K) > 1 else None
    check(lib().tyr_skinny_gemm_bf16(ptr(x2), ptr(w), ptr(b), ptr(y), ptr(ws), x2.stride(0), w.stride(0), y.stride(0), M, N, K, cur_stream(x2.device)), "skinny_gemm_bf16")
    return y


_SWIGLU = os.environ.get("TYR_SKINNY_SWIGLU", "1") != "0"


def swiglu_supported(x2: torch.Tensor, gate_w: torch.Tensor, up_w: torch.Tensor) -> bool:
    # the gated form replaces a library product plus two element-wise launches and stays ahead of them up to 32 rows
    return (_SWIGLU and supported(x2, gate_w, MAX_ROWS) and supported(x2, up_w, MAX_ROWS) and gate_w.shape == up_w.shape and gate_w.stride(0) == up_w.stride(0)
            and hasattr(lib(), "tyr_skinny_swiglu_bf16"))


def skinny_swiglu(x2: torch.Tensor, gate_w: torch.Tensor, up_w: torch.Tensor) -> torch.Tensor:
    """x2: [M <= 32, K] bf16 -> silu(x2 gate_w^T) * (x2 up_w^T) as [M, N] bf16: both matrices streamed once, one launch."""
    M, K = x2.shape
    N = gate_w.shape[0]
    if not x2.is_cuda:
        return (torch.nn.functional.silu(x2.float() @ gate_w.float().T) * (x2.float() @ up_w.float().T)).to(x2.dtype)
    y = torch.empty((M, N), dtype=torch.bfloat16, device=x2.device)
    check(lib().tyr_skinny_swiglu_bf16(ptr(x2), ptr(gate_w), ptr(up_w), ptr(y), x2.stride(0), gate_w.stride(0), N, M, N, K, cur_stream(x2.device)),
          "skinny_swiglu")
    return y


def skinny_xielu(x2: torch.Tensor, w: torch.Tensor, a: float, b: float) -> torch.Tensor:
    """x2: [M <= 32, K] bf16 -> xIELU of ``x2 w^T`` (factors ``a`` above zero, ``b`` below) as [M, N] bf16, in the product's epilogue."""
    M, K = x2.shape
    N = w.shape[0]
    y = torch.empty((M, N), dtype=torch.bfloat16, device=x2.device)
    ws = _workspace(x2.device, M, N) if lib().tyr_skinny_gemm_splits(N, K) > 1 else None
    check(lib().tyr_skinny_gemm_act_bf16(ptr(x2), ptr(w), None, ptr(y), ptr(ws), x2.stride(0), w.stride(0), N, M, N, K, 6, a, b, cur_stream(x2.device)),
          "skinny_xielu")
    return y


def skinny_gelu_mul(x2: torch.Tensor, w: torch.Tensor, e: torch.Tensor) -> torch.Tensor:
    """x2: [M <= 32, K] bf16 -> tanh-GELU of ``x2 w^T`` times ``e`` [M, N] (rows may be strided) as [M, N] bf16, in the product's epilogue."""
    M, K = x2.shape
    N = w.shape[0]
    assert e.shape == (M, N) and e.dtype == torch.bfloat16 and e.stride(1) == 1
    y = torch.empty((M, N), dtype=torch.bfloat16, device=x2.device)
    ws = _workspace(x2.device, M, N) if lib().tyr_skinny_gemm_splits(N, K) > 1 else None
    check(lib().tyr_skinny_gelu_mul_bf16(ptr(x2), ptr(w), ptr(e), ptr(y), ptr(ws), x2.stride(0), w.stride(0), e.stride(0), N, M, N, K, cur_stream(x2.device)),
          "skinny_gelu_mul")
    return y


def head_products_supported(x: torch.Tensor, w: torch.Tensor) -> bool:
    return (x.is_cuda and x.dtype == w.dtype == torch.bfloat16 and w.shape[2] % 32 == 0 and x.stride(2) == w.stride(2) == 1
            and all(s % 8 == 0 for s in (*x.stride()[:2], *w.stride()[:2])) and x.data_ptr() % 16 == w.data_ptr() % 16 == 0)


def head_products(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """A matrix of its own for each head: out[m, h, :N] = x[m, h, :K] w[h]^T.  x: [M, H, >= K] and out: [M, H, >= N] (views with contiguous
    channels), w: [H, N, K].  Channels of x past K and of out past N are left alone."""
    M, H = x.shape[:2]
    _, N, K = w.shape
    if not head_products_supported(x, w):
        out[..., :N] = torch.einsum("mhk,hnk->mhn", x[..., :K], w) if x.is_cuda else torch.einsum("mhk,hnk->mhn", x[..., :K].float(), w.float()).to(out.dtype)
        return out
    assert x.shape[2] >= K and out.shape[:2] == (M, H) and out.shape[2] >= N and out.stride(2) == 1 and out.dtype == x.dtype
    for m in range(0, M, MAX_ROWS):
        n = min(MAX_ROWS, M - m)
        check(lib().tyr_skinny_heads_bf16(ptr(x[m:]), ptr(w), ptr(out[m:]), x.stride(0), x.stride(1), w.stride(0), w.stride(1), out.stride(0), out.stride(1),
                                          H, n, N, K, cur_stream(x.device)), "skinny_heads")
    return out
