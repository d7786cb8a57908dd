"""Activations of two operands alone (csrc/gates.cu), and a projection with one in its epilogue.  Plain PyTorch computes the same off the
GPU."""
from __future__ import annotations

import ctypes

import torch

from .._native import register_signatures
from . import skinny as _skinny
from .gemm import clamped_swiglu as _clamped_swiglu, gemm as _gemm
from ._common import check, cur_stream, lib, ptr

_KIND = {torch.bfloat16: 0, torch.float32: 1}
MIN_GEMM_ROWS = 128


@register_signatures
def _sigs(lib_):
    P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
    for name, args in (("tyr_clamped_swiglu", [P, L, P, L, I, I, F, F, I, P]), ("tyr_gelu_mul", [P, L, P, L, P, L, I, I, P])):
        fn = getattr(lib_, name, None)
        if fn is not None:
            fn.argtypes, fn.restype = args, I


def clamped_swiglu(z: torch.Tensor, n: int, limit: float, slope: float, block: int = 0) -> torch.Tensor:
    """z: [rows, 2 n] gate columns, then up columns (``block`` > 0: blocks of that many gate columns and the matching up columns) -> [rows, n]."""
    block = block or n
    if not z.is_cuda:
        b = z.reshape(z.shape[0], -1, 2, block)
        return _clamped_swiglu(b[:, :, 0], b[:, :, 1], limit, slope).reshape(z.shape[0], -1)[:, :n].to(z.dtype)
    out = torch.empty((z.shape[0], n), dtype=z.dtype, device=z.device)
    check(lib().tyr_clamped_swiglu(ptr(z), z.stride(0), ptr(out), z.shape[0], n, block, limit, slope, _KIND[z.dtype], cur_stream(z.device)), "clamped_swiglu")
    return out


def gelu_mul(z: torch.Tensor, e: torch.Tensor) -> torch.Tensor:
    """tanh-GELU of z times e, [rows, n] each (rows may be strided)."""
    if not z.is_cuda:
        return (torch.nn.functional.gelu(z.float(), approximate="tanh") * e.float()).to(z.dtype)
    assert z.shape == e.shape and z.dtype == e.dtype and z.stride(1) == e.stride(1) == 1
    out = torch.empty(z.shape, dtype=z.dtype, device=z.device)
    check(lib().tyr_gelu_mul(ptr(z), z.stride(0), ptr(e), e.stride(0), ptr(out), z.shape[0], z.shape[1], _KIND[z.dtype], cur_stream(z.device)), "gelu_mul")
    return out


def gelu_mul_project(x: torch.Tensor, w: torch.Tensor, e: torch.Tensor) -> torch.Tensor:
    """tanh-GELU of ``x w^T`` times e: x [rows, K], w [n, K], e [rows, n] (rows may be strided) -> [rows, n], in the product's epilogue where
    one applies."""
    if x.is_cuda and x.dtype == w.dtype == e.dtype == torch.bfloat16 and e.stride(1) == 1:
        if (x.shape[0] >= MIN_GEMM_ROWS and w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0 and e.stride(0) % 8 == 0 and e.data_ptr() % 16 == 0
                and w.is_contiguous()):
            return _gemm(x.contiguous(), w, act="gelu_mul", aux=e)
        if _skinny.supported(x, w):
            return _skinny.skinny_gelu_mul(x, w, e)
    return gelu_mul(torch.nn.functional.linear(x, w), e)
