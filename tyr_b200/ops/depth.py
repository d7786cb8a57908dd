"""Average over depth (csrc/depth_average.cu): a layer's last residual add (its norm included), the stored result, the weighted sum over all
stored results and the next norm in one launch.  Plain PyTorch computes the same off the GPU."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from .._native import register_signatures
from ._common import check, cur_stream, lib, ptr
from .norm import rms_norm_ref

_KIND = {torch.bfloat16: 0, torch.float32: 1}


@register_signatures
def _sigs(lib_):
    P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
    fn = getattr(lib_, "tyr_depth_average", None)
    if fn is not None:
        fn.argtypes, fn.restype = [P, L, P, P, P, L, P, P, P, L, I, I, I, F, I, I, P], I


def depth_average(y: Optional[torch.Tensor], post: Optional[torch.Tensor], x: torch.Tensor, history: torch.Tensor, n: int, weights: torch.Tensor,
                  gain: torch.Tensor, eps: float, out_dtype: torch.dtype, store: bool = True) -> torch.Tensor:
    """``X_n = x + norm(y) post`` (``y`` itself without ``post``), kept as ``history[n]`` with ``store``; ``x = sum_{j<=n} weights[j] X_j`` IN PLACE
    over the results ``history[:n]`` and X_n; returns ``norm(x) gain`` in ``out_dtype``.  x: fp32 [..., D]; history: fp32 [layers, ..., D]
    (its first dimension may have any stride); y like x in any dtype."""
    D = x.shape[-1]
    if not x.is_cuda:
        if y is not None:
            y = y.float()
            x = x.add_(y if post is None else rms_norm_ref(y, eps) * post)
        if store:
            history[n].copy_(x)
        x.copy_(torch.tensordot(weights[:n], history[:n], dims=1) + weights[n] * x)
        return (rms_norm_ref(x, eps) * gain).to(out_dtype)
    assert x.dtype == history.dtype == weights.dtype == gain.dtype == torch.float32 and x.is_contiguous() and history[0].is_contiguous()
    assert history.shape[1:] == x.shape and history.shape[0] >= n + (1 if store else 0) and weights.numel() == n + 1 and gain.is_contiguous()
    y2 = None if y is None else y.reshape(-1, D)
    out = torch.empty(x.shape, dtype=out_dtype, device=x.device)
    check(lib().tyr_depth_average(ptr(y2), 0 if y2 is None else y2.stride(0), ptr(post), ptr(x), ptr(history), history.stride(0), ptr(weights), ptr(gain), ptr(out),
                                  x.numel() // D, D, n, 1 if store else 0, eps, _KIND[out_dtype if y2 is None else y2.dtype], _KIND[out_dtype],
                                  cur_stream(x.device)), "depth_average")
    return out
