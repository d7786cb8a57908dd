"""Selective scan (csrc/selective_scan.cu): per channel c and state n

    delta = softplus(dt + dt_bias[c]);  S[c, n] <- exp(delta A[c, n]) S[c, n] + delta x B[n];  y = sum_n S[c, n] C[n] + D[c] x
    out = scale * y * silu(z)

with an fp32 state that is carried from token to token.  Plain PyTorch computes the same off the GPU."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from .._native import register_signatures
from ._common import check, cur_stream, lib, ptr, row_stride

MAX_STATES = 256


@register_signatures
def _sigs(lib_):
    P, I = ctypes.c_void_p, ctypes.c_int
    fn = getattr(lib_, "tyr_selective_scan", None)
    if fn is not None:
        fn.argtypes = [P] * 5 + [ctypes.POINTER(ctypes.c_longlong)] + [P] * 6 + [I] * 6 + [ctypes.c_float, I, P]
        fn.restype = I


def _plain(x, dt, z, b, c, A, D, dt_bias, state, out, lens, scale):
    B, S, C = x.shape
    delta = torch.nn.functional.softplus(dt.float() + dt_bias)
    xf, y = x.float(), torch.zeros(B, S, C)
    for r in range(B):
        for t in range(S if lens is None else int(lens[r])):
            state[r] = torch.exp(delta[r, t][:, None] * A) * state[r] + (delta[r, t] * xf[r, t])[:, None] * b[r, t].float()
            y[r, t] = state[r] @ c[r, t].float() + D * xf[r, t]
    out.copy_((scale * y * torch.nn.functional.silu(z.float())).to(out.dtype))


def _run(x, dt, z, b, c, A, D, dt_bias, state, out, lens, scale, fresh, step):
    B, S, C = x.shape
    N = A.shape[1]
    if N > MAX_STATES:
        raise ValueError(f"selective scan holds at most {MAX_STATES} states per channel, got {N}")
    if not x.is_cuda:
        if fresh:
            state.zero_()
        return _plain(x, dt, z, b, c, A, D, dt_bias, state, out, lens, scale)
    assert x.dtype == dt.dtype == z.dtype == b.dtype == c.dtype == out.dtype and x.dtype in (torch.bfloat16, torch.float32)
    assert all(t.dtype == torch.float32 and t.is_contiguous() for t in (A, D, dt_bias, state)) and state.shape == (B, C, N)
    if row_stride(b) != row_stride(c):
        raise ValueError("B and C of a selective scan must be windows of rows with one stride")
    ld = (ctypes.c_longlong * 5)(*[row_stride(t) for t in (x, dt, z, b, out)])
    check(lib().tyr_selective_scan(ptr(x), ptr(dt), ptr(z), ptr(b), ptr(c), ld, ptr(A), ptr(D), ptr(dt_bias), ptr(state), ptr(out), ptr(lens),
                                   B, S, C, N, 1 if fresh else 0, 1 if step else 0, scale, 1 if x.dtype == torch.float32 else 0, cur_stream(x.device)),
          "selective_scan")


def scan_prompt(x, dt, z, b, c, A, D, dt_bias, state, out, lens: Optional[torch.Tensor] = None, scale: float = 1.0, fresh: bool = True) -> None:
    """x, dt, z: [B, S, C]; b, c: [B, S, N]; A fp32 [C, N]; D, dt_bias fp32 [C] -> ``out`` [B, S, C] (rows of a view may be strided).  ``state``
    fp32 [B, C, N] receives the state after each row's ``lens`` tokens; it starts at zero when ``fresh``.  Rows of ``out`` past ``lens`` are
    of no meaning."""
    _run(x, dt, z, b, c, A, D, dt_bias, state, out, lens, scale, fresh, False)


def scan_step(x, dt, z, b, c, A, D, dt_bias, state, out, scale: float = 1.0) -> None:
    """One token per row ([B, 1, .] operands); ``state`` is advanced in place."""
    _run(x, dt, z, b, c, A, D, dt_bias, state, out, None, scale, False, True)
