"""The step between a layer's input projection and its mixers (csrc/mix_conv.cu): column segments of the projection, each with an
optional short causal convolution, activation and position-dependent factor, written where its consumer reads it.  One launch for
all segments of a layer; plain PyTorch computes the same off the GPU."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Sequence

import torch

from .._native import register_signatures
from ._common import check, cur_stream, lib

MAX_SEGMENTS = 6
_ACT = {None: 0, "silu": 1, "relu2": 2, "xielu": 3}


class _Seg(ctypes.Structure):
    _fields_ = [("col", ctypes.c_int), ("heads", ctypes.c_int), ("d_in", ctypes.c_int), ("d_out", ctypes.c_int), ("taps", ctypes.c_int),
                ("act", ctypes.c_int), ("w", ctypes.c_void_p), ("bias", ctypes.c_void_p), ("window", ctypes.c_void_p), ("out", ctypes.c_void_p),
                ("out_ld", ctypes.c_longlong), ("store", ctypes.c_void_p), ("cap", ctypes.c_int), ("store_d", ctypes.c_int),
                ("temp_coef", ctypes.c_float), ("temp_every", ctypes.c_float), ("act_a", ctypes.c_float), ("act_b", ctypes.c_float)]


class _Args(ctypes.Structure):
    _fields_ = [("x", ctypes.c_void_p), ("x_sb", ctypes.c_longlong), ("x_ss", ctypes.c_longlong), ("lens", ctypes.c_void_p),
                ("pos", ctypes.c_void_p), ("B", ctypes.c_int), ("S", ctypes.c_int), ("n_seg", ctypes.c_int), ("groups", ctypes.c_int),
                ("seg", _Seg * MAX_SEGMENTS)]


@register_signatures
def _sigs(lib_):
    fn = getattr(lib_, "tyr_mix_conv", None)
    if fn is not None:
        fn.argtypes = [ctypes.POINTER(_Args), ctypes.c_int, ctypes.c_int, ctypes.c_void_p]
        fn.restype = ctypes.c_int


@dataclass
class Segment:
    """Columns [col, col + heads * d) of the projection -> ``out`` [B, S, heads * d_out] (evenly spaced rows, contiguous channels; the
    channels of a head past d are zero).  ``w`` fp32 [heads * d, taps] and ``bias`` fp32: causal convolution whose last ``taps`` inputs
    are the ``window`` [B, heads * d, taps].  ``temp`` (coef, every): the result is multiplied by
    1 + coef ln(floor((p + 1) / every) + 1) at position p.  ``act`` "silu", "relu2" or "xielu" (``act_args`` (a, b): a z^2 + z / 2 above
    zero, b (e^z - 1 - z) + z / 2 below).  ``store`` [B, heads, cap, d_store] receives whole prompts by position."""
    col: int
    heads: int
    d: int
    out: torch.Tensor
    d_out: Optional[int] = None
    w: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None
    window: Optional[torch.Tensor] = None
    act: Optional[str] = None
    temp: Optional[tuple] = None
    store: Optional[torch.Tensor] = None
    act_args: tuple = (0.0, 0.0)


def xielu(z: torch.Tensor, a: float, b: float) -> torch.Tensor:
    """a z^2 + z / 2 above zero, b (e^z - 1 - z) + z / 2 below."""
    low = z.clamp_max(0.0)
    return torch.where(z > 0, a * z * z, b * (torch.expm1(low) - low)) + 0.5 * z


def temperature(p: torch.Tensor, coef: float, every: float) -> torch.Tensor:
    """fp32 factors of the positions ``p``."""
    return 1.0 + coef * torch.log(torch.floor((p.float() + 1.0) / every) + 1.0)


def _plain(x, segments, lens, pos, step):
    B, S, _ = x.shape
    for s in segments:
        C = s.heads * s.d
        u = x[..., s.col:s.col + C]
        if s.w is None:
            y = u.float()
        else:
            K = s.w.shape[1]
            if step:
                s.window.copy_(torch.cat([s.window[:, :, 1:], u.transpose(1, 2)], 2))
                hist = s.window.transpose(1, 2)                                            # [B, K, C]
            else:
                hist = torch.cat([torch.zeros(B, K - 1, C, dtype=x.dtype), u], 1)
                for b in range(B):
                    n = S if lens is None else int(lens[b])
                    if s.window is not None:
                        s.window[b] = torch.cat([torch.zeros(K, C, dtype=x.dtype), u[b, :n]])[-K:].T
            y = sum(hist[:, j:j + S].float() * s.w[:, j] for j in range(K))
            if s.bias is not None:
                y = y + s.bias
        if s.act == "silu":
            y = torch.nn.functional.silu(y)
        elif s.act == "relu2":
            y = torch.relu(y).square()
        elif s.act == "xielu":
            y = xielu(y, *s.act_args)
        if s.temp is not None:
            p = pos[:, None] if step else torch.arange(S)[None]
            y = y * temperature(p, *s.temp)[:, :, None]
        y = y.to(x.dtype).reshape(B, S, s.heads, s.d)
        d_out = s.d_out or s.d
        s.out.copy_(torch.nn.functional.pad(y, (0, d_out - s.d)).reshape(B, S, s.heads * d_out))
        if s.store is not None and not step:
            for b in range(B):
                n = S if lens is None else int(lens[b])
                s.store[b, :, :n, :s.d] = y[b, :n].transpose(0, 1)


def _run(x, segments: Sequence[Segment], lens, pos, step: bool):
    B, S, _ = x.shape
    if not x.is_cuda:
        return _plain(x, segments, lens, pos, step)
    assert len(segments) <= MAX_SEGMENTS and x.stride(2) == 1 and x.dtype in (torch.bfloat16, torch.float32)
    a = _Args()
    p = lambda t: None if t is None else t.data_ptr()
    a.x, a.x_sb, a.x_ss, a.lens, a.pos, a.B, a.S, a.n_seg = x.data_ptr(), x.stride(0), x.stride(1), p(lens), p(pos), B, S, len(segments)
    for r, s in zip(a.seg, segments):
        C, d_out = s.heads * s.d, s.d_out or s.d
        o = s.out
        assert o.shape == (B, S, s.heads * d_out) and o.stride(2) == 1 and o.dtype == x.dtype and (B == 1 or S == 1 or o.stride(0) == S * o.stride(1))
        r.col, r.heads, r.d_in, r.d_out, r.act = s.col, s.heads, s.d, d_out, _ACT[s.act]
        r.out, r.out_ld = o.data_ptr(), o.stride(1) if S > 1 else o.stride(0)
        if s.w is not None:
            assert s.w.dtype == torch.float32 and s.w.is_contiguous() and s.w.shape[0] == C and (s.bias is None or s.bias.dtype == torch.float32)
            r.taps, r.w, r.bias, r.window = s.w.shape[1], s.w.data_ptr(), p(s.bias), p(s.window)
            assert s.window is None or (s.window.is_contiguous() and s.window.dtype == x.dtype and s.window.shape == (B, C, r.taps))
        if s.store is not None and not step:
            assert s.store.is_contiguous() and s.store.dtype == x.dtype and s.store.shape[:2] == (B, s.heads)
            r.store, r.cap, r.store_d = s.store.data_ptr(), s.store.shape[2], s.store.shape[3]
        if s.temp is not None:
            r.temp_coef, r.temp_every = s.temp
        r.act_a, r.act_b = s.act_args
    check(lib().tyr_mix_conv(ctypes.byref(a), 1 if step else 0, 1 if x.dtype == torch.float32 else 0, cur_stream(x.device)), "mix_conv")


def mix_prompt(x: torch.Tensor, segments: Sequence[Segment], lens: Optional[torch.Tensor] = None) -> None:
    """x: [B, S, columns] (contiguous channels) of fresh prompts; ``lens`` int32 [B] where rows end earlier."""
    _run(x, segments, lens, None, False)


def mix_step(x: torch.Tensor, segments: Sequence[Segment], pos: torch.Tensor) -> None:
    """x: [B, 1, columns]; ``pos`` int32 [B] positions of the new tokens."""
    _run(x, segments, None, pos, True)


def activate(x: torch.Tensor, act: str, act_args: tuple = (0.0, 0.0)) -> torch.Tensor:
    """An activation alone, of contiguous rows [..., C]."""
    rows = x.numel() // x.shape[-1]
    flat = x.view(rows, 1, -1) if rows < 4096 else x.view(1, rows, -1)        # few rows: a thread each instead of a thread per 64
    y = torch.empty_like(flat)
    mix_prompt(flat, [Segment(0, 1, x.shape[-1], y, act=act, act_args=act_args)])
    return y.view(x.shape)
