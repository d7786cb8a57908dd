"""Attention with a logarithmic distance penalty on the scores and an optional sliding window:

    score(i, j) = scale q_i . k_j - r1_h ln(1 + r2_h (i - j)),   0 <= i - j < window.

``prompt_attention`` runs over whole prompts (tcgen05 flash kernel), ``step_attention`` over one new token per row with the K/V
append fused in (split-KV kernel, a position per row, plain or ring store).  Shapes and dtypes those do not take go to the
one-warp-per-query kernel of csrc/attention_general.cu, which also norms q / k and fills the store (``qk_norm_store``).  Plain
PyTorch computes the same off the GPU."""
from __future__ import annotations

import ctypes
from typing import Optional, Tuple

import torch

from .._native import register_signatures
from . import decode_attention as da
from . import flash
from ._common import check, cur_stream, err_word, lib, ptr, row_stride

MAX_HEAD = 256


@register_signatures
def _sigs(lib_):
    P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
    for name, args in (("tyr_qk_norm_store", [P, L] + [P] * 10 + [I] * 10 + [F, I, P]),
                       ("tyr_general_attention", [P] * 7 + [ctypes.POINTER(L)] + [I] * 10 + [F, I, P, P])):
        fn = getattr(lib_, name, None)
        if fn is not None:
            fn.argtypes = args
            fn.restype = I


def _dt(t: torch.Tensor) -> int:
    if t.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"attention kernels take bf16 or fp32, got {t.dtype}")
    return 0 if t.dtype == torch.bfloat16 else 1


def store_dims(H: int, G: int, dk: int, dv: int, dtype, device) -> Tuple[int, int]:
    """Row lengths of the K and V stores: padded to what the split-KV kernel reads where it applies, else the sizes themselves."""
    if torch.device(device).type != "cuda" or dtype != torch.bfloat16 or dk > 128 or dv > 128 or H // G > 16:
        return dk, dv
    up = lambda d: 64 if d <= 64 else 128
    return up(dk), up(dv)


def penalty(r1: torch.Tensor, r2: torch.Tensor, dist: torch.Tensor) -> torch.Tensor:
    """[H, ...] penalties of the distances ``dist``."""
    shape = (-1,) + (1,) * dist.dim()
    return r1.reshape(shape) * torch.log1p(r2.reshape(shape) * dist.float())


def qk_norm_store(y: torch.Tensor, q_w: Optional[torch.Tensor], k_w: Optional[torch.Tensor], H: int, G: int, dk: int, dv: int, eps: float, *,
                  dkp: int, dvp: int, store=None, pos: Optional[torch.Tensor] = None, lens: Optional[torch.Tensor] = None,
                  want_v: bool = True, bias: Optional[torch.Tensor] = None):
    """y: [B, S, >= (H + G) dk + G dv] rows q | k | v (G = 0: q alone), to which ``bias`` (fp32, one per column) is
    added.  Per-head RMSNorm of q and k with the fp32 weights (None: no weight);
    returns (q [B, S, H, dkp], k [B, S, G, dkp], v [B, S, G, dvp]) with zeros in the padded channels.  ``store`` (a ``KVCache``)
    receives k and v of the first ``lens[b]`` tokens of every row at positions ``pos[b]`` + s (a ring store: its last ``cap``)."""
    B, S, _ = y.shape
    F_ = torch.nn.functional
    if not y.is_cuda:
        dt, y = y.dtype, y[..., :(H + G) * dk + G * dv].float() + (0.0 if bias is None else bias)
        norm = lambda t, w: (t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * (1.0 if w is None else w)).to(dt)
        q = F_.pad(norm(y[..., :H * dk].reshape(B, S, H, dk), q_w), (0, dkp - dk))
        if G == 0:
            return q, None, None
        k = F_.pad(norm(y[..., H * dk:(H + G) * dk].reshape(B, S, G, dk), k_w), (0, dkp - dk))
        v = F_.pad(y[..., (H + G) * dk:(H + G) * dk + G * dv].reshape(B, S, G, dv), (0, dvp - dv)).to(dt)
        if store is not None:
            for b in range(B):
                n, p0 = S if lens is None else int(lens[b]), 0 if pos is None else int(pos[b])
                s0 = max(0, n - store.cap) if store.ring else 0
                slots = torch.arange(p0 + s0, p0 + n) % store.cap if store.ring else torch.arange(p0, p0 + n)
                store.k[b, :, slots] = k[b, s0:n].transpose(0, 1)
                store.v[b, :, slots] = v[b, s0:n].transpose(0, 1)
        return q, k, v
    q = torch.empty((B, S, H, dkp), dtype=y.dtype, device=y.device)
    k = torch.empty((B, S, G, dkp), dtype=y.dtype, device=y.device) if G else None
    v = torch.empty((B, S, G, dvp), dtype=y.dtype, device=y.device) if G and want_v else None
    check(lib().tyr_qk_norm_store(ptr(y), row_stride(y), ptr(q_w), ptr(k_w), ptr(bias), ptr(q), ptr(k), ptr(v), ptr(store.k) if store is not None else None,
                                  ptr(store.v) if store is not None else None, ptr(pos), ptr(lens), B, S, H, G, dk, dv, dkp, dvp,
                                  store.cap if store is not None else 0, 1 if store is not None and store.ring else 0, eps, _dt(y),
                                  cur_stream(y.device)), "qk_norm_store")
    return q, k, v


def _general(q, k, v, strides, r1, r2, pos, G, dv, cap, ring, window, keys, scale):
    B, S, H, dk = q.shape
    out = torch.empty((B, S, H, dv), dtype=q.dtype, device=q.device)
    st = (ctypes.c_longlong * 9)(*(q.stride()[:3] + strides))
    check(lib().tyr_general_attention(ptr(q), ptr(k), ptr(v), ptr(out), ptr(pos), ptr(r1), ptr(r2), st, B, S, H, G, dk, dv, cap, 1 if ring else 0,
                                      int(window or 0), keys, scale, _dt(q), ptr(err_word(q.device)), cur_stream(q.device)), "general_attention")
    return out


def prompt_attention(q, k, v, r1, r2, *, window: Optional[int], scale: float) -> torch.Tensor:
    """q: [B, S, H, dk], k: [B, S, G, dk], v: [B, S, G, dv] of whole prompts (rows may end earlier: padding at the end only feeds
    padding) -> [B, S, H, dv]."""
    if q.is_cuda:
        if flash.biased_supported(q, k, v):
            return flash.flash_fwd_biased(q, k, v, r1, r2, window=window, scale=scale)
        S = q.shape[1]
        return _general(q, k, v, k.stride()[:3] + v.stride()[:3], r1, r2, None, k.shape[2], v.shape[3], S, False, window, S, scale)
    B, S, H, _ = q.shape
    G = k.shape[2]
    s = torch.einsum("bighd,bjgd->bghij", q.float().reshape(B, S, G, H // G, -1), k.float()) * scale
    dist = torch.arange(S)[:, None] - torch.arange(S)[None, :]
    s = s - penalty(r1, r2, dist.clamp_min(0)).reshape(1, G, H // G, S, S)
    seen = (dist >= 0) if window is None else (dist >= 0) & (dist < window)
    p = torch.softmax(s.masked_fill(~seen, float("-inf")), -1)
    return torch.einsum("bghij,bjgd->bighd", p, v.float()).reshape(B, S, H, -1).to(q.dtype)


def step_fused(q: torch.Tensor, G: int, store) -> bool:
    """The split-KV kernel takes this step (and does the append): bf16 stores of 64 or 128 channels."""
    H = q.shape[2]
    return (q.is_cuda and q.dtype == torch.bfloat16 and H % G == 0 and H // G <= 16 and store.k.shape[3] in (64, 128) and store.v.shape[3] in (64, 128)
            and hasattr(lib(), "tyr_decode_attention_biased"))


def step_attention(q, k_new, v_new, store, pos: torch.Tensor, r1, r2, *, window: Optional[int], scale: float, append: bool) -> torch.Tensor:
    """One new token per row.  q: [B, 1, H, dkp]; k_new / v_new: [B, 1, G, .] in the store's row layout; pos: int32 [B] positions of
    the new tokens.  Attends the last ``window`` positions held by ``store`` (a ``KVCache``; all of them without a window), the new
    one included -> [B, 1, H, dvp].  ``append`` False when the store already holds the new token (a layer that reads another
    layer's keys)."""
    B, _, H, dkp = q.shape
    G, cap = store.k.shape[1], store.cap
    dvp = store.v.shape[3]
    if step_fused(q, G, store):
        keys = min(cap, window) if window else cap
        splits = da.pick_splits(B, G, keys)
        key = (q.device.index, B, H, G, dvp, splits)
        ws = da._workspaces.get(key)
        if ws is None:
            ws = da._workspaces[key] = torch.zeros(lib().tyr_decode_attention_workspace_bytes(B, H, G, dvp, splits) // 4, dtype=torch.int32, device=q.device)
        out = torch.empty((B, 1, H, dvp), dtype=q.dtype, device=q.device)
        check(lib().tyr_decode_attention_biased(ptr(q), ptr(k_new), ptr(v_new), ptr(store.k), ptr(store.v), ptr(pos), 1, ptr(out), ptr(ws), q.stride(0),
                                                k_new.stride(0), v_new.stride(0), B, H, G, dkp, dvp, cap, 1 if store.ring else 0, int(window or 0), splits,
                                                1 if append else 0, scale, ptr(r1), ptr(r2), ptr(err_word(q.device)), cur_stream(q.device)),
              "decode_attention_biased")
        return out
    if append:
        rows = torch.arange(B, device=q.device)
        slots = (pos % cap if store.ring else pos).long()
        store.k[rows, :, slots] = k_new[:, 0]
        store.v[rows, :, slots] = v_new[:, 0]
    if q.is_cuda:
        st = tuple(t.stride(i) for t in (store.k, store.v) for i in (0, 2, 1))
        return _general(q, store.k, store.v, st, r1, r2, pos, G, dvp, cap, store.ring, window, cap, scale)
    out = torch.empty(B, 1, H, dvp, dtype=q.dtype)
    for b in range(B):
        p = int(pos[b])
        n = p + 1 if window is None else min(p + 1, window)
        if store.ring:
            n = min(n, cap)
        at = torch.arange(p + 1 - n, p + 1)
        slots = at % cap if store.ring else at
        k, v = store.k[b][:, slots].float(), store.v[b][:, slots].float()
        s = torch.einsum("ghd,gjd->ghj", q[b, 0].float().reshape(G, H // G, -1), k) * scale - penalty(r1, r2, p - at).reshape(G, H // G, n)
        out[b, 0] = torch.einsum("ghj,gjd->ghd", torch.softmax(s, -1), v).reshape(H, dvp).to(q.dtype)
    return out
