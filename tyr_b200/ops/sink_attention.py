"""Causal attention whose softmax has a sink, with an output gate:

    o_i = sum_j exp(scale q_i . k_j) v_j / (sum_j exp(scale q_i . k_j) + exp(sink_h)),   j <= i
    out = out_scale * sigmoid(gate) * o

``prompt_attention`` runs over whole prompts (tcgen05 flash kernel), ``step_attention`` over one new token per row with the K/V append
fused in (split-KV kernel, a position per row).  Sink and gate are applied inside the kernels.  The values may be the keys themselves
(the same tensor, or a ``KVCache`` whose two stores are one).  Shapes and dtypes the fast kernels do not take go to the
one-warp-per-query kernel of csrc/attention_general.cu; plain PyTorch computes the same off the GPU."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from .._native import register_signatures
from . import decode_attention as da
from . import flash
from ._common import check, cur_stream, err_word, lib, ptr, row_stride

MAX_HEAD = 256


@register_signatures
def _sigs(lib_):
    P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
    for name, args in (("tyr_general_attention_sink", [P] * 7 + [ctypes.POINTER(L)] + [I] * 7 + [F, F, I, P, P]),
                       ("tyr_decode_attention_sink", [P] * 8 + [L, L, L] + [I] * 9 + [F, P, P, L, L, F, P, P])):
        fn = getattr(lib_, name, None)
        if fn is not None:
            fn.argtypes = args
            fn.restype = I


def _finish(o, gate, out_scale, out):
    """o fp32 [B, S, H * dv] -> gated and scaled into ``out``."""
    if gate is not None:
        o = o * torch.sigmoid(gate.float())
    return out.copy_((o * out_scale).to(out.dtype))


def _general(q, k, v, kv_strides, sink, gate, out, pos, G, dv, keys, scale, out_scale):
    B, S, H, dk = q.shape
    if dk > MAX_HEAD or dv > MAX_HEAD:
        raise ValueError(f"attention heads hold at most {MAX_HEAD} channels, got {dk} and {dv}")
    st = (ctypes.c_longlong * 11)(*q.stride()[:3], *kv_strides, 0 if gate is None else row_stride(gate), row_stride(out))
    kind = {torch.bfloat16: 0, torch.float32: 1}[q.dtype]
    check(lib().tyr_general_attention_sink(ptr(q), ptr(k), ptr(v), ptr(out), ptr(pos), ptr(sink), ptr(gate), st, B, S, H, G, dk, dv, keys, scale,
                                           out_scale, kind, ptr(err_word(q.device)), cur_stream(q.device)), "general_attention_sink")
    return out


def prompt_attention(q, k, v, *, scale: float, sink: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None, out_scale: float = 1.0,
                     out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q: [B, S, H, dk], k: [B, S, G, dk], v: [B, S, G, dv] of whole prompts (rows may end earlier: padding at the end only feeds
    padding), sink fp32 [H], gate [B, S, H * dv] -> [B, S, H * dv] (``gate`` and ``out`` may be views with evenly spaced rows)."""
    B, S, H, _ = q.shape
    G, dv = k.shape[2], v.shape[3]
    if out is None:
        out = torch.empty((B, S, H * dv), dtype=q.dtype, device=q.device)
    if q.is_cuda:
        if scale > 0.0 and flash.sink_supported(q, k, v, gate, out):
            return flash.flash_fwd_sink(q, k, v, scale=scale, sink=sink, gate=gate, out_scale=out_scale, out=out)
        return _general(q, k, v, k.stride()[:3] + v.stride()[:3], sink, gate, out, None, G, dv, S, scale, out_scale)
    s = torch.einsum("bighd,bjgd->bghij", q.float().reshape(B, S, G, H // G, -1), k.float()) * scale
    s = s.masked_fill(torch.ones(S, S, dtype=torch.bool).triu(1), float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink.reshape(1, G, H // G, 1, 1).expand(B, -1, -1, S, 1)], -1)
    p = torch.softmax(s, -1)[..., :S]
    return _finish(torch.einsum("bghij,bjgd->bighd", p, v.float()).reshape(B, S, H * dv), gate, out_scale, out)


def store_dim(H: int, G: int, d: int, dtype, device) -> int:
    """Row length of a store (and of the step's queries and new keys): padded to what the split-KV kernel reads where it applies."""
    if torch.device(device).type != "cuda" or dtype != torch.bfloat16 or d > 128 or H // G > 16:
        return d
    return 64 if d <= 64 else 128


def pick_splits(B: int, G: int, keys: int) -> int:
    """Slices of the keys for one (row, K/V head).  The merge costs about as much as 512 keys, so slices are no shorter and one per (row,
    head) is best once those fill the SMs; far beyond that, three even out the last wave (measured)."""
    want = max(1, 192 // (B * G)) if B * G <= 192 else 3
    return max(1, min(want, -(-keys // 512), 32))


def step_fused(q, G: int, store) -> bool:
    """The split-KV kernel takes this step: bf16 stores of 64 or 128 channels."""
    H, d = q.shape[2], q.shape[3]
    return (q.is_cuda and q.dtype == torch.bfloat16 and H % G == 0 and H // G <= 16 and d in (64, 128) and store.k.shape[3] == store.v.shape[3] == d
            and hasattr(lib(), "tyr_decode_attention_sink"))


def step_attention(q, k_new, v_new, store, pos: torch.Tensor, dv: int, *, scale: float, sink: Optional[torch.Tensor] = None,
                   gate: Optional[torch.Tensor] = None, out_scale: float = 1.0, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One new token per row.  q: [B, 1, H, .]; k_new / v_new: [B, 1, G, .] in the row length of ``store`` (a plain ``KVCache``), which they
    are appended to; pos: int32 [B] positions of the new tokens; ``dv`` real value channels of a head -> [B, 1, H * dv]."""
    B, _, H, dkp = q.shape
    G, cap = store.k.shape[1], store.cap
    if out is None:
        out = torch.empty((B, 1, H * dv), dtype=q.dtype, device=q.device)
    if step_fused(q, G, store):
        splits = pick_splits(B, G, cap)
        key = (q.device.index, B, H, G, dkp, splits)
        ws = da._workspaces.get(key)
        if ws is None:
            ws = da._workspaces[key] = torch.zeros(lib().tyr_decode_attention_workspace_bytes(B, H, G, dkp, splits) // 4, dtype=torch.int32, device=q.device)
        check(lib().tyr_decode_attention_sink(ptr(q), ptr(k_new), ptr(v_new), ptr(store.k), ptr(store.v), ptr(pos), ptr(out), ptr(ws), q.stride(0),
                                              k_new.stride(0), v_new.stride(0), B, H, G, dkp, dv, cap, splits, 1, 1, scale, ptr(sink), ptr(gate),
                                              0 if gate is None else gate.stride(0), out.stride(0), out_scale, ptr(err_word(q.device)),
                                              cur_stream(q.device)), "decode_attention_sink")
        return out
    rows = torch.arange(B, device=q.device)
    store.k[rows, :, pos.long()] = k_new[:, 0]
    if store.v is not store.k:
        store.v[rows, :, pos.long()] = v_new[:, 0]
    if q.is_cuda:
        st = tuple(t.stride(i) for t in (store.k, store.v) for i in (0, 2, 1))
        return _general(q, store.k, store.v, st, sink, gate, out, pos, G, dv, cap, scale, out_scale)
    o = torch.empty(B, 1, H * dv)
    for b in range(B):
        n = int(pos[b]) + 1
        k, v = store.k[b, :, :n].float(), store.v[b, :, :n, :dv].float()
        s = torch.einsum("ghd,gjd->ghj", q[b, 0].float().reshape(G, H // G, -1), k) * scale
        if sink is not None:
            s = torch.cat([s, sink.reshape(G, H // G, 1)], -1)
        o[b, 0] = torch.einsum("ghj,gjd->ghd", torch.softmax(s, -1)[..., :n], v).reshape(-1)
    return _finish(o, gate, out_scale, out)
