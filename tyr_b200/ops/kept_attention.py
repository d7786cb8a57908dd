"""Causal attention over a sliding window that leaves the first positions visible:

    o_i = softmax over j of (scale q_i . k_j) v_j,   j <= i and (i - j < window or j < keep)

with values that may be rotated by their positions (every output is then turned back by the query's angles) and one output gate
per head.  ``rotary_store`` rotates queries and keys, norms and rotates values and fills the store; ``prompt_attention`` runs over whole
prompts (tcgen05 flash kernel), ``step_attention`` over one new token per row (split-KV kernel, a position per row, a plain store
or one of kept slots followed by a ring).  Shapes and dtypes those do not take go to the one-warp-per-query kernel of
csrc/attention_general.cu.  Plain PyTorch computes the same off the GPU."""
from __future__ import annotations

import ctypes
import math
from typing import Optional, Tuple

import torch

from .._native import register_signatures
from . import decode_attention as da
from . import flash
from ._common import check, cur_stream, err_word, lib, ptr, row_stride
from .norm import rms_norm_ref

MAX_HEAD = 256
_KIND = {torch.bfloat16: 0, torch.float32: 1}


@register_signatures
def _sigs(lib_):
    P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
    for name, args in (("tyr_rotary_store", [P, L] + [P] * 9 + [ctypes.POINTER(I), F, I, P, P]),
                       ("tyr_general_attention_kept", [P] * 7 + [I, ctypes.POINTER(L)] + [I] * 11 + [F, I, P, P]),
                       ("tyr_decode_attention_kept", [P] * 6 + [I, P, P, L, L, L] + [I] * 12 + [F, P, L, P, I, L, P, P])):
        fn = getattr(lib_, name, None)
        if fn is not None:
            fn.argtypes, fn.restype = args, I


def turn_table(dims: int, base: float, factor: float, positions: int, device) -> Optional[torch.Tensor]:
    """fp32 [positions, dims / 2, 2]: cosine and sine of p base^(-2i / dims) / factor, angles in double; None without dims."""
    if dims == 0:
        return None
    i = torch.arange(dims // 2, dtype=torch.float64, device=device)
    turns = base ** (-2.0 * i / dims) / (factor * 2.0 * math.pi)
    angle = 2.0 * math.pi * torch.frac(torch.arange(positions, dtype=torch.float64, device=device)[:, None] * turns)
    return torch.stack([torch.cos(angle), torch.sin(angle)], -1).float().contiguous()


def rotate(x: torch.Tensor, table: Optional[torch.Tensor], p: torch.Tensor, back: bool = False) -> torch.Tensor:
    """x: [B, S, H, d] in fp32; the pairs (i, i + half) turn by their angles at positions p [B, S] (``back``: the other way)."""
    if table is None:
        return x
    cs = table[p.long()].unsqueeze(2)
    c, s = cs[..., 0], -cs[..., 1] if back else cs[..., 1]
    half = table.shape[1]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def _positions(B, S, pos):
    p = torch.arange(S)[None].expand(B, S)
    return p if pos is None else p + pos[:, None].long()


def step_dims(H: int, G: int, dk: int, dv: int, dtype, device) -> Tuple[int, int]:
    """Row lengths of the stores (and of a step's queries): padded to what the split-KV kernel reads where it applies, else the sizes."""
    if torch.device(device).type != "cuda" or dtype != torch.bfloat16 or dk > 128 or dv > 128 or H // G > 16:
        return dk, dv
    up = lambda d: 64 if d <= 64 else 128
    return up(dk), up(dv)


def rotary_store(y: torch.Tensor, H: int, G: int, dk: int, dv: int, key_table: Optional[torch.Tensor], value_table: Optional[torch.Tensor], eps: float, *,
                 store=None, pos: Optional[torch.Tensor] = None, lens: Optional[torch.Tensor] = None, norm_v: bool = True):
    """y: [B, S, >= (H + G) dk + G dv] rows q | k | v.  Queries and keys turn by ``key_table``, values are divided by their root mean square
    (``norm_v``) and turn by ``value_table``.  ``store`` (a ``KVCache``) receives keys and values of the first ``lens[b]`` tokens of every row at
    positions ``pos[b]`` + s.  Without ``pos`` (prompts) returns q [B, S, H, dk], k [B, S, G, dk], v [B, S, G, dv]; with it (steps) q in the
    store's row length and None twice."""
    B, S, _ = y.shape
    step = pos is not None
    if not y.is_cuda:
        yf, p = y.float(), _positions(B, S, pos)
        part = lambda a, n, d: yf[..., a:a + n * d].reshape(B, S, n, d)
        q, k = (rotate(t, key_table, p).to(y.dtype) for t in (part(0, H, dk), part(H * dk, G, dk)))
        v = part((H + G) * dk, G, dv)
        v = rotate(rms_norm_ref(v, eps) if norm_v else v, value_table, p).to(y.dtype)
        if store is not None:
            for b in range(B):
                n, p0 = S if lens is None else int(lens[b]), 0 if pos is None else int(pos[b])
                at = store.held(p0, p0 + n - 1)
                store.k[b, :, store.slots(at), :dk] = k[b, at - p0].transpose(0, 1)
                store.v[b, :, store.slots(at), :dv] = v[b, at - p0].transpose(0, 1)
        return (torch.nn.functional.pad(q, (0, store.k.shape[3] - dk)), None, None) if step else (q, k, v)
    new = lambda n, d: torch.empty((B, S, n, d), dtype=y.dtype, device=y.device)
    dkp, dvp = (store.k.shape[3], store.v.shape[3]) if store is not None else (dk, dv)
    q = new(H, dkp if step else dk)
    k, v = (None, None) if step else (new(G, dk), new(G, dv))
    half = lambda t: 0 if t is None else t.shape[1]
    tables = [t for t in (key_table, value_table) if t is not None]
    assert all(t.dtype == torch.float32 and t.is_contiguous() for t in tables)
    sizes = (ctypes.c_int * 18)(B, S, H, G, dk, dv, q.shape[3], dk, dv, dkp, dvp, store.cap if store is not None else 0, 1 if store is not None and store.ring else 0,
                                store.keep if store is not None else 0, half(key_table), half(value_table), min([t.shape[0] for t in tables], default=1 << 30),
                                1 if norm_v else 0)
    check(lib().tyr_rotary_store(ptr(y), row_stride(y), ptr(key_table), ptr(value_table), ptr(q), ptr(k), ptr(v), ptr(store.k) if store is not None else None,
                                 ptr(store.v) if store is not None else None, ptr(pos), ptr(lens), sizes, eps, _KIND[y.dtype], ptr(err_word(y.device)),
                                 cur_stream(y.device)), "rotary_store")
    return q, k, v


def _general(q, k, v, kv_strides, head_gate, back, pos, G, dk, dv, cap, ring, window, keep, keys, scale):
    B, S, H, _ = q.shape
    if dk > MAX_HEAD or dv > MAX_HEAD:
        raise ValueError(f"attention heads hold at most {MAX_HEAD} channels, got {dk} and {dv}")
    out = torch.empty((B, S, H * dv), dtype=q.dtype, device=q.device)
    st = (ctypes.c_longlong * 11)(*q.stride()[:3], *kv_strides, 0 if head_gate is None else row_stride(head_gate), row_stride(out))
    check(lib().tyr_general_attention_kept(ptr(q), ptr(k), ptr(v), ptr(out), ptr(pos), ptr(head_gate), ptr(back), 0 if back is None else back.shape[0], st, B, S, H, G, dk, dv,
                                           cap, 1 if ring else 0,
                                           int(window or 0), keep, keys, scale, _KIND[q.dtype], ptr(err_word(q.device)), cur_stream(q.device)),
          "general_attention_kept")
    return out


def prompt_attention(q, k, v, *, scale: float, window: Optional[int] = None, keep: int = 0, head_gate: Optional[torch.Tensor] = None,
                     back: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q: [B, S, H, dk], k: [B, S, G, dk], v: [B, S, G, dv] of whole prompts (rows may end earlier: padding at the end only feeds padding),
    ``head_gate`` [B, S, H] logits, ``back`` the values' table of turns -> [B, S, H * dv]."""
    B, S, H, dk = q.shape
    G, dv = k.shape[2], v.shape[3]
    if q.is_cuda:
        if scale > 0.0 and flash.biased_supported(q, k, v) and hasattr(lib(), "tyr_flash_fwd_kept") and (back is None or dv % 16 == 0):
            return flash.flash_fwd_kept(q, k, v, scale=scale, window=window, keep=keep, head_gate=head_gate, back=back)
        return _general(q, k, v, k.stride()[:3] + v.stride()[:3], head_gate, back, None, G, dk, dv, S, False, window, keep, S, scale)
    s = torch.einsum("bighd,bjgd->bghij", q.float().reshape(B, S, G, H // G, dk), k.float()) * scale
    i, j = torch.arange(S)[:, None], torch.arange(S)[None, :]
    seen = (j <= i) if window is None else (j <= i) & ((i - j < window) | (j < keep))
    p = torch.softmax(s.masked_fill(~seen, float("-inf")), -1)
    return _finish(torch.einsum("bghij,bjgd->bighd", p, v.float()).reshape(B, S, H, dv), head_gate, back, _positions(B, S, None), q.dtype)


def _finish(o, head_gate, back, p, dtype):
    o = rotate(o, back, p, back=True)
    if head_gate is not None:
        o = o * torch.sigmoid(head_gate.float())[..., None]
    return o.flatten(2).to(dtype)


def step_fused(q: torch.Tensor, G: int, store) -> bool:
    """The split-KV kernel takes this step: bf16 stores of 64 or 128 channels."""
    H = q.shape[2]
    return (q.is_cuda and q.dtype == torch.bfloat16 and H % G == 0 and H // G <= 16 and store.k.shape[3] in (64, 128) and store.v.shape[3] in (64, 128)
            and q.shape[3] == store.k.shape[3] and hasattr(lib(), "tyr_decode_attention_kept"))


def step_attention(q, store, pos: torch.Tensor, dk: int, dv: int, *, scale: float, window: Optional[int] = None, keep: int = 0,
                   head_gate: Optional[torch.Tensor] = None, back: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One new token per row, whose key and value ``store`` holds already.  q: [B, 1, H, .] in the store's row length (dk channels count);
    pos: int32 [B] positions of the new tokens; ``head_gate`` [B, 1, H] -> [B, 1, H * dv]."""
    B, _, H, dkp = q.shape
    G, cap = store.k.shape[1], store.cap
    dvp = store.v.shape[3]
    assert not store.ring or store.keep == keep
    if step_fused(q, G, store):
        keys = min(cap, window + keep) if window else cap
        splits = da.pick_splits(B, G, keys)
        key = (q.device.index, B, H, G, dvp, splits)
        ws = da._workspaces.get(key)
        if ws is None:
            ws = da._workspaces[key] = torch.zeros(lib().tyr_decode_attention_workspace_bytes(B, H, G, dvp, splits) // 4, dtype=torch.int32, device=q.device)
        out = torch.empty((B, 1, H * dv), dtype=q.dtype, device=q.device)
        check(lib().tyr_decode_attention_kept(ptr(q), None, None, ptr(store.k), ptr(store.v), ptr(pos), 1, ptr(out), ptr(ws), q.stride(0), 0, 0, B, H, G, dkp, dvp,
                                              dv, cap, 1 if store.ring else 0, int(window or 0), keep, splits, 0, scale, ptr(head_gate),
                                              0 if head_gate is None else head_gate.stride(0), ptr(back), 0 if back is None else back.shape[0], out.stride(0), ptr(err_word(q.device)),
                                              cur_stream(q.device)), "decode_attention_kept")
        return out
    if q.is_cuda:
        st = tuple(t.stride(i) for t in (store.k, store.v) for i in (0, 2, 1))
        return _general(q, store.k, store.v, st, head_gate, back, pos, G, dk, dv, cap, store.ring, window, keep, cap, scale)
    o = torch.empty(B, 1, H, dv)
    for b in range(B):
        p = int(pos[b])
        at = store.held(0, p)
        if window is not None:
            at = at[(p - at < window) | (at < keep)]
        k, v = store.k[b][:, store.slots(at), :dk].float(), store.v[b][:, store.slots(at), :dv].float()
        s = torch.einsum("ghd,gjd->ghj", q[b, 0, :, :dk].float().reshape(G, H // G, dk), k) * scale
        o[b, 0] = torch.einsum("ghj,gjd->ghd", torch.softmax(s, -1), v).reshape(H, dv)
    return _finish(o, head_gate, back, pos[:, None].long(), q.dtype)
