"""Causal attention in which all heads of a query are worked on together (csrc/joint_attention.cu):

    s_g(i, j) = softcap tanh(scale temp_g q_g . k_j / softcap) + rel[bucket(i - j), g]
    score_h   = sum_g talk[h, g] s_g,    0 <= i - j < window

``talking_prompt`` / ``talking_step`` mix the heads' scores before the softmax (``Talk``); ``latent_step`` lets every head read one
shared row per position whose first channels are its value.  The steps read a ``KVCache`` that already holds the new token.  Plain
PyTorch computes the same off the GPU."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from .._native import register_signatures
from ._common import check, cur_stream, err_word, lib, ptr


class _Scores(ctypes.Structure):
    _fields_ = [("temp", ctypes.c_void_p), ("rel", ctypes.c_void_p), ("bucket", ctypes.c_void_p), ("talk", ctypes.c_void_p),
                ("reach", ctypes.c_int), ("rows", ctypes.c_int), ("talk_exact", ctypes.c_int), ("scale", ctypes.c_float), ("softcap", ctypes.c_float)]


@register_signatures
def _sigs(lib_):
    P, I, L = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong
    S, LL = ctypes.POINTER(_Scores), ctypes.POINTER(L)
    for name, args in (("tyr_joint_attention", [P, P, P, P, P, S, LL] + [I] * 11 + [P, P]), ("tyr_joint_prompt_form", [I] * 6),
                       ("tyr_joint_prompt", [P, P, P, P, S, LL] + [I] * 7 + [P]), ("tyr_joint_step_heads", [I] * 8),
                       ("tyr_joint_step", [P, P, P, P, P, S, P, LL] + [I] * 10 + [P, P]), ("tyr_keymajor_heads", [I] * 5),
                       ("tyr_keymajor_prompt", [P] * 6 + [I, LL] + [I] * 7 + [P, P]),
                       ("tyr_keymajor_step", [P] * 7 + [I, ctypes.c_float, P, LL] + [I] * 10 + [P, P])):
        fn = getattr(lib_, name, None)
        if fn is not None:
            fn.argtypes, fn.restype = args, I
    fn = getattr(lib_, "tyr_joint_step_workspace_bytes", None)
    if fn is not None:
        fn.argtypes, fn.restype = [I, I, I, I], L


def distance_buckets(rows: int, reach: int) -> torch.Tensor:
    """int32 [reach + 1]: the row of a table of ``rows`` for the distances 0 .. reach; every distance from ``reach`` on has the last row.
    Half of the rows stand for one distance each, the others for logarithmic steps up to ``reach``."""
    half = rows // 2
    if half < 1 or reach <= half:
        raise ValueError(f"a distance table needs at least 2 rows and a reach beyond half of them, got {rows} and {reach}")
    steps, out, x = rows - half, [], 0
    for n in range(reach + 1):
        # floor(steps ln(n / half) / ln(reach / half)), decided in whole numbers: x + 1 is reached when (n / half)^steps >= (reach / half)^(x + 1)
        while x < steps - 1 and n > half and n ** steps * half ** (x + 1) >= reach ** (x + 1) * half ** steps:
            x += 1
        out.append(n if n < half else half + x)
    return torch.tensor(out, dtype=torch.int32)


@dataclass
class Talk:
    """What happens to the scores of one layer before the softmax."""
    temp: torch.Tensor            # fp32 [H]
    rel: torch.Tensor             # fp32 [rows, H]
    bucket: torch.Tensor          # int32 [reach + 1]: row of rel for a distance
    mix: torch.Tensor             # fp32 [H, H]
    softcap: float

    def __post_init__(self):
        self._plans: dict = {}
        self.exact = bool((self.mix.bfloat16().float() == self.mix).all())     # entries that TF32 holds as they are

    def scores(self, dots: torch.Tensor, dist: torch.Tensor) -> torch.Tensor:
        """dots: scaled products [..., H, i, j], dist: [i, j] -> mixed scores."""
        s = self.softcap * torch.tanh(dots * self.temp[:, None, None] / self.softcap)
        s = s + self.rel[self.bucket[dist.clamp(0, self.bucket.numel() - 1).long()].long()].permute(2, 0, 1)
        return torch.einsum("hg,...gij->...hij", self.mix, s)

    def plan(self, scale: float, dot_bound: Optional[float]):
        """The scores in log2 units against a fixed reference, score_h - reference_h = init_h + near_h[distance] + sum_g w[h, g] / (1 + exp2(k2_g x)):
        (w [HT, HT], init [HT] and k2 [HT] in one host tensor, near [H, reach + 1]), or None where their range could leave fp32 exponents.
        ``dot_bound``: largest |q . k| (None: only the cap bounds a score)."""
        key = (scale, dot_bound)
        if key not in self._plans:
            log2e, dev, H = 1.4426950408889634, self.mix.device, self.temp.numel()
            T, temp, cap = self.mix.double(), self.temp.double(), self.softcap
            near = (T @ self.rel.double()[self.bucket.long()].T) * log2e                      # [H, reach + 1], reference: the last distance
            near = near - near[:, -1:]
            top = torch.full_like(temp, cap) if dot_bound is None else cap * torch.tanh(dot_bound * abs(scale) * temp.abs() / cap)
            reach = float((T.abs() @ top * log2e + near.abs().amax(1)).max())
            if not reach <= 100.0:
                self._plans[key] = None
            else:
                HT = 8 if H <= 8 else 16 if H <= 16 else 32
                grow = lambda t, *n: torch.nn.functional.pad(t, [x for d, m in zip(reversed(t.shape), reversed(n)) for x in (0, m - d)]).flatten()
                host = torch.cat([grow(-2.0 * cap * log2e * T, HT, HT), grow(cap * log2e * T.sum(1), HT), grow(2.0 * log2e * scale * temp / cap, HT)])
                self._plans[key] = (host.float().cpu().contiguous(), near.float().contiguous().to(dev))
        return self._plans[key]

    def args(self, scale: float) -> _Scores:
        assert all(t.dtype == torch.float32 and t.is_contiguous() for t in (self.temp, self.rel, self.mix)) and self.bucket.dtype == torch.int32
        a = _Scores(scale=scale, softcap=self.softcap, reach=self.bucket.numel() - 1, rows=self.rel.shape[0], talk_exact=1 if self.exact else 0)
        a.temp, a.rel, a.bucket, a.talk = (t.data_ptr() for t in (self.temp, self.rel, self.bucket, self.mix))
        return a


def store_dims(dk: int, dv: int, dtype, device) -> tuple:
    """Row lengths of the K and V stores (and of the queries and new keys): multiples of 16 for the tensor-core forms, else the sizes
    themselves."""
    if torch.device(device).type != "cuda" or dtype != torch.bfloat16:
        return dk, dv
    return -(-dk // 16) * 16, -(-dv // 16) * 16


_workspaces: dict = {}


def _prompt_fused(q, k, v, talk: Talk) -> bool:
    """The tensor-core form takes these prompts: bf16, heads of a token adjacent in rows that are multiples of 16."""
    if q.dtype != torch.bfloat16 or not q.dtype == k.dtype == v.dtype:
        return False
    H, G, dk, dvp = q.shape[2], k.shape[2], q.shape[3], v.stride(2)
    ok = lambda t, d: t.stride(3) == 1 and t.stride(2) == d and t.stride(0) % 8 == 0 and t.stride(1) % 8 == 0 and t.data_ptr() % 16 == 0
    return (ok(q, dk) and ok(k, dk) and ok(v, dvp) and dvp >= v.shape[3] and v.stride(1) >= G * dvp
            and lib().tyr_joint_prompt_form(H, G, dk, dvp, talk.rel.shape[0], talk.bucket.numel() - 1) != 0)


def pick_splits(B: int, blocks: int, keys: int) -> int:
    """Slices of the keys for one (row, block of heads): one CTA fills an SM, and a slice should outweigh its part of the merge."""
    return max(1, min(148 // (B * blocks), -(-keys // 128), 32))


def _step_heads(q, store, dv: int, talk: Optional[Talk]) -> int:
    """Heads of a CTA of the tensor-core step, 0 where it does not apply."""
    if q.dtype != torch.bfloat16 or store.k.dtype != q.dtype or q.shape[3] != store.k.shape[3] or q.stride(3) != 1:
        return 0
    shared = store.v is store.k
    if shared != (talk is None) or any(s % 8 for s in (q.stride(0), q.stride(2))) or q.data_ptr() % 16:
        return 0
    return lib().tyr_joint_step_heads(0 if talk is None else 1, q.shape[2], store.k.shape[1], q.shape[3], dv, store.v.shape[3], 1 if shared else 0,
                                      0 if talk is None else talk.rel.shape[0])


def _kind(t: torch.Tensor) -> int:
    if t.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"attention kernels take bf16 or fp32, got {t.dtype}")
    return 0 if t.dtype == torch.bfloat16 else 1


def _general(q, k, v, kv_strides, scores: _Scores, out, pos, G, dk, dv, cap, ring, window, keys):
    B, S, H, _ = q.shape
    st = (ctypes.c_longlong * 11)(*q.stride()[:3], *kv_strides, out.stride(1) if S > 1 else out.stride(0), out.stride(2))
    check(lib().tyr_joint_attention(ptr(q), ptr(k), ptr(v), ptr(out), ptr(pos), ctypes.byref(scores), st, B, S, H, G, dk, dv, cap, 1 if ring else 0,
                                    int(window or 0), keys, _kind(q), ptr(err_word(q.device)), cur_stream(q.device)), "joint_attention")
    return out


def _rows_ok(*ts) -> bool:
    """bf16 head rows that TMA and vector loads take: contiguous channels, strides that are multiples of 8, 16-byte aligned."""
    return all(t.dtype == torch.bfloat16 and t.stride(3) == 1 and all(x % 8 == 0 for x in t.stride()[:3]) and t.data_ptr() % 16 == 0 for t in ts)


def _keymajor_prompt(q, k, v, out, scale, talk: Talk, dot_bound) -> bool:
    B, S, H, dk = q.shape
    G, dv = k.shape[2], v.shape[3]
    dvp = -(-dv // 8) * 8
    if not _rows_ok(q, k, v) or v.stride(2) < dvp or not lib().tyr_keymajor_heads(0, H, G, dk, dv):
        return False
    plan = talk.plan(scale, dot_bound)
    if plan is None:
        return False
    st = (ctypes.c_longlong * 12)(*[t.stride(i) for t in (q, k, v, out) for i in range(3)])
    check(lib().tyr_keymajor_prompt(ptr(q), ptr(k), ptr(v), ptr(out), *(ptr(t) for t in plan), plan[1].shape[1] - 1, st, B, S, H, G, dk, dv, dvp,
                                    ptr(err_word(q.device)), cur_stream(q.device)), "keymajor_prompt")
    return True


def _workspace(q, H, dv, splits):
    key = (q.device.index, q.shape[0], H, dv, splits)
    ws = _workspaces.get(key)
    if ws is None and splits > 1:
        ws = _workspaces[key] = torch.zeros(lib().tyr_joint_step_workspace_bytes(q.shape[0], H, dv, splits) // 4, dtype=torch.int32, device=q.device)
    return ws


def _keymajor_step(q, store, pos, out, dv, scale, window, talk: Optional[Talk], dot_bound) -> bool:
    B, _, H, dk = q.shape
    G, cap, dvp = store.k.shape[1], store.cap, store.v.shape[3]
    shared = store.v is store.k
    if not _rows_ok(q, store.k, store.v) or not (store.k.is_contiguous() and store.v.is_contiguous()) or dk != store.k.shape[3] or shared != (talk is None):
        return False
    if store.ring and (talk is not None or (window is not None and window < cap)) or (talk is not None and window is not None):
        return False
    hb = lib().tyr_keymajor_heads(2 if shared else 1, H, G, dk, dv)
    plan = (None,) * 2 if shared else talk.plan(scale, dot_bound)
    if not hb or plan is None:
        return False
    splits = pick_splits(B, -(-H // hb), min(cap, window) if window else cap)
    st = (ctypes.c_longlong * 4)(q.stride(0), q.stride(2), out.stride(0), out.stride(2))
    check(lib().tyr_keymajor_step(ptr(q), ptr(store.k), ptr(store.v), ptr(out), ptr(pos), *(ptr(t) for t in plan), 0 if shared else plan[1].shape[1] - 1, scale,
                                  ptr(_workspace(q, H, dv, splits)), st, B, H, G, dk, dv, dvp, cap, 1 if store.ring else 0, int(window or 0), splits,
                                  ptr(err_word(q.device)), cur_stream(q.device)), "keymajor_step")
    return True


def prompt_attention(q, k, v, *, scale: float, window: Optional[int] = None, talk: Optional[Talk] = None,
                     dot_bound: Optional[float] = None) -> torch.Tensor:
    """Whole prompts (rows may end earlier: padding at the end only feeds padding).  q: [B, S, H, dk], k: [B, S, G, dk], v: [B, S, G, dv]
    -> [B, S, H * dv].  ``talk``: mixed scores; ``dot_bound``: largest |q . k| there can be, where one is known (unit queries and keys)."""
    B, S, H, dk = q.shape
    G, dv = k.shape[2], v.shape[3]
    if q.is_cuda:
        out = torch.empty((B, S, H, dv), dtype=q.dtype, device=q.device)
        scores = _Scores(scale=scale) if talk is None else talk.args(scale)
        if talk is not None and window is None and _keymajor_prompt(q, k, v, out, scale, talk, dot_bound):
            return out.flatten(2)
        if talk is not None and window is None and _prompt_fused(q, k, v, talk):
            st = (ctypes.c_longlong * 6)(*[t.stride(i) for t in (q, k, v) for i in range(2)])
            check(lib().tyr_joint_prompt(ptr(q), ptr(k), ptr(v), ptr(out), ctypes.byref(scores), st, B, S, H, G, dk, dv, v.stride(2), cur_stream(q.device)),
                  "joint_prompt")
            return out.flatten(2)
        return _general(q, k, v, (*k.stride()[:3], *v.stride()[:3]), scores, out, None, G, dk, dv, S, False, window, S).flatten(2)
    s = torch.einsum("bighd,bjgd->bghij", q.float().reshape(B, S, G, H // G, dk), k.float()).reshape(B, H, S, S) * scale
    dist = torch.arange(S)[:, None] - torch.arange(S)[None, :]
    if talk is not None:
        s = talk.scores(s, dist)
    seen = (dist >= 0) if window is None else (dist >= 0) & (dist < window)
    p = torch.softmax(s.masked_fill(~seen, float("-inf")), -1).reshape(B, G, H // G, S, S)
    return torch.einsum("bghij,bjgd->bighd", p, v.float()).reshape(B, S, H * dv).to(q.dtype)


def step_attention(q, store, pos: torch.Tensor, dv: int, *, scale: float, window: Optional[int] = None, talk: Optional[Talk] = None,
                   out: Optional[torch.Tensor] = None, dot_bound: Optional[float] = None) -> torch.Tensor:
    """One token per row against a ``KVCache`` (plain or ring) that holds it.  q: [B, 1, H, dk]; pos: int32 [B]; ``dv`` value channels (of
    a shared store: the first of the keys) -> [B, 1, H, dv], into ``out`` (a view with contiguous channels) if given."""
    B, _, H, dk = q.shape
    G, cap = store.k.shape[1], store.cap
    if out is None:
        out = torch.empty((B, 1, H, dv), dtype=q.dtype, device=q.device)
    if q.is_cuda:
        st = tuple(t.stride(i) for t in (store.k, store.v) for i in (0, 2, 1))
        scores = _Scores(scale=scale) if talk is None else talk.args(scale)
        if _keymajor_step(q, store, pos, out, dv, scale, window, talk, dot_bound):
            return out
        hb = _step_heads(q, store, dv, talk)
        if hb:
            splits = pick_splits(B, -(-H // hb), min(cap, window) if window else cap)
            ws = _workspace(q, H, dv, splits)
            so = (ctypes.c_longlong * 4)(q.stride(0), q.stride(2), out.stride(0), out.stride(2))
            check(lib().tyr_joint_step(ptr(q), ptr(store.k), None if talk is None else ptr(store.v), ptr(out), ptr(pos), ctypes.byref(scores), ptr(ws), so, B, H, G,
                                       dk, dv, store.v.shape[3], cap, 1 if store.ring else 0, int(window or 0), splits, ptr(err_word(q.device)),
                                       cur_stream(q.device)), "joint_step")
            return out
        return _general(q, store.k, store.v, st, scores, out, pos, G, dk, dv, cap, store.ring, window, cap)
    for b in range(B):
        p = int(pos[b])
        n = p + 1 if window is None else min(p + 1, window)
        if store.ring:
            n = min(n, cap)
        at = torch.arange(p + 1 - n, p + 1)
        slots = at % cap if store.ring else at
        k, v = store.k[b][:, slots, :dk].float(), store.v[b][:, slots, :dv].float()
        s = torch.einsum("ghd,gjd->ghj", q[b, 0].float().reshape(G, H // G, dk), k).reshape(H, 1, n) * scale
        if talk is not None:
            s = talk.scores(s, (p - at)[None])
        w = torch.softmax(s[:, 0], -1).reshape(G, H // G, n)
        out[b, 0] = torch.einsum("ghj,gjd->ghd", w, v).reshape(H, dv).to(q.dtype)
    return out
