"""Gated delta rule (Qwen3.5 GatedDeltaNet core): chunked prefill, recurrent oracle, fused decode step.

q, k: [B, S, H, dk]; v: [B, S, H, dv]; g (log decay, <= 0) and beta: [B, S, H]; state [B, H, dk, dv] fp32.
Semantics: cc/src/tyr_qwen35.cpp:12-170 of the reference (L2-normalised q/k, q scaled by dk^-1/2).
"""
from __future__ import annotations

import os
from typing import Optional, Tuple

import torch

from .._native import register_signatures
from ._common import check, cur_stream, err_word, lib, ptr, row_stride


@register_signatures
def _sigs(lib_):
    import ctypes
    P, I, L = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong
    fn = getattr(lib_, "tyr_gdr_decode", None)
    if fn is not None:
        fn.argtypes = [P, P, P, P, P, P, P, I, I, I, I, I, L, L, P]
        fn.restype = ctypes.c_int
    fn = getattr(lib_, "tyr_gdr_decode_norm", None)
    if fn is not None:
        fn.argtypes = [P, P, P, P, P, P, P, I, I, I, I, I, L, L, P, L, P, ctypes.c_float, P]
        fn.restype = ctypes.c_int
    fn = getattr(lib_, "tyr_gdr_decode_tile", None)
    if fn is not None:
        fn.argtypes = [P, P, P, P, P, P, P, I, I, I, I, L, L, P, L, P, ctypes.c_float, I, P, P]
        fn.restype = ctypes.c_int
    fn = getattr(lib_, "tyr_gdn_conv_gates", None)
    if fn is not None:
        fn.argtypes = [P] * 3 + [L, L, L] + [P] * 8 + [I, I, I, I, P]
        fn.restype = ctypes.c_int
    fn = getattr(lib_, "tyr_gdr_chunk_scan", None)
    if fn is not None:
        fn.argtypes = [P] * 9 + [I, I, I, I, I, I, I, I, I, P]
        fn.restype = ctypes.c_int
    fn = getattr(lib_, "tyr_gdr_chunk_prepare_channel", None)
    if fn is not None:
        fn.argtypes = [P] * 14 + [ctypes.POINTER(L), I, I, I, I, I, I, P]
        fn.restype = ctypes.c_int
    fn = getattr(lib_, "tyr_gdr_decode_tile_channel", None)
    if fn is not None:
        fn.argtypes = [P] * 11 + [ctypes.POINTER(L), I, I, I, I, ctypes.c_float, P, P]
        fn.restype = ctypes.c_int
    fn = getattr(lib_, "tyr_gdr_chunk_prepare", None)
    if fn is not None:
        fn.argtypes = [P] * 12 + [ctypes.POINTER(L), I, I, I, I, I, I, P]
        fn.restype = ctypes.c_int
    fn = getattr(lib_, "tyr_causal_conv1d_silu", None)
    if fn is not None:
        fn.argtypes = [P, P, P, P, I, I, I, I, L, L, P]
        fn.restype = ctypes.c_int
    F = ctypes.c_float
    for name, args in (("tyr_conv_silu", [P, P, P, I, I, I, I, L, L, I, P]),
                       ("tyr_delta_conv_gates", [P, P, P, L, L, L] + [P] * 7 + [I, I, I, I, I, P]),
                       ("tyr_delta_gates", [P, P, L, L, P, P, P, P, L, I, I, P]),
                       ("tyr_gdr_recurrent", [P] * 8 + [ctypes.POINTER(L), I, I, I, I, I, I, I, P]),
                       ("tyr_gdr_recurrent_channel", [P] * 10 + [ctypes.POINTER(L), I, I, I, I, I, I, I, P]),
                       ("tyr_gated_norm", [P, P, L, P, P, L, L, I, I, F, I, I, P])):
        fn = getattr(lib_, name, None)
        if fn is not None:
            fn.argtypes = args
            fn.restype = ctypes.c_int


def _dt(t: torch.Tensor) -> int:
    """Activation type code of csrc/delta_general.cu."""
    if t.dtype == torch.bfloat16:
        return 0
    if t.dtype == torch.float32:
        return 1
    raise TypeError(f"delta rule kernels take bf16 or fp32 activations, got {t.dtype}")


_CHUNK_KERNEL = os.environ.get("TYR_GDR_CHUNK_KERNEL", "1") != "0"


def l2norm(x: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    return x * torch.rsqrt((x * x).sum(-1, keepdim=True) + eps)


def recurrent_gated_delta_rule(q, k, v, g, beta, state: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """Token-by-token recurrence in fp32 (oracle and the multi-token fallback with an initial state)."""
    dt = q.dtype
    qf = l2norm(q.float()).transpose(1, 2) * (q.shape[-1] ** -0.5)
    kf = l2norm(k.float()).transpose(1, 2)
    vf, bf, gf = v.float().transpose(1, 2), beta.float().transpose(1, 2), g.float().transpose(1, 2)
    B, H, S, dk = kf.shape
    dv = vf.shape[-1]
    st = torch.zeros(B, H, dk, dv, device=q.device) if state is None else state.float().clone()
    out = torch.empty(B, H, S, dv, device=q.device)
    for i in range(S):
        st = st * gf[:, :, i].exp()[..., None, None]
        kv = (st * kf[:, :, i].unsqueeze(-1)).sum(-2)
        delta = (vf[:, :, i] - kv) * bf[:, :, i].unsqueeze(-1)
        st = st + kf[:, :, i].unsqueeze(-1) * delta.unsqueeze(-2)
        out[:, :, i] = (st * qf[:, :, i].unsqueeze(-1)).sum(-2)
    return out.transpose(1, 2).contiguous().to(dt), st


def chunk_kernels_supported(q, k, v, chunk_size: int = 64) -> bool:
    """Both chunk kernels (csrc/delta_rule.cu) apply: bf16 on CUDA, dk and dv multiples of 8 up to 128, chunk 64, 16-byte aligned
    q / k / v rows; q and k may carry fewer heads than v (grouped keys)."""
    dk, dv = q.shape[-1], v.shape[-1]
    ok_view = lambda t: t.stride(3) == 1 and all(x % 8 == 0 for x in t.stride()[:3]) and t.data_ptr() % 16 == 0
    return (_CHUNK_KERNEL and q.is_cuda and q.dtype == k.dtype == v.dtype == torch.bfloat16 and 0 < dk <= 128 and dk % 8 == 0 and 0 < dv <= 128 and dv % 8 == 0
            and chunk_size == 64 and v.shape[2] % q.shape[2] == 0 and q.shape[2] == k.shape[2] and ok_view(q) and ok_view(k) and ok_view(v)
            and hasattr(lib(), "tyr_gdr_chunk_prepare") and hasattr(lib(), "tyr_gdr_chunk_scan"))


def chunk_gated_delta_rule_fused(q, k, v, g, beta, state: Optional[torch.Tensor] = None, lens: Optional[torch.Tensor] = None,
                                 exact: bool = False, state_out: Optional[torch.Tensor] = None):
    """Two launches: the chunk-local quantities (normalisation, decay, the two 64 x 64 products, the triangular solve) and the
    recurrence over the chunks.  q, k: [B, S, Hk, dk] with Hk dividing Hv (keys are not repeated); see :func:`chunk_kernels_supported`.
    ``lens`` (int32 [B]): tokens of each row; the padding after them leaves the state alone.  ``exact``: split-TF32 products
    against the state and an fp32 read-out."""
    import ctypes
    B, S, Hk, dk = q.shape
    Hv, dv = v.shape[2], v.shape[3]
    n, BH, dev = (S + 63) // 64, B * Hv, q.device
    f32 = lambda *shape: torch.empty(shape, dtype=torch.float32, device=dev)
    u, w, qg, kd, intra, glast = f32(BH, n, 64, -(-dv // 64) * 64), f32(BH, n, 64, 128), f32(BH, n, 64, 128), f32(BH, n, 64, 128), f32(BH, n, 64, 64), f32(BH, n)
    strides = (ctypes.c_longlong * 9)(*[t.stride(i) for t in (q, k, v) for i in range(3)])
    gc, bc = g.float().contiguous(), beta.float().contiguous()
    st = cur_stream(dev)
    check(lib().tyr_gdr_chunk_prepare(ptr(q), ptr(k), ptr(v), ptr(gc), ptr(bc), ptr(u), ptr(w), ptr(qg), ptr(kd), ptr(intra), ptr(glast), ptr(lens), strides,
                                      B, S, Hk, Hv, dk, dv, st), "gdr_chunk_prepare")
    st_in = None if state is None else state.float().contiguous()
    st_out = f32(B, Hv, dk, dv) if state_out is None else state_out
    out = torch.empty((B, S, Hv, dv), dtype=torch.float32 if exact else torch.bfloat16, device=dev)   # the layer's layout, from the scan kernel
    check(lib().tyr_gdr_chunk_scan(ptr(u), ptr(w), ptr(qg), ptr(kd), ptr(intra), ptr(glast), ptr(st_in), ptr(st_out), ptr(out), BH, n, dk, dv, 64, S, Hv, 1 if exact else 0, 0, st),
          "gdr_chunk_scan")
    return out, st_out


def causal_conv1d_silu(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x: [B, S, C] (channels last), weight: [C, K] -> silu(causal depthwise conv + bias) as [B, S, C], zero history."""
    B, S, C = x.shape
    K = weight.shape[-1]
    if x.is_cuda and bias is None and x.stride(2) == 1 and (x.dtype == torch.float32 or K > 4 or C % 8):
        y = torch.empty((B, S, C), dtype=x.dtype, device=x.device)
        wf = weight.reshape(C, K).float().contiguous()
        check(lib().tyr_conv_silu(ptr(x), ptr(wf), ptr(y), B, S, C, K, x.stride(0), x.stride(1), _dt(x), cur_stream(x.device)), "conv_silu")
        return y
    if (x.is_cuda and x.dtype == torch.bfloat16 and C % 8 == 0 and K <= 4 and x.stride(2) == 1 and x.stride(0) % 8 == 0 and x.stride(1) % 8 == 0
            and x.data_ptr() % 16 == 0 and hasattr(lib(), "tyr_causal_conv1d_silu")):
        y = torch.empty((B, S, C), dtype=x.dtype, device=x.device)
        wf = weight.reshape(C, K).float().contiguous()
        bf = None if bias is None else bias.float().contiguous()
        check(lib().tyr_causal_conv1d_silu(ptr(x), ptr(wf), ptr(bf), ptr(y), B, S, C, K, x.stride(0), x.stride(1), cur_stream(x.device)), "causal_conv1d_silu")
        return y
    xc = x.transpose(1, 2)
    y = torch.nn.functional.conv1d(torch.nn.functional.pad(xc, (K - 1, 0)), weight.reshape(C, 1, K).to(xc.dtype), None if bias is None else bias.to(xc.dtype), groups=C)
    return torch.nn.functional.silu(y).transpose(1, 2)


def chunk_gated_delta_rule(q, k, v, g, beta, chunk_size: int = 64, state: Optional[torch.Tensor] = None):
    """Chunk-parallel form: the intra-chunk triangular system is solved with one batched
    unit-lower-triangular solve; chunks are chained through the [dk, dv] state."""
    if chunk_kernels_supported(q, k, v, chunk_size):
        return chunk_gated_delta_rule_fused(q, k, v, g, beta, state)
    if q.shape[2] != v.shape[2]:
        rep = v.shape[2] // q.shape[2]
        q, k = q.repeat_interleave(rep, dim=2), k.repeat_interleave(rep, dim=2)
    dt = q.dtype
    qf = l2norm(q.float()).transpose(1, 2) * (q.shape[-1] ** -0.5)
    kf = l2norm(k.float()).transpose(1, 2)
    vf, bf, gf = v.float().transpose(1, 2), beta.float().transpose(1, 2), g.float().transpose(1, 2)
    B, H, S, dk = kf.shape
    dv = vf.shape[-1]
    pad = (-S) % chunk_size
    if pad:
        P = lambda t, d: torch.nn.functional.pad(t, (0, 0, 0, pad) if d else (0, pad))
        qf, kf, vf, bf, gf = P(qf, 1), P(kf, 1), P(vf, 1), P(bf, 0), P(gf, 0)
    n, C = (S + pad) // chunk_size, chunk_size
    rs = lambda t: t.reshape(B, H, n, C, *t.shape[3:])
    qf, kf, vf, bf, gf = rs(qf), rs(kf), rs(vf), rs(bf), rs(gf)
    gc = gf.cumsum(-1)
    decay = torch.tril((gc.unsqueeze(-1) - gc.unsqueeze(-2))).exp().tril()
    kb, vb = kf * bf.unsqueeze(-1), vf * bf.unsqueeze(-1)
    L = (kb @ kf.transpose(-1, -2) * decay).tril(-1)                           # strictly lower
    eye = torch.eye(C, device=q.device)
    rhs = torch.cat([vb, kb * gc.exp().unsqueeze(-1)], dim=-1)
    sol = torch.linalg.solve_triangular(eye + L, rhs, upper=False, unitriangular=True)
    u, w = sol[..., :dv], sol[..., dv:]                                          # "value" and "k_cumdecay"
    intra = (qf @ kf.transpose(-1, -2) * decay).tril()
    st = torch.zeros(B, H, dk, dv, device=q.device) if state is None else state.float().clone()
    out = torch.empty(B, H, n, C, dv, device=q.device)
    for i in range(n):
        v_new = u[:, :, i] - w[:, :, i] @ st
        out[:, :, i] = (qf[:, :, i] * gc[:, :, i].exp().unsqueeze(-1)) @ st + intra[:, :, i] @ v_new
        g_last = gc[:, :, i, -1]
        st = st * g_last.exp()[..., None, None] + (kf[:, :, i] * (g_last.unsqueeze(-1) - gc[:, :, i]).exp().unsqueeze(-1)).transpose(-1, -2) @ v_new
    out = out.reshape(B, H, n * C, dv)[:, :, :S].transpose(1, 2).contiguous().to(dt)
    return out, st


def gdr_decode_step(q, k, v, g, beta, state: torch.Tensor) -> torch.Tensor:
    """One token: q, k [B, 1, Hk, dk] (un-repeated key heads), v [B, 1, Hv, dv], g/beta [B, 1, Hv];
    ``state`` fp32 [B, Hv, dk, dv] is updated IN PLACE.  Returns [B, 1, Hv, dv]."""
    B, _, Hk, dk = q.shape
    Hv, dv = v.shape[2], v.shape[3]
    if (q.is_cuda and q.dtype == torch.bfloat16 and dk in (64, 128) and state.dtype == torch.float32
            and state.is_contiguous() and q.stride(-1) == 1 and k.stride(-1) == 1 and v.stride(-1) == 1
            and q.stride(2) == dk and k.stride(2) == dk and v.stride(2) == dv and q.stride(0) == k.stride(0)):
        out = torch.empty((B, 1, Hv, dv), dtype=q.dtype, device=q.device)
        gc, bc = g.float().contiguous(), beta.float().contiguous()
        if _tile_ok(dv, v, None, B * Hv):
            check(lib().tyr_gdr_decode_tile(ptr(q), ptr(k), ptr(v), ptr(gc), ptr(bc), ptr(state), ptr(out), B, Hk, Hv, dk,
                                            q.stride(0), v.stride(0), None, 0, None, 0.0, 1, ptr(err_word(q.device)),
                                            cur_stream(q.device)), "gdr_decode_tile")
            return out
        check(lib().tyr_gdr_decode(ptr(q), ptr(k), ptr(v), ptr(gc), ptr(bc), ptr(state), ptr(out), B, Hk, Hv, dk, dv,
                                   q.stride(0), v.stride(0), cur_stream(q.device)), "gdr_decode")
        return out
    rep = Hv // Hk
    qr, kr = q.repeat_interleave(rep, dim=2), k.repeat_interleave(rep, dim=2)
    out, st = recurrent_gated_delta_rule(qr, kr, v, g, beta, state)
    state.copy_(st)
    return out


_GDN_FUSED = os.environ.get("TYR_GDN_DECODE_FUSED", "1") != "0"
_GDR_TILE = os.environ.get("TYR_GDR_DECODE_TILE", "1") != "0"      # 0: the register-resident form of the decode step
# Fewer (batch, head) tiles than this: the register-resident form.  The tile form was faster at every size measured (8 to 64
# rows x 48 heads) once the weight-streaming GEMMs state their own shared-memory / L1 split (csrc/skinny_gemm.cu): its
# 64 KB tiles leave the SMs configured for shared memory.
_GDR_TILE_MIN_TILES = int(os.environ.get("TYR_GDR_TILE_MIN_TILES", "0"))


def _tile_ok(dv: int, v: torch.Tensor, z: Optional[torch.Tensor], tiles: int) -> bool:
    """The shared-memory tile form of the decode step: dv == 128, 8-byte aligned v / z rows, enough tiles."""
    if not (_GDR_TILE and dv == 128 and tiles >= _GDR_TILE_MIN_TILES and hasattr(lib(), "tyr_gdr_decode_tile")):
        return False
    for t in (v, z):
        if t is not None and (t.data_ptr() % 8 or t.stride(0) % 4):
            return False
    return True


def gdn_decode_fused_supported(mixed, conv_state, rec_state, dk: int, dv: int) -> bool:
    return (_GDN_FUSED and mixed.is_cuda and mixed.dtype == torch.bfloat16 and mixed.shape[1] == 1 and mixed.stride(-1) == 1
            and conv_state is not None and conv_state.dtype == torch.bfloat16 and conv_state.is_contiguous()
            and rec_state is not None and rec_state.dtype == torch.float32 and rec_state.is_contiguous()
            and dk in (64, 128) and dv == 128 and hasattr(lib(), "tyr_gdn_conv_gates") and hasattr(lib(), "tyr_gdr_decode_norm"))


def gdn_decode_fused(mixed, z, b, a, conv_state, conv_w, conv_b, dt_bias, a_log, norm_w, eps: float, rec_state,
                     Hk: int, Hv: int, dk: int, dv: int, exact: bool = False) -> torch.Tensor:
    """One GatedDeltaNet decode token between the input and output projections in two launches.

    ``mixed`` [B, 1, cd] (q | k | v channels), ``z`` [B, 1, Hv*dv], ``b`` / ``a`` [B, 1, Hv]: column windows of one projection
    output or separate tensors (rows may be strided).  Kernel 1: causal conv + bias + SiLU with ``conv_state`` ([B, cd, K] bf16) shifted in place,
    beta = sigmoid(b), g = -softplus(a + dt_bias) * exp(a_log).  Kernel 2: the recurrent step on ``rec_state`` (fp32
    [B, Hv, dk, dv], in place; L2-normalised q / k inside) with the gated RMSNorm ``norm(o) * norm_w * silu(z)`` in its
    epilogue (``exact``: of the fp32 read-out, else of the read-out rounded to bf16; tile form only).  Returns [B, 1, Hv*dv].  Model.lean:642-779 of the reference, which issues library ops."""
    B, _, cd = mixed.shape
    K = conv_state.shape[-1]
    assert b.stride(-1) == 1 and a.stride(-1) == 1 and z.stride(-1) == 1 and b.dtype == a.dtype == z.dtype == torch.bfloat16
    dev = mixed.device
    conv_out = torch.empty((B, cd), dtype=torch.bfloat16, device=dev)
    g = torch.empty((B, Hv), dtype=torch.float32, device=dev)
    beta = torch.empty((B, Hv), dtype=torch.float32, device=dev)
    w = conv_w.reshape(cd, K)
    if w.dtype != torch.bfloat16 or not w.is_contiguous():
        w = w.to(torch.bfloat16).contiguous()
    cb = None if conv_b is None else conv_b.to(torch.bfloat16).contiguous()
    check(lib().tyr_gdn_conv_gates(ptr(mixed), ptr(b), ptr(a), mixed.stride(0), b.stride(0), a.stride(0), ptr(conv_state), ptr(w), ptr(cb), ptr(dt_bias.float().contiguous()),
                                   ptr(a_log.float().contiguous()), ptr(conv_out), ptr(g), ptr(beta), B, cd, K, Hv, cur_stream(dev)),
          "gdn_conv_gates")
    kd = Hk * dk
    q, k, v = conv_out[:, :kd], conv_out[:, kd:2 * kd], conv_out[:, 2 * kd:]
    out = torch.empty((B, 1, Hv * dv), dtype=torch.bfloat16, device=dev)
    nw = norm_w if (norm_w.dtype == torch.bfloat16 and norm_w.is_contiguous()) else norm_w.to(torch.bfloat16).contiguous()
    if _tile_ok(dv, v, z, B * Hv):
        check(lib().tyr_gdr_decode_tile(ptr(q), ptr(k), ptr(v), ptr(g), ptr(beta), ptr(rec_state), ptr(out), B, Hk, Hv, dk, cd, cd,
                                        ptr(z), z.stride(0), ptr(nw), eps, 0 if exact else 1, ptr(err_word(dev)), cur_stream(dev)), "gdr_decode_tile")
        return out
    check(lib().tyr_gdr_decode_norm(ptr(q), ptr(k), ptr(v), ptr(g), ptr(beta), ptr(rec_state), ptr(out), B, Hk, Hv, dk, dv, cd, cd,
                                    ptr(z), z.stride(0), ptr(nw), eps, cur_stream(dev)), "gdr_decode_norm")
    return out


# ---- any head size, bf16 or fp32, rows of unequal length (csrc/delta_general.cu; plain PyTorch off the GPU) ---------------------
def delta_gates(b: torch.Tensor, a: torch.Tensor, dt_bias: torch.Tensor, a_log: torch.Tensor):
    """b, a: [B, S, Hv] projections (rows may be strided) -> fp32 (g, beta): log decay ``-exp(a_log) softplus(a + dt_bias)`` and
    write strength ``sigmoid(b)``."""
    if not b.is_cuda:
        return -torch.exp(a_log.float()) * torch.nn.functional.softplus(a.float() + dt_bias.float()), torch.sigmoid(b.float())
    B, S, Hv = b.shape
    g = torch.empty((B, S, Hv), dtype=torch.float32, device=b.device)
    beta = torch.empty_like(g)
    assert b.dtype == a.dtype
    check(lib().tyr_delta_gates(ptr(b), ptr(a), row_stride(b), row_stride(a), ptr(dt_bias), ptr(a_log), ptr(g), ptr(beta), B * S, Hv, _dt(b),
                                cur_stream(b.device)), "delta_gates")
    return g, beta


def recurrent_delta(q, k, v, g, beta, state: torch.Tensor, lens: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The recurrence token by token with fp32 state, arithmetic and read-out.  q, k: [B, S, Hk, dk]; v: [B, S, Hv, dv] (views with
    contiguous channels); ``state`` fp32 [B, Hv, dk, dv] is advanced IN PLACE over the first ``lens[b]`` tokens of row b; the
    read-out [B, S, Hv, dv] is zero past them."""
    B, S, Hk, dk = q.shape
    Hv, dv = v.shape[2], v.shape[3]
    if not q.is_cuda:
        rep = Hv // Hk
        n = lens.tolist() if lens is not None else [S] * B
        out = torch.zeros(B, S, Hv, dv, dtype=torch.float32)
        for r in range(B):
            sl = lambda t: t[r:r + 1, :n[r]].float()
            o, st = recurrent_gated_delta_rule(sl(q).repeat_interleave(rep, 2), sl(k).repeat_interleave(rep, 2), sl(v), sl(g), sl(beta), state[r:r + 1])
            out[r, :n[r]] = o[0]
            state[r] = st[0]
        return out
    import ctypes
    assert state.dtype == torch.float32 and state.is_contiguous() and q.stride(3) == k.stride(3) == v.stride(3) == 1 and q.dtype == k.dtype == v.dtype
    out = torch.empty((B, S, Hv, dv), dtype=torch.float32, device=q.device)
    strides = (ctypes.c_longlong * 9)(*[t.stride(i) for t in (q, k, v) for i in range(3)])
    check(lib().tyr_gdr_recurrent(ptr(q), ptr(k), ptr(v), ptr(g.contiguous()), ptr(beta.contiguous()), ptr(state), ptr(out), ptr(lens), strides,
                                  B, S, Hk, Hv, dk, dv, _dt(q), cur_stream(q.device)), "gdr_recurrent")
    return out


def delta_prefill(q, k, v, g, beta, state: torch.Tensor, lens: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Fresh prompts (the state starts at zero): fp32 read-out [B, S, Hv, dv]; ``state`` receives the state after each row's last
    token.  The tensor-core chunk form where it applies, else the recurrence."""
    if q.is_cuda and q.shape[1] > 1 and chunk_kernels_supported(q, k, v):
        return chunk_gated_delta_rule_fused(q, k, v, g, beta, None, lens, exact=True, state_out=state)[0]
    state.zero_()
    return recurrent_delta(q, k, v, g, beta, state, lens)


def gated_norm(o: torch.Tensor, z: torch.Tensor, w: torch.Tensor, eps: float, act: str = "silu", out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``o / sqrt(mean(o^2) + eps) * w * act(z)`` per head, ``act`` SiLU or sigmoid: o fp32 [B, S, Hv, dv], z [B, S, Hv*dv] (rows may be
    strided), w fp32 [dv] -> [B, S, Hv*dv] in z's dtype (``out``: a view with evenly spaced rows)."""
    B, S, Hv, dv = o.shape
    if not o.is_cuda:
        y = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * w.float()
        f = torch.sigmoid if act == "sigmoid" else torch.nn.functional.silu
        y = (y * f(z.float()).reshape(B, S, Hv, dv)).reshape(B, S, Hv * dv).to(z.dtype)
        return y if out is None else out.copy_(y)
    assert o.is_contiguous()
    y = torch.empty((B, S, Hv * dv), dtype=z.dtype, device=z.device) if out is None else out
    assert y.dtype == z.dtype and y.shape == (B, S, Hv * dv)
    check(lib().tyr_gated_norm(ptr(o), ptr(z), row_stride(z), ptr(w), ptr(y), row_stride(y), B * S, Hv, dv, eps, {"silu": 0, "sigmoid": 1}[act], _dt(z),
                               cur_stream(z.device)), "gated_norm")
    return y


def conv_window(x: torch.Tensor, K: int, lens: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The last K inputs of every channel at the end of each row ([B, S, C] -> [B, C, K], zeros before the start): the state a
    decode step continues from."""
    B, S, C = x.shape
    end = torch.full((B,), S, device=x.device, dtype=torch.long) if lens is None else lens.long()
    t = end[:, None] - K + torch.arange(K, device=x.device)
    win = torch.gather(x, 1, t.clamp_min(0)[:, :, None].expand(B, K, C))
    return (win * (t >= 0).to(x.dtype)[:, :, None]).transpose(1, 2).contiguous()


def delta_decode(mixed, z, b, a, conv_state, conv_w, dt_bias, a_log, norm_w, eps: float, rec_state, Hk: int, Hv: int, dk: int, dv: int):
    """One token of a gated delta layer between its input and output projections: convolution window and state advanced in
    place, fp32 gates, recurrence, read-out and norm.  Shapes as in :func:`gdn_decode_fused` (no convolution bias)."""
    if gdn_decode_fused_supported(mixed, conv_state, rec_state, dk, dv) and conv_state.shape[-1] <= 8 and _tile_ok(dv, mixed, z, mixed.shape[0] * Hv):
        return gdn_decode_fused(mixed, z, b, a, conv_state, conv_w, None, dt_bias, a_log, norm_w, eps, rec_state, Hk, Hv, dk, dv, exact=True)
    B, _, C = mixed.shape
    K = conv_state.shape[-1]
    if mixed.is_cuda:
        dev = mixed.device
        y = torch.empty((B, 1, C), dtype=mixed.dtype, device=dev)
        g = torch.empty((B, 1, Hv), dtype=torch.float32, device=dev)
        beta = torch.empty_like(g)
        assert conv_state.is_contiguous() and conv_state.dtype == mixed.dtype and mixed.stride(2) == b.stride(2) == a.stride(2) == 1
        check(lib().tyr_delta_conv_gates(ptr(mixed), ptr(b), ptr(a), mixed.stride(0), b.stride(0), a.stride(0), ptr(conv_state), ptr(conv_w.float()),
                                         ptr(dt_bias), ptr(a_log), ptr(y), ptr(g), ptr(beta), B, C, K, Hv, _dt(mixed), cur_stream(dev)), "delta_conv_gates")
    else:
        conv_state.copy_(torch.cat([conv_state[:, :, 1:], mixed.transpose(1, 2)], dim=2))
        y = torch.nn.functional.silu((conv_state.float() * conv_w.float()).sum(-1)).to(mixed.dtype).unsqueeze(1)
        g, beta = delta_gates(b, a, dt_bias, a_log)
    kd = Hk * dk
    q, k, v = y[..., :kd].reshape(B, 1, Hk, dk), y[..., kd:2 * kd].reshape(B, 1, Hk, dk), y[..., 2 * kd:].reshape(B, 1, Hv, dv)
    return gated_norm(recurrent_delta(q, k, v, g, beta, rec_state), z, norm_w.float(), eps)


# ---- a decay per key channel ------------------------------------------------------------------------------------------------------
def channel_log_decay(a: torch.Tensor, dt_bias: torch.Tensor, a_log: torch.Tensor) -> torch.Tensor:
    """a: [B, S, Hv * dk] -> fp32 [B, S, Hv, dk]: ``-exp(a_log) softplus(a + dt_bias)``."""
    z = torch.nn.functional.softplus(a.float() + dt_bias).reshape(*a.shape[:2], a_log.numel(), -1)
    return -torch.exp(a_log.float())[:, None] * z


def recurrent_channel_delta(q, k, v, a, b, dt_bias, a_log, state: torch.Tensor, lens: Optional[torch.Tensor] = None) -> torch.Tensor:
    """:func:`recurrent_delta` with a decay per key channel: ``a`` [B, S, Hv * dk] and ``b`` [B, S, Hv] are the projections of decay and
    write strength (rows may be strided), dt_bias fp32 [Hv * dk], a_log fp32 [Hv]."""
    import ctypes
    B, S, Hk, dk = q.shape
    Hv, dv = v.shape[2], v.shape[3]
    if not q.is_cuda:
        rep = Hv // Hk
        decay, beta = torch.exp(channel_log_decay(a, dt_bias, a_log)), torch.sigmoid(b.float())
        qf, kf = (l2norm(t.float()).repeat_interleave(rep, 2) for t in (q, k))
        qf = qf * dk ** -0.5
        out = torch.zeros(B, S, Hv, dv, dtype=torch.float32)
        for r in range(B):
            st = state[r]
            for t in range(S if lens is None else int(lens[r])):
                st = st * decay[r, t][..., None]
                u = beta[r, t][:, None] * (v[r, t].float() - torch.einsum("hd,hdv->hv", kf[r, t], st))
                st = st + kf[r, t][..., None] * u[:, None]
                out[r, t] = torch.einsum("hd,hdv->hv", qf[r, t], st)
            state[r] = st
        return out
    assert state.dtype == torch.float32 and state.is_contiguous() and q.stride(3) == k.stride(3) == v.stride(3) == 1 and q.dtype == k.dtype == v.dtype == a.dtype == b.dtype
    out = torch.empty((B, S, Hv, dv), dtype=torch.float32, device=q.device)
    strides = (ctypes.c_longlong * 11)(*[t.stride(i) for t in (q, k, v) for i in range(3)], row_stride(a), row_stride(b))
    check(lib().tyr_gdr_recurrent_channel(ptr(q), ptr(k), ptr(v), ptr(a), ptr(b), ptr(dt_bias), ptr(a_log), ptr(state), ptr(out), ptr(lens), strides,
                                          B, S, Hk, Hv, dk, dv, _dt(q), cur_stream(q.device)), "gdr_recurrent_channel")
    return out


def chunk_channel_delta_fused(q, k, v, a, b, dt_bias, a_log, state: torch.Tensor, lens: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The two chunk kernels with a decay per key channel, the exact form of the scan: fp32 read-out [B, S, Hv, dv] of fresh prompts;
    ``state`` receives the state after each row's last token.  Operands of :func:`recurrent_channel_delta`, shapes of
    :func:`chunk_kernels_supported`."""
    import ctypes
    B, S, Hk, dk = q.shape
    Hv, dv = v.shape[2], v.shape[3]
    n, BH, dev = (S + 63) // 64, B * Hv, q.device
    f32 = lambda *shape: torch.empty(shape, dtype=torch.float32, device=dev)
    u, w, qg, kd, intra, glast = f32(BH, n, 64, -(-dv // 64) * 64), f32(BH, n, 64, 128), f32(BH, n, 64, 128), f32(BH, n, 64, 128), f32(BH, n, 64, 64), f32(BH, n, 128)
    assert a.dtype == b.dtype == q.dtype and dt_bias.dtype == a_log.dtype == torch.float32 and state.dtype == torch.float32 and state.is_contiguous()
    strides = (ctypes.c_longlong * 11)(*[t.stride(i) for t in (q, k, v) for i in range(3)], row_stride(a), row_stride(b))
    st = cur_stream(dev)
    check(lib().tyr_gdr_chunk_prepare_channel(ptr(q), ptr(k), ptr(v), ptr(a), ptr(b), ptr(dt_bias), ptr(a_log), ptr(u), ptr(w), ptr(qg), ptr(kd), ptr(intra),
                                              ptr(glast), ptr(lens), strides, B, S, Hk, Hv, dk, dv, st), "gdr_chunk_prepare_channel")
    out = f32(B, S, Hv, dv)
    check(lib().tyr_gdr_chunk_scan(ptr(u), ptr(w), ptr(qg), ptr(kd), ptr(intra), ptr(glast), None, ptr(state), ptr(out), BH, n, dk, dv, 64, S, Hv, 1, 1, st),
          "gdr_chunk_scan")
    return out


def channel_delta_prefill(q, k, v, a, b, dt_bias, a_log, state: torch.Tensor, lens: Optional[torch.Tensor] = None) -> torch.Tensor:
    """:func:`delta_prefill` with a decay per key channel (operands of :func:`recurrent_channel_delta`)."""
    if q.is_cuda and q.shape[1] > 1 and chunk_kernels_supported(q, k, v) and hasattr(lib(), "tyr_gdr_chunk_prepare_channel"):
        return chunk_channel_delta_fused(q, k, v, a, b, dt_bias, a_log, state, lens)
    state.zero_()
    return recurrent_channel_delta(q, k, v, a, b, dt_bias, a_log, state, lens)


def channel_delta_decode(q, k, v, a, b, z, dt_bias, a_log, norm_w: torch.Tensor, norm_lp: torch.Tensor, eps: float, state: torch.Tensor, out: torch.Tensor) -> None:
    """One token per row: recurrence on ``state`` (in place), norm of the read-out and sigmoid gate ``z`` [B, 1, Hv * dv] -> ``out`` (rows
    may be strided).  norm_w: fp32 [dv], norm_lp: the same in the activations' type."""
    import ctypes
    B, _, Hk, dk = q.shape
    Hv, dv = v.shape[2], v.shape[3]
    if (q.is_cuda and q.dtype == torch.bfloat16 and dk in (64, 128) and q.stride(0) == k.stride(0) and q.stride(2) == k.stride(2) == dk
            and v.stride(2) == dv and _tile_ok(dv, v, z, B * Hv) and out.stride(0) % 4 == 0 and out.data_ptr() % 8 == 0
            and hasattr(lib(), "tyr_gdr_decode_tile_channel")):
        strides = (ctypes.c_longlong * 6)(q.stride(0), v.stride(0), a.stride(0), b.stride(0), z.stride(0), out.stride(0))
        check(lib().tyr_gdr_decode_tile_channel(ptr(q), ptr(k), ptr(v), ptr(a), ptr(b), ptr(dt_bias), ptr(a_log), ptr(state), ptr(out), ptr(z), ptr(norm_lp),
                                                strides, B, Hk, Hv, dk, eps, ptr(err_word(q.device)), cur_stream(q.device)), "gdr_decode_tile_channel")
        return
    gated_norm(recurrent_channel_delta(q, k, v, a, b, dt_bias, a_log, state), z, norm_w, eps, "sigmoid", out)
