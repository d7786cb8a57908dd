"""Plain implementation of the Zatorax design for the tests: one function per mechanism, one token or one head at a time, in
the dtype of the weights it is given (float32 or float64), on the CPU.  It shares no code with the package."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rms_unit(x, eps):
    """x over its root mean square (last axis)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def short_conv(x, w):
    """x: [T, C]; w: [C, taps], last column for the current token; zeros before the start; silu."""
    T, C = x.shape
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return silu(out)


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, decay, beta, state=None):
    """q, k: [T, Hk, dk] (already unit vectors, q scaled), v: [T, Hv, dv], decay and beta: [T, Hv].  Returns ([T, Hv, dv], state)."""
    T, Hv, dv = v.shape
    rep = Hv // q.shape[1]
    S = torch.zeros(Hv, q.shape[2], dv, dtype=v.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        for h in range(Hv):
            kk, qq = k[t, h // rep], q[t, h // rep]
            S[h] = decay[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ kk)
            S[h] = S[h] + torch.outer(kk, u)
            out[t, h] = S[h].T @ qq
    return out, S


def delta_mixer(w: Dict[str, torch.Tensor], p: str, mix: dict, x, eps):
    """x: [T, width] -> [T, width]."""
    T = x.shape[0]
    Hk, Hv, dk, dv = mix["kv_heads"], mix["heads"], mix["dim"], mix["vdim"]
    q = short_conv(x @ w[p + "q"].T, w[p + "q.conv"]).reshape(T, Hk, dk)
    k = short_conv(x @ w[p + "k"].T, w[p + "k.conv"]).reshape(T, Hk, dk)
    v = short_conv(x @ w[p + "v"].T, w[p + "v.conv"]).reshape(T, Hv, dv)
    q = unit_vectors(q) * dk ** -0.5
    k = unit_vectors(k)
    beta = sigmoid(x @ w[p + "b"].T)
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(x @ w[p + "a"].T + w[p + "dt_bias"]))
    o, _ = delta_recurrence(q, k, v, decay, beta)
    o = rms_unit(o, eps) * w[p + "norm"]
    o = o * silu(x @ w[p + "g"].T).reshape(T, Hv, dv)
    return o.reshape(T, Hv * dv) @ w[p + "o"].T


def window_attention(q, k, v, scale, r1, r2, window: Optional[int]):
    """q: [T, H, d], k: [T, G, d], v: [T, G, dv]; one query and head at a time.  The score of a key at distance n loses
    r1 ln(1 + r2 n); distances of ``window`` and more are not seen."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=v.dtype)
    for i in range(T):
        lo = 0 if window is None else max(0, i - window + 1)
        dist = torch.arange(i - lo, -1, -1, dtype=v.dtype)
        for h in range(H):
            g = h // rep
            s = (k[lo:i + 1, g] @ q[i, h]) * scale - r1[h] * torch.log(1 + r2[h] * dist)
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[lo:i + 1, g]
    return out


def attention_keys(w, p, mix, x, eps):
    T = x.shape[0]
    k = (x @ w[p + "k"].T).reshape(T, mix["kv_heads"], mix["dim"])
    return rms_unit(k, eps) * w[p + "k.norm"], (x @ w[p + "v"].T).reshape(T, mix["kv_heads"], mix["vdim"])


def attention_mixer(w, p, mix, x, eps, k, v):
    T = x.shape[0]
    q = (x @ w[p + "q"].T).reshape(T, mix["heads"], mix["dim"])
    q = rms_unit(q, eps) * w[p + "q.norm"]
    mask = mix.get("mask")
    o = window_attention(q, k, v, mix["scale"], w[p + "r1"], w[p + "r2"], mask["size"] if mask else None)
    return o.reshape(T, -1) @ w[p + "o"].T


def choose_experts(scores, correction, top, groups: Optional[dict]):
    """Indices of the chosen experts of one token, best choice score first."""
    choice = (scores + correction).clone()
    E = len(choice)
    if groups is not None:
        n = E // groups["count"]
        best = [(-float(choice[g * n:(g + 1) * n].max()), g) for g in range(groups["count"])]
        kept = {g for _, g in sorted(best)[:groups["keep"]]}
        for e in range(E):
            if e // n not in kept:
                choice[e] = -math.inf
    return sorted(range(E), key=lambda e: (-float(choice[e]), e))[:top]


def gated_ff(w, p, x):
    return (silu(x @ w[p + ".gate"].T) * (x @ w[p + ".up"].T)) @ w[p + ".down"].T


def expert_mixture(w, p, mlp, x):
    r = mlp["router"]
    s = torch.softmax(x @ w[p + "router"].T, -1)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e in choose_experts(s[t], w[p + "correction"], r["top"], r.get("groups")):
            out[t] += s[t, e] * gated_ff(w, f"{p}e{e}", x[t])
    if mlp.get("shared"):
        out = out + gated_ff(w, p + "shared", x)
    return out


def residual_stream(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> List[torch.Tensor]:
    """The residual stream of one sequence after every layer, [T, width] each."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    keys, out = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        if layer["type"] == "delta":
            y = delta_mixer(w, p + "mix.", mix, x, eps)
        else:
            src = mix.get("kv_from")
            if src is None:
                keys[i] = attention_keys(w, p + "mix.", mix, x, eps)
            k, v = keys[i if src is None else src]
            y = attention_mixer(w, p + "mix.", mix, x, eps, k, v)
        x = x + rms_unit(y, eps) * w[p + "norm1"]
        if layer.get("mlp"):
            x = x + rms_unit(expert_mixture(w, p + "mlp.", layer["mlp"], x), eps) * w[p + "norm2"]
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """[T, vocab]."""
    x = residual_stream(cfg, w, tokens)[-1]
    return (rms_unit(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T
