"""Plain implementation of the Kinetar design for the tests: one function per mechanism, one token at a time where there is a
recurrence, in the dtype of the weights it is given (float32 or float64), on the CPU.  It shares no code with the package."""
from __future__ import annotations

import math
from typing import Dict, List

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


def zero_centred_norm(x, w, eps):
    return rms_unit(x, eps) * (1 + w)


def position_vectors(T, width, dtype):
    """[T, width]: channel 2i holds sin(p / 10000^(2i / width)), channel 2i + 1 the cosine."""
    out = torch.zeros(T, width, dtype=torch.float64)
    p = torch.arange(T, dtype=torch.float64)
    for c in range(width):
        angle = p * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.cos(angle) if c % 2 else torch.sin(angle)
    return out.to(dtype)


def embedding(w, tokens, scale):
    e = w["embed"][torch.tensor(tokens)]
    return e * scale + position_vectors(len(tokens), e.shape[1], e.dtype)


def short_conv(x, w, bias=None):
    """x: [T, C]; w: [C, taps], last column for the current token; zeros before the start; no activation."""
    T, C = x.shape
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j] * x[:T - back]
    return out if bias is None else out + bias


def query_temperature(T, coef, every, dtype):
    return torch.tensor([1 + coef * math.log((p + 1) // every + 1) for p in range(T)], dtype=dtype)


def sink_attention(q, k, v, scale, sink):
    """q: [T, H, d], k: [T, G, d], v: [T, G, dv]; causal softmax whose denominator also holds exp(sink[h])."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=v.dtype)
    for i in range(T):
        for h in range(H):
            g = h // rep
            s = (k[:i + 1, g] @ q[i, h]) * scale
            m = torch.maximum(s.max(), sink[h])
            e = torch.exp(s - m)
            out[i, h] = (e / (e.sum() + torch.exp(sink[h] - m))) @ v[:i + 1, g]
    return out


def attention_mixer(w: Dict[str, torch.Tensor], p: str, mix: dict, h):
    T = h.shape[0]
    q = short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).reshape(T, mix["heads"], mix["dim"])
    k = short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).reshape(T, mix["kv_heads"], mix["dim"])
    t = mix["q_temp"]
    q = q * query_temperature(T, t["coef"], t["every"], q.dtype)[:, None, None]
    o = sink_attention(q, k, k, mix["scale"], w[p + "sink"]).reshape(T, -1)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def selective_scan(x, dt, A, B, C, D, state=None):
    """x, dt: [T, c]; A: [c, n]; B, C: [T, n]; D: [c].  Returns ([T, c], state [c, n])."""
    S = torch.zeros_like(A) if state is None else state.clone()
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out, S


def scan_mixer(w, p, mix, h):
    n, r, inner = mix["state"], mix["dt_rank"], mix["inner"]
    xz = h @ w[p + "in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(short_conv(x, w[p + "conv"], w[p + "conv.b"]))
    proj = x @ w[p + "x"].T
    dt = softplus(proj[:, :r] @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), proj[:, r:r + n], proj[:, r + n:r + 2 * n], w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


def parallel_mixer(w, p, mix, h):
    return mix["left_scale"] * attention_mixer(w, p + "left.", mix["left"], h) + mix["right_scale"] * scan_mixer(w, p + "right.", mix["right"], h)


def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_delta_recurrence(q, k, v, decay, beta, state=None):
    """q, k: [T, Hk, dk] (already unit vectors, q scaled), v: [T, H, dv], decay: [T, H, dk], beta: [T, H]."""
    T, H, dv = v.shape
    rep = H // q.shape[1]
    S = torch.zeros(H, q.shape[2], dv, dtype=v.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    of = torch.arange(H) // rep
    for t in range(T):
        kk, qq = k[t, of], q[t, of]
        S = decay[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, kk))
        S = S + kk[:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, qq)
    return out, S


def channel_decay(a, dt_bias, A_log):
    """a: [T, H * dk] -> decays [T, H, dk]."""
    H = A_log.shape[0]
    z = softplus(a + dt_bias).reshape(a.shape[0], H, -1)
    return torch.exp(-torch.exp(A_log)[None, :, None] * z)


def delta_mixer(w, p, mix, h, eps):
    T = h.shape[0]
    Hk, H, dk, dv = mix["kv_heads"], mix["heads"], mix["dim"], mix["vdim"]
    q = silu(short_conv(h @ w[p + "q"].T, w[p + "q.conv"])).reshape(T, Hk, dk)
    k = silu(short_conv(h @ w[p + "k"].T, w[p + "k.conv"])).reshape(T, Hk, dk)
    v = silu(short_conv(h @ w[p + "v"].T, w[p + "v.conv"])).reshape(T, H, dv)
    beta = sigmoid(h @ w[p + "b"].T)
    decay = channel_decay((h @ w[p + "a1"].T) @ w[p + "a2"].T, w[p + "dt_bias"], w[p + "A_log"])
    o, _ = channel_delta_recurrence(unit_vectors(q) * dk ** -0.5, unit_vectors(k), v, decay, beta)
    o = rms_unit(o, eps) * w[p + "norm"]
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return (o.reshape(T, H * dv) * gate) @ w[p + "o"].T


def feed_forward(w, p, h):
    u = torch.clamp(h @ w[p + "up"].T, min=0)
    return (u * u) @ w[p + "down"].T


def residual_stream(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> List[torch.Tensor]:
    """The residual stream of one sequence after every layer, [T, width] each."""
    eps = cfg["norm"]["eps"]
    x = embedding(w, tokens, cfg["embedding"]["scale"])
    out = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = zero_centred_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "parallel":
            y = parallel_mixer(w, p + "mix.", layer["mixer"], h)
        else:
            y = delta_mixer(w, p + "mix.", layer["mixer"], h, eps)
        if layer.get("mlp"):
            y = y + feed_forward(w, p + "mlp.", h)
        x = x + y
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """[T, vocab]."""
    x = residual_stream(cfg, w, tokens)[-1]
    return (zero_centred_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T) * cfg["logit_scale"]
