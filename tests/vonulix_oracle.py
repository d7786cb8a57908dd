"""Plain implementation of the Vonulix design for the tests: one function per mechanism, one query or one token at a time where the
mechanism has one, in the dtype of the weights it is given (float32 or float64), on the CPU.  It shares no code with the package."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def over_rms(x, eps):
    """x over its root mean square (last axis)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    return over_rms(x, eps) * (1.0 + w)


def turn(x, p, dims, base, factor=1.0):
    """One head's vector x at position p (negative: turned back): channel i < dims / 2 and channel i + dims / 2 turn by p base^(-2i / dims) / factor."""
    y, half = x.clone(), dims // 2
    for i in range(half):
        a = p * base ** (-2.0 * i / dims) / factor
        c, s = math.cos(a), math.sin(a)
        y[..., i] = x[..., i] * c - x[..., i + half] * s
        y[..., i + half] = x[..., i + half] * c + x[..., i] * s
    return y


def visible(i, size: Optional[int], keep):
    """The positions a query at position i sees."""
    return [j for j in range(i + 1) if size is None or i - j < size or j < keep]


def attend(q, k, v, scale, size, keep, first=0):
    """q: [n, H, d] at positions ``first`` .., k: [T, G, d], v: [T, G, dv] at 0 .. -> [n, H, dv]."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=v.dtype)
    for i in range(n):
        js = torch.tensor(visible(first + i, size, keep))
        for h in range(H):
            s = (k[js, h // rep] @ q[i, h]) * scale
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[js, h // rep]
    return out


def attention_mixer(w: Dict[str, torch.Tensor], p: str, mix: dict, x, eps):
    """x: [T, width] -> [T, width]."""
    T, H, G, d, dv = x.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    rot, mask = mix["rot"], mix.get("mask") or {}
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    q = (x @ w[p + "q"].T).reshape(T, H, d)
    k = (x @ w[p + "k"].T).reshape(T, G, d)
    v = over_rms((x @ w[p + "v"].T).reshape(T, G, dv), eps)
    q = torch.stack([turn(q[t], t, rot["dims"], rot["base"], factor) for t in range(T)])
    k = torch.stack([turn(k[t], t, rot["dims"], rot["base"], factor) for t in range(T)])
    v = torch.stack([turn(v[t], t, dv, rot["base"]) for t in range(T)])
    o = attend(q, k, v, mix["scale"], mask.get("size"), mask.get("keep_first", 0))
    o = torch.stack([turn(o[t], -t, dv, rot["base"]) for t in range(T)])
    o = o * sigmoid(x @ w[p + "g"].T)[..., None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def expert(w, p, limit, x):
    g = torch.clamp(x @ w[p + ".gate"].T, max=limit)
    u = torch.clamp(x @ w[p + ".up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + ".down"].T


def choose(scores, top):
    """Indices of the largest scores of one token, the largest first."""
    return sorted(range(len(scores)), key=lambda e: (-float(scores[e]), e))[:top]


def expert_mixture(w, p, mlp, x):
    s = sigmoid(x @ w[p + "router"].T)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e in choose(s[t], mlp["router"]["top"]):
            out[t] += expert(w, f"{p}e{e}", mlp["expert"]["limit"], s[t, e] * x[t])
    if mlp.get("shared"):
        out = out + sigmoid(x @ w[p + "shared.sg"].T) * expert(w, p + "shared", mlp["shared"]["limit"], x)
    return out


def token_input(w, p, table, x, tokens, layer, dim, eps):
    e = table[torch.tensor(tokens)][:, layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return x + over_rms(y, eps) * w[p + "side.norm"]


def depth_average(weights, streams):
    out = torch.zeros_like(streams[0])
    for a, x in zip(weights, streams):
        out = out + a * x
    return out


def residual_stream(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> List[torch.Tensor]:
    """What goes on after every layer of one sequence, [T, width] each."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    results, out = [x], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + attention_mixer(w, p + "mix.", layer["mixer"], norm_around_zero(x, w[p + "norm1"], eps), eps)
        if layer.get("mlp"):
            x = x + expert_mixture(w, p + "mlp.", layer["mlp"], norm_around_zero(x, w[p + "norm2"], eps))
        x = token_input(w, p, w["side.embed"], x, tokens, i, cfg["token_side"]["dim"], eps)
        results.append(x)
        x = depth_average(w[p + "dwa"], results)
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """[T, vocab]."""
    x = residual_stream(cfg, w, tokens)[-1]
    return norm_around_zero(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
