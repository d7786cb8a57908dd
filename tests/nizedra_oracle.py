"""Plain implementation of the Nizedra design for the tests: one function per mechanism, one token at a time where there is a
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


def norm(x, w, eps):
    return rms_unit(x, eps) * w


def xielu(z, pq):
    """Quadratic above zero, an integrated ELU below, both with slope 1/2 at zero."""
    above = softplus(pq[0]) * z * z
    low = torch.clamp(z, max=0)
    below = (0.5 + softplus(pq[1])) * (torch.exp(low) - 1 - low)
    return torch.where(z > 0, above, below) + z / 2


def feed_forward(w, p, h):
    return xielu(h @ w[p + "up"].T, w[p + "act"]) @ w[p + "down"].T


# ---- lightning ----------------------------------------------------------------------------------------------------
def decayed_recurrence(q, k, v, decay, state=None):
    """q, k: [T, H, d], v: [T, H, dv], decay: [H].  S <- decay S + k v^T, o = S^T q."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=v.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def lightning_mixer(w, p, mix, h, eps):
    T, H = h.shape[0], mix["heads"]
    q, k = (silu(h @ w[p + n].T).reshape(T, H, mix["dim"]) for n in "qk")
    v = silu(h @ w[p + "v"].T).reshape(T, H, mix["vdim"])
    o, _ = decayed_recurrence(q, k, v, torch.tensor(mix["decay"], dtype=h.dtype))
    return (norm(o.reshape(T, -1), w[p + "norm"], eps) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- latent attention ---------------------------------------------------------------------------------------------
def rotate(x, base, dims, first=0):
    """x: [T, ..., d]; the channel pairs (2i, 2i + 1) of the first ``dims`` turn by position * base^(-2i / dims)."""
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = (first + t) * base ** (-2.0 * i / dims)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[t, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def window_attention(q, k, v, scale, window=None):
    """q, k: [T, H, d], v: [T, H, dv]; query i sees the keys j with 0 <= i - j < window."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=v.dtype)
    for i in range(q.shape[0]):
        lo = 0 if window is None else max(0, i - window + 1)
        s = torch.einsum("hd,jhd->hj", q[i], k[lo:i + 1]) * scale
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhd->hd", e / e.sum(-1, keepdim=True), v[lo:i + 1])
    return out


def latent_mixer(w, p, mix, h, eps):
    T, H, d, r, c = h.shape[0], mix["heads"], mix["dim"], mix["rot_dim"], mix["kv_rank"]
    q = (norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, d + r)
    down = h @ w[p + "dkv"].T
    lat = norm(down[:, :c], w[p + "dkv.norm"], eps)
    rot = mix["rot"]
    k_rot = rotate(down[:, c:], rot["base"], rot["dims"])
    q = torch.cat([q[..., :d], rotate(q[..., d:], rot["base"], rot["dims"])], -1)
    k = torch.cat([(lat @ w[p + "uk"].T).reshape(T, H, d), k_rot[:, None].expand(T, H, r)], -1)
    v = (lat @ w[p + "uv"].T).reshape(T, H, mix["vdim"])
    return window_attention(q, k, v, mix["scale"], mix["mask"]["size"]).reshape(T, -1) @ w[p + "o"].T


# ---- attention with mixed heads -----------------------------------------------------------------------------------
def distance_bucket(n, rows, reach):
    """Row of the table for a distance: one each up to half the rows, logarithmic up to ``reach``, the last row beyond."""
    half = rows // 2
    if n < half:
        return n
    # the largest step x whose lower end half * (reach / half)^(x / steps) is not past n, in whole numbers
    steps, x = rows - half, 0
    while x < steps - 1 and n ** steps * half ** (x + 1) >= reach ** (x + 1) * half ** steps:
        x += 1
    return half + x


def talking_scores(q, k, mix, temp, rel, talk, i):
    """Scores [H, i + 1] of query i.  q: [T, H, d], k: [T, G, d], both already of unit root mean square."""
    H = q.shape[1]
    of = torch.arange(H) // (H // k.shape[1])
    s = torch.einsum("hd,jhd->hj", q[i], k[:i + 1][:, of]) * mix["scale"] * temp[:, None]
    s = mix["softcap"] * torch.tanh(s / mix["softcap"])
    rows = [distance_bucket(i - j, rel.shape[0], mix["bias_max"]) for j in range(i + 1)]
    return talk @ (s + rel[rows].T)


def talking_attention(q, k, v, mix, temp, rel, talk, first=0):
    """Rows before query ``first`` stay zero."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=v.dtype)
    of = torch.arange(q.shape[1]) // (q.shape[1] // k.shape[1])
    for i in range(first, q.shape[0]):
        s = talking_scores(q, k, mix, temp, rel, talk, i)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhd->hd", e / e.sum(-1, keepdim=True), v[:i + 1][:, of])
    return out


def attention_mixer(w, p, mix, h, eps):
    T = h.shape[0]
    linear = lambda n, x: x @ w[p + n].T + w[p + n + ".b"]
    q = rms_unit(linear("q", h).reshape(T, mix["heads"], mix["dim"]), eps)
    k = rms_unit(linear("k", h).reshape(T, mix["kv_heads"], mix["dim"]), eps)
    v = linear("v", h).reshape(T, mix["kv_heads"], mix["vdim"])
    return linear("o", talking_attention(q, k, v, mix, w[p + "temp"], w[p + "rel"], w[p + "talk"]).reshape(T, -1))


MIXERS = {"lightning": lightning_mixer, "latent_attention": latent_mixer, "attention": attention_mixer}


# ---- the model ----------------------------------------------------------------------------------------------------
def layer_runs(cfg):
    """(layer, opens a pass) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def residual_stream(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> List[torch.Tensor]:
    """The residual stream of one sequence after every layer run, [T, width] each."""
    eps = cfg["norm"]["eps"]
    x = x0 = w["embed"][torch.tensor(tokens)]
    out = []
    for i, opens in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if opens:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T
        y = MIXERS[layer["type"]](w, p + "mix.", layer["mixer"], norm(x, w[p + "norm1"], eps), eps)
        x = x + norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(w, p + "mlp.", norm(x, w[p + "norm2"], eps))
            x = x + norm(y, w[p + "norm2b"], eps)
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """[T, vocab]."""
    return norm(residual_stream(cfg, w, tokens)[-1], w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
