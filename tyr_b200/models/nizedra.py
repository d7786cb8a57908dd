"""Nizedra: looped hybrid decoder with a norm before and after every sublayer and an fp32 residual stream:

    x += norm1b(mix(norm1(x)));   x += norm2b(down(xielu(up(norm2(x)))))

A mixer is ``lightning`` (linear attention with one decay per head), ``latent_attention`` (keys and values from a shared low-rank latent,
one rotated key part for all heads, sliding window) or ``attention`` (unit queries and keys, soft-capped scores with a learned
distance bias, mixed across the heads before the softmax).  A range of layers may run several times in a row with the same weights; each
pass starts from a product of the stream and the embedding output, and has a cache and state of its own.

The residual add, the norm after a sublayer, an output bias and the norm before the next sublayer are one launch.  Latent attention
expands keys and values for prompts (one product, whose weight also copies the shared rotated part to every head) and reads the latents
themselves when it decodes (queries and outputs go through the key and value matrices instead).  The decode step is captured as a CUDA
graph.  Rows of a batch may have prompts of different lengths (padded at the end)."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Sequence, Tuple, Union

import torch
import torch.nn.functional as F

from ..io import safetensors as st
from ..ops import delta_rule as dr
from ..ops import flash
from ..ops import joint_attention as ja
from ..ops import latent as lt
from ..ops import lightning as lg
from ..ops.biased_attention import qk_norm_store
from ..ops.embed import position_turns
from ..ops.norm import add_norm, sandwich_norm
from ..ops.skinny import head_products
from .common import KVCache, LinearState, lin, project, xielu_mlp
from .generation import SamplingStrategy, StreamCallback, generate_cached
from .session import HybridSession

LIGHTNING, LATENT, ATTENTION = "lightning", "latent_attention", "attention"


def _up(n: int, multiple: int) -> int:
    return -(-n // multiple) * multiple


# ---- configuration ------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class LightningSpec:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int                              # unrotated query / key channels of a head
    rot_dim: int                          # rotated ones; the key's are shared by all heads
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int                         # of the rotated part, the channels that turn
    window: Optional[int] = None          # keys a query sees, itself included

    # row lengths: of a query or key head, of a value head, of the store (latent | rotated part)
    @property
    def head_row(self): return max(_up(self.dim, 32), _up(self.dim + self.rot_dim, 8))
    @property
    def value_row(self): return _up(self.vdim, 8)
    @property
    def store_row(self): return _up(self.kv_rank + self.rot_dim, 32)


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    bias_max: int                         # distances from here on share the last row of the distance table


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[LightningSpec, LatentSpec, AttentionSpec]
    ff: int = 0                           # 0: no feed-forward


@dataclass(frozen=True)
class Loop:
    """Layers start .. stop - 1 run ``times`` times in a row."""
    start: int
    stop: int
    times: int


def _fields(j: dict, what: str, required: Sequence[str], optional: Sequence[str] = ()) -> dict:
    j = {k: v for k, v in j.items() if v is not None}
    missing = [k for k in required if k not in j]
    unknown = [k for k in j if k not in required and k not in optional]
    if missing or unknown:
        raise ValueError(f"Invalid Nizedra config: {what} " + "; ".join(
            [f"lacks {', '.join(missing)}"] * bool(missing) + [f"has unknown {', '.join(unknown)}"] * bool(unknown)))
    return j


@dataclass
class NizedraConfig:
    vocab: int
    width: int
    eps: float
    layers: List[LayerSpec]
    loop: Optional[Loop] = None

    def __post_init__(self):
        e = lambda i, m: ValueError(f"Invalid Nizedra config: layer {i}: {m}")
        if min(self.vocab, self.width) <= 0 or not self.layers:
            raise ValueError("Invalid Nizedra config: vocab, width and the number of layers must be positive")
        for i, l in enumerate(self.layers):
            m = l.mixer
            if min(m.heads, m.dim, m.vdim) <= 0:
                raise e(i, "head counts and sizes must be positive")
            if isinstance(m, LightningSpec) and len(m.decay) != m.heads:
                raise e(i, "decay needs one number per head")
            if isinstance(m, LatentSpec):
                if min(m.q_rank, m.kv_rank) <= 0 or m.rot_dim < 0 or (m.window is not None and m.window <= 0):
                    raise e(i, "ranks and mask.size must be positive")
                if m.rot_dims % 2 or not 0 <= m.rot_dims <= m.rot_dim:
                    raise e(i, "rot.dims must be even and at most rot_dim")
            if isinstance(m, AttentionSpec):
                if m.kv_heads <= 0 or m.heads % m.kv_heads:
                    raise e(i, "heads must be a multiple of kv_heads")
                if m.softcap <= 0:
                    raise e(i, "softcap must be positive")
            if l.ff < 0:
                raise e(i, "ff must not be negative")
        if self.loop is not None and not (0 <= self.loop.start < self.loop.stop <= len(self.layers) and self.loop.times > 0):
            raise ValueError("Invalid Nizedra config: loop must name a range of layers and run it at least once")

    def runs(self) -> List[Tuple[int, bool]]:
        """(layer, opens a pass of the loop) in the order they run."""
        lo, hi, times = (len(self.layers), len(self.layers), 0) if self.loop is None else (self.loop.start, self.loop.stop, self.loop.times)
        return ([(i, False) for i in range(lo)] + [(i, i == lo) for _ in range(times) for i in range(lo, hi)]
                + [(i, False) for i in range(hi, len(self.layers))])

    @staticmethod
    def from_json(j: dict) -> "NizedraConfig":
        layers = []
        for i, l in enumerate(j["layers"]):
            kind = l.get("type")
            if kind == LIGHTNING:
                m = _fields(l["mixer"], f"layer {i} mixer", ("heads", "dim", "vdim", "decay"))
                mixer = LightningSpec(m["heads"], m["dim"], m["vdim"], tuple(float(d) for d in m["decay"]))
            elif kind == LATENT:
                m = _fields(l["mixer"], f"layer {i} mixer", ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot"), ("mask",))
                rot = _fields(m.pop("rot"), f"layer {i} rot", ("base", "dims"))
                mask = _fields(m.pop("mask"), f"layer {i} mask", ("size",)) if "mask" in m else {}
                mixer = LatentSpec(**m, rot_base=float(rot["base"]), rot_dims=rot["dims"], window=mask.get("size"))
            elif kind == ATTENTION:
                mixer = AttentionSpec(**_fields(l["mixer"], f"layer {i} mixer", ("heads", "kv_heads", "dim", "vdim", "scale", "softcap", "bias_max")))
            else:
                raise ValueError(f'Invalid Nizedra config: layer {i} has unknown type "{kind}"; expected {LIGHTNING}, {LATENT} or {ATTENTION}')
            ff = 0
            if l.get("mlp") is not None:
                p = _fields(l["mlp"], f"layer {i} mlp", ("kind", "ff"))
                if p["kind"] != "dense":
                    raise ValueError(f'Invalid Nizedra config: layer {i} has unknown mlp kind "{p["kind"]}"; expected dense')
                ff = p["ff"]
                if ff <= 0:
                    raise ValueError(f"Invalid Nizedra config: layer {i}: ff must be positive")
            layers.append(LayerSpec(mixer, ff))
        loop = None if j.get("loop") is None else Loop(**_fields(j["loop"], "loop", ("start", "stop", "times")))
        return NizedraConfig(int(j["vocab"]), int(j["width"]), float(j["norm"]["eps"]), layers, loop)

    def to_json(self) -> dict:
        layers = []
        for l in self.layers:
            m, mix = l.mixer, dict(vars(l.mixer))
            if isinstance(m, LightningSpec):
                kind, mix["decay"] = LIGHTNING, list(m.decay)
            elif isinstance(m, LatentSpec):
                kind, mix["rot"] = LATENT, {"base": mix.pop("rot_base"), "dims": mix.pop("rot_dims")}
                window = mix.pop("window")
                if window is not None:
                    mix["mask"] = {"size": window}
            else:
                kind = ATTENTION
            layers.append({"type": kind, "mixer": mix, "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None})
        out = {"architecture": "Nizedra", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": layers}
        if self.loop is not None:
            out["loop"] = dict(vars(self.loop))
        return out

    @staticmethod
    def load_from_pretrained_dir(model_dir: str) -> "NizedraConfig":
        with open(os.path.join(model_dir, "config.json")) as f:
            return NizedraConfig.from_json(json.load(f))


# ---- parameters ---------------------------------------------------------------------------------------------------
@dataclass
class LightningMixer:
    w_in: torch.Tensor            # [q | k | v | g] rows
    decay: torch.Tensor           # double [heads]
    norm: torch.Tensor            # fp32 [heads * vdim]
    w_out: torch.Tensor


@dataclass
class LatentMixer:
    w_down: torch.Tensor          # [query latent | key/value latent | rotated part] rows, padded to a multiple of 8
    q_norm: torch.Tensor          # fp32 [q_rank]
    kv_norm: torch.Tensor         # fp32 [kv_rank]
    turns: torch.Tensor           # rotation frequencies over 2 pi, double
    w_q: torch.Tensor             # [heads * head_row, q_rank padded]
    w_kv: torch.Tensor            # [heads * head_row | heads * value_row, store_row]: a store row to every head's key and value
    w_absorb: torch.Tensor        # [heads, kv_rank, dim padded]: a query head to the latent's channels
    w_value: torch.Tensor         # [heads, value_row, kv_rank padded]
    w_out: torch.Tensor           # [width, heads * value_row]


@dataclass
class AttentionMixer:
    w_in: torch.Tensor            # [q | k | v] rows, padded to a multiple of 8
    b_in: torch.Tensor            # fp32 [q | k | v]
    talk: ja.Talk
    w_out: torch.Tensor
    b_out: torch.Tensor           # fp32 [width]


@dataclass
class FeedForward:
    up: torch.Tensor
    down: torch.Tensor
    act: Tuple[float, float]      # factors of the activation above and below zero
    raw_act: torch.Tensor         # the two numbers they come from
    pre: torch.Tensor             # fp32 norm2, norm2b
    post: torch.Tensor


@dataclass
class Layer:
    pre: torch.Tensor             # fp32 norm1, norm1b
    post: torch.Tensor
    mixer: Union[LightningMixer, LatentMixer, AttentionMixer]
    ffn: Optional[FeedForward]


@dataclass
class NizedraForCausalLM:
    cfg: NizedraConfig
    embed: torch.Tensor
    loop_in: Optional[torch.Tensor]       # [width, 2 width]: stream first, embedding output second
    layers: List[Layer]
    norm: torch.Tensor            # fp32 [width]
    head: torch.Tensor

    @property
    def device(self): return self.embed.device
    @property
    def dtype(self): return self.embed.dtype


def tensor_shapes(cfg: NizedraConfig) -> Dict[str, Tuple[Optional[int], ...]]:
    """Checkpoint names and shapes.  The rows of the distance tables are not part of the configuration: None."""
    h = cfg.width
    out: Dict[str, Tuple[Optional[int], ...]] = {"embed": (cfg.vocab, h)}
    if cfg.loop is not None:
        out["loop.in"] = (h, 2 * h)
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        x = p + "mix."
        out[p + "norm1"] = out[p + "norm1b"] = (h,)
        if isinstance(m, LightningSpec):
            dk, dv = m.heads * m.dim, m.heads * m.vdim
            out.update({x + "q": (dk, h), x + "k": (dk, h), x + "v": (dv, h), x + "g": (dv, h), x + "o": (h, dv), x + "norm": (dv,)})
        elif isinstance(m, LatentSpec):
            out.update({x + "dq": (m.q_rank, h), x + "dq.norm": (m.q_rank,), x + "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                        x + "dkv": (m.kv_rank + m.rot_dim, h), x + "dkv.norm": (m.kv_rank,), x + "uk": (m.heads * m.dim, m.kv_rank),
                        x + "uv": (m.heads * m.vdim, m.kv_rank), x + "o": (h, m.heads * m.vdim)})
        else:
            for n, d in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                out[x + n], out[x + n + ".b"] = (d, h), (d,)
            out.update({x + "rel": (None, m.heads), x + "talk": (m.heads, m.heads), x + "temp": (m.heads,), x + "o": (h, m.heads * m.vdim), x + "o.b": (h,)})
        if l.ff:
            out[p + "norm2"] = out[p + "norm2b"] = (h,)
            out.update({p + "mlp.up": (l.ff, h), p + "mlp.down": (h, l.ff), p + "mlp.act": (2,)})
    out["final.norm"], out["head"] = (h,), (cfg.vocab, h)
    return out


def _pad(w: torch.Tensor, *sizes: int) -> torch.Tensor:
    """Zeros after the last dimensions up to ``sizes``."""
    pads = [p for n, s in zip(reversed(w.shape), reversed(sizes)) for p in (0, s - n)]
    return F.pad(w, pads).contiguous()


def _rows(ws: Sequence[torch.Tensor]) -> torch.Tensor:
    w = torch.cat(list(ws), 0)
    return _pad(w, _up(w.shape[0], 8), w.shape[1])


def _latent_mixer(s: LatentSpec, take, f32, p: str) -> LatentMixer:
    H, dk, R = s.heads, s.dim + s.rot_dim, s.kv_rank
    uk, uv = take(p + "uk").reshape(H, s.dim, R), take(p + "uv").reshape(H, s.vdim, R)
    w_k = uk.new_zeros(H, s.head_row, s.store_row)
    w_k[:, :s.dim, :R] = uk
    w_k[:, s.dim:dk, R:R + s.rot_dim] = torch.eye(s.rot_dim, dtype=uk.dtype, device=uk.device)      # the shared part as it is
    w_v = _pad(uv, s.value_row, s.store_row)
    w_q = _pad(take(p + "uq").reshape(H, dk, s.q_rank), s.head_row, _up(s.q_rank, 32))
    w_out = take(p + "o")
    w_out = _pad(w_out.reshape(w_out.shape[0], H, s.vdim), s.value_row).flatten(1)
    return LatentMixer(_rows([take(p + "dq"), take(p + "dkv")]), f32(p + "dq.norm"), f32(p + "dkv.norm"),
                       position_turns(s.rot_dims, s.rot_base, uk.device), w_q.flatten(0, 1), torch.cat([w_k.flatten(0, 1), w_v.flatten(0, 1)]),
                       _pad(uk.transpose(1, 2), R, _up(s.dim, 32)), _pad(uv, s.value_row, _up(R, 32)), w_out)


def build(cfg: NizedraConfig, get: Callable[[str], torch.Tensor], device="cpu", dtype=torch.bfloat16) -> NizedraForCausalLM:
    """Assemble the model from ``get(name) -> tensor`` (checkpoint names)."""
    shapes = tensor_shapes(cfg)

    def take(name, dt=dtype):
        t = get(name)
        want = shapes[name]
        if t.dim() != len(want) or any(w is not None and w != n for w, n in zip(want, t.shape)):
            raise st.SafeTensorsError(f"{name}: expected shape {list(want)}, got {list(t.shape)}")
        return t.to(device=device, dtype=dt)
    f32 = lambda name: take(name, torch.float32).contiguous()
    layers = []
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.mix.", l.mixer
        if isinstance(m, LightningSpec):
            mixer = LightningMixer(_rows([take(p + n) for n in "qkvg"]), torch.tensor(m.decay, dtype=torch.float64, device=device), f32(p + "norm"),
                                   take(p + "o").contiguous())
        elif isinstance(m, LatentSpec):
            mixer = _latent_mixer(m, take, f32, p)
        else:
            rel = f32(p + "rel")
            talk = ja.Talk(f32(p + "temp"), rel, ja.distance_buckets(rel.shape[0], m.bias_max).to(device), f32(p + "talk"), float(m.softcap))
            mixer = AttentionMixer(_rows([take(p + n) for n in "qkv"]), torch.cat([f32(f"{p}{n}.b") for n in "qkv"]), talk, take(p + "o").contiguous(),
                                   f32(p + "o.b"))
        ffn = None
        if l.ff:
            p = f"l{i}.mlp."
            raw = take(p + "act", torch.float32)
            above, below = F.softplus(raw.double()).tolist()
            ffn = FeedForward(take(p + "up").contiguous(), take(p + "down").contiguous(), (above, 0.5 + below), raw, f32(f"l{i}.norm2"), f32(f"l{i}.norm2b"))
        layers.append(Layer(f32(f"l{i}.norm1"), f32(f"l{i}.norm1b"), mixer, ffn))
    loop_in = take("loop.in").contiguous() if cfg.loop is not None else None
    return NizedraForCausalLM(cfg, take("embed").contiguous(), loop_in, layers, f32("final.norm"), take("head").contiguous())


def load(cfg: NizedraConfig, source, device="cpu", dtype=torch.bfloat16, log=None) -> NizedraForCausalLM:
    """Load from a safetensors ``Source`` (file or directory)."""
    src = source if isinstance(source, st.Source) else st.Source.open(source)
    m = build(cfg, src.load, device, dtype)
    if log is not None:
        log(f"  loaded {len(m.layers)} layers")
    return m


def load_pretrained(model_dir: str, device="cpu", dtype=torch.bfloat16, log=None) -> NizedraForCausalLM:
    return load(NizedraConfig.load_from_pretrained_dir(model_dir), model_dir, device, dtype, log)


def random_tensor(name: str, shape: Tuple[int, ...], gen: torch.Generator) -> torch.Tensor:
    """Random-init value of one checkpoint tensor (fp32)."""
    dev = gen.device
    last = name.rsplit(".", 1)[-1]
    if "norm" in last or last == "temp":
        return torch.ones(shape, device=dev)
    if last in ("b", "act"):
        return torch.zeros(shape, device=dev)
    if last == "talk":
        return torch.eye(shape[0], device=dev) + torch.randn(shape, generator=gen, device=dev) * (0.1 * shape[0] ** -0.5)
    if last == "rel":
        return torch.randn(shape, generator=gen, device=dev) * 0.1
    return torch.randn(shape, generator=gen, device=dev) * (1.0 if name == "embed" else shape[-1] ** -0.5)


def init(cfg: NizedraConfig, device="cpu", dtype=torch.float32, seed: int = 0, rows: int = 32) -> NizedraForCausalLM:
    """Random weights; ``rows`` of the distance tables."""
    gen = torch.Generator(device=device).manual_seed(seed)
    shapes = tensor_shapes(cfg)
    return build(cfg, lambda n: random_tensor(n, tuple(rows if d is None else d for d in shapes[n]), gen).to(dtype), device, dtype)


def state_dict(m: NizedraForCausalLM) -> Dict[str, torch.Tensor]:
    """Checkpoint-format tensors (inverse of ``load``)."""
    cfg = m.cfg
    out = {"embed": m.embed, "final.norm": m.norm, "head": m.head}
    if m.loop_in is not None:
        out["loop.in"] = m.loop_in
    for i, (s, l) in enumerate(zip(cfg.layers, m.layers)):
        p, x, w = f"l{i}.mix.", s.mixer, l.mixer
        out[f"l{i}.norm1"], out[f"l{i}.norm1b"] = l.pre, l.post
        if isinstance(x, LightningSpec):
            dk, dv = x.heads * x.dim, x.heads * x.vdim
            out.update({p + n: t for n, t in zip("qkvg", torch.split(w.w_in[:2 * (dk + dv)], [dk, dk, dv, dv]))})
            out.update({p + "norm": w.norm, p + "o": w.w_out})
        elif isinstance(x, LatentSpec):
            H, R, dk = x.heads, x.kv_rank, x.dim + x.rot_dim
            out.update({p + "dq": w.w_down[:x.q_rank], p + "dkv": w.w_down[x.q_rank:x.q_rank + R + x.rot_dim], p + "dq.norm": w.q_norm, p + "dkv.norm": w.kv_norm,
                        p + "uq": w.w_q.reshape(H, x.head_row, -1)[:, :dk, :x.q_rank].flatten(0, 1),
                        p + "uk": w.w_absorb[..., :x.dim].transpose(1, 2).flatten(0, 1), p + "uv": w.w_value[:, :x.vdim, :R].flatten(0, 1),
                        p + "o": w.w_out.reshape(cfg.width, H, -1)[..., :x.vdim].flatten(1)})
        else:
            sizes = [x.heads * x.dim, x.kv_heads * x.dim, x.kv_heads * x.vdim]
            out.update({p + n: t for n, t in zip("qkv", torch.split(w.w_in[:sum(sizes)], sizes))})
            out.update({f"{p}{n}.b": t for n, t in zip("qkv", torch.split(w.b_in, sizes))})
            out.update({p + "rel": w.talk.rel, p + "talk": w.talk.mix, p + "temp": w.talk.temp, p + "o": w.w_out, p + "o.b": w.b_out})
        if l.ffn is not None:
            f = l.ffn
            out.update({f"l{i}.norm2": f.pre, f"l{i}.norm2b": f.post, f"l{i}.mlp.up": f.up, f"l{i}.mlp.down": f.down, f"l{i}.mlp.act": f.raw_act})
    return {k: v.contiguous() for k, v in out.items()}


# ---- blocks -------------------------------------------------------------------------------------------------------
@dataclass
class Tokens:
    """The tokens of one pass: whole prompts (``lens`` where rows end earlier) or one token per row at ``pos``."""
    lens: Optional[torch.Tensor] = None
    pos: Optional[torch.Tensor] = None

    @property
    def step(self): return self.pos is not None


def lightning_mixer(s: LightningSpec, m: LightningMixer, h: torch.Tensor, state: LinearState, t: Tokens, eps: float) -> torch.Tensor:
    dk, n = s.heads * s.dim, s.heads * (2 * s.dim + s.vdim)
    if t.step:                                             # one product; the step takes the activation
        y = lin(h, m.w_in)
        y, gate = y[..., :n], y[..., n:n + s.heads * s.vdim]
    else:                                                  # activated in the product's epilogue
        y, gate = project(h, m.w_in[:n], act="silu"), project(h, m.w_in[n:n + s.heads * s.vdim])
    q, k, v = (y[..., a:b].unflatten(2, (s.heads, -1)) for a, b in ((0, dk), (dk, 2 * dk), (2 * dk, n)))
    o = lg.step(q, k, v, m.decay, state.rec) if t.step else lg.prefill(q, k, v, m.decay, state.rec, t.lens)
    return lin(dr.gated_norm(o.flatten(2).unsqueeze(2), gate, m.norm, eps, "sigmoid"), m.w_out)


def latent_mixer(s: LatentSpec, m: LatentMixer, h: torch.Tensor, store: KVCache, t: Tokens, eps: float) -> torch.Tensor:
    B, S, _ = h.shape
    H, dk, R = s.heads, s.dim + s.rot_dim, s.kv_rank
    cq, rows = lt.latent_norm_store(lin(h, m.w_down), m.q_norm, m.kv_norm, m.turns, s.rot_dim, eps, q_width=m.w_q.shape[1], width=s.store_row,
                                    store=store, pos=t.pos, lens=t.lens, want_rows=not t.step)
    q = lin(cq, m.w_q).unflatten(2, (H, s.head_row))
    if not t.step:
        lt.rotate_heads(q[..., s.dim:dk], m.turns)
        kv = lin(rows, m.w_kv)
        k, v = kv[..., :H * s.head_row].unflatten(2, (H, -1)), kv[..., H * s.head_row:].unflatten(2, (H, -1))
        d8 = _up(dk, 8)
        if flash.sink_supported(q[..., :d8], k[..., :d8], v, None, None) and s.scale > 0.0:
            o = flash.flash_fwd_sink(q[..., :d8], k[..., :d8], v, scale=s.scale, window=s.window)
        else:
            o = ja.prompt_attention(q[..., :dk], k[..., :dk], v, scale=s.scale, window=s.window)
        return lin(o, m.w_out)
    new = torch.empty if R % 32 == 0 else torch.zeros
    ql = torch.empty((B, 1, H, s.store_row), dtype=h.dtype, device=h.device)
    lat = new((B, 1, H, m.w_value.shape[2]), dtype=h.dtype, device=h.device)
    o = torch.empty((B, H, s.value_row), dtype=h.dtype, device=h.device)
    head_products(q[:, 0], m.w_absorb, ql[:, 0])
    lt.rotate_heads(q[..., s.dim:dk], m.turns, t.pos, ql[..., R:])
    ja.step_attention(ql, store, t.pos, R, scale=s.scale, window=s.window, out=lat[..., :R])
    head_products(lat[:, 0], m.w_value, o)
    return lin(o.reshape(B, 1, -1), m.w_out)


def attention_mixer(s: AttentionSpec, m: AttentionMixer, h: torch.Tensor, store: KVCache, t: Tokens, eps: float) -> torch.Tensor:
    """Without the output bias, which the norm that follows adds."""
    dkp, dvp = store.k.shape[3], store.v.shape[3]
    bound = 1.02 * s.dim                                   # queries and keys of unit root mean square, rounded
    q, k, v = qk_norm_store(lin(h, m.w_in), None, None, s.heads, s.kv_heads, s.dim, s.vdim, eps, dkp=dkp, dvp=dvp, store=store, pos=t.pos, lens=t.lens,
                            bias=m.b_in)
    if t.step:
        o = ja.step_attention(q, store, t.pos, s.vdim, scale=s.scale, talk=m.talk, dot_bound=bound).flatten(2)
    else:
        o = ja.prompt_attention(q, k, v[..., :s.vdim], scale=s.scale, talk=m.talk, dot_bound=bound)
    return lin(o, m.w_out)


class CacheSession(HybridSession):
    """A store or state for every layer run (each pass of the loop has its own): latent rows (a ring of the window), K/V of the attention
    layers, lightning states; ``retain`` gives finished rows back."""
    name = "Nizedra"

    def __init__(self, m: NizedraForCausalLM, batch: int, max_len: int):
        super().__init__(batch, max_len, m.device)
        self.m, self.runs = m, m.cfg.runs()
        for i, _ in self.runs:
            s = m.cfg.layers[i].mixer
            kv = state = None
            if isinstance(s, LightningSpec):
                state = LinearState(rec=torch.zeros((batch, s.heads, s.dim, s.vdim), device=m.device))
            elif isinstance(s, LatentSpec):
                ring = s.window is not None and s.window < max_len
                kv = KVCache.allocate(batch, 1, s.window if ring else max_len, s.store_row, m.device, m.dtype, ring=ring, shared=True)
            else:
                dkp, dvp = ja.store_dims(s.dim, s.vdim, m.dtype, m.device)
                kv = KVCache.allocate(batch, s.kv_heads, max_len, dkp, m.device, m.dtype, v_dim=dvp)
            self.kv.append(kv)
            self.lin.append(state)

    def _forward(self, ids: torch.Tensor, t: Tokens, layer_done=None) -> torch.Tensor:
        """Normed hidden states after all layers."""
        m, eps, W = self.m, self.m.cfg.eps, self.m.cfg.width
        e = F.embedding(ids, m.embed)
        x = e.to(torch.float32, copy=True)
        both = None
        if m.loop_in is not None:
            both = torch.cat([e, e], -1)                   # (stream | embedding output), the input of every pass

        def open_pass(layer: Layer) -> torch.Tensor:
            return sandwich_norm(lin(both, m.loop_in), None, layer.pre, eps, x, m.dtype, replace=True)

        def after(k: int) -> dict:
            """What the norm after run k leaves for the next: its input, or the stream for the next pass."""
            if k + 1 == len(self.runs):
                return {"gain": m.norm}
            j, opens = self.runs[k + 1]
            return {"gain": None, "out": both[..., :W]} if opens else {"gain": m.layers[j].pre}
        first = m.layers[self.runs[0][0]]
        h = open_pass(first) if self.runs[0][1] else add_norm(None, first.pre, eps, x, m.dtype)
        for k, (i, _) in enumerate(self.runs):
            s, l = m.cfg.layers[i].mixer, m.layers[i]
            bias = None
            if isinstance(s, LightningSpec):
                y = lightning_mixer(s, l.mixer, h, self.lin[k], t, eps)
            elif isinstance(s, LatentSpec):
                y = latent_mixer(s, l.mixer, h, self.kv[k], t, eps)
            else:
                y, bias = attention_mixer(s, l.mixer, h, self.kv[k], t, eps), l.mixer.b_out
            nxt = after(k)
            if l.ffn is not None:
                h = sandwich_norm(y, l.post, l.ffn.pre, eps, x, m.dtype, bias=bias)
                y, bias = xielu_mlp(h, l.ffn.up, l.ffn.down, *l.ffn.act), None
            h = sandwich_norm(y, l.post if l.ffn is None else l.ffn.post, resid=x, eps=eps, out_dtype=m.dtype, bias=bias, **nxt)
            if layer_done is not None:
                layer_done(k, x)
            if nxt["gain"] is None:
                h = open_pass(m.layers[self.runs[k + 1][0]])
        return h

    @torch.no_grad()
    def hidden(self, ids: torch.Tensor, lengths: Optional[Sequence[int]] = None, layer_done=None) -> torch.Tensor:
        B, S = ids.shape
        if B != self.batch or S == 0 or self.pos > 0:
            raise ValueError("Nizedra prefills a fresh session with one prompt per row")
        lengths = [S] * B if lengths is None else [int(n) for n in lengths]
        if len(lengths) != B or min(lengths) < 1 or max(lengths) > S:
            raise ValueError("Nizedra prompt lengths must be between 1 and the padded length")
        self._check_room(max(lengths))
        lens = None if min(lengths) == S else torch.tensor(lengths, dtype=torch.int32, device=self.device)
        h = self._forward(ids, Tokens(lens=lens), layer_done)
        self._advance(lengths)
        return h

    def head(self, h: torch.Tensor) -> torch.Tensor:
        return lin(h, self.m.head)

    # -- decode ----------------------------------------------------------------------------------------------------
    def device_step_supported(self) -> bool:
        return True

    def graph_supported(self) -> bool:
        return super().graph_supported() and self.m.embed.is_cuda and self.m.dtype == torch.bfloat16

    def _positions(self) -> torch.Tensor:
        return torch.tensor(self.lengths, dtype=torch.int32, device=self.device)

    def _device_step(self, tok: torch.Tensor) -> torch.Tensor:
        h = self._forward(tok.reshape(-1, 1), Tokens(pos=self.pos_t))
        self.pos_t += 1
        return self.head(h[:, -1])


# ---- whole sequences and generation -------------------------------------------------------------------------------
@torch.no_grad()
def forward(m: NizedraForCausalLM, input_ids: torch.Tensor, lengths: Optional[Sequence[int]] = None) -> torch.Tensor:
    """Logits [B, S, V] of whole sequences."""
    s = CacheSession(m, input_ids.shape[0], input_ids.shape[1])
    return s.head(s.hidden(input_ids, lengths))


def generate(m: NizedraForCausalLM, input_ids: torch.Tensor, max_new_tokens: int = 64, strategy: SamplingStrategy = SamplingStrategy(),
             eos_token_ids: Sequence[int] = (), on_step: Optional[StreamCallback] = None, generator=None,
             lengths: Optional[Sequence[int]] = None) -> torch.Tensor:
    """``input_ids`` [B, S], rows shorter than S padded at the end with ``lengths`` given; the new tokens of every row follow in
    columns S, S + 1, ..."""
    sess = CacheSession(m, input_ids.shape[0], input_ids.shape[1] + max_new_tokens)
    return generate_cached(lambda ids: sess.prefill(ids, lengths), sess.step, input_ids, max_new_tokens, strategy, eos_token_ids, on_step, generator)


def generate_greedy(m, input_ids, max_new_tokens=64, eos_token_ids=(), lengths=None):
    return generate(m, input_ids, max_new_tokens, SamplingStrategy.greedy(), eos_token_ids, lengths=lengths)


def generate_stream(m, input_ids, on_step, max_new_tokens=64, strategy=SamplingStrategy(), eos_token_ids=()):
    return generate(m, input_ids, max_new_tokens, strategy, eos_token_ids, on_step)
