"""Kinetar: hybrid decoder whose layers run their mixer and their feed-forward side by side on one norm's output, with an fp32
residual stream and sinusoidal positions on the embedding:

    h = norm1(x);   x += mix(h) + down(relu(up(h))^2)

A mixer is either ``parallel`` (grouped-query attention with short convolutions on queries and keys, values that are the keys, a query
temperature, a softmax sink and an output gate, next to a selective scan) or ``channel_delta`` (gated delta rule with a decay per key
channel).

Everything that reads h is one product, and everything that is added to x is one product: the mixers write their gated and scaled
outputs and the feed-forward its activations into column windows of one buffer, which a single output projection (its weight the
mixers' and the feed-forward's side by side) sums in fp32.  Between the two lie one launch for all convolutions and activations
and the mixers' own kernels.  The decode step is captured as a CUDA graph.  Rows of a batch may have prompts of different lengths
(padded at the end)."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Sequence, Tuple, Union

import torch
import torch.nn.functional as F

from ..io import safetensors as st
from ..ops import delta_rule as dr
from ..ops import selective_scan as ss
from ..ops import sink_attention as sa
from ..ops.embed import embed_positions, position_turns
from ..ops.mix_conv import Segment, mix_prompt, mix_step
from ..ops.norm import add_norm
from .common import KVCache, LinearState, lin, project
from .generation import SamplingStrategy, StreamCallback, generate_cached
from .session import HybridSession

PARALLEL, CHANNEL_DELTA = "parallel", "channel_delta"


# ---- configuration ------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int                             # the values are the keys: equal to dim
    conv: int
    scale: float
    temp_coef: float
    temp_every: float


@dataclass(frozen=True)
class ScanSpec:
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass(frozen=True)
class ParallelSpec:
    left: AttentionSpec
    right: ScanSpec
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class ChannelDeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @property
    def key_dim(self): return self.kv_heads * self.dim
    @property
    def value_dim(self): return self.heads * self.vdim
    @property
    def conv_dim(self): return 2 * self.key_dim + self.value_dim


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[ParallelSpec, ChannelDeltaSpec]
    ff: int = 0                           # 0: no feed-forward


def _fields(j: dict, what: str, required: Sequence[str], optional: Sequence[str] = ()) -> dict:
    j = {k: v for k, v in j.items() if v is not None}
    missing = [k for k in required if k not in j]
    unknown = [k for k in j if k not in required and k not in optional]
    if missing or unknown:
        raise ValueError(f"Invalid Kinetar config: {what} " + "; ".join(
            [f"lacks {', '.join(missing)}"] * bool(missing) + [f"has unknown {', '.join(unknown)}"] * bool(unknown)))
    return j


@dataclass
class KinetarConfig:
    vocab: int
    width: int
    eps: float
    layers: List[LayerSpec]
    embedding_scale: float = 1.0
    logit_scale: float = 1.0

    def __post_init__(self):
        e = lambda i, m: ValueError(f"Invalid Kinetar config: layer {i}: {m}")
        if min(self.vocab, self.width) <= 0 or not self.layers:
            raise ValueError("Invalid Kinetar config: vocab, width and the number of layers must be positive")
        for i, l in enumerate(self.layers):
            m = l.mixer
            heads = m.left if isinstance(m, ParallelSpec) else m
            if min(heads.heads, heads.kv_heads, heads.dim, heads.vdim) <= 0 or heads.heads % heads.kv_heads:
                raise e(i, "head counts and sizes must be positive and heads a multiple of kv_heads")
            if heads.conv <= 0 or (isinstance(m, ParallelSpec) and m.right.conv <= 0):
                raise e(i, "the convolutions need at least one tap")
            if isinstance(m, ParallelSpec):
                if m.left.vdim != m.left.dim:
                    raise e(i, "the values are the keys: vdim must equal dim")
                if m.left.temp_every <= 0:
                    raise e(i, "q_temp.every must be positive")
                if min(m.right.inner, m.right.state, m.right.dt_rank) <= 0:
                    raise e(i, "sizes of the scan must be positive")
            if l.ff < 0:
                raise e(i, "ff must not be negative")

    @staticmethod
    def from_json(j: dict) -> "KinetarConfig":
        layers = []
        for i, l in enumerate(j["layers"]):
            kind = l.get("type")
            if kind == CHANNEL_DELTA:
                mixer = ChannelDeltaSpec(**_fields(l["mixer"], f"layer {i} mixer", ("heads", "kv_heads", "dim", "vdim", "conv")))
            elif kind == PARALLEL:
                m = _fields(l["mixer"], f"layer {i} mixer", ("left", "right", "left_scale", "right_scale"))
                a = _fields(m["left"], f"layer {i} left", ("heads", "kv_heads", "dim", "vdim", "conv", "scale", "q_temp"))
                t = _fields(a.pop("q_temp"), f"layer {i} q_temp", ("coef", "every"))
                right = ScanSpec(**_fields(m["right"], f"layer {i} right", ("inner", "state", "dt_rank", "conv")))
                mixer = ParallelSpec(AttentionSpec(**a, temp_coef=t["coef"], temp_every=t["every"]), right, m["left_scale"], m["right_scale"])
            else:
                raise ValueError(f'Invalid Kinetar config: layer {i} has unknown type "{kind}"; expected {PARALLEL} or {CHANNEL_DELTA}')
            ff = 0
            if l.get("mlp") is not None:
                p = _fields(l["mlp"], f"layer {i} mlp", ("kind", "ff"))
                if p["kind"] != "dense":
                    raise ValueError(f'Invalid Kinetar config: layer {i} has unknown mlp kind "{p["kind"]}"; expected dense')
                ff = p["ff"]
                if ff <= 0:
                    raise ValueError(f"Invalid Kinetar config: layer {i}: ff must be positive")
            layers.append(LayerSpec(mixer, ff))
        return KinetarConfig(int(j["vocab"]), int(j["width"]), float(j["norm"]["eps"]), layers, float(j["embedding"]["scale"]), float(j["logit_scale"]))

    def to_json(self) -> dict:
        layers = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, ChannelDeltaSpec):
                kind, mix = CHANNEL_DELTA, dict(vars(m))
            else:
                a = dict(vars(m.left))
                a["q_temp"] = {"coef": a.pop("temp_coef"), "every": a.pop("temp_every")}
                kind, mix = PARALLEL, {"left": a, "right": dict(vars(m.right)), "left_scale": m.left_scale, "right_scale": m.right_scale}
            layers.append({"type": kind, "mixer": mix, "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None})
        return {"architecture": "Kinetar", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "embedding": {"scale": self.embedding_scale},
                "logit_scale": self.logit_scale, "layers": layers}

    @staticmethod
    def load_from_pretrained_dir(model_dir: str) -> "KinetarConfig":
        with open(os.path.join(model_dir, "config.json")) as f:
            return KinetarConfig.from_json(json.load(f))


# ---- parameters ---------------------------------------------------------------------------------------------------
@dataclass
class Columns:
    """Named column windows of a buffer, each starting at a multiple of 8; ``total`` is a multiple of 32."""
    at: Dict[str, int]
    width: Dict[str, int]
    total: int

    @staticmethod
    def lay_out(parts: Sequence[Tuple[str, int]], multiple: int = 32) -> "Columns":
        at, end = {}, 0
        for n, w in parts:
            at[n] = end
            end += -(-w // 8) * 8
        return Columns(at, dict(parts), -(-end // multiple) * multiple)

    def __getitem__(self, n: str) -> slice:
        return slice(self.at[n], self.at[n] + self.width[n])

    @property
    def padded(self) -> bool:
        return sum(self.width.values()) != self.total

    def buffer(self, B: int, S: int, device, dtype) -> torch.Tensor:
        """[B, S, total]; columns that belong to no window are zero."""
        make = torch.zeros if self.padded else torch.empty
        return make((B, S, self.total), device=device, dtype=dtype)


@dataclass
class AttentionMixer:
    q_conv: torch.Tensor          # fp32 [heads * dim, taps]
    k_conv: torch.Tensor
    sink: torch.Tensor            # fp32 [heads]


@dataclass
class ScanMixer:
    conv: torch.Tensor            # fp32 [inner, taps]
    conv_b: torch.Tensor          # fp32 [inner]
    w_x: torch.Tensor             # [dt | B | C] rows by ``proj``
    proj: Columns
    w_dt: torch.Tensor            # [inner, columns of dt, padded]
    dt_b: torch.Tensor            # fp32
    a: torch.Tensor               # fp32 [inner, state]: -exp(A_log)
    d: torch.Tensor               # fp32


@dataclass
class DeltaMixer:
    conv: Dict[str, torch.Tensor]     # fp32, q / k / v
    w_a: torch.Tensor                 # [heads * dim, rank of a, padded]
    w_g: torch.Tensor                 # [value_dim, rank of g, padded]
    a_log: torch.Tensor               # fp32
    dt_bias: torch.Tensor
    norm: torch.Tensor                # fp32 [vdim]
    norm_lp: torch.Tensor             # the same in the compute dtype


@dataclass
class Layer:
    gain: torch.Tensor            # fp32 [width]: 1 + weight of norm1
    w_in: torch.Tensor            # rows by ``cols``: everything that reads h; the feed-forward's rows come last
    cols: Columns
    w_out: torch.Tensor           # [width, act.total]: everything that is added to x
    act: Columns
    mixer: Tuple                  # (AttentionMixer, ScanMixer) | (DeltaMixer,)
    raw: Dict[str, torch.Tensor]  # checkpoint tensors that the fields above hold only in another form


@dataclass
class KinetarForCausalLM:
    cfg: KinetarConfig
    embed: torch.Tensor
    turns: torch.Tensor           # sinusoid frequencies
    layers: List[Layer]
    gain: torch.Tensor            # fp32 [width]: (1 + final norm weight) * logit_scale
    head: torch.Tensor
    raw: Dict[str, torch.Tensor]

    @property
    def device(self): return self.embed.device
    @property
    def dtype(self): return self.embed.dtype


def tensor_shapes(cfg: KinetarConfig) -> Dict[str, Tuple[Optional[int], ...]]:
    """Checkpoint names and shapes.  The ranks of the low-rank projections are not part of the configuration: None."""
    h = cfg.width
    out: Dict[str, Tuple[Optional[int], ...]] = {"embed": (cfg.vocab, h)}
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        out[p + "norm1"] = (h,)
        x = p + "mix."
        if isinstance(m, ChannelDeltaSpec):
            for n, d in (("q", m.key_dim), ("k", m.key_dim), ("v", m.value_dim)):
                out[x + n], out[x + n + ".conv"] = (d, h), (d, m.conv)
            hk = m.heads * m.dim
            out.update({x + "b": (m.heads, h), x + "A_log": (m.heads,), x + "norm": (m.vdim,), x + "a1": (None, h), x + "a2": (hk, None),
                        x + "dt_bias": (hk,), x + "g1": (None, h), x + "g2": (m.value_dim, None), x + "o": (h, m.value_dim)})
        else:
            a, s, y = m.left, m.right, x + "left."
            hd, gd = a.heads * a.dim, a.kv_heads * a.dim
            out.update({y + "q": (hd, h), y + "k": (gd, h), y + "q.conv": (hd, a.conv), y + "k.conv": (gd, a.conv), y + "sink": (a.heads,),
                        y + "g": (a.heads * a.vdim, h), y + "o": (h, a.heads * a.vdim)})
            y = x + "right."
            out.update({y + "in": (2 * s.inner, h), y + "conv": (s.inner, s.conv), y + "conv.b": (s.inner,), y + "x": (s.dt_rank + 2 * s.state, s.inner),
                        y + "dt": (s.inner, s.dt_rank), y + "dt.b": (s.inner,), y + "A_log": (s.inner, s.state), y + "D": (s.inner,),
                        y + "o": (h, s.inner)})
        if l.ff:
            out[p + "mlp.up"], out[p + "mlp.down"] = (l.ff, h), (h, l.ff)
    out["final.norm"], out["head"] = (h,), (cfg.vocab, h)
    return out


def _rows(cols: Columns, parts: Dict[str, torch.Tensor]) -> torch.Tensor:
    """Weight whose output columns are laid out by ``cols``."""
    first = next(iter(parts.values()))
    w = torch.zeros((cols.total, first.shape[1]), dtype=first.dtype, device=first.device)
    for n, t in parts.items():
        w[cols[n]] = t
    return w


def _pad_cols(w: torch.Tensor, multiple: int = 32) -> torch.Tensor:
    return F.pad(w, (0, (-w.shape[1]) % multiple)).contiguous()


def build(cfg: KinetarConfig, get: Callable[[str], torch.Tensor], device="cpu", dtype=torch.bfloat16) -> KinetarForCausalLM:
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
        raw = {}

        def keep(name):
            raw[name] = take(name, torch.float32)
            return raw[name]
        if isinstance(m, ChannelDeltaSpec):
            a1, a2, g1, g2 = (take(p + n) for n in ("a1", "a2", "g1", "g2"))
            if a1.shape[0] != a2.shape[1] or g1.shape[0] != g2.shape[1]:
                raise st.SafeTensorsError(f"{p}a1 / a2 / g1 / g2: the ranks of a pair differ")
            w_a, w_g = _pad_cols(a2), _pad_cols(g2)
            cols = [("q", m.key_dim), ("k", m.key_dim), ("v", m.value_dim), ("b", m.heads), ("a1", w_a.shape[1]), ("g1", w_g.shape[1])]
            rows = {n: take(p + n) for n in "qkvb"}
            rows["a1"], rows["g1"] = (F.pad(t, (0, 0, 0, w.shape[1] - t.shape[0])) for t, w in ((a1, w_a), (g1, w_g)))
            raw["rank"] = torch.tensor([a1.shape[0], g1.shape[0]])
            mixer = (DeltaMixer({n: f32(f"{p}{n}.conv") for n in "qkv"}, w_a, w_g, f32(p + "A_log"), f32(p + "dt_bias"), f32(p + "norm"), take(p + "norm")),)
            act, outs = [("mix", m.value_dim)], {"mix": take(p + "o")}
        else:
            a, s = m.left, m.right
            proj = Columns.lay_out([("dt", -(-s.dt_rank // 32) * 32), ("b", s.state), ("c", s.state)], 8)
            wx = take(p + "right.x")
            w_dt = _pad_cols(take(p + "right.dt"))
            w_x = _rows(proj, {"dt": F.pad(wx[:s.dt_rank], (0, 0, 0, proj.width["dt"] - s.dt_rank)), "b": wx[s.dt_rank:s.dt_rank + s.state],
                               "c": wx[s.dt_rank + s.state:]})
            xz = take(p + "right.in")
            cols = [("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("g", a.heads * a.vdim), ("x", s.inner), ("z", s.inner)]
            rows = {**{n: take(f"{p}left.{n}") for n in "qkg"}, "x": xz[:s.inner], "z": xz[s.inner:]}
            left = AttentionMixer(f32(p + "left.q.conv"), f32(p + "left.k.conv"), f32(p + "left.sink"))
            right = ScanMixer(f32(p + "right.conv"), f32(p + "right.conv.b"), w_x, proj, w_dt, f32(p + "right.dt.b"),
                              -torch.exp(keep(p + "right.A_log")), f32(p + "right.D"))
            mixer = (left, right)
            act, outs = [("left", a.heads * a.vdim), ("right", s.inner)], {"left": take(p + "left.o"), "right": take(p + "right.o")}
        if l.ff:
            cols, rows["up"] = cols + [("up", l.ff)], take(f"l{i}.mlp.up")
            act, outs["up"] = act + [("up", l.ff)], take(f"l{i}.mlp.down")
        cols, act = Columns.lay_out(cols, 8), Columns.lay_out(act)
        w_out = _rows(act, {n: t.T for n, t in outs.items()}).T.contiguous()
        layers.append(Layer(1.0 + keep(f"l{i}.norm1"), _rows(cols, rows), cols, w_out, act, mixer, raw))
    final = take("final.norm", torch.float32)
    return KinetarForCausalLM(cfg, take("embed").contiguous(), position_turns(cfg.width, device=device), layers, (1.0 + final) * cfg.logit_scale,
                              take("head").contiguous(), {"final.norm": final})


def load(cfg: KinetarConfig, source, device="cpu", dtype=torch.bfloat16, log=None) -> KinetarForCausalLM:
    """Load from a safetensors ``Source`` (file or directory)."""
    src = source if isinstance(source, st.Source) else st.Source.open(source)
    m = build(cfg, src.load, device, dtype)
    if log is not None:
        log(f"  loaded {len(m.layers)} layers")
    return m


def load_pretrained(model_dir: str, device="cpu", dtype=torch.bfloat16, log=None) -> KinetarForCausalLM:
    return load(KinetarConfig.load_from_pretrained_dir(model_dir), model_dir, device, dtype, log)


def random_tensor(name: str, shape: Tuple[int, ...], gen: torch.Generator) -> torch.Tensor:
    """Random-init value of one checkpoint tensor (fp32)."""
    dev = gen.device
    last = name.rsplit(".", 1)[-1]
    uniform = lambda lo, hi: torch.rand(shape, generator=gen, device=dev) * (hi - lo) + lo
    if name.endswith("mix.norm") or last == "D":
        return torch.ones(shape, device=dev)
    if last in ("norm1", "norm", "sink") or name.endswith("conv.b"):
        return torch.zeros(shape, device=dev)
    if last == "A_log":
        return torch.log(uniform(0.05, 4.0))
    if last == "dt_bias" or name.endswith("dt.b"):
        return uniform(-4.0, -1.0)
    return torch.randn(shape, generator=gen, device=dev) * (1.0 if name == "embed" else shape[-1] ** -0.5)


def init(cfg: KinetarConfig, device="cpu", dtype=torch.float32, seed: int = 0, rank: Optional[int] = None) -> KinetarForCausalLM:
    """Random weights; ``rank`` of the low-rank projections (default: the key size)."""
    gen = torch.Generator(device=device).manual_seed(seed)
    shapes = tensor_shapes(cfg)

    def get(name):
        r = rank
        if r is None and None in shapes[name]:
            r = cfg.layers[int(name[1:name.index(".")])].mixer.dim
        return random_tensor(name, tuple(r if n is None else n for n in shapes[name]), gen).to(dtype)
    return build(cfg, get, device, dtype)


def state_dict(m: KinetarForCausalLM) -> Dict[str, torch.Tensor]:
    """Checkpoint-format tensors (inverse of ``load``)."""
    out = {"embed": m.embed, "head": m.head, **m.raw}
    for i, (s, l) in enumerate(zip(m.cfg.layers, m.layers)):
        p, x = f"l{i}.mix.", s.mixer
        rows = {n: l.w_in[l.cols[n]] for n in l.cols.at}
        outs = {n: l.w_out[:, l.act[n]] for n in l.act.at}
        out[f"l{i}.norm1"] = l.raw[f"l{i}.norm1"]
        if isinstance(x, ChannelDeltaSpec):
            d = l.mixer[0]
            ra, rg = l.raw["rank"].tolist()
            out.update({p + n: rows[n] for n in "qkvb"})
            out.update({f"{p}{n}.conv": t for n, t in d.conv.items()})
            out.update({p + "a1": rows["a1"][:ra], p + "g1": rows["g1"][:rg], p + "a2": d.w_a[:, :ra], p + "g2": d.w_g[:, :rg], p + "A_log": d.a_log,
                        p + "dt_bias": d.dt_bias, p + "norm": d.norm, p + "o": outs["mix"]})
        else:
            a, c = l.mixer
            out.update({f"{p}left.{n}": rows[n] for n in "qkg"})
            out.update({p + "left.q.conv": a.q_conv, p + "left.k.conv": a.k_conv, p + "left.sink": a.sink, p + "left.o": outs["left"]})
            y, r = p + "right.", x.right.dt_rank
            out.update({y + "in": torch.cat([rows["x"], rows["z"]]), y + "conv": c.conv, y + "conv.b": c.conv_b,
                        y + "x": torch.cat([c.w_x[c.proj["dt"]][:r], c.w_x[c.proj["b"]], c.w_x[c.proj["c"]]]), y + "dt": c.w_dt[:, :r],
                        y + "dt.b": c.dt_b, y + "A_log": l.raw[y + "A_log"], y + "D": c.d, y + "o": outs["right"]})
        if s.ff:
            out[f"l{i}.mlp.up"], out[f"l{i}.mlp.down"] = rows["up"], outs["up"]
    return {k: v.contiguous() for k, v in out.items()}


# ---- blocks -------------------------------------------------------------------------------------------------------
@dataclass
class MixerState:
    """What a layer carries from token to token."""
    kv: Optional[KVCache]
    lin: Tuple[LinearState, ...]          # parallel: queries' and keys' windows, then the scan; channel_delta: q, k, v windows and state


@dataclass
class Tokens:
    """The tokens of one pass: whole prompts (``lens`` where rows end earlier) or one token per row at ``pos``."""
    lens: Optional[torch.Tensor] = None
    pos: Optional[torch.Tensor] = None

    @property
    def step(self): return self.pos is not None


def _inputs(l: Layer, h: torch.Tensor, act: torch.Tensor, segments: List[Segment], t: Tokens) -> torch.Tensor:
    """Input projection and, in one launch, everything up to the mixers: convolutions, activations, stores.  For prompts the
    feed-forward's half of the product takes its activation in the product's epilogue and goes straight to ``act``."""
    if t.step:
        y = lin(h, l.w_in)
        if "up" in l.cols.at:
            segments = segments + [Segment(l.cols.at["up"], 1, l.cols.width["up"], act[..., l.act["up"]], act="relu2")]
        mix_step(y, segments, t.pos)
        return y
    n = l.cols.at.get("up", l.cols.total)
    y = project(h, l.w_in[:n])
    if "up" in l.cols.at:
        project(h, l.w_in[n:n + l.cols.width["up"]], act="relu2", out=act[..., l.act["up"]])
    mix_prompt(y, segments, t.lens)
    return y


def parallel_mixer(s: ParallelSpec, l: Layer, h: torch.Tensor, act: torch.Tensor, state: MixerState, t: Tokens) -> None:
    """Both mixers' gated and scaled outputs and the feed-forward's activations -> ``act``."""
    a, r, (left, right), at = s.left, s.right, l.mixer, l.cols.at
    B, S, _ = h.shape
    new = lambda *shape: torch.empty((B, S, *shape), device=h.device, dtype=h.dtype)
    d = state.kv.k.shape[3] if t.step else a.dim
    q, k, x = new(a.heads, d), new(a.kv_heads, d), new(r.inner)
    qs, ks, xs = state.lin
    y = _inputs(l, h, act, [
        Segment(at["q"], a.heads, a.dim, q.flatten(2), d, w=left.q_conv, window=qs.conv, temp=(a.temp_coef, a.temp_every)),
        Segment(at["k"], a.kv_heads, a.dim, k.flatten(2), d, w=left.k_conv, window=ks.conv, store=state.kv.k),
        Segment(at["x"], 1, r.inner, x, w=right.conv, bias=right.conv_b, window=xs.conv, act="silu")], t)
    kw = dict(scale=a.scale, sink=left.sink, gate=y[..., l.cols["g"]], out_scale=s.left_scale, out=act[..., l.act["left"]])
    if t.step:
        sa.step_attention(q, k, k, state.kv, t.pos, a.vdim, **kw)
    else:
        sa.prompt_attention(q, k, k, **kw)
    p = project(x, right.w_x)
    dt = project(p[..., right.proj["dt"]], right.w_dt)
    args = (x, dt, y[..., l.cols["z"]], p[..., right.proj["b"]], p[..., right.proj["c"]], right.a, right.d, right.dt_b, xs.rec, act[..., l.act["right"]])
    if t.step:
        ss.scan_step(*args, scale=s.right_scale)
    else:
        ss.scan_prompt(*args, lens=t.lens, scale=s.right_scale)


def channel_delta_mixer(s: ChannelDeltaSpec, l: Layer, h: torch.Tensor, act: torch.Tensor, state: MixerState, t: Tokens, eps: float) -> None:
    m, at = l.mixer[0], l.cols.at
    B, S, _ = h.shape
    heads = {"q": (s.kv_heads, s.dim), "k": (s.kv_heads, s.dim), "v": (s.heads, s.vdim)}
    bufs = {n: torch.empty((B, S, *hd), device=h.device, dtype=h.dtype) for n, hd in heads.items()}
    y = _inputs(l, h, act, [Segment(at[n], *heads[n], bufs[n].flatten(2), w=m.conv[n], window=w.conv, act="silu") for n, w in zip("qkv", state.lin)], t)
    a, z = project(y[..., l.cols["a1"]], m.w_a), project(y[..., l.cols["g1"]], m.w_g)
    args = (bufs["q"], bufs["k"], bufs["v"], a, y[..., l.cols["b"]])
    rec, out = state.lin[3].rec, act[..., l.act["mix"]]
    if t.step:
        dr.channel_delta_decode(*args, z, m.dt_bias, m.a_log, m.norm, m.norm_lp, eps, rec, out)
    else:
        dr.gated_norm(dr.channel_delta_prefill(*args, m.dt_bias, m.a_log, rec, t.lens), z, m.norm, eps, "sigmoid", out)


class CacheSession(HybridSession):
    """K stores of the attention mixers (their values are the keys: one store), convolution windows, scan and delta-rule states;
    ``retain`` gives finished rows back."""
    name = "Kinetar"

    def __init__(self, m: KinetarForCausalLM, batch: int, max_len: int):
        super().__init__(batch, max_len, m.device)
        self.m = m
        self.states: List[MixerState] = []
        window = lambda channels, taps: LinearState(torch.zeros((batch, channels, taps), device=m.device, dtype=m.dtype))
        f32 = lambda *shape: torch.zeros((batch, *shape), device=m.device)
        for l in m.cfg.layers:
            s = l.mixer
            if isinstance(s, ChannelDeltaSpec):
                kv = None
                states = (window(s.key_dim, s.conv), window(s.key_dim, s.conv), window(s.value_dim, s.conv), LinearState(rec=f32(s.heads, s.dim, s.vdim)))
            else:
                a, r = s.left, s.right
                d = sa.store_dim(a.heads, a.kv_heads, a.dim, m.dtype, m.device)
                kv = KVCache.allocate(batch, a.kv_heads, max_len, d, m.device, m.dtype, shared=True)
                scan = window(r.inner, r.conv)
                scan.rec = f32(r.inner, r.state)
                states = (window(a.heads * a.dim, a.conv), window(a.kv_heads * a.dim, a.conv), scan)
            self.kv.append(kv)
            self.lin.extend(states)
            self.states.append(MixerState(kv, states))

    def _forward(self, ids: torch.Tensor, t: Tokens, layer_done=None) -> torch.Tensor:
        """Residual stream (fp32) after all layers."""
        m, cfg = self.m, self.m.cfg
        B, S = ids.shape
        x = embed_positions(ids, m.embed, m.turns, cfg.embedding_scale, t.pos)
        h = add_norm(None, m.layers[0].gain, cfg.eps, x, m.dtype)
        for i, (s, l, state) in enumerate(zip(cfg.layers, m.layers, self.states)):
            act = l.act.buffer(B, S, m.device, m.dtype)
            if isinstance(s.mixer, ParallelSpec):
                parallel_mixer(s.mixer, l, h, act, state, t)
            else:
                channel_delta_mixer(s.mixer, l, h, act, state, t, cfg.eps)
            h = add_norm(lin(act, l.w_out), m.layers[i + 1].gain if i + 1 < len(m.layers) else m.gain, cfg.eps, x, m.dtype)
            if layer_done is not None:
                layer_done(i, x)
        return h

    @torch.no_grad()
    def hidden(self, ids: torch.Tensor, lengths: Optional[Sequence[int]] = None, layer_done=None) -> torch.Tensor:
        B, S = ids.shape
        if B != self.batch or S == 0 or self.pos > 0:
            raise ValueError("Kinetar prefills a fresh session with one prompt per row")
        lengths = [S] * B if lengths is None else [int(n) for n in lengths]
        if len(lengths) != B or min(lengths) < 1 or max(lengths) > S:
            raise ValueError("Kinetar prompt lengths must be between 1 and the padded length")
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
def forward(m: KinetarForCausalLM, input_ids: torch.Tensor, lengths: Optional[Sequence[int]] = None) -> torch.Tensor:
    """Logits [B, S, V] of whole sequences."""
    s = CacheSession(m, input_ids.shape[0], input_ids.shape[1])
    return s.head(s.hidden(input_ids, lengths))


def generate(m: KinetarForCausalLM, input_ids: torch.Tensor, max_new_tokens: int = 64, strategy: SamplingStrategy = SamplingStrategy(),
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
