"""Zatorax: hybrid decoder of gated delta-rule layers and sliding-window attention with a logarithmic distance penalty, group-limited
mixture of experts with a shared expert, norms with a single gain on the sublayers' outputs, fp32 residual stream.

    x += norm1(mix(x));   x += norm2(moe(x))

An attention layer may read the keys and values of an earlier one (``kv_from``): it has queries, window and penalty of its own and
no store.  Prompts run through the chunked delta-rule kernels and the flash kernel with the penalty table; a decode step through
the fused convolution / recurrence step, the split-KV kernel with a position per row, and one norm-and-add kernel per sublayer,
captured as a CUDA graph.  Rows of a batch may have prompts of different lengths (padded at the end).
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn.functional as F

from ..io import safetensors as st
from ..ops import biased_attention as ba
from ..ops import delta_rule as dr
from ..ops import moe as moe_ops
from ..ops.gemm import gemm
from ..ops.norm import post_norm_residual
from .common import TCGEN05_MIN_ROWS, KVCache, LinearState, lin, swiglu_mlp
from .generation import SamplingStrategy, StreamCallback, generate_cached
from .session import HybridSession

DELTA, ATTENTION = "delta", "attention"


# ---- configuration ------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class DeltaSpec:
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
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None          # keys a query sees, itself included
    kv_from: Optional[int] = None         # layer whose keys and values this one reads


@dataclass(frozen=True)
class MoeSpec:
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0


@dataclass(frozen=True)
class LayerSpec:
    mixer: object                         # DeltaSpec | AttentionSpec
    mlp: Optional[MoeSpec] = None


def _fields(j: dict, what: str, required: Sequence[str], optional: Sequence[str] = ()) -> dict:
    j = {k: v for k, v in j.items() if v is not None}
    missing = [k for k in required if k not in j]
    unknown = [k for k in j if k not in required and k not in optional]
    if missing or unknown:
        raise ValueError(f"Invalid Zatorax config: {what} " + "; ".join(
            [f"lacks {', '.join(missing)}"] * bool(missing) + [f"has unknown {', '.join(unknown)}"] * bool(unknown)))
    return j


@dataclass
class ZatoraxConfig:
    vocab: int
    width: int
    eps: float
    layers: List[LayerSpec]

    def __post_init__(self):
        e = lambda i, m: ValueError(f"Invalid Zatorax config: layer {i}: {m}")
        if min(self.vocab, self.width) <= 0 or not self.layers:
            raise ValueError("Invalid Zatorax config: vocab, width and the number of layers must be positive")
        for i, l in enumerate(self.layers):
            m = l.mixer
            if min(m.heads, m.kv_heads, m.dim, m.vdim) <= 0 or m.heads % m.kv_heads:
                raise e(i, "head counts and sizes must be positive and heads a multiple of kv_heads")
            if isinstance(m, DeltaSpec):
                if m.conv <= 0:
                    raise e(i, "the convolution needs at least one tap")
            else:
                if m.window is not None and m.window <= 0:
                    raise e(i, "mask.size must be positive")
                if m.kv_from is not None:
                    src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                    if not isinstance(src, AttentionSpec) or src.kv_from is not None:
                        raise e(i, "kv_from must name an earlier attention layer that has keys of its own")
                    if (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                        raise e(i, "kv_from must name a layer with the same kv_heads, dim and vdim")
            if l.mlp is not None:
                p = l.mlp
                if not (0 < p.top <= p.experts) or p.ff <= 0 or p.groups <= 0 or p.experts % p.groups or not (0 < p.keep <= p.groups):
                    raise e(i, "experts must split into equal groups and top, ff and keep be positive and within bounds")
                if p.top > p.keep * (p.experts // p.groups):
                    raise e(i, "top experts must fit the kept groups")

    def kv_users(self, i: int) -> List[AttentionSpec]:
        """The layers that read layer i's keys: itself and every layer with ``kv_from`` i."""
        return [l.mixer for k, l in enumerate(self.layers) if isinstance(l.mixer, AttentionSpec) and (k == i or l.mixer.kv_from == i)]

    def kv_reach(self, i: int) -> Optional[int]:
        """Positions layer i's store must hold back from the newest (None: all)."""
        w = [m.window for m in self.kv_users(i)]
        return None if None in w else max(w)

    @staticmethod
    def from_json(j: dict) -> "ZatoraxConfig":
        layers = []
        for i, l in enumerate(j["layers"]):
            kind = l.get("type")
            sizes = ("heads", "kv_heads", "dim", "vdim")
            if kind == DELTA:
                mixer = DeltaSpec(**_fields(l["mixer"], f"layer {i} mixer", (*sizes, "conv")))
            elif kind == ATTENTION:
                m = _fields(l["mixer"], f"layer {i} mixer", (*sizes, "scale"), ("mask", "kv_from"))
                mask = _fields(m.pop("mask"), f"layer {i} mask", ("size",)) if "mask" in m else {}
                mixer = AttentionSpec(**m, window=mask.get("size"))
            else:
                raise ValueError(f'Invalid Zatorax config: layer {i} has unknown type "{kind}"; expected {DELTA} or {ATTENTION}')
            mlp = None
            if l.get("mlp") is not None:
                p = _fields(l["mlp"], f"layer {i} mlp", ("kind", "expert", "router"), ("shared",))
                if p["kind"] != "moe":
                    raise ValueError(f'Invalid Zatorax config: layer {i} has unknown mlp kind "{p["kind"]}"; expected moe')
                r = _fields(p["router"], f"layer {i} router", ("experts", "top"), ("groups",))
                g = _fields(r["groups"], f"layer {i} groups", ("count", "keep")) if "groups" in r else {"count": 1, "keep": 1}
                shared = _fields(p["shared"], f"layer {i} shared expert", ("ff",))["ff"] if "shared" in p else 0
                mlp = MoeSpec(r["experts"], r["top"], _fields(p["expert"], f"layer {i} expert", ("ff",))["ff"], g["count"], g["keep"], shared)
            layers.append(LayerSpec(mixer, mlp))
        return ZatoraxConfig(int(j["vocab"]), int(j["width"]), float(j["norm"]["eps"]), layers)

    def to_json(self) -> dict:
        layers = []
        for l in self.layers:
            m = l.mixer
            mix = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim}
            if isinstance(m, DeltaSpec):
                kind, mix["conv"] = DELTA, m.conv
            else:
                kind, mix["scale"] = ATTENTION, m.scale
                if m.window is not None:
                    mix["mask"] = {"size": m.window}
                if m.kv_from is not None:
                    mix["kv_from"] = m.kv_from
            mlp = None
            if l.mlp is not None:
                p = l.mlp
                mlp = {"kind": "moe", "expert": {"ff": p.ff}, "router": {"experts": p.experts, "top": p.top}}
                if p.groups > 1:
                    mlp["router"]["groups"] = {"count": p.groups, "keep": p.keep}
                if p.shared_ff:
                    mlp["shared"] = {"ff": p.shared_ff}
            layers.append({"type": kind, "mixer": mix, "mlp": mlp})
        return {"architecture": "Zatorax", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": layers}

    @staticmethod
    def load_from_pretrained_dir(model_dir: str) -> "ZatoraxConfig":
        with open(os.path.join(model_dir, "config.json")) as f:
            return ZatoraxConfig.from_json(json.load(f))


# ---- parameters ---------------------------------------------------------------------------------------------------
@dataclass
class DeltaMixer:
    w_in: torch.Tensor            # [q | k | v | g | b | a] rows, padded to a multiple of 8
    conv: torch.Tensor            # [conv_dim, taps]: q, k, v channels
    a_log: torch.Tensor           # fp32 [heads]
    dt_bias: torch.Tensor         # fp32 [heads]
    norm: torch.Tensor            # [vdim]
    w_out: torch.Tensor


@dataclass
class AttentionMixer:
    w_in: torch.Tensor            # [q | k | v] rows (q alone with kv_from), padded to a multiple of 8
    q_norm: torch.Tensor          # fp32 [dim]
    k_norm: Optional[torch.Tensor]
    r1: torch.Tensor              # fp32 [heads]
    r2: torch.Tensor
    w_out: torch.Tensor           # [width, heads * vdim], vdim padded to the K/V store's row length


@dataclass
class Experts:
    router: torch.Tensor          # fp32 [E, width]
    router_lp: torch.Tensor       # the same in the compute dtype
    correction: torch.Tensor      # fp32 [E], added to the scores for the choice only
    bank: moe_ops.ExpertBank
    shared: Optional[Tuple[torch.Tensor, torch.Tensor, torch.Tensor]]    # gate, up, down


@dataclass
class Layer:
    mixer: object
    norm1: torch.Tensor           # fp32 [1]
    ffn: Optional[Experts]
    norm2: Optional[torch.Tensor]


@dataclass
class ZatoraxForCausalLM:
    cfg: ZatoraxConfig
    embed: torch.Tensor
    layers: List[Layer]
    norm: torch.Tensor            # fp32 [1]
    head: torch.Tensor

    @property
    def device(self): return self.embed.device
    @property
    def dtype(self): return self.embed.dtype


def tensor_shapes(cfg: ZatoraxConfig) -> Dict[str, Tuple[int, ...]]:
    """Checkpoint names and shapes."""
    h = cfg.width
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, h)}
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        out[p + "norm1"] = ()
        x = p + "mix."
        if isinstance(m, DeltaSpec):
            for n, d in (("q", m.key_dim), ("k", m.key_dim), ("v", m.value_dim)):
                out[x + n], out[x + n + ".conv"] = (d, h), (d, m.conv)
            out.update({x + "b": (m.heads, h), x + "A_log": (m.heads,), x + "norm": (m.vdim,), x + "a": (m.heads, h), x + "dt_bias": (m.heads,),
                        x + "g": (m.value_dim, h), x + "o": (h, m.value_dim)})
        else:
            out[x + "q"], out[x + "q.norm"] = (m.heads * m.dim, h), (m.dim,)
            if m.kv_from is None:
                out.update({x + "k": (m.kv_heads * m.dim, h), x + "v": (m.kv_heads * m.vdim, h), x + "k.norm": (m.dim,)})
            out.update({x + "r1": (m.heads,), x + "r2": (m.heads,), x + "o": (h, m.heads * m.vdim)})
        if l.mlp is not None:
            out[p + "norm2"] = ()
            x, s = p + "mlp.", l.mlp
            ffs = [(f"e{e}", s.ff) for e in range(s.experts)] + ([("shared", s.shared_ff)] if s.shared_ff else [])
            for n, ff in ffs:
                out.update({f"{x}{n}.gate": (ff, h), f"{x}{n}.up": (ff, h), f"{x}{n}.down": (h, ff)})
            out[x + "router"], out[x + "correction"] = (s.experts, h), (s.experts,)
    out["final.norm"], out["head"] = (), (cfg.vocab, h)
    return out


def _pad_rows(ws: Sequence[torch.Tensor]) -> torch.Tensor:
    w = torch.cat(list(ws), 0)
    return F.pad(w, (0, 0, 0, (-w.shape[0]) % 8)).contiguous()


def build(cfg: ZatoraxConfig, get, device="cpu", dtype=torch.bfloat16) -> ZatoraxForCausalLM:
    """Assemble the model from ``get(name) -> tensor`` (checkpoint names)."""
    shapes = tensor_shapes(cfg)

    def take(name, dt=dtype):
        t = get(name)
        if tuple(t.shape) != shapes[name]:
            raise st.SafeTensorsError(f"{name}: expected shape {list(shapes[name])}, got {list(t.shape)}")
        return t.to(device=device, dtype=dt)
    f32 = lambda name: take(name, torch.float32)
    one = lambda name: f32(name).reshape(1)
    layers = []
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.mix.", l.mixer
        if isinstance(m, DeltaSpec):
            mixer = DeltaMixer(_pad_rows([take(p + n) for n in "qkvgba"]), torch.cat([take(p + n + ".conv") for n in "qkv"], 0).contiguous(),
                               f32(p + "A_log"), f32(p + "dt_bias"), take(p + "norm"), take(p + "o"))
        else:
            own = m.kv_from is None
            _, dvp = ba.store_dims(m.heads, m.kv_heads, m.dim, m.vdim, dtype, device)
            wo = F.pad(take(p + "o").reshape(cfg.width, m.heads, m.vdim), (0, dvp - m.vdim)).reshape(cfg.width, -1).contiguous()
            mixer = AttentionMixer(_pad_rows([take(p + n) for n in ("qkv" if own else "q")]), f32(p + "q.norm"), f32(p + "k.norm") if own else None,
                                   f32(p + "r1"), f32(p + "r2"), wo)
        ffn = None
        if l.mlp is not None:
            p, s = f"l{i}.mlp.", l.mlp
            gu = torch.stack([torch.cat([take(f"{p}e{e}.gate"), take(f"{p}e{e}.up")], 0) for e in range(s.experts)])
            dn = torch.stack([take(f"{p}e{e}.down") for e in range(s.experts)])
            shared = tuple(take(f"{p}shared.{n}") for n in ("gate", "up", "down")) if s.shared_ff else None
            ffn = Experts(f32(p + "router"), take(p + "router"), f32(p + "correction"), moe_ops.ExpertBank(gu, dn), shared)
        layers.append(Layer(mixer, one(f"l{i}.norm1"), ffn, one(f"l{i}.norm2") if ffn is not None else None))
    return ZatoraxForCausalLM(cfg, take("embed"), layers, one("final.norm"), take("head"))


def load(cfg: ZatoraxConfig, source, device="cpu", dtype=torch.bfloat16, log=None) -> ZatoraxForCausalLM:
    """Load from a safetensors ``Source`` (file or directory)."""
    src = source if isinstance(source, st.Source) else st.Source.open(source)
    m = build(cfg, src.load, device, dtype)
    if log is not None:
        log(f"  loaded {len(m.layers)} layers")
    return m


def load_pretrained(model_dir: str, device="cpu", dtype=torch.bfloat16, log=None) -> ZatoraxForCausalLM:
    return load(ZatoraxConfig.load_from_pretrained_dir(model_dir), model_dir, device, dtype, log)


def random_tensor(name: str, shape: Tuple[int, ...], gen: torch.Generator) -> torch.Tensor:
    """Random-init value of one checkpoint tensor (fp32)."""
    dev = gen.device
    last = name.rsplit(".", 1)[-1]
    if last in ("norm", "norm1", "norm2"):
        return torch.ones(shape, device=dev)
    if last == "A_log":
        return torch.log(torch.rand(shape, generator=gen, device=dev) * 4.0 + 0.05)
    if last == "dt_bias":
        return torch.rand(shape, generator=gen, device=dev) * 3.0 - 4.0
    if last == "r1":
        return torch.rand(shape, generator=gen, device=dev) * 2.0
    if last == "r2":
        return torch.rand(shape, generator=gen, device=dev) * 0.5
    if last == "correction":
        return torch.randn(shape, generator=gen, device=dev) * 0.01
    return torch.randn(shape, generator=gen, device=dev) * (1.0 if name == "embed" else shape[-1] ** -0.5)


def init(cfg: ZatoraxConfig, device="cpu", dtype=torch.float32, seed: int = 0) -> ZatoraxForCausalLM:
    gen = torch.Generator(device=device).manual_seed(seed)
    shapes = tensor_shapes(cfg)
    return build(cfg, lambda n: random_tensor(n, shapes[n], gen).to(dtype), device, dtype)


def state_dict(m: ZatoraxForCausalLM) -> Dict[str, torch.Tensor]:
    """Checkpoint-format tensors (inverse of ``load``)."""
    cfg = m.cfg
    out = {"embed": m.embed, "final.norm": m.norm.reshape(()), "head": m.head}
    for i, (s, l) in enumerate(zip(cfg.layers, m.layers)):
        p, x = f"l{i}.mix.", s.mixer
        if isinstance(x, DeltaSpec):
            rows = dict(zip("qkvgba", torch.split(l.mixer.w_in[:x.conv_dim + x.value_dim + 2 * x.heads],
                                                  [x.key_dim, x.key_dim, x.value_dim, x.value_dim, x.heads, x.heads])))
            conv = dict(zip("qkv", torch.split(l.mixer.conv, [x.key_dim, x.key_dim, x.value_dim])))
            out.update({p + n: t for n, t in rows.items()})
            out.update({f"{p}{n}.conv": t for n, t in conv.items()})
            out.update({p + "A_log": l.mixer.a_log, p + "dt_bias": l.mixer.dt_bias, p + "norm": l.mixer.norm, p + "o": l.mixer.w_out})
        else:
            hq, hk, hv = x.heads * x.dim, x.kv_heads * x.dim, x.kv_heads * x.vdim
            out[p + "q"], out[p + "q.norm"] = l.mixer.w_in[:hq], l.mixer.q_norm
            if x.kv_from is None:
                out[p + "k"], out[p + "v"], out[p + "k.norm"] = l.mixer.w_in[hq:hq + hk], l.mixer.w_in[hq + hk:hq + hk + hv], l.mixer.k_norm
            out[p + "r1"], out[p + "r2"] = l.mixer.r1, l.mixer.r2
            out[p + "o"] = l.mixer.w_out.reshape(cfg.width, x.heads, -1)[..., :x.vdim].reshape(cfg.width, -1)
        out[f"l{i}.norm1"] = l.norm1.reshape(())
        if l.ffn is not None:
            out[f"l{i}.norm2"] = l.norm2.reshape(())
            p, gu, dn = f"l{i}.mlp.", l.ffn.bank.gate_up, l.ffn.bank.down
            for e in range(gu.shape[0]):
                out[f"{p}e{e}.gate"], out[f"{p}e{e}.up"] = gu[e].chunk(2, 0)
                out[f"{p}e{e}.down"] = dn[e]
            out[p + "router"], out[p + "correction"] = l.ffn.router_lp, l.ffn.correction
            if l.ffn.shared is not None:
                out.update({f"{p}shared.{n}": t for n, t in zip(("gate", "up", "down"), l.ffn.shared)})
    return {k: v.contiguous() for k, v in out.items()}


# ---- blocks -------------------------------------------------------------------------------------------------------
def _delta_parts(s: DeltaSpec, y: torch.Tensor):
    """(conv input q|k|v, output gate, b, a) windows of a delta layer's input projection."""
    c, v = s.conv_dim, s.value_dim
    return y[..., :c], y[..., c:c + v], y[..., c + v:c + v + s.heads], y[..., c + v + s.heads:c + v + 2 * s.heads]


def delta_prompt(s: DeltaSpec, m: DeltaMixer, h: torch.Tensor, eps: float, state: LinearState, lens: Optional[torch.Tensor]) -> torch.Tensor:
    B, S, _ = h.shape
    mixed, z, b, a = _delta_parts(s, lin(h, m.w_in))
    y = dr.causal_conv1d_silu(mixed, m.conv)
    state.conv.copy_(dr.conv_window(mixed, s.conv, lens))
    g, beta = dr.delta_gates(b, a, m.dt_bias, m.a_log)
    q, k, v = (t.reshape(B, S, n, -1) for t, n in zip(torch.split(y, [s.key_dim, s.key_dim, s.value_dim], -1), (s.kv_heads, s.kv_heads, s.heads)))
    o = dr.delta_prefill(q, k, v, g, beta, state.rec, lens)
    return lin(dr.gated_norm(o, z, m.norm.float(), eps), m.w_out)


def delta_step(s: DeltaSpec, m: DeltaMixer, h: torch.Tensor, eps: float, state: LinearState) -> torch.Tensor:
    mixed, z, b, a = _delta_parts(s, lin(h, m.w_in))
    return lin(dr.delta_decode(mixed, z, b, a, state.conv, m.conv, m.dt_bias, m.a_log, m.norm, eps, state.rec, s.kv_heads, s.heads, s.dim, s.vdim),
               m.w_out)


def _project_qkv(s: AttentionSpec, m: AttentionMixer, h, eps, store=None, lens=None):
    dkp, dvp = ba.store_dims(s.heads, s.kv_heads, s.dim, s.vdim, h.dtype, h.device)
    return ba.qk_norm_store(lin(h, m.w_in), m.q_norm, m.k_norm, s.heads, 0 if m.k_norm is None else s.kv_heads, s.dim, s.vdim, eps,
                            dkp=dkp, dvp=dvp, store=store, lens=lens)


def attention_prompt(s: AttentionSpec, m: AttentionMixer, h, eps, store: Optional[KVCache], lens, shared):
    """``shared``: keys and values of the layer named by ``kv_from``.  Returns (output, keys, values)."""
    q, k, v = _project_qkv(s, m, h, eps, store, lens)
    if s.kv_from is not None:
        k, v = shared
    o = ba.prompt_attention(q, k, v, m.r1, m.r2, window=s.window, scale=s.scale)
    return lin(o.flatten(2), m.w_out), k, v


def attention_step(s: AttentionSpec, m: AttentionMixer, h, eps, store: KVCache, pos: torch.Tensor, shared):
    q, k, v = _project_qkv(s, m, h, eps)
    if s.kv_from is not None:
        k, v = shared
    o = ba.step_attention(q, k, v, store, pos, m.r1, m.r2, window=s.window, scale=s.scale, append=s.kv_from is None)
    return lin(o.flatten(2), m.w_out), k, v


def route(s: MoeSpec, m: Experts, x2: torch.Tensor):
    """Softmax over all experts in fp32, group-limited choice on corrected scores, weights the plain scores."""
    kw = dict(softmax=True, bias=m.correction, renorm=False, groups=s.groups, keep=s.keep)
    if moe_ops.route_fused_supported(x2, m.router):
        return moe_ops.route_fused(x2, m.router, s.top, **kw)
    if x2.is_cuda and x2.dtype == torch.bfloat16 and x2.shape[0] >= TCGEN05_MIN_ROWS and s.experts % 8 == 0 and x2.shape[1] % 8 == 0:
        logits = gemm(x2, m.router_lp, out_dtype=torch.float32)       # bf16 operands are exact here: fp32 sums of fp32 products
    else:
        logits = F.linear(x2.float(), m.router)
    return moe_ops.route(logits, s.top, **kw)


def experts_forward(s: MoeSpec, m: Experts, h: torch.Tensor) -> torch.Tensor:
    x2 = h.reshape(-1, h.shape[-1])
    ids, w, counts = route(s, m, x2)
    shared = swiglu_mlp(x2, *m.shared) if m.shared is not None else None
    return moe_ops.moe_bank_forward(x2, ids, w, m.bank, counts=counts, add=shared).reshape(h.shape)


class CacheSession(HybridSession):
    """K/V stores of the layers with keys of their own (ring stores of the widest window that reads them) and convolution /
    recurrent states of the delta layers; ``retain`` gives finished rows back."""
    name = "Zatorax"

    def __init__(self, m: ZatoraxForCausalLM, batch: int, max_len: int):
        super().__init__(batch, max_len, m.device)
        self.m = m
        for i, l in enumerate(m.cfg.layers):
            s = l.mixer
            kv = state = None
            if isinstance(s, DeltaSpec):
                state = LinearState(torch.zeros((batch, s.conv_dim, s.conv), device=m.device, dtype=m.dtype),
                                    torch.zeros((batch, s.heads, s.dim, s.vdim), device=m.device, dtype=torch.float32))
            elif s.kv_from is None:
                reach = m.cfg.kv_reach(i)
                ring = reach is not None and reach < max_len
                dkp, dvp = ba.store_dims(s.heads, s.kv_heads, s.dim, s.vdim, m.dtype, m.device)
                kv = KVCache.allocate(batch, s.kv_heads, reach if ring else max_len, dkp, m.device, m.dtype, ring=ring, v_dim=dvp)
            self.kv.append(kv)
            self.lin.append(state)

    def _forward(self, ids: torch.Tensor, mix, layer_done=None) -> torch.Tensor:
        """Residual stream (fp32) after all layers.  ``mix(i, h, shared) -> (y, k, v)`` runs layer i's mixer."""
        m, cfg = self.m, self.m.cfg
        h = F.embedding(ids, m.embed)
        x = h.float() if h.dtype != torch.float32 else h
        keys: Dict[int, Tuple[torch.Tensor, torch.Tensor]] = {}
        for i, (s, l) in enumerate(zip(cfg.layers, m.layers)):
            src = getattr(s.mixer, "kv_from", None)
            y, k, v = mix(i, h, keys.get(src))
            if k is not None and src is None and len(cfg.kv_users(i)) > 1:
                keys[i] = (k, v)
            h = post_norm_residual(y, l.norm1, cfg.eps, x, m.dtype)
            if l.ffn is not None:
                h = post_norm_residual(experts_forward(s.mlp, l.ffn, h), l.norm2, cfg.eps, x, m.dtype)
            if layer_done is not None:
                layer_done(i, x)
        return x

    @torch.no_grad()
    def hidden(self, ids: torch.Tensor, lengths: Optional[Sequence[int]] = None, layer_done=None) -> torch.Tensor:
        B, S = ids.shape
        if B != self.batch or S == 0 or self.pos > 0:
            raise ValueError("Zatorax prefills a fresh session with one prompt per row")
        lengths = [S] * B if lengths is None else [int(n) for n in lengths]
        if len(lengths) != B or min(lengths) < 1 or max(lengths) > S:
            raise ValueError("Zatorax prompt lengths must be between 1 and the padded length")
        self._check_room(max(lengths))
        lens = None if min(lengths) == S else torch.tensor(lengths, dtype=torch.int32, device=self.device)
        cfg = self.m.cfg

        def mix(i, h, shared):
            s, p = cfg.layers[i].mixer, self.m.layers[i].mixer
            if isinstance(s, DeltaSpec):
                return delta_prompt(s, p, h, cfg.eps, self.lin[i], lens), None, None
            return attention_prompt(s, p, h, cfg.eps, self.kv[i], lens, shared)
        x = self._forward(ids, mix, layer_done)
        self._advance(lengths)
        return post_norm_residual(x, self.m.norm, cfg.eps, out_dtype=self.m.dtype)

    def head(self, h: torch.Tensor) -> torch.Tensor:
        return lin(h, self.m.head)

    # -- decode ----------------------------------------------------------------------------------------------------
    def device_step_supported(self) -> bool:
        return True

    def graph_supported(self) -> bool:
        m = self.m
        grouped = all(l.ffn is None or moe_ops.grouped_supported(m.embed, l.ffn.bank.moe_int) for l in m.layers)
        return super().graph_supported() and m.embed.is_cuda and m.dtype == torch.bfloat16 and grouped

    def _positions(self) -> torch.Tensor:
        return torch.tensor(self.lengths, dtype=torch.int32, device=self.device)

    def _device_step(self, tok: torch.Tensor) -> torch.Tensor:
        cfg = self.m.cfg

        def mix(i, h, shared):
            s, p = cfg.layers[i].mixer, self.m.layers[i].mixer
            if isinstance(s, DeltaSpec):
                return delta_step(s, p, h, cfg.eps, self.lin[i]), None, None
            store = self.kv[i if s.kv_from is None else s.kv_from]
            return attention_step(s, p, h, cfg.eps, store, self.pos_t, shared)
        x = self._forward(tok.reshape(-1, 1), mix)
        self.pos_t += 1
        return self.head(post_norm_residual(x[:, -1], self.m.norm, cfg.eps, out_dtype=self.m.dtype))


# ---- whole sequences and generation -------------------------------------------------------------------------------
@torch.no_grad()
def forward(m: ZatoraxForCausalLM, input_ids: torch.Tensor, lengths: Optional[Sequence[int]] = None) -> torch.Tensor:
    """Logits [B, S, V] of whole sequences."""
    s = CacheSession(m, input_ids.shape[0], input_ids.shape[1])
    return s.head(s.hidden(input_ids, lengths))


def generate(m: ZatoraxForCausalLM, input_ids: torch.Tensor, max_new_tokens: int = 64, strategy: SamplingStrategy = SamplingStrategy(),
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
