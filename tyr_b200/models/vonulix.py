"""Vonulix: windowed-attention decoder with an input of every layer by token and an average over depth, fp32 residual stream:

    x += attention(norm1(x));   x += experts(norm2(x));   X_{i+1} = x + norm(proj(gelu(gate x) * e_i[token]));   x = sum_{j <= i+1} a_ij X_j

X_0 is the embedding output; norms have the gain 1 + w.  Attention sees a sliding window and the first positions, its values are
unit-normed and rotated by their positions (the outputs are turned back), every head has an output gate.  Experts take the token times its
sigmoid score; a shared expert is gated by one number per token.

A layer is: one product for queries, keys, values and gates; rotation, value norm and store in one launch; attention, which turns
back and gates; the output product; residual add and norm; routing (the shared expert's gate is one more row of the router); the experts' two
products (a few tokens: weight-streaming, the shared expert in the same launches); the sum of the experts into the stream; the token
input's two products (activation and embedding in the first one's epilogue); and norm, add, depth average and the next norm in one launch.
The decode step is captured as a CUDA graph.  Rows of a batch may have prompts of different lengths (padded at the end)."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn.functional as F

from ..io import safetensors as st
from ..ops import kept_attention as ka
from ..ops import moe as moe_ops
from ..ops.depth import depth_average
from ..ops.embed import embed_positions
from ..ops.gates import gelu_mul_project
from ..ops.gemm import gemm
from ..ops.norm import add_norm, sandwich_norm
from .common import KVCache, TCGEN05_MIN_ROWS, config_fields, lin
from .generation import SamplingStrategy, StreamCallback, generate_cached
from .session import HybridSession

ATTENTION = "attention"
GATE_SLOPE = 1.702                        # of the experts' gate


def _up(n: int, multiple: int) -> int:
    return -(-n // multiple) * multiple


# ---- configuration ------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int
    rot_factor: float = 1.0               # divides the frequencies of queries and keys
    window: Optional[int] = None          # keys a query sees, itself included
    keep: int = 0                         # first positions that stay visible


@dataclass(frozen=True)
class MoeSpec:
    experts: int
    top: int
    ff: int
    limit: float
    shared_ff: int = 0                    # 0: no shared expert
    shared_limit: float = 0.0


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec
    mlp: Optional[MoeSpec] = None


@dataclass
class VonulixConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    side_dim: int                         # channels of a layer's token input
    layers: List[LayerSpec]

    def __post_init__(self):
        e = lambda i, m: ValueError(f"Invalid Vonulix config: layer {i}: {m}")
        if min(self.vocab, self.width, self.side_dim) <= 0 or not self.layers:
            raise ValueError("Invalid Vonulix config: vocab, width, token_side.dim and the number of layers must be positive")
        for i, l in enumerate(self.layers):
            m, p = l.mixer, l.mlp
            if min(m.heads, m.kv_heads, m.dim, m.vdim) <= 0 or m.heads % m.kv_heads:
                raise e(i, "head counts and sizes must be positive and heads a multiple of kv_heads")
            if m.rot_dims % 2 or not 0 <= m.rot_dims <= m.dim or m.vdim % 2:
                raise e(i, "rot.dims and vdim must be even and rot.dims at most dim")
            if m.rot_factor <= 0 or m.rot_base <= 0:
                raise e(i, "rot.base and rot.scaling.factor must be positive")
            if (m.window is not None and m.window <= 0) or m.keep < 0:
                raise e(i, "mask.size must be positive and mask.keep_first not negative")
            if p is not None:
                if not 0 < p.top <= p.experts or p.ff <= 0 or p.shared_ff < 0:
                    raise e(i, "top must lie between 1 and the number of experts and ff be positive")

    @staticmethod
    def from_json(j: dict) -> "VonulixConfig":
        fields = lambda *a: config_fields("Vonulix", *a)
        layers = []
        for i, l in enumerate(j["layers"]):
            if l.get("type") != ATTENTION:
                raise ValueError(f'Invalid Vonulix config: layer {i} has unknown type "{l.get("type")}"; expected {ATTENTION}')
            m = fields(l["mixer"], f"layer {i} mixer", ("heads", "kv_heads", "dim", "vdim", "scale", "rot"), ("mask",))
            rot = fields(m.pop("rot"), f"layer {i} rot", ("base", "dims"), ("scaling",))
            factor = fields(rot["scaling"], f"layer {i} rot.scaling", ("factor",))["factor"] if "scaling" in rot else 1.0
            mask = fields(m.pop("mask"), f"layer {i} mask", ("size",), ("keep_first",)) if "mask" in m else {}
            mixer = AttentionSpec(**m, rot_base=float(rot["base"]), rot_dims=rot["dims"], rot_factor=float(factor), window=mask.get("size"),
                                  keep=mask.get("keep_first", 0))
            mlp = None
            if l.get("mlp") is not None:
                p = fields(l["mlp"], f"layer {i} mlp", ("kind", "expert", "router"), ("shared",))
                if p["kind"] != "moe":
                    raise ValueError(f'Invalid Vonulix config: layer {i} has unknown mlp kind "{p["kind"]}"; expected moe')
                r = fields(p["router"], f"layer {i} router", ("experts", "top"))
                x = fields(p["expert"], f"layer {i} expert", ("ff", "limit"))
                s = fields(p["shared"], f"layer {i} shared expert", ("ff", "limit")) if "shared" in p else {"ff": 0, "limit": 0.0}
                mlp = MoeSpec(r["experts"], r["top"], x["ff"], float(x["limit"]), s["ff"], float(s["limit"]))
            layers.append(LayerSpec(mixer, mlp))
        return VonulixConfig(int(j["vocab"]), int(j["width"]), float(j["norm"]["eps"]), float(j["embedding"]["scale"]), int(j["token_side"]["dim"]), layers)

    def to_json(self) -> dict:
        layers = []
        for l in self.layers:
            m, p = l.mixer, l.mlp
            mix = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                   "rot": {"base": m.rot_base, "dims": m.rot_dims, "scaling": {"factor": m.rot_factor}}}
            if m.window is not None:
                mix["mask"] = {"size": m.window, "keep_first": m.keep}
            mlp = None
            if p is not None:
                mlp = {"kind": "moe", "expert": {"ff": p.ff, "limit": p.limit}, "router": {"experts": p.experts, "top": p.top}}
                if p.shared_ff:
                    mlp["shared"] = {"ff": p.shared_ff, "limit": p.shared_limit}
            layers.append({"type": ATTENTION, "mixer": mix, "mlp": mlp})
        return {"architecture": "Vonulix", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "embedding": {"scale": self.embed_scale},
                "token_side": {"dim": self.side_dim}, "layers": layers}

    @staticmethod
    def load_from_pretrained_dir(model_dir: str) -> "VonulixConfig":
        with open(os.path.join(model_dir, "config.json")) as f:
            return VonulixConfig.from_json(json.load(f))


# ---- parameters ---------------------------------------------------------------------------------------------------
class Norm:
    """A norm's weight, stored around zero, and its gain (fp32)."""

    def __init__(self, w: torch.Tensor):
        self.w, self.gain = w, 1.0 + w


@dataclass
class Attention:
    w_in: torch.Tensor            # [q | k | v | g] rows, padded to a multiple of 8
    w_out: torch.Tensor


@dataclass
class Experts:
    router: torch.Tensor          # fp32 [E (+ 1), width]: the last row is the shared expert's gate
    router_lp: torch.Tensor       # the same in the compute dtype, padded to a multiple of 8 rows
    bank: moe_ops.ExpertBank
    form: moe_ops.ClampedExpert
    shared: Optional[moe_ops.ExpertBank]
    shared_form: Optional[moe_ops.ClampedExpert]


@dataclass
class Layer:
    norm1: Norm
    mixer: Attention
    norm2: Optional[Norm]
    ffn: Optional[Experts]
    side_gate: torch.Tensor
    side_proj: torch.Tensor
    side_norm: torch.Tensor       # fp32 [width]
    depth: torch.Tensor           # fp32 [layer + 2]


@dataclass
class VonulixForCausalLM:
    cfg: VonulixConfig
    embed: torch.Tensor
    side_embed: torch.Tensor      # [vocab, layers * side_dim]
    layers: List[Layer]
    norm: Norm
    head: torch.Tensor

    def __post_init__(self):
        self._turns: Dict[Tuple[int, float, float], torch.Tensor] = {}

    @property
    def device(self): return self.embed.device
    @property
    def dtype(self): return self.embed.dtype

    def turns(self, dims: int, base: float, factor: float, positions: int) -> Optional[torch.Tensor]:
        """The rotation table of at least that many positions; layers with the same constants share one."""
        key = (dims, base, factor)
        t = self._turns.get(key)
        if dims and (t is None or t.shape[0] < positions):
            t = self._turns[key] = ka.turn_table(dims, base, factor, positions, self.device)
        return t


def tensor_shapes(cfg: VonulixConfig) -> Dict[str, Tuple[int, ...]]:
    """Checkpoint names and shapes."""
    h, sd = cfg.width, cfg.side_dim
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, h), "side.embed": (cfg.vocab, len(cfg.layers) * sd)}
    for i, l in enumerate(cfg.layers):
        p, m, s = f"l{i}.", l.mixer, l.mlp
        x = p + "mix."
        out.update({p + "norm1": (h,), x + "q": (m.heads * m.dim, h), x + "k": (m.kv_heads * m.dim, h), x + "v": (m.kv_heads * m.vdim, h), x + "g": (m.heads, h),
                    x + "o": (h, m.heads * m.vdim)})
        if s is not None:
            x, out[p + "norm2"] = p + "mlp.", (h,)
            for n, ff in [(f"e{e}", s.ff) for e in range(s.experts)] + [("shared", s.shared_ff)] * bool(s.shared_ff):
                out.update({f"{x}{n}.gate": (ff, h), f"{x}{n}.up": (ff, h), f"{x}{n}.down": (h, ff)})
            out[x + "router"] = (s.experts, h)
            if s.shared_ff:
                out[x + "shared.sg"] = (1, h)
        out.update({p + "side.gate": (sd, h), p + "side.proj": (h, sd), p + "side.norm": (h,), p + "dwa": (i + 2,)})
    out["final.norm"], out["head"] = (h,), (cfg.vocab, h)
    return out


def _rows(ws: Sequence[torch.Tensor]) -> torch.Tensor:
    w = torch.cat(list(ws), 0)
    return F.pad(w, (0, 0, 0, -w.shape[0] % 8)).contiguous()


def build(cfg: VonulixConfig, get: Callable[[str], torch.Tensor], device="cpu", dtype=torch.bfloat16) -> VonulixForCausalLM:
    """Assemble the model from ``get(name) -> tensor`` (checkpoint names)."""
    shapes = tensor_shapes(cfg)

    def take(name, dt=dtype):
        t = get(name)
        if tuple(t.shape) != shapes[name]:
            raise st.SafeTensorsError(f"{name}: expected shape {list(shapes[name])}, got {list(t.shape)}")
        return t.to(device=device, dtype=dt)
    f32 = lambda name: take(name, torch.float32).contiguous()

    def bank(names):
        return moe_ops.ExpertBank(torch.stack([torch.cat([take(n + ".gate"), take(n + ".up")], 0) for n in names]), torch.stack([take(n + ".down") for n in names]))
    layers = []
    for i, l in enumerate(cfg.layers):
        p, s = f"l{i}.", l.mlp
        ffn = None
        if s is not None:
            x = p + "mlp."
            router = torch.cat([f32(x + "router")] + ([f32(x + "shared.sg")] if s.shared_ff else []))
            ffn = Experts(router, _rows([router.to(dtype)]), bank([f"{x}e{e}" for e in range(s.experts)]), moe_ops.ClampedExpert(s.limit, GATE_SLOPE),
                          bank([x + "shared"]) if s.shared_ff else None, moe_ops.ClampedExpert(s.shared_limit, GATE_SLOPE) if s.shared_ff else None)
        layers.append(Layer(Norm(f32(p + "norm1")), Attention(_rows([take(f"{p}mix.{n}") for n in "qkvg"]), take(p + "mix.o").contiguous()),
                            Norm(f32(p + "norm2")) if s is not None else None, ffn, take(p + "side.gate").contiguous(), take(p + "side.proj").contiguous(),
                            f32(p + "side.norm"), f32(p + "dwa")))
    return VonulixForCausalLM(cfg, take("embed").contiguous(), take("side.embed").contiguous(), layers, Norm(f32("final.norm")), take("head").contiguous())


def load(cfg: VonulixConfig, source, device="cpu", dtype=torch.bfloat16, log=None) -> VonulixForCausalLM:
    """Load from a safetensors ``Source`` (file or directory)."""
    src = source if isinstance(source, st.Source) else st.Source.open(source)
    m = build(cfg, src.load, device, dtype)
    if log is not None:
        log(f"  loaded {len(m.layers)} layers")
    return m


def load_pretrained(model_dir: str, device="cpu", dtype=torch.bfloat16, log=None) -> VonulixForCausalLM:
    return load(VonulixConfig.load_from_pretrained_dir(model_dir), model_dir, device, dtype, log)


def random_tensor(name: str, shape: Tuple[int, ...], gen: torch.Generator) -> torch.Tensor:
    """Random-init value of one checkpoint tensor (fp32): norms at one, every layer's average at its own result."""
    dev = gen.device
    last = name.rsplit(".", 1)[-1]
    if last == "dwa":
        return F.pad(torch.ones(1, device=dev), (shape[0] - 1, 0))
    if name.endswith("side.norm"):
        return torch.ones(shape, device=dev)
    if "norm" in last:
        return torch.zeros(shape, device=dev)
    return torch.randn(shape, generator=gen, device=dev) * (1.0 if name in ("embed", "side.embed") else shape[-1] ** -0.5)


def init(cfg: VonulixConfig, device="cpu", dtype=torch.float32, seed: int = 0) -> VonulixForCausalLM:
    gen = torch.Generator(device=device).manual_seed(seed)
    shapes = tensor_shapes(cfg)
    return build(cfg, lambda n: random_tensor(n, shapes[n], gen).to(dtype), device, dtype)


def state_dict(m: VonulixForCausalLM) -> Dict[str, torch.Tensor]:
    """Checkpoint-format tensors (inverse of ``load``)."""
    out = {"embed": m.embed, "side.embed": m.side_embed, "final.norm": m.norm.w, "head": m.head}

    def experts(names, bank):
        gu, dn = bank.gate_up, bank.down
        for e, n in enumerate(names):
            out[n + ".gate"], out[n + ".up"] = gu[e].chunk(2, 0)
            out[n + ".down"] = dn[e]
    for i, (s, l) in enumerate(zip(m.cfg.layers, m.layers)):
        p, x = f"l{i}.", s.mixer
        sizes = [x.heads * x.dim, x.kv_heads * x.dim, x.kv_heads * x.vdim, x.heads]
        out.update({f"{p}mix.{n}": t for n, t in zip("qkvg", torch.split(l.mixer.w_in[:sum(sizes)], sizes))})
        out.update({p + "mix.o": l.mixer.w_out, p + "norm1": l.norm1.w, p + "side.gate": l.side_gate, p + "side.proj": l.side_proj, p + "side.norm": l.side_norm,
                    p + "dwa": l.depth})
        if l.ffn is not None:
            f, E = l.ffn, s.mlp.experts
            out[p + "norm2"], out[p + "mlp.router"] = l.norm2.w, f.router[:E]
            experts([f"{p}mlp.e{e}" for e in range(E)], f.bank)
            if f.shared is not None:
                experts([p + "mlp.shared"], f.shared)
                out[p + "mlp.shared.sg"] = f.router[E:]
    return {k: v.contiguous() for k, v in out.items()}


# ---- blocks -------------------------------------------------------------------------------------------------------
@dataclass
class Tokens:
    """The tokens of one pass: whole prompts (``lens`` where rows end earlier) or one token per row at ``pos``."""
    lens: Optional[torch.Tensor] = None
    pos: Optional[torch.Tensor] = None

    @property
    def step(self): return self.pos is not None


def attention_mixer(s: AttentionSpec, m: Attention, h: torch.Tensor, store: KVCache, tables, t: Tokens, eps: float) -> torch.Tensor:
    """``tables``: turns of queries and keys, and of values."""
    y = lin(h, m.w_in)
    n = (s.heads + s.kv_heads) * s.dim + s.kv_heads * s.vdim
    gate = y[..., n:n + s.heads]
    q, k, v = ka.rotary_store(y, s.heads, s.kv_heads, s.dim, s.vdim, *tables, eps, store=store, pos=t.pos, lens=t.lens)
    kw = dict(scale=s.scale, window=s.window, keep=s.keep, head_gate=gate, back=tables[1])
    o = ka.step_attention(q, store, t.pos, s.dim, s.vdim, **kw) if t.step else ka.prompt_attention(q, k, v, **kw)
    return lin(o, m.w_out)


def route(s: MoeSpec, m: Experts, x2: torch.Tensor):
    """(experts, their sigmoid scores, rows per expert, logits with the shared expert's gate in the last column)."""
    kw = dict(softmax=False, renorm=False, experts=s.experts)
    if moe_ops.route_fused_supported(x2, m.router):
        return moe_ops.route_fused(x2, m.router, s.top, want_logits=True, **kw)
    if x2.is_cuda and x2.dtype == torch.bfloat16 and x2.shape[0] >= TCGEN05_MIN_ROWS and x2.shape[1] % 8 == 0:
        logits = gemm(x2, m.router_lp, out_dtype=torch.float32)       # bf16 operands are exact here: fp32 sums of fp32 products
    else:
        logits = F.linear(x2.float(), m.router)
    return (*moe_ops.route(logits, s.top, **kw), logits)


def experts_into(s: MoeSpec, m: Experts, h: torch.Tensor, x: torch.Tensor) -> torch.Tensor:
    """Adds the experts' output for h to the stream x; the stream in h's dtype."""
    h2 = h.reshape(-1, h.shape[-1])
    ids, w, counts, logits = route(s, m, h2)
    gate = logits[:, s.experts] if m.shared is not None else None
    return moe_ops.weighted_input_experts(h2, ids, w, m.bank, m.form, x.view(h2.shape), shared=m.shared, shared_form=m.shared_form, shared_gate=gate,
                                          counts=counts).reshape(h.shape)


class CacheSession(HybridSession):
    """A K/V store per layer: plain, or where the window is shorter than the session a ring behind the kept first positions; ``retain`` gives
    finished rows back."""
    name = "Vonulix"

    def __init__(self, m: VonulixForCausalLM, batch: int, max_len: int):
        super().__init__(batch, max_len, m.device)
        self.m = m
        self.tables = []
        for l in m.cfg.layers:
            s = l.mixer
            ring = s.window is not None and s.keep + s.window < max_len
            dkp, dvp = ka.step_dims(s.heads, s.kv_heads, s.dim, s.vdim, m.dtype, m.device)
            self.kv.append(KVCache.allocate(batch, s.kv_heads, s.keep + s.window if ring else max_len, dkp, m.device, m.dtype, ring=ring, v_dim=dvp,
                                            keep=s.keep if ring else 0))
            self.tables.append((m.turns(s.rot_dims, s.rot_base, s.rot_factor, max_len), m.turns(s.vdim, s.rot_base, 1.0, max_len)))

    def _forward(self, ids: torch.Tensor, t: Tokens, layer_done=None) -> torch.Tensor:
        """Normed hidden states after all layers."""
        m, cfg, eps, dt = self.m, self.m.cfg, self.m.cfg.eps, self.m.dtype
        L, sd = len(m.layers), cfg.side_dim
        history = torch.empty((L, *ids.shape, cfg.width), dtype=torch.float32, device=ids.device)       # the results X_0 .. X_{L-1}
        embed_positions(ids, m.embed, None, cfg.embed_scale, out=history[0])
        x = torch.empty_like(history[0])
        h = sandwich_norm(history[0], None, m.layers[0].norm1.gain, eps, x, dt, replace=True)
        side = F.embedding(ids, m.side_embed).flatten(0, 1)
        for i, (s, l) in enumerate(zip(cfg.layers, m.layers)):
            y = attention_mixer(s.mixer, l.mixer, h, self.kv[i], self.tables[i], t, eps)
            if l.ffn is not None:
                out = experts_into(s.mlp, l.ffn, add_norm(y, l.norm2.gain, eps, x, dt), x)
            else:
                out = sandwich_norm(y, None, None, eps, x, dt)
            g = gelu_mul_project(out.flatten(0, 1), l.side_gate, side[:, i * sd:(i + 1) * sd])
            y = lin(g, l.side_proj).view(x.shape)
            nxt = m.layers[i + 1].norm1 if i + 1 < L else m.norm
            h = depth_average(y, l.side_norm, x, history, i + 1, l.depth, nxt.gain, eps, dt, store=i + 1 < L)
            if layer_done is not None:
                layer_done(i, x)
        return h

    @torch.no_grad()
    def hidden(self, ids: torch.Tensor, lengths: Optional[Sequence[int]] = None, layer_done=None) -> torch.Tensor:
        B, S = ids.shape
        if B != self.batch or S == 0 or self.pos > 0:
            raise ValueError("Vonulix prefills a fresh session with one prompt per row")
        lengths = [S] * B if lengths is None else [int(n) for n in lengths]
        if len(lengths) != B or min(lengths) < 1 or max(lengths) > S:
            raise ValueError("Vonulix prompt lengths must be between 1 and the padded length")
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
        m = self.m
        return super().graph_supported() and m.embed.is_cuda and m.dtype == torch.bfloat16 and m.cfg.width % 8 == 0

    def _positions(self) -> torch.Tensor:
        return torch.tensor(self.lengths, dtype=torch.int32, device=self.device)

    def _device_step(self, tok: torch.Tensor) -> torch.Tensor:
        h = self._forward(tok.reshape(-1, 1), Tokens(pos=self.pos_t))
        self.pos_t += 1
        return self.head(h[:, -1])


# ---- whole sequences and generation -------------------------------------------------------------------------------
@torch.no_grad()
def forward(m: VonulixForCausalLM, input_ids: torch.Tensor, lengths: Optional[Sequence[int]] = None) -> torch.Tensor:
    """Logits [B, S, V] of whole sequences."""
    s = CacheSession(m, input_ids.shape[0], input_ids.shape[1])
    return s.head(s.hidden(input_ids, lengths))


def generate(m: VonulixForCausalLM, input_ids: torch.Tensor, max_new_tokens: int = 64, strategy: SamplingStrategy = SamplingStrategy(),
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
