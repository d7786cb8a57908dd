"""Kinetar against Qwen3.5 (dense) at equal size: prefill and decode throughput of 8-layer stacks with random weights, and the kernels
of the new design beside the like kernels of the older models.

    python bench.py --workload kinetar --steps 10 --warmup 3          # one JSON line
    python -m benchmarks.kinetar_bench kernels ["prompt attention"]   # the kernels alone (cases whose name starts so)

Both stacks have the same width, heads of 128, vocabulary and order of layers (attention or parallel, then delta rule); the
feed-forward of Qwen3.5 is sized so that both hold the same number of parameters (Kinetar's parallel layers also carry a selective
scan).  CUDA events around every step, 256 MB written between steps (L2 flush, outside the events), median of the steps."""
from __future__ import annotations

import json
import sys

import torch

from .zatorax_bench import Timer

SIZES = {      # width, query heads, K/V heads, delta key heads, delta value heads, scan channels, dense ff
    "small": (1024, 8, 2, 8, 8, 2048, 4096),
    "medium": (2048, 16, 4, 16, 16, 4096, 8192),
    "large": (4096, 32, 8, 16, 32, 8192, 16384),
}
LAYERS, VOCAB, STATES = 8, 32768, 16


def kinetar_config(size: str):
    from tyr_b200.models import kinetar as K
    h, H, G, Hk, Hv, inner, ff = SIZES[size]
    p = K.ParallelSpec(K.AttentionSpec(H, G, 128, 128, 4, 128 ** -0.5, 0.1, 8192), K.ScanSpec(inner, STATES, h // 16, 4), 0.7, 0.7)
    d = K.ChannelDeltaSpec(Hv, Hk, 128, 128, 4)
    return K.KinetarConfig(VOCAB, h, 1e-6, [K.LayerSpec(d if i % 2 else p, ff) for i in range(LAYERS)])


def parameters(size: str) -> int:
    from tyr_b200.models import kinetar as K
    n = 0
    for s in K.tensor_shapes(kinetar_config(size)).values():
        t = 1
        for x in s:
            t *= 128 if x is None else x
        n += t
    return n


def qwen_config(size: str):
    from tyr_b200.models import qwen35 as Q
    h, H, G, Hk, Hv, _, _ = SIZES[size]
    full = h * (2 * H + 2 * G) * 128 + H * 128 * h
    linear = h * (2 * Hk + 2 * Hv) * 128 + Hv * 128 * h
    left = parameters(size) - 2 * VOCAB * h - LAYERS // 2 * (full + linear)
    ff = round(left / (3 * h * LAYERS) / 256) * 256
    types = [Q.LINEAR if i % 2 else Q.FULL for i in range(LAYERS)]
    return Q.Qwen35Config(vocab_size=VOCAB, hidden_size=h, intermediate_size=ff, num_hidden_layers=LAYERS, num_attention_heads=H, num_key_value_heads=G,
                          head_dim=128, linear_num_key_heads=Hk, linear_num_value_heads=Hv, layer_types=types)


@torch.no_grad()
def model_case(which: str, size: str, prompt=(4, 2048), decode_batches=(1, 32), warmup=3, steps=10, device="cuda") -> dict:
    if which == "kinetar":
        from tyr_b200.models import kinetar as K
        m, make = K.init(kinetar_config(size), device, torch.bfloat16, rank=128), K.CacheSession
    else:
        from tyr_b200.models import qwen35 as Q
        m, make = Q.init(qwen_config(size), device, torch.bfloat16), Q.HybridCache
    t = Timer(device, warmup, steps)
    B, S = prompt
    ids = lambda b, s: torch.randint(0, VOCAB, (b, s), device=device)
    x = ids(B, S)
    out = {"prefill_tokens": B * S, "prefill_ms": t(lambda: make(m, B, S + 8).prefill(x))}
    out["prefill_tokens_per_s"] = B * S / out["prefill_ms"] * 1e3
    for b in decode_batches:
        s = make(m, b, 1024 + warmup + steps + 16)
        tok = s.prefill(ids(b, 1024)).argmax(-1)
        state = {"tok": s.step(tok).argmax(-1)}

        def one():
            state["tok"] = s.step(state["tok"]).argmax(-1)
        ms = t(one)
        out[f"decode_b{b}_ms"], out[f"decode_b{b}_tokens_per_s"] = ms, b / ms * 1e3
    from tyr_b200.ops._common import raise_on_device_error
    raise_on_device_error(device)
    return out


def run(warmup: int = 3, steps: int = 10, sizes=tuple(SIZES)) -> dict:
    from tyr_b200.ops import _common as opc
    l0 = opc.LAUNCH_COUNT[0]
    cases = {}
    for size in sizes:
        cases[size] = {"parameters": parameters(size)}
        for which in ("kinetar", "qwen35"):
            cases[size][which] = model_case(which, size, warmup=warmup, steps=steps)
            torch.cuda.empty_cache()
    mid = cases["medium" if "medium" in cases else sizes[0]]["kinetar"]
    return {"metric": "kinetar_prefill_tokens_per_s", "value": mid["prefill_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": steps,
            "warmup": max(3, warmup), "ms_per_step": mid["prefill_ms"], "higher_is_better": True, "dtype": "bf16",
            "data": "synthetic uniform token ids, random-init weights", "gpu_launches": opc.LAUNCH_COUNT[0] - l0,
            "config": {"layers": LAYERS, "vocab": VOCAB, "states": STATES, "prompt": "4 x 2048", "decode_context": 1024,
                       "sizes": {s: dict(zip(("width", "heads", "kv_heads", "delta_key_heads", "delta_value_heads", "scan_channels", "ff"), SIZES[s])) for s in sizes},
                       "l2": "256 MB buffer written between steps"},
            "cases": cases}


@torch.no_grad()
def kernels(only: str = "", warmup: int = 3, steps: int = 20, device="cuda") -> dict:
    """{case: {"new", "floor", "like", "like_floor"}} in ms: a kernel of the new design and the like kernel of the older models on the
    same shapes, each with the time of its algorithmic bytes or operations at the measured peaks."""
    from tyr_b200.models.common import KVCache
    from tyr_b200.ops import decode_attention as da
    from tyr_b200.ops import delta_rule as dr
    from tyr_b200.ops import flash
    from tyr_b200.ops import selective_scan as ss
    from tyr_b200.ops import sink_attention as sa
    from tyr_b200.ops.embed import embed_positions, position_turns
    from tyr_b200.ops.mix_conv import Segment, mix_prompt, mix_step
    from tyr_b200.ops.norm import add_norm, rms_norm_weighted
    try:
        peaks = json.load(open("MEASURED_PEAKS.json"))
    except OSError:
        peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    gb = lambda n: n / peaks["hbm_gbs"] / 1e6
    tf = lambda n: n / peaks["bf16_tflops"] / 1e9
    t, out, bf = Timer(device, warmup, steps), {}, torch.bfloat16
    mk = lambda *s, dt=bf: torch.randn(*s, device=device).to(dt)
    f32 = lambda *s: torch.randn(*s, device=device)

    def case(name, new, floor, like=None, like_floor=None):
        if not name.startswith(only):
            return
        r = out[name] = {"new": t(new), "floor": floor, "like": t(like) if like else None, "like_floor": floor if like_floor is None else like_floor}
        us = lambda x: f"{x * 1e3:.1f}"
        txt = f"{name}: new {us(r['new'])} us (floor {us(floor)}, x{r['new'] / floor:.2f})"
        if like:
            txt += f", like {us(r['like'])} us (floor {us(r['like_floor'])}, x{r['like'] / r['like_floor']:.2f}), ratio of distances " \
                   f"{r['new'] / floor / (r['like'] / r['like_floor']):.2f}"
        print(txt, flush=True)

    # attention over prompts: sink, gate, values that are the keys / plain flash kernel
    for B, S, H, G in ((4, 2048, 16, 4), (4, 4096, 32, 8), (1, 2048, 16, 4)):
        q, k, v, y, sink = mk(B, S, H, 128), mk(B, S, G, 128), mk(B, S, G, 128), mk(B, S, 2 * H * 128), f32(H)
        o = mk(B, S, 2 * H * 128)
        case(f"prompt attention {B}x{S}, {H}/{G} heads", lambda: sa.prompt_attention(q, k, k, scale=0.09, sink=sink, gate=y[..., :H * 128], out_scale=0.7, out=o[..., :H * 128]),
             tf(B * H * S * (S + 1) / 2 * 4 * 128), lambda: flash.flash_fwd_bthd(q, k, v, causal=True, window=None, scale=0.09, need_lse=False))
    # one token per row over 1024 keys
    for B, H, G, n in ((32, 16, 4, 1024), (64, 32, 8, 2048), (1, 16, 4, 1024)):
        q, kn, vn = mk(B, 1, H, 128), mk(B, 1, G, 128), mk(B, 1, G, 128)
        kc, vc, pos = mk(B, G, n + 8, 128), mk(B, G, n + 8, 128), torch.full((B,), n, dtype=torch.int32, device=device)
        y, sink, st = mk(B, 1, 2 * H * 128), f32(H), KVCache(kc, kc)
        case(f"step attention batch {B}, {H}/{G} heads, {n} keys", lambda: sa.step_attention(q, kn, kn, st, pos, 128, scale=0.09, sink=sink, gate=y[..., :H * 128], out_scale=0.7),
             gb(B * G * n * 128 * 2), lambda: da.decode_attention(q[:, 0], kn[:, 0], vn[:, 0], kc, vc, pos[:1], scale=0.09, elem_gate=y[:, 0, :H * 128].unflatten(1, (H, 128))),
             gb(B * G * n * 128 * 4))
    # delta rule over prompts: decay per key channel / per head, both exact
    for B, S, Hk, Hv in ((4, 2048, 16, 16), (4, 2048, 16, 32), (1, 8192, 16, 32)):
        q, k, v, a, b = mk(B, S, Hk, 128), mk(B, S, Hk, 128), mk(B, S, Hv, 128), mk(B, S, Hv * 128), mk(B, S, Hv)
        bias, al = f32(Hv * 128) - 2.0, f32(Hv) * 0.3
        g, beta, state = -torch.rand(B, S, Hv, device=device), torch.rand(B, S, Hv, device=device), torch.zeros(B, Hv, 128, 128, device=device)
        flops = B * Hv * S * (2 * 64 * 128 * 2 + 64 * 256 + 3 * 2 * 128 * 128 + 2 * 64 * 128)
        qkvo = 2 * (2 * q.numel() + 2 * v.numel())
        case(f"delta prompt {B}x{S}, {Hk}/{Hv} heads", lambda: dr.channel_delta_prefill(q, k, v, a, b, bias, al, state), max(tf(flops), gb(qkvo + 2 * a.numel())),
             lambda: dr.delta_prefill(q, k, v, g, beta, state), max(tf(flops), gb(qkvo)))
    # delta rule, one token per row: convolutions, recurrence, norm and gate
    for B, Hk, Hv in ((32, 16, 32), (64, 16, 32), (1, 16, 16)):
        C = (2 * Hk + Hv) * 128
        y = mk(B, 1, C + 2 * Hv * 128 + 2 * Hv)
        rec, pos = torch.zeros(B, Hv, 128, 128, device=device), torch.zeros(B, dtype=torch.int32, device=device)
        conv, w, nw, nw32 = mk(B, C, 4), mk(C, 4), mk(128), f32(128)
        bias, al, biasc, o = f32(Hv), f32(Hv) * 0.3, f32(Hv * 128) - 2.0, mk(B, 1, 2 * Hv * 128)
        z, e = C + Hv * 128, C + 2 * Hv * 128
        q, k, v = mk(B, 1, Hk, 128), mk(B, 1, Hk, 128), mk(B, 1, Hv, 128)
        wins = [mk(B, n, 4) for n in (Hk * 128, Hk * 128, Hv * 128)]
        segs = [Segment(c, h, 128, x.flatten(2), w=f32(h * 128, 4), window=win, act="silu")
                for c, h, x, win in zip((0, Hk * 128, 2 * Hk * 128), (Hk, Hk, Hv), (q, k, v), wins)]

        def new():
            mix_step(y, segs, pos)
            dr.channel_delta_decode(q, k, v, y[..., z:e], y[..., e:e + Hv], y[..., C:z], biasc, al, nw32, nw, 1e-6, rec, o[..., :Hv * 128])
        args = (y[..., :C], y[..., C:z], y[..., e:e + Hv], y[..., e + Hv:e + 2 * Hv], conv, w)
        case(f"delta step batch {B}, {Hk}/{Hv} heads", new, gb(2 * rec.numel() * 4),
             lambda: dr.gdn_decode_fused(*args, None, bias, al, nw, 1e-6, rec, Hk, Hv, 128, 128))
    # selective scan (no like kernel: the delta rule's prompt and step kernels are the nearest)
    for B, S, C in ((4, 2048, 4096), (4, 2048, 8192), (1, 2048, 4096)):
        x, dt, y, bc, o = mk(B, S, C), mk(B, S, C), mk(B, S, 2 * C), mk(B, S, 2 * STATES + 256), mk(B, S, 2 * C)
        A, D, bias, state = -torch.rand(C, STATES, device=device) * 4 - 0.05, f32(C), f32(C) - 3.0, torch.zeros(B, C, STATES, device=device)
        q, k, v, st = mk(B, S, C // 256, 128), mk(B, S, C // 256, 128), mk(B, S, C // 128, 128), torch.zeros(B, C // 128, 128, 128, device=device)
        g, beta = -torch.rand(B, S, C // 128, device=device), torch.rand(B, S, C // 128, device=device)
        case(f"scan prompt {B}x{S}, {C} channels", lambda: ss.scan_prompt(x, dt, y[..., :C], bc[..., 256:256 + STATES], bc[..., 256 + STATES:], A, D, bias, state, o[..., :C]),
             gb(B * S * C * 8), lambda: dr.delta_prefill(q, k, v, g, beta, st), gb(2 * (2 * q.numel() + 2 * v.numel())))
    for B, C in ((32, 4096), (64, 8192), (1, 4096)):
        x, dt, y, bc, o = mk(B, 1, C), mk(B, 1, C), mk(B, 1, 2 * C), mk(B, 1, 2 * STATES + 256), mk(B, 1, 2 * C)
        A, D, bias, state = -torch.rand(C, STATES, device=device) * 4 - 0.05, f32(C), f32(C) - 3.0, torch.zeros(B, C, STATES, device=device)
        H = max(1, C * STATES // 16384)                   # as many bytes of state
        rec, q, k, v = torch.zeros(B, H, 128, 128, device=device), mk(B, 1, H, 128), mk(B, 1, H, 128), mk(B, 1, H, 128)
        g, beta = -torch.rand(B, 1, H, device=device), torch.rand(B, 1, H, device=device)
        case(f"scan step batch {B}, {C} channels", lambda: ss.scan_step(x, dt, y[..., :C], bc[..., 256:256 + STATES], bc[..., 256 + STATES:], A, D, bias, state, o[..., :C]),
             gb(2 * state.numel() * 4 + A.numel() * 4 + B * C * 8), lambda: dr.gdr_decode_step(q, k, v, g, beta, rec), gb(2 * rec.numel() * 4))
    # convolutions and activations
    for B, S, H, G, C in ((4, 2048, 16, 4, 4096), (4, 2048, 32, 8, 8192)):
        n = (H + G) * 128 + C
        y, q, k, x, store = mk(B, S, 2 * n), mk(B, S, H * 128), mk(B, S, G * 128), mk(B, S, C), mk(B, G, S, 128)
        segs = [Segment(0, H, 128, q, w=f32(H * 128, 4), window=mk(B, H * 128, 4), temp=(0.1, 64)),
                Segment(H * 128, G, 128, k, w=f32(G * 128, 4), window=mk(B, G * 128, 4), store=store),
                Segment((H + G) * 128, 1, C, x, w=f32(C, 4), bias=f32(C), window=mk(B, C, 4), act="silu")]
        w = mk(n, 4)
        case(f"convolutions {B}x{S}, {n} channels", lambda: mix_prompt(y, segs), gb(B * S * (4 * n + G * 128 * 2)), lambda: dr.causal_conv1d_silu(y[..., :n], w), gb(B * S * 4 * n))
    # residual add and norm; embedding
    for T, D in ((8192, 2048), (8192, 4096), (32, 2048)):
        x, r32, r16, g1, gd = mk(T, D), f32(T, D), mk(T, D), torch.ones(D, device=device), mk(D)
        case(f"add and norm {T}x{D} (fp32 stream against bf16 stream)", lambda: add_norm(x, g1, 1e-6, r32, bf), gb(T * D * 12),
             lambda: rms_norm_weighted(x, gd, 1e-6, residual=r16, return_residual=True), gb(T * D * 8))
    for B, S, D in ((4, 2048, 2048), (32, 1, 2048)):
        ids, table, turns = torch.randint(0, VOCAB, (B, S), device=device), mk(VOCAB, D), position_turns(D, device=device)
        pos = torch.full((B,), 1000, dtype=torch.int32, device=device) if S == 1 else None
        case(f"embedding {B}x{S}, width {D}", lambda: embed_positions(ids, table, turns, 0.5, pos), gb(B * S * D * 6),
             lambda: torch.nn.functional.embedding(ids, table), gb(B * S * D * 4))
    return out


if __name__ == "__main__":
    if sys.argv[1:2] == ["kernels"]:
        kernels(*sys.argv[2:3])
    else:
        print(json.dumps(run()))
