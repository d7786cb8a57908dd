"""Vonulix against Zatorax (its attention layers alone) at equal size: prefill and decode throughput of 8-layer stacks with random weights,
and the kernels of the new design beside the like kernels of the older models.

    python bench.py --workload vonulix --steps 10 --warmup 3          # one JSON line
    python -m benchmarks.vonulix_bench kernels ["prompt attention"]   # the kernels alone (cases whose name starts so)

Both stacks have the same width, head counts, head size 128, window, expert count, top-k, expert and shared FFN, vocabulary and number of
layers; Vonulix also has its kept positions, gates, token inputs (256 channels a layer) and averages over depth.  CUDA events around every
step, 256 MB written between steps (L2 flush, outside the events), median of the steps."""
from __future__ import annotations

import json
import sys

import torch

from .zatorax_bench import Timer

SIZES = {      # width, query heads, K/V heads, experts, top, expert ff, window
    "small": (1024, 8, 2, 32, 4, 512, 512),
    "medium": (2048, 16, 4, 64, 8, 768, 1024),
    "large": (4096, 32, 8, 64, 8, 1024, 2048),
}
LAYERS, VOCAB, KEEP, SIDE = 8, 32768, 4, 256


def vonulix_config(size: str):
    from tyr_b200.models import vonulix as V
    h, H, G, E, top, ff, window = SIZES[size]
    layer = V.LayerSpec(V.AttentionSpec(H, G, 128, 128, 128 ** -0.5, 1e4, 64, 2.0, window, KEEP), V.MoeSpec(E, top, ff, 7.0, ff, 7.0))
    return V.VonulixConfig(VOCAB, h, 1e-6, 1.0, SIDE, [layer] * LAYERS)


def zatorax_config(size: str):
    from tyr_b200.models import zatorax as Z
    h, H, G, E, top, ff, window = SIZES[size]
    layer = Z.LayerSpec(Z.AttentionSpec(H, G, 128, 128, 128 ** -0.5, window), Z.MoeSpec(E, top, ff, shared_ff=ff))
    return Z.ZatoraxConfig(VOCAB, h, 1e-6, [layer] * LAYERS)


@torch.no_grad()
def model_case(which: str, size: str, prompt=(4, 2048), decode_batches=(1, 32), warmup=3, steps=10, device="cuda") -> dict:
    if which == "vonulix":
        from tyr_b200.models import vonulix as M
        m = M.init(vonulix_config(size), device, torch.bfloat16)
    else:
        from tyr_b200.models import zatorax as M
        m = M.init(zatorax_config(size), device, torch.bfloat16)
    t = Timer(device, warmup, steps)
    B, S = prompt
    ids = lambda b, s: torch.randint(0, VOCAB, (b, s), device=device)
    x = ids(B, S)
    out = {"prefill_tokens": B * S, "prefill_ms": t(lambda: M.CacheSession(m, B, S + 8).prefill(x))}
    out["prefill_tokens_per_s"] = B * S / out["prefill_ms"] * 1e3
    for b in decode_batches:
        s = M.CacheSession(m, b, 1024 + warmup + steps + 16)
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
        cases[size] = {}
        for which in ("vonulix", "zatorax"):
            cases[size][which] = model_case(which, size, warmup=warmup, steps=steps)
            torch.cuda.empty_cache()
    mid = cases["medium" if "medium" in cases else sizes[0]]["vonulix"]
    return {"metric": "vonulix_prefill_tokens_per_s", "value": mid["prefill_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": steps,
            "warmup": max(3, warmup), "ms_per_step": mid["prefill_ms"], "higher_is_better": True, "dtype": "bf16",
            "data": "synthetic uniform token ids, random-init weights", "gpu_launches": opc.LAUNCH_COUNT[0] - l0,
            "config": {"layers": LAYERS, "vocab": VOCAB, "kept_positions": KEEP, "token_input": SIDE, "prompt": "4 x 2048", "decode_context": 1024,
                       "sizes": {s: dict(zip(("width", "heads", "kv_heads", "experts", "top", "ff", "window"), SIZES[s])) for s in sizes},
                       "l2": "256 MB buffer written between steps"},
            "cases": cases}


@torch.no_grad()
def kernels(only: str = "", warmup: int = 3, steps: int = 20, device="cuda") -> dict:
    """{case: {"new", "floor", "like", "like_floor"}} in ms: a kernel of the new design and the like kernel of the older models on the
    same shapes, each with the time of its algorithmic bytes or operations at the measured peaks."""
    from tyr_b200.models.common import KVCache
    from tyr_b200.ops import biased_attention as ba
    from tyr_b200.ops import flash, gates, moe
    from tyr_b200.ops import kept_attention as ka
    from tyr_b200.ops.depth import depth_average
    from tyr_b200.ops.embed import embed_positions, position_turns
    from tyr_b200.ops.gemm import gemm
    from tyr_b200.ops.norm import add_norm, post_norm_residual
    from tyr_b200.ops.skinny import skinny_linear
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

    # prompts: kept positions, turned values, gate per head / the flash kernel with a window (and without kept positions)
    for B, S, H, G, w in ((4, 2048, 8, 2, 512), (4, 2048, 16, 4, 1024), (4, 2048, 32, 8, 2048), (1, 8192, 16, 4, 1024)):
        q, k, v, g = mk(B, S, H, 128), mk(B, S, G, 128), mk(B, S, G, 128), mk(B, S, H)
        table = ka.turn_table(128, 1e4, 1.0, S, device)
        pairs = B * H * (w * (w + 1) / 2 + (S - w) * w) if w < S else B * H * S * (S + 1) / 2
        case(f"prompt attention {B}x{S}, {H}/{G} heads, window {w}", lambda: ka.prompt_attention(q, k, v, scale=0.09, window=w, keep=KEEP, head_gate=g, back=table),
             tf(pairs * 4 * 128), lambda: flash.flash_fwd_sink(q, k, v, scale=0.09, window=w))
    # one token per row / the penalised step
    for B, H, G, w in ((1, 8, 2, 512), (32, 8, 2, 512), (1, 16, 4, 1024), (32, 16, 4, 1024), (64, 32, 8, 2048)):
        q, kn, vn, g = mk(B, 1, H, 128), mk(B, 1, G, 128), mk(B, 1, G, 128), mk(B, 1, H)
        st = KVCache(mk(B, G, w + KEEP, 128), mk(B, G, w + KEEP, 128), True, keep=KEEP)
        s2 = KVCache(mk(B, G, w, 128), mk(B, G, w, 128), True)
        pos, table = torch.full((B,), 3 * w + 5, dtype=torch.int32, device=device), ka.turn_table(128, 1e4, 1.0, 3 * w + 8, device)
        r1, r2 = torch.rand(H, device=device) * 2, torch.rand(H, device=device) * 0.5
        case(f"step attention batch {B}, {H}/{G} heads, window {w}", lambda: ka.step_attention(q, st, pos, 128, 128, scale=0.09, window=w, keep=KEEP, head_gate=g, back=table),
             gb(B * G * (w + KEEP) * 128 * 4), lambda: ba.step_attention(q, kn, vn, s2, pos, r1, r2, window=w, scale=0.09, append=True), gb(B * G * w * 128 * 4))
    # rotation, value norm and store / query and key norm and store
    for B, S, H, G in ((4, 2048, 16, 4), (4, 2048, 32, 8), (1, 1, 16, 4), (32, 1, 16, 4)):
        n = (H + 2 * G) * 128
        y, w1 = mk(B, S, n + 16), torch.ones(128, device=device)
        st, s2 = (KVCache.allocate(B, G, 4096, 128, device, bf) for _ in range(2))
        kt, vt = ka.turn_table(64, 1e4, 2.0, 4096, device), ka.turn_table(128, 1e4, 1.0, 4096, device)
        pos = torch.full((B,), 3000, dtype=torch.int32, device=device) if S == 1 else None
        rows = B * S * (n + H * 128 + (2 if S > 1 else 1) * 2 * G * 128) * 2
        case(f"rotation and store {B}x{S}, {H}/{G} heads", lambda: ka.rotary_store(y, H, G, 128, 128, kt, vt, 1e-6, store=st, pos=pos), gb(rows),
             lambda: ba.qk_norm_store(y, w1, w1, H, G, 128, 128, 1e-6, dkp=128, dvp=128, store=s2, pos=pos), gb(B * S * (2 * n + 2 * G * 128) * 2))
    # experts of the weighted input, shared expert and add / experts and shared expert (sum in 16 bits)
    for T, h, E, k, ff in ((8192, 1024, 32, 4, 512), (8192, 2048, 64, 8, 768), (8192, 4096, 64, 8, 1024), (1, 1024, 32, 4, 512), (1, 2048, 64, 8, 768), (32, 1024, 32, 4, 512),
                           (32, 2048, 64, 8, 768), (64, 2048, 64, 8, 768), (32, 4096, 64, 8, 1024)):
        from tyr_b200.models.common import swiglu_mlp
        x, resid, gate = mk(T, h), f32(T, h), f32(T)
        ids = torch.stack([torch.randperm(E, device=device)[:k] for _ in range(T)]).int()
        wt, counts = torch.rand(T, k, device=device), moe.count_experts(ids, E)
        bank, shared = (moe.ExpertBank(mk(n, 2 * ff, h) * h ** -0.5, mk(n, h, ff) * ff ** -0.5) for n in (E, 1))
        b2 = moe.ExpertBank(*(x.clone() for x in (bank.gate_up, bank.down)))
        sg, su = (x.contiguous() for x in shared.gate_up[0].chunk(2))
        sd, form = shared.down[0].contiguous(), moe.ClampedExpert(7.0, 1.702)
        active = int((counts > 0).sum())
        floor = max(tf((T * k + T) * 6 * h * ff), gb((active + 1) * 6 * h * ff + T * h * 10))
        case(f"experts {T} tokens, width {h}, {E} top {k}, ff {ff}",
             lambda: moe.weighted_input_experts(x, ids, wt, bank, form, resid, shared=shared, shared_form=form, shared_gate=gate, counts=counts), floor,
             lambda: moe.moe_bank_forward(x, ids, wt, b2, counts=counts, add=swiglu_mlp(x, sg, su, sd)))
        del bank, shared, b2, sg, su, sd
        torch.cuda.empty_cache()
    # routing with one more row
    for T, h, E, k in ((8192, 2048, 64, 8), (32, 2048, 64, 8), (1, 2048, 64, 8)):
        x, w, corr = mk(T, h), f32(E + 1, h), torch.randn(E, device=device) * 0.1
        w0 = w[:E].contiguous()
        if T > moe.ROUTE_FUSED_MAX_TOKENS:
            wide = f32(T, E + 8)
            plain = wide[:, :E].contiguous()
            case(f"routing {T} tokens, {E} experts top {k}", lambda: moe.route(wide, k, renorm=False, experts=E), gb(T * (E + 2 * k) * 4),
                 lambda: moe.route(plain, k, softmax=True, bias=corr, renorm=False))
        else:
            case(f"routing {T} tokens, {E} experts top {k}", lambda: moe.route_fused(x, w, k, renorm=False, experts=E, want_logits=True), gb(E * h * 4 + T * h * 2),
                 lambda: moe.route_fused(x, w0, k, softmax=True, bias=corr, renorm=False))
    # token input: product with GELU and factor / the plain product
    for T, h, n in ((8192, 2048, SIDE), (8192, 4096, SIDE), (1, 2048, SIDE), (16, 2048, SIDE), (32, 2048, SIDE)):
        x, w, e = mk(T, h), mk(n, h) * h ** -0.5, mk(T, LAYERS * n)
        like = (lambda: gemm(x, w)) if T >= 128 else (lambda: skinny_linear(x, w))
        floor = max(tf(2 * T * h * n), gb((T * h + n * h + 2 * T * n) * 2))
        case(f"token input {T} rows, width {h}, {n} channels", lambda: gates.gelu_mul_project(x, w, e[:, n:2 * n]), floor, like, max(tf(2 * T * h * n), gb((T * h + n * h + T * n) * 2)))
    # depth average after layer n - 1, with norm, add and next norm / norm, add and copy
    for T, D, n in ((8192, 2048, 1), (8192, 2048, 8), (8192, 4096, 8), (1, 2048, 8), (32, 2048, 8), (32, 4096, 32)):
        y, x, hist, w, g = mk(T, D), f32(T, D), f32(n + 1, T, D), torch.rand(n + 1, device=device) / n, torch.ones(D, device=device)
        case(f"depth average {T}x{D} over {n + 1}", lambda: depth_average(y, g, x, hist, n, w, g, 1e-6, bf), gb(T * D * (2 + 4 * n + 4 + 4 + 4 + 2)),
             lambda: post_norm_residual(y, g, 1e-6, x, bf), gb(T * D * 12))
    for T, D in ((8192, 2048), (32, 2048)):
        ids, table, x, turns = torch.randint(0, VOCAB, (1, T), device=device), mk(VOCAB, D), f32(1, T, D), position_turns(D, device=device)
        case(f"scaled embedding {T}x{D}", lambda: embed_positions(ids, table, None, 2.0, out=x), gb(T * D * 6), lambda: embed_positions(ids, table, turns, 2.0, out=x))
        y, g = mk(1, T, D), torch.ones(D, device=device)
        case(f"add and norm {T}x{D}", lambda: add_norm(y, g, 1e-6, x, bf), gb(T * D * 12), lambda: post_norm_residual(y, g, 1e-6, x, bf))
    return out


if __name__ == "__main__":
    if sys.argv[1:2] == ["kernels"]:
        kernels(*sys.argv[2:3])
    else:
        print(json.dumps(run()))
