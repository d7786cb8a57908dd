"""Zatorax against Qwen3.5 MoE at equal size: prefill and decode throughput of 8-layer stacks with random weights, and the kernels
of the new design beside the like kernels of the older models.

    python bench.py --workload zatorax --steps 10 --warmup 3          # one JSON line
    python -m benchmarks.zatorax_bench kernels ["prompt attention"]   # the kernels alone (cases whose name starts so)

Both stacks have the same width, head counts, head size 128, expert count, top-k, expert and shared FFN, vocabulary and order
of layers (three delta-rule layers, then one attention layer).  Qwen3.5 attends the whole prompt, Zatorax a window.  CUDA events
around every step, 256 MB written between steps (L2 flush, outside the events), median of the steps."""
from __future__ import annotations

import json
import statistics
import sys

import torch

SIZES = {      # width, query heads, K/V heads, delta key heads, delta value heads, experts, top, expert ff, window
    "small": (1024, 8, 2, 8, 16, 32, 4, 512, 512),
    "medium": (2048, 16, 4, 16, 32, 64, 8, 768, 1024),
    "large": (4096, 32, 8, 16, 48, 64, 8, 1024, 2048),
}
LAYERS, VOCAB = 8, 32768


class Timer:
    def __init__(self, device, warmup: int, steps: int):
        self.flush = torch.empty(256 * 1024 * 1024, dtype=torch.uint8, device=device)
        self.warmup, self.steps = max(3, warmup), steps

    def __call__(self, fn) -> float:
        """Median milliseconds of ``fn``."""
        ms = []
        for i in range(self.warmup + self.steps):
            self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            if i >= self.warmup:
                ms.append(a.elapsed_time(b))
        return statistics.median(ms)


def zatorax_config(size: str):
    from tyr_b200.models import zatorax as Z
    h, H, G, Hk, Hv, E, top, ff, window = SIZES[size]
    mlp = Z.MoeSpec(E, top, ff, groups=8, keep=4, shared_ff=ff)
    d, a = Z.DeltaSpec(Hv, Hk, 128, 128, 4), Z.AttentionSpec(H, G, 128, 128, 128 ** -0.5, window)
    return Z.ZatoraxConfig(VOCAB, h, 1e-6, [Z.LayerSpec(a if i % 4 == 3 else d, mlp) for i in range(LAYERS)])


def qwen_config(size: str):
    from tyr_b200.models import qwen35 as Q
    h, H, G, Hk, Hv, E, top, ff, _ = SIZES[size]
    return Q.Qwen35Config(vocab_size=VOCAB, hidden_size=h, intermediate_size=0, num_hidden_layers=LAYERS, num_attention_heads=H, num_key_value_heads=G,
                          head_dim=128, linear_num_key_heads=Hk, linear_num_value_heads=Hv, moe_intermediate_size=ff, shared_expert_intermediate_size=ff,
                          num_experts=E, num_experts_per_tok=top)


@torch.no_grad()
def model_case(which: str, size: str, prompt=(4, 2048), decode_batches=(1, 32), warmup=3, steps=10, device="cuda") -> dict:
    if which == "zatorax":
        from tyr_b200.models import zatorax as Z
        m, make = Z.init(zatorax_config(size), device, torch.bfloat16), Z.CacheSession
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
        cases[size] = {}
        for which in ("zatorax", "qwen35_moe"):
            cases[size][which] = model_case(which, size, warmup=warmup, steps=steps)
            torch.cuda.empty_cache()
    mid = cases["medium" if "medium" in cases else sizes[0]]["zatorax"]
    return {"metric": "zatorax_prefill_tokens_per_s", "value": mid["prefill_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": steps,
            "warmup": max(3, warmup), "ms_per_step": mid["prefill_ms"], "higher_is_better": True, "dtype": "bf16",
            "data": "synthetic uniform token ids, random-init weights", "gpu_launches": opc.LAUNCH_COUNT[0] - l0,
            "config": {"layers": LAYERS, "vocab": VOCAB, "prompt": "4 x 2048", "decode_context": 1024,
                       "sizes": {s: dict(zip(("width", "heads", "kv_heads", "delta_key_heads", "delta_value_heads", "experts", "top", "ff", "window"), SIZES[s]))
                                 for s in sizes}, "l2": "256 MB buffer written between steps"},
            "cases": cases}


@torch.no_grad()
def kernels(only: str = "", warmup: int = 3, steps: int = 20, device="cuda") -> dict:
    """{case: {"new": ms, "like": ms, "floor": ms}}: a kernel of the new design, the like kernel of the older models on the same
    shapes, and the time of the algorithmic bytes or operations at the measured peaks."""
    from tyr_b200.models.common import KVCache
    from tyr_b200.ops import biased_attention as ba
    from tyr_b200.ops import decode_attention as da
    from tyr_b200.ops import delta_rule as dr
    from tyr_b200.ops import flash, moe
    from tyr_b200.ops.norm import post_norm_residual, rms_norm_weighted
    try:
        peaks = json.load(open("MEASURED_PEAKS.json"))
    except OSError:
        peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    gb = lambda n: n / peaks["hbm_gbs"] / 1e6
    tf = lambda n: n / peaks["bf16_tflops"] / 1e9
    t, out, bf = Timer(device, warmup, steps), {}, torch.bfloat16
    mk = lambda *s, dt=bf: torch.randn(*s, device=device).to(dt)

    def case(name, new, like, floor):
        if not name.startswith(only):
            return
        out[name] = {"new": t(new), "like": t(like), "floor": floor}
        print(f"{name}: new {out[name]['new'] * 1e3:.1f} us, like {out[name]['like'] * 1e3:.1f} us, floor {floor * 1e3:.1f} us", flush=True)

    # attention over prompts: flash kernel with and without the penalty, same window
    for B, S, H, G, w in ((4, 2048, 16, 4, 1024), (4, 4096, 32, 8, 2048), (4, 2048, 16, 4, 512)):
        q, k, v, r1, r2 = mk(B, S, H, 128), mk(B, S, G, 128), mk(B, S, G, 128), torch.rand(H, device=device) * 2, torch.rand(H, device=device) * 0.5
        pairs = B * H * (S * w - w * (w - 1) / 2)
        case(f"prompt attention {B}x{S}, {H}/{G} heads, window {w}", lambda: flash.flash_fwd_biased(q, k, v, r1, r2, window=w, scale=0.09),
             lambda: flash.flash_fwd_bthd(q, k, v, causal=True, window=w, scale=0.09, need_lse=False), tf(pairs * 4 * 128))
    # one token per row: split-KV kernel
    for B, H, G, w in ((32, 16, 4, 1024), (64, 32, 8, 2048), (1, 16, 4, 1024)):
        q, kn, vn = mk(B, 1, H, 128), mk(B, 1, G, 128), mk(B, 1, G, 128)
        st, pos = KVCache(mk(B, G, w, 128), mk(B, G, w, 128), True), torch.full((B,), 3 * w + 5, dtype=torch.int32, device=device)
        r1, r2 = torch.rand(H, device=device) * 2, torch.rand(H, device=device) * 0.5
        case(f"step attention batch {B}, {H}/{G} heads, window {w}",
             lambda: ba.step_attention(q, kn, vn, st, pos, r1, r2, window=w, scale=0.09, append=True),
             lambda: da.decode_attention(q[:, 0], kn[:, 0], vn[:, 0], st.k, st.v, pos[:1], ring=True, scale=0.09), gb(B * G * w * 128 * 4))
    # delta rule over prompts: chunk kernels, 32-bit form against the TF32 form
    for B, S, Hk, Hv in ((4, 2048, 16, 32), (8, 2048, 16, 48), (1, 8192, 16, 32)):
        q, k, v = mk(B, S, Hk, 128), mk(B, S, Hk, 128), mk(B, S, Hv, 128)
        g, beta = -torch.rand(B, S, Hv, device=device), torch.rand(B, S, Hv, device=device)
        state = torch.zeros(B, Hv, 128, 128, device=device)
        flops = B * Hv * S * (2 * 64 * 128 * 2 + 64 * 256 + 3 * 2 * 128 * 128 + 2 * 64 * 128)
        case(f"delta prompt {B}x{S}, {Hk}/{Hv} heads", lambda: dr.delta_prefill(q, k, v, g, beta, state),
             lambda: dr.chunk_gated_delta_rule(q, k, v, g, beta), max(tf(flops), gb(2 * (2 * q.numel() + 2 * v.numel()))))
    # delta rule, one token per row
    for B, Hk, Hv in ((32, 16, 32), (64, 16, 48), (1, 16, 32)):
        C = (2 * Hk + Hv) * 128
        y = mk(B, 1, C + Hv * 128 + 2 * Hv)
        conv, rec = mk(B, C, 4), torch.zeros(B, Hv, 128, 128, device=device)
        w, nw, bias, al = mk(C, 4), mk(128), torch.randn(Hv, device=device), torch.randn(Hv, device=device)
        z = C + Hv * 128
        args = (y[..., :C], y[..., C:z], y[..., z:z + Hv], y[..., z + Hv:], conv, w)
        case(f"delta step batch {B}, {Hk}/{Hv} heads", lambda: dr.delta_decode(*args, bias, al, nw, 1e-6, rec, Hk, Hv, 128, 128),
             lambda: dr.gdn_decode_fused(*args, None, bias, al, nw, 1e-6, rec, Hk, Hv, 128, 128), gb(2 * rec.numel() * 4))
    # sublayer norm, residual add and 16-bit copy
    for T, D in ((8192, 2048), (8192, 4096), (32, 2048)):
        x, r32, r16, g1, gd = mk(T, D), mk(T, D, dt=torch.float32), mk(T, D), torch.ones(1, device=device), mk(D)
        case(f"norm and add {T}x{D} (fp32 stream against bf16 stream)", lambda: post_norm_residual(x, g1, 1e-6, r32, bf),
             lambda: rms_norm_weighted(x, gd, 1e-6, residual=r16, return_residual=True), gb(T * D * 12))
    # routing
    for T, h, E, k in ((8192, 2048, 64, 8), (32, 2048, 64, 8)):
        x, w, corr = mk(T, h), mk(E, h), torch.randn(E, device=device) * 0.1
        w32, logits = w.float(), mk(T, E, dt=torch.float32)
        if T > moe.ROUTE_FUSED_MAX_TOKENS:
            new = lambda: moe.route(logits, k, softmax=True, bias=corr, renorm=False, groups=8, keep=4)
            like = lambda: moe.route(logits, k, softmax=True, renorm=True)
            floor = gb(T * (E + 2 * k) * 4)
        else:
            new = lambda: moe.route_fused(x, w32, k, softmax=True, bias=corr, renorm=False, groups=8, keep=4)
            like = lambda: moe.route_fused(x, w32, k, softmax=True, renorm=True)
            floor = gb(E * h * 4 + T * h * 2)
        case(f"routing {T} tokens, {E} experts top {k}", new, like, floor)
    return out


if __name__ == "__main__":
    if sys.argv[1:2] == ["kernels"]:
        kernels(*sys.argv[2:3])
    else:
        print(json.dumps(run()))
