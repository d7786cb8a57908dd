"""Nizedra against Qwen3.5 (dense) at equal size: prefill and decode throughput of 8-layer stacks with random weights, and the kernels
of the new design beside the like kernels of the older models.

    python bench.py --workload nizedra --steps 10 --warmup 3          # one JSON line
    python -m benchmarks.nizedra_bench kernels ["talking prompt"]     # the kernels alone (cases whose name starts so)

Both stacks have the same width, vocabulary and number of layers, every second one linear attention with heads of 128; Nizedra's other
layers are latent attention and attention with mixed heads in turn, the middle ones inside a loop of one pass.  The feed-forward of
Qwen3.5 is sized so that both hold the same number of parameters.  CUDA events around every step, 256 MB written between steps (L2
flush, outside the events), median of the steps."""
from __future__ import annotations

import json
import sys

import torch

from .zatorax_bench import Timer

SIZES = {      # width, linear heads, latent (heads, unrotated, rotated, value, query rank, key/value rank), mixed (heads, K/V heads, size), dense ff
    "small": (1024, 8, (16, 64, 32, 64, 384, 256), (16, 4, 64), 4096),
    "medium": (2048, 16, (32, 64, 32, 64, 768, 512), (16, 4, 128), 8192),
    "large": (4096, 32, (32, 96, 32, 128, 1536, 512), (32, 8, 128), 16384),
}
LAYERS, VOCAB, WINDOW, ROWS, REACH = 8, 32768, 1024, 32, 128


def nizedra_config(size: str):
    from tyr_b200.models import nizedra as N
    h, Hl, (H, d, r, v, qr, kr), (Ha, G, da), ff = SIZES[size]
    light = N.LightningSpec(Hl, 128, 128, tuple(1.0 - 2.0 ** -(3 + 8 * i / Hl) for i in range(Hl)))
    lat = N.LatentSpec(H, d, r, v, qr, kr, (d + r) ** -0.5, 1e4, r, WINDOW)
    talk = N.AttentionSpec(Ha, G, da, da, da ** -0.5, 50.0, REACH)
    return N.NizedraConfig(VOCAB, h, 1e-6, [N.LayerSpec(m, ff) for m in (light, lat, light, talk)] * 2, N.Loop(2, 6, 1))


def parameters(size: str) -> int:
    from tyr_b200.models import nizedra as N
    n = 0
    for s in N.tensor_shapes(nizedra_config(size)).values():
        t = 1
        for x in s:
            t *= ROWS if x is None else x
        n += t
    return n


def qwen_config(size: str):
    from tyr_b200.models import qwen35 as Q
    h, Hl, _, _, _ = SIZES[size]
    H, G = h // 128, max(2, h // 512)
    full = h * (2 * H + 2 * G) * 128 + H * 128 * h
    linear = h * 4 * Hl * 128 + Hl * 128 * h
    left = parameters(size) - 2 * VOCAB * h - LAYERS // 2 * (full + linear)
    ff = round(left / (3 * h * LAYERS) / 256) * 256
    types = [Q.FULL if i % 2 else Q.LINEAR for i in range(LAYERS)]
    return Q.Qwen35Config(vocab_size=VOCAB, hidden_size=h, intermediate_size=ff, num_hidden_layers=LAYERS, num_attention_heads=H, num_key_value_heads=G,
                          head_dim=128, linear_num_key_heads=Hl, linear_num_value_heads=Hl, layer_types=types)


@torch.no_grad()
def model_case(which: str, size: str, prompt=(4, 2048), decode_batches=(1, 32), warmup=3, steps=10, device="cuda") -> dict:
    if which == "nizedra":
        from tyr_b200.models import nizedra as N
        m, make = N.init(nizedra_config(size), device, torch.bfloat16, rows=ROWS), N.CacheSession
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
        for which in ("nizedra", "qwen35"):
            cases[size][which] = model_case(which, size, warmup=warmup, steps=steps)
            torch.cuda.empty_cache()
    mid = cases["medium" if "medium" in cases else sizes[0]]["nizedra"]
    return {"metric": "nizedra_prefill_tokens_per_s", "value": mid["prefill_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": steps,
            "warmup": max(3, warmup), "ms_per_step": mid["prefill_ms"], "higher_is_better": True, "dtype": "bf16",
            "data": "synthetic uniform token ids, random-init weights", "gpu_launches": opc.LAUNCH_COUNT[0] - l0,
            "config": {"layers": LAYERS, "vocab": VOCAB, "window": WINDOW, "prompt": "4 x 2048", "decode_context": 1024,
                       "sizes": {s: dict(zip(("width", "linear_heads", "latent", "mixed", "ff"), SIZES[s])) for s in sizes},
                       "l2": "256 MB buffer written between steps"},
            "cases": cases}


@torch.no_grad()
def kernels(only: str = "", warmup: int = 3, steps: int = 20, device="cuda") -> dict:
    """{case: {"new", "floor", "like", "like_floor"}} in ms: a kernel of the new design and the like kernel of the older models on the
    same shapes, each with the time of its algorithmic bytes or operations at the measured peaks.  The floor of mixed heads is the sum of
    its products (bf16 for Q K^T and P V, half that rate for the mix of the scores in two TF32 terms) or its three special-function
    operations a score, whichever is longer."""
    from tyr_b200.models.common import KVCache, lin
    from tyr_b200.ops import decode_attention as da
    from tyr_b200.ops import delta_rule as dr
    from tyr_b200.ops import flash
    from tyr_b200.ops import joint_attention as ja
    from tyr_b200.ops import latent as lt
    from tyr_b200.ops import lightning as lg
    from tyr_b200.ops import skinny
    from tyr_b200.ops.biased_attention import qk_norm_store
    from tyr_b200.ops.embed import position_turns
    from tyr_b200.ops.gemm import gemm
    from tyr_b200.ops.norm import rms_norm_weighted, sandwich_norm
    try:
        peaks = json.load(open("MEASURED_PEAKS.json"))
    except OSError:
        peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    gb = lambda n: n / peaks["hbm_gbs"] / 1e6
    tf = lambda n: n / peaks["bf16_tflops"] / 1e9
    sfu = lambda n: n / (148 * 16 * 1.965e9) * 1e3
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

    bound = 130.0                    # of unit queries and keys

    def talk(H):
        return ja.Talk(torch.ones(H, device=device), f32(ROWS, H) * 0.1, ja.distance_buckets(ROWS, REACH).to(device),
                       (torch.eye(H, device=device) + 0.1 * f32(H, H)).bfloat16().float(), 50.0)

    # mixed heads over prompts / plain flash kernel (heads of 128)
    for B, S, H, G, d in ((4, 2048, 16, 4, 64), (4, 2048, 16, 4, 128), (4, 2048, 32, 8, 128), (1, 2048, 16, 4, 128), (1, 8192, 16, 4, 128)):
        q, k, v, tk = mk(B, S, H, d), mk(B, S, G, d), mk(B, S, G, d), talk(H)
        q1, k1, v1 = mk(B, S, H, 128), mk(B, S, G, 128), mk(B, S, G, 128)
        pairs = B * S * (S + 1) / 2
        case(f"talking prompt {B}x{S}, {H}/{G} heads of {d}", lambda: ja.prompt_attention(q, k, v, scale=0.09, talk=tk, dot_bound=bound),
             max(tf(pairs * H * (4 * d + 2 * 2 * 2 * H)), sfu(pairs * H * 3)), lambda: flash.flash_fwd_bthd(q1, k1, v1, causal=True, window=None, scale=0.09, need_lse=False),
             max(tf(pairs * H * 4 * 128), sfu(pairs * H)))
    # mixed heads, one token per row / split-KV kernel
    for B, H, G, n in ((32, 16, 4, 1024), (64, 32, 8, 2048), (1, 16, 4, 1024), (1, 16, 4, 16384)):
        q, kn, vn = mk(B, 1, H, 128), mk(B, 1, G, 128), mk(B, 1, G, 128)
        kc, vc, pos, tk = mk(B, G, n + 8, 128), mk(B, G, n + 8, 128), torch.full((B,), n, dtype=torch.int32, device=device), talk(H)
        st = KVCache(kc, vc)
        case(f"talking step batch {B}, {H}/{G} heads, {n} keys", lambda: ja.step_attention(q, st, pos, 128, scale=0.09, talk=tk, dot_bound=bound), gb(B * G * n * 128 * 4),
             lambda: da.decode_attention(q[:, 0], kn[:, 0], vn[:, 0], kc, vc, pos[:1], scale=0.09))
    # latent attention over prompts: windowed flash kernel with its head sizes / heads of 128, the same window
    for B, S, H, dk, dv in ((4, 2048, 32, 96, 64), (4, 2048, 32, 128, 128), (1, 8192, 32, 96, 64)):
        q, k, v = mk(B, S, H, dk), mk(B, S, H, dk), mk(B, S, H, dv)
        q1, k1, v1 = mk(B, S, H, 128), mk(B, S, H, 128), mk(B, S, H, 128)
        pairs = B * (WINDOW * (WINDOW + 1) / 2 + (S - WINDOW) * WINDOW)
        case(f"latent prompt {B}x{S}, {H} heads of {dk}/{dv}", lambda: flash.flash_fwd_sink(q, k, v, scale=0.1, window=WINDOW), tf(pairs * H * 2 * (dk + dv)),
             lambda: flash.flash_fwd_bthd(q1, k1, v1, causal=True, window=WINDOW, scale=0.09, need_lse=False), tf(pairs * H * 4 * 128))
    # latent rows, one token per row / split-KV kernel over as many keys
    for B, H, R, n in ((32, 32, 512, 1024), (64, 32, 512, 4096), (1, 32, 512, 1024), (32, 16, 256, 1024), (64, 128, 512, 4096)):
        row = R + (32 if R == 256 else 64)
        q, st, pos = mk(B, 1, H, row), mk(B, 1, n, row), torch.full((B,), 3 * n // 2, dtype=torch.int32, device=device)
        kv = KVCache(st, st, ring=True)
        q1, kn, kc, vc, p1 = mk(B, 16, 128), mk(B, 4, 128), mk(B, 4, n + 8, 128), mk(B, 4, n + 8, 128), pos.clone().fill_(n)
        case(f"latent step batch {B}, {H} heads over {row}, {n} keys", lambda: ja.step_attention(q, kv, pos, R, scale=0.05, window=n),
             max(gb(B * n * row * 2), tf(B * n * H * 2 * (row + R))), lambda: da.decode_attention(q1, kn, kn, kc, vc, p1[:1], scale=0.09), gb(B * 4 * n * 128 * 4))
    # lightning over prompts / exact gated delta rule
    for B, S, H in ((4, 2048, 8), (4, 2048, 16), (4, 2048, 32), (1, 8192, 32)):
        y, dec, state = mk(B, S, 3 * H * 128), torch.linspace(0.9, 0.999, H, dtype=torch.float64, device=device), torch.zeros(B, H, 128, 128, device=device)
        q, k, v = (y[..., i * H * 128:(i + 1) * H * 128].unflatten(2, (H, 128)) for i in range(3))
        g, beta = -torch.rand(B, S, H, device=device), torch.rand(B, S, H, device=device)
        case(f"lightning prompt {B}x{S}, {H} heads", lambda: lg.prefill(q, k, v, dec, state), gb(B * S * H * 128 * 10), lambda: dr.delta_prefill(q, k, v, g, beta, state),
             gb(B * S * H * 128 * 10))
    for B, H in ((32, 16), (64, 32), (1, 16)):
        y, dec, rec = mk(B, 1, 4 * H * 128), torch.linspace(0.9, 0.999, H, dtype=torch.float64, device=device), torch.zeros(B, H, 128, 128, device=device)
        q, k, v = (y[..., i * H * 128:(i + 1) * H * 128].unflatten(2, (H, 128)) for i in range(3))
        qc, kc, vc = (x.contiguous() for x in (q, k, v))
        g, beta, z, w = -torch.rand(B, 1, H, device=device), torch.rand(B, 1, H, device=device), y[..., 3 * H * 128:], torch.ones(H * 128, device=device)
        case(f"lightning step batch {B}, {H} heads", lambda: dr.gated_norm(lg.step(q, k, v, dec, rec).flatten(2).unsqueeze(2), z, w, 1e-6, "sigmoid"),
             gb(2 * rec.numel() * 4), lambda: dr.gated_norm(dr.gdr_decode_step(qc, kc, vc, g, beta, rec).float(), z, w[:128], 1e-6), gb(2 * rec.numel() * 4))
    # norms, rotation, products per head
    for T, D in ((8192, 2048), (8192, 4096), (32, 2048)):
        x, r32, r16, g1, gd = mk(1, T, D), f32(1, T, D), mk(1, T, D), torch.ones(D, device=device), mk(D)
        case(f"norm, add and norm {T}x{D} (fp32 stream against bf16 add and norm)", lambda: sandwich_norm(x, g1, g1, 1e-6, r32, bf), gb(T * D * 12),
             lambda: rms_norm_weighted(x, gd, 1e-6, residual=r16, return_residual=True), gb(T * D * 8))
        o, z = f32(1, T, 1, D), mk(1, T, D)
        case(f"norm over heads and gate {T}x{D}", lambda: dr.gated_norm(o, z, g1, 1e-6, "sigmoid"), gb(T * D * 8),
             lambda: dr.gated_norm(o.view(1, T, D // 128, 128), z, g1[:128], 1e-6, "sigmoid"), gb(T * D * 8))
    for B, S in ((4, 2048), (32, 1)):
        y, qw, kw, turns = mk(B, S, 768 + 512 + 64), torch.ones(768, device=device), torch.ones(512, device=device), position_turns(64, device=device)
        st = KVCache.allocate(B, 1, 1024, 576, device, bf, ring=True, shared=True)
        pos = torch.full((B,), 5000, dtype=torch.int32, device=device) if S == 1 else None
        case(f"latent norms, rotation and store {B}x{S}", lambda: lt.latent_norm_store(y, qw, kw, turns, 64, 1e-6, q_width=768, width=576, store=st, pos=pos),
             gb(B * S * (1344 * 4 + min(1.0, 1024 / S) * 576 * 2)), lambda: rms_norm_weighted(y, None, 1e-6), gb(B * S * 1344 * 4))
        q, x, bias = mk(B, S, 32, 128), mk(B, S, 24 * 128), f32(24 * 128)
        case(f"rotation of query heads {B}x{S}, 32 heads, 32 of 128 channels", lambda: lt.rotate_heads(q[..., 96:], turns[:16], pos), gb(B * S * 32 * 32 * 4))
        case(f"unit queries and keys and store {B}x{S}, 16/4 heads", lambda: qk_norm_store(x, None, None, 16, 4, 128, 128, 1e-6, dkp=128, dvp=128, bias=bias),
             gb(B * S * 24 * 128 * 4), lambda: rms_norm_weighted(x, None, 1e-6), gb(B * S * 24 * 128 * 4))
    for M, H, N, K in ((1, 32, 512, 64), (32, 32, 512, 64), (32, 32, 64, 512), (32, 128, 512, 128)):
        x, w, y, w2 = mk(M, H, K), mk(H, N, K), mk(M, H, N), mk(H * N * K // 2048, 2048)
        x2 = mk(M, 2048)
        case(f"product per head, {M} rows, {H} x {N} x {K}", lambda: skinny.head_products(x, w, y), gb(2 * (x.numel() + w.numel() + y.numel())),
             lambda: lin(x2, w2), gb(2 * (x2.numel() + w2.numel() + M * w2.shape[0])))
    for M, N, K in ((8192, 8192, 2048),):
        x, w = mk(M, K), mk(N, K)
        case(f"product with xIELU {M}x{N}x{K}", lambda: gemm(x, w, act="xielu", alpha=0.7, beta=1.2), tf(2 * M * N * K), lambda: gemm(x, w, act="relu2"))
    return out


if __name__ == "__main__":
    if sys.argv[1:2] == ["kernels"]:
        kernels(*sys.argv[2:3])
    else:
        print(json.dumps(run()))
