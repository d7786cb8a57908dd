"""Vonulix end to end: configuration and weights, whole prompts, decoding through the session, batches of unequal requests, generation
through the framework's loop and command line, and trace replay, against the plain implementation in ``vonulix_oracle``."""
import json

import pytest
import torch

import vonulix_oracle as O
from tyr_b200.cli import model_runner, trace_run
from tyr_b200.io import safetensors as st
from tyr_b200.models import registry
from tyr_b200.models import vonulix as V
from tyr_b200.models.generation import SamplingStrategy

GPU = pytest.mark.gpu
PLACES = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU), pytest.param(("cuda", torch.bfloat16), marks=GPU)]


def attn(heads, kv_heads, dim, vdim, scale, base, dims, factor, mask):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if factor is not None:
        out["rot"]["scaling"] = {"factor": factor}
    if mask is not None:
        out["mask"] = dict(zip(("size", "keep_first"), mask))
    return out


def experts(n, top, ff, limit, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": n, "top": top}}
    if shared:
        out["shared"] = dict(zip(("ff", "limit"), shared))
    return out


def config(vocab, width, eps, scale, side, layers):
    return {"architecture": "Vonulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "token_side": {"dim": side},
            "layers": [{"type": "attention", "mixer": m, "mlp": p} for m, p in layers]}


CONFIGS = {
    # unequal sizes everywhere, a layer without feed-forward, one without a shared expert, more kept positions than the window, no window
    "mixed": config(88, 48, 1e-3, 2.5, 12, [
        (attn(6, 3, 24, 40, 0.3, 300.0, 16, 1.5, (7, 3)), experts(8, 3, 20, 0.8, (36, 1.2))), (attn(4, 4, 16, 8, 0.4, 50.0, 16, None, (11, 0)), None),
        (attn(8, 1, 32, 16, 0.2, 1e4, 8, 3.0, (5, 13)), experts(5, 1, 40, 0.5)), (attn(2, 1, 8, 24, 0.5, 20.0, 4, 1.0, None), experts(4, 4, 12, 2.0, (8, 0.3)))]),
    # every count that can be one is one
    "ones": config(40, 16, 1e-6, 1.0, 1, [(attn(1, 1, 2, 2, 1.0, 10.0, 2, 1.0, (1, 1)), experts(1, 1, 1, 1.0, (1, 1.0)))]),
    # sizes no tensor-core kernel tiles
    "odd": config(77, 50, 1e-5, 3.0, 5, [
        (attn(3, 3, 140, 18, 0.1, 2000.0, 20, 2.0, (13, 2)), experts(6, 2, 13, 0.9, (11, 0.6))), (attn(18, 1, 21, 6, 0.25, 80.0, 10, 1.2, (6, 1)), experts(3, 1, 7, 1.5)),
        (attn(2, 1, 10, 134, 0.3, 500.0, 0, 1.0, (30, 5)), None)]),
    # sizes of the fused kernels; windows and kept positions over more than one block of keys
    "wide": config(120, 128, 1e-5, 2.0, 32, [
        (attn(8, 2, 64, 64, 0.125, 1e4, 32, 4.0, (40, 6)), experts(16, 4, 96, 0.7, (160, 1.1))), (attn(6, 2, 96, 48, 0.1, 1e3, 96, 2.0, (70, 130)), experts(8, 2, 128, 1.0, (64, 0.5))),
        (attn(4, 4, 128, 128, 0.09, 1e5, 64, 1.0, (129, 1)), experts(4, 1, 64, 0.4)), (attn(16, 1, 32, 80, 0.2, 100.0, 32, 8.0, (33, 20)), None)]),
    # many thin layers for the average over depth
    "deep": config(96, 64, 1e-5, 1.5, 8, [(attn(2, 1, 32, 32, 0.2, 1e3, 16, 1.0, (9 + i, i % 3)), experts(4, 1 + i % 3, 32, 1.0, (32, 1.0)) if i % 4 else None) for i in range(11)]),
}
TOL = {torch.float32: 1e-4, torch.bfloat16: 0.04}
KINDS = 4                                 # the tokens fall into kinds; a channel for each decides the experts


def weights(name, seed=0):
    """Exact in bf16.  Averages over depth with weight on every earlier result.  The first channels of the embedding tell a token's kind, no
    layer writes them, and the routers read little else, so that 16-bit arithmetic cannot turn a choice of experts."""
    cfg, gen = CONFIGS[name], torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in V.tensor_shapes(V.VonulixConfig.from_json(cfg)).items():
        last = n.rsplit(".", 1)[-1]
        t = torch.randn(shape, generator=gen)
        if n.endswith("side.norm"):
            t = 0.5 + 0.2 * t
            t[:KINDS] = 0
        elif "norm" in last:
            t = 0.3 * t
            t[:KINDS] = 0
        elif last == "dwa":
            t = 0.3 * t
            t[0] = t[0].abs() + 0.4
            t[-1] = 0.8
        elif last == "router":
            t = 0.003 * t
            for c in range(KINDS):
                t[torch.randperm(shape[0], generator=gen), c] = torch.linspace(-1.2, 1.2, shape[0]) if shape[0] > 1 else torch.ones(1)
        elif n == "embed":
            t = t / cfg["embedding"]["scale"]
            t[:, :KINDS] = 2.5 / cfg["embedding"]["scale"] * torch.eye(KINDS)[torch.arange(shape[0]) % KINDS]
        elif n != "side.embed":
            t = t * shape[-1] ** -0.5
            if last in ("o", "down", "proj"):
                t[:KINDS] = 0
        out[n] = t.bfloat16()
    return out


def tokens(name, n, seed=1):
    return torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


_known = {}


def expected(name, toks):
    key = (name, tuple(toks))
    if key not in _known:
        _known[key] = O.logits(CONFIGS[name], {k: v.double() for k, v in weights(name).items()}, toks)
    return _known[key]


def model(name, place):
    return V.build(V.VonulixConfig.from_json(CONFIGS[name]), weights(name).__getitem__, *place)


def close(got, want, dtype):
    """Root mean square of the logits' difference at every position."""
    d = got.detach().double().cpu() - want
    err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std()
    assert bool((err < TOL[dtype]).all()) and (err.numel() < 8 or float(err.median()) < TOL[dtype] / 3), err


# ---- configuration, weights, registry -----------------------------------------------------------------------------
@pytest.mark.parametrize("name", CONFIGS)
def test_config_round_trip(name):
    cfg = V.VonulixConfig.from_json(CONFIGS[name])
    assert V.VonulixConfig.from_json(cfg.to_json()) == cfg
    assert registry.detect(CONFIGS[name]).name == "vonulix"


def test_config_errors():
    def broken(edit, match):
        j = json.loads(json.dumps(CONFIGS["mixed"]))
        edit(j["layers"])
        with pytest.raises(ValueError, match=match):
            V.VonulixConfig.from_json(j)
    broken(lambda l: l[0].update(type="delta"), "unknown type")
    broken(lambda l: l[0]["mixer"].pop("scale"), "lacks scale")
    broken(lambda l: l[0]["mixer"].update(softcap=3), "unknown softcap")
    broken(lambda l: l[0]["mixer"].update(heads=5), "multiple of kv_heads")
    broken(lambda l: l[1]["mixer"].update(vdim=0), "must be positive")
    broken(lambda l: l[1]["mixer"].update(vdim=7), "must be even")
    broken(lambda l: l[2]["mixer"]["rot"].update(dims=34), "at most dim")
    broken(lambda l: l[2]["mixer"]["rot"].update(dims=3), "must be even")
    broken(lambda l: l[2]["mixer"]["rot"].pop("base"), "lacks base")
    broken(lambda l: l[2]["mixer"]["rot"]["scaling"].update(factor=0.0), "factor must be positive")
    broken(lambda l: l[2]["mixer"]["mask"].update(size=0), "mask.size must be positive")
    broken(lambda l: l[2]["mixer"]["mask"].update(keep_first=-1), "keep_first not negative")
    broken(lambda l: l[0]["mlp"].update(kind="dense"), "unknown mlp kind")
    broken(lambda l: l[0]["mlp"]["router"].update(top=9), "top must lie")
    broken(lambda l: l[0]["mlp"]["expert"].pop("limit"), "lacks limit")
    with pytest.raises(ValueError, match="token_side.dim"):
        V.VonulixConfig.from_json({**CONFIGS["mixed"], "token_side": {"dim": 0}})


def test_kinds_decide_the_experts():
    """What the 16-bit tests rest on: no choice of experts is a close call."""
    for name, n in (("mixed", 60), ("wide", 60), ("odd", 40), ("deep", 40)):
        cfg, w, gap = CONFIGS[name], {k: v.double() for k, v in weights(name).items()}, []
        seen = O.expert_mixture

        def watch(w, p, mlp, x):
            z = (x @ w[p + "router"].T).sort(-1, descending=True).values
            if mlp["router"]["top"] < z.shape[1]:
                gap.append(float((z[:, mlp["router"]["top"] - 1] - z[:, mlp["router"]["top"]]).min()))
            return seen(w, p, mlp, x)
        O.expert_mixture = watch
        try:
            O.residual_stream(cfg, w, tokens(name, n))
        finally:
            O.expert_mixture = seen
        assert min(gap) > 0.04, (name, gap)


def save(tmp_path, name):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS[name]))
    st.save_file(weights(name), str(tmp_path / "model.safetensors"))
    return str(tmp_path)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", CONFIGS)
def test_weights_round_trip(tmp_path, name, dtype):
    m = registry.detect_dir(save(tmp_path, name)).load(str(tmp_path), "cpu", dtype)
    sd, w = V.state_dict(m), weights(name)
    assert set(sd) == set(w)
    for k in w:
        assert sd[k].shape == w[k].shape and torch.equal(sd[k].float(), w[k].float()), k


@GPU
def test_weights_round_trip_after_the_experts_took_their_layout():
    m = model("wide", ("cuda", torch.bfloat16))
    V.forward(m, torch.tensor([tokens("wide", 9)], device="cuda"))
    sd, w = V.state_dict(m), weights("wide")
    assert all(torch.equal(sd[k].float().cpu(), w[k].float()) for k in w)


def test_missing_or_misshapen_weights_are_named(tmp_path):
    cfg = V.VonulixConfig.from_json(CONFIGS["mixed"])

    def broken(name, edit, match):
        w = weights("mixed")
        w[name] = edit(w[name])
        with pytest.raises(st.SafeTensorsError, match=match):
            V.build(cfg, w.__getitem__, "cpu", torch.float32)
    broken("l1.mix.q", lambda t: t[:4], "l1.mix.q: expected shape")
    broken("l2.dwa", lambda t: t[:3], "l2.dwa: expected shape")
    broken("side.embed", lambda t: t[:, :12], "side.embed: expected shape")
    w = weights("mixed")
    del w["l3.mlp.shared.sg"]
    st.save_file(w, str(tmp_path / "model.safetensors"))
    with pytest.raises(Exception, match="l3.mlp.shared.sg"):
        V.load(cfg, str(tmp_path / "model.safetensors"), "cpu", torch.float32)


# ---- whole prompts and decoding -----------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name,n", [("mixed", 75), ("ones", 20), ("odd", 40), ("wide", 300), ("mixed", 1), ("mixed", 2), ("mixed", 140), ("wide", 3), ("wide", 64), ("deep", 40)])
def test_whole_prompt(place, name, n):
    toks = tokens(name, n)
    got = V.forward(model(name, place), torch.tensor([toks], device=place[0]))
    close(got[0], expected(name, toks), place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["mixed", "deep"])
def test_residual_stream_after_every_layer(place, name):
    toks = tokens(name, 30)
    m, seen = model(name, place), []
    V.CacheSession(m, 1, 30).hidden(torch.tensor([toks], device=m.device), layer_done=lambda i, x: seen.append((i, x[0].clone())))
    want = O.residual_stream(CONFIGS[name], {k: v.double() for k, v in weights(name).items()}, toks)
    assert [i for i, _ in seen] == list(range(len(want))) and all(x.dtype == torch.float32 for _, x in seen)
    for (_, x), w in zip(seen, want):
        close(x, w, place[1])


def run_split(m, toks, first):
    """Logits of every position from ``first`` - 1 on: a prompt of ``first`` tokens, then one by one."""
    s = V.CacheSession(m, 1, len(toks))
    out = [s.prefill(torch.tensor([toks[:first]], device=m.device))[0].clone()]
    for t in toks[first:]:
        out.append(s.step(torch.tensor([t], device=m.device))[0].clone())
    return torch.stack(out)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name,n,first", [("mixed", 75, 1), ("mixed", 75, 2), ("mixed", 75, 4), ("mixed", 75, 10), ("mixed", 75, 40), ("ones", 20, 1), ("odd", 40, 5), ("wide", 300, 128),
                                          ("wide", 300, 46), ("wide", 300, 199), ("wide", 300, 200), ("wide", 300, 201), ("deep", 40, 9)])
def test_decoding_continues_a_prompt(place, name, n, first):
    """Cuts before, at and past the windows and the kept positions; windows that pass over decoded tokens."""
    toks = tokens(name, n)
    close(run_split(model(name, place), toks, first), expected(name, toks)[first - 1:], place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name,lens", [("mixed", (40, 1, 23, 9)), ("wide", (3, 170, 64)), ("odd", (2, 20))])
def test_unequal_requests_in_one_batch(place, name, lens):
    """Every request of a batch as alone: prompts, 20 decoded tokens, requests that end early and give their rows back."""
    m, steps = model(name, place), 20
    seqs = [tokens(name, n + steps, seed=7 + i) for i, n in enumerate(lens)]
    pad = max(lens)
    ids = torch.tensor([s[:n] + [0] * (pad - n) for s, n in zip(seqs, lens)], device=m.device)
    sess = V.CacheSession(m, len(lens), pad + steps)
    out = [[x] for x in sess.prefill(ids, lens).clone()]
    rows, stop = list(range(len(lens))), {0: 5, 2: 11}
    for t in range(steps):
        gone = [r for r in rows if stop.get(r) == t]
        if gone:
            before = sess.state_bytes()
            sess.retain([i for i, r in enumerate(rows) if r not in gone])
            rows = [r for r in rows if r not in gone]
            assert sess.state_bytes() * (len(rows) + len(gone)) == before * len(rows)
        lg = sess.step(torch.tensor([seqs[r][lens[r] + t] for r in rows], device=m.device)).clone()
        for i, r in enumerate(rows):
            out[r].append(lg[i])
    got = torch.cat([torch.stack(o) for o in out])
    want = torch.cat([expected(name, s[:n + len(o) - 1])[n - 1:] for s, n, o in zip(seqs, lens, out)])
    close(got, want, place[1])


@GPU
def test_a_batch_too_large_for_the_weight_streaming_experts():
    """70 rows decode through the sorted experts, as each row does alone."""
    m, seqs = model("wide", ("cuda", torch.bfloat16)), [tokens("wide", 12, seed=i) for i in range(70)]
    s = V.CacheSession(m, 70, 12)
    out = [s.prefill(torch.tensor([q[:8] for q in seqs], device="cuda")).clone()]
    for t in range(8, 12):
        out.append(s.step(torch.tensor([q[t] for q in seqs], device="cuda")).clone())
    got = torch.stack(out, 1)
    for r in (0, 33, 69):
        close(got[r], expected("wide", seqs[r])[7:], torch.bfloat16)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding(place, name):
    toks = tokens(name, 300, seed=3)
    close(run_split(model(name, place), toks, 4)[-90:], expected(name, toks)[-90:], place[1])


@pytest.mark.parametrize("place", PLACES)
def test_a_new_session_sees_nothing_of_the_last(place):
    """The same memory used again: a session's logits do not depend on what ran before it, and other rows do not matter."""
    m = model("wide", place)
    toks = tokens("wide", 90, seed=5)
    alone = run_split(m, toks, 80)
    noise = V.CacheSession(m, 3, 200)
    noise.prefill(torch.tensor([tokens("wide", 150, seed=s) for s in (6, 7, 8)], device=m.device))
    noise.step(torch.tensor([1, 2, 3], device=m.device))
    del noise
    close(run_split(m, toks, 80), alone.double().cpu(), torch.float32)


@pytest.mark.parametrize("place", PLACES)
def test_session_rules(place):
    m = model("mixed", place)
    s = V.CacheSession(m, 2, 10)
    ids = torch.zeros(2, 9, dtype=torch.long, device=place[0])
    with pytest.raises(ValueError, match="lengths"):
        s.hidden(ids, [9, 10])
    with pytest.raises(ValueError, match="fresh session"):
        s.hidden(ids[:1])
    s.prefill(ids)
    with pytest.raises(ValueError, match="fresh session"):
        s.hidden(ids)
    s.step(ids[:, 0])
    with pytest.raises(ValueError, match="overflow"):
        s.step(ids[:, 0])
    with pytest.raises(ValueError, match="capacity"):
        V.CacheSession(m, 1, 0)


def test_stores_hold_the_window_and_the_kept_positions():
    m = model("mixed", ("cpu", torch.float32))
    assert [(c.cap, c.ring, c.keep) for c in V.CacheSession(m, 2, 100).kv] == [(10, True, 3), (11, True, 0), (18, True, 13), (100, False, 0)]
    assert [(c.cap, c.ring, c.keep) for c in V.CacheSession(m, 2, 11).kv] == [(10, True, 3), (11, False, 0), (11, False, 0), (11, False, 0)]
    s = V.CacheSession(m, 3, 100)
    s.retain([2, 0])
    assert all(c.k.shape[0] == c.v.shape[0] == 2 for c in s.kv)
    assert m.turns(8, 50.0, 1.0, 50) is m.turns(8, 50.0, 1.0, 100)          # tables are shared and only grow


# ---- generation ---------------------------------------------------------------------------------------------------
def greedy_oracle(name, prompt, n):
    seq = list(prompt)
    w = {k: v.double() for k, v in weights(name).items()}
    for _ in range(n):
        seq.append(int(O.logits(CONFIGS[name], w, seq)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("place", PLACES[:2])
def test_greedy_generation_of_unequal_prompts(place):
    m = model("mixed", place)
    prompts = [tokens("mixed", n, seed=20 + n) for n in (11, 3, 18)]
    ids, lengths = model_runner.right_pad(prompts, 0)
    out = V.generate_greedy(m, ids.to(place[0]), 8, lengths=lengths)[:, ids.shape[1]:].tolist()
    for p, row in zip(prompts, out):
        assert row == greedy_oracle("mixed", p, 8)


@GPU
def test_generation_through_the_captured_step():
    """16-bit generation: every token is the argmax of the session's own logits, and those are the oracle's."""
    m = model("wide", ("cuda", torch.bfloat16))
    p = tokens("wide", 30, seed=9)
    got = V.generate_greedy(m, torch.tensor([p], device="cuda"), 12)[0].tolist()
    assert got[:30] == p
    lg = run_split(m, got, 30)
    assert lg[:-1].argmax(-1).tolist() == got[30:]
    close(lg, expected("wide", got)[29:], torch.bfloat16)


def test_sampling_and_stop_tokens():
    m = model("mixed", ("cpu", torch.float32))
    ids = torch.tensor([tokens("mixed", 5)])
    first = greedy_oracle("mixed", ids[0].tolist(), 1)[0]
    assert V.generate(m, ids, 6, SamplingStrategy.greedy(), eos_token_ids=[first]).shape[1] == 6
    g = lambda: torch.Generator().manual_seed(5)
    a, b = (V.generate(m, ids, 6, SamplingStrategy.multinomial(0.8, 20, 0.9), generator=g()) for _ in range(2))
    assert torch.equal(a, b) and a.shape[1] == 11


def test_command_line_generates_from_token_ids(tmp_path, capsys):
    d = save(tmp_path, "mixed")
    p = tokens("mixed", 6)
    (tmp_path / "prompts.txt").write_text(" ".join(map(str, p)) + "\n" + ", ".join(map(str, p[:2])) + "\n")
    assert model_runner.main(["--source", d, "--prompt-file", str(tmp_path / "prompts.txt"), "--batch-size", "2", "--max-new-tokens", "4", "--device", "cpu"]) == 0
    lines = capsys.readouterr().out.splitlines()
    got = [[int(t) for t in l.split()] for l in lines if not l.startswith(">")]
    assert got == [greedy_oracle("mixed", p, 4), greedy_oracle("mixed", p[:2], 4)]


# ---- trace replay -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
def test_trace_replay(tmp_path, capsys, place):
    d = save(tmp_path, "mixed")
    a, b, c = (tokens("mixed", n, seed=n) for n in (30, 14, 22))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}, {"id": "b", "tokens": b[:12], "want": [11]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [b[12]], "want": [0]}, {"id": "a", "tokens": [a[20]], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[21]], "want": []}, {"id": "b", "tokens": [b[13]], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": c[:21]}], "end": []},
             {"step": 4, "entries": [{"id": "a", "tokens": [a[22]], "want": [0]}], "end": ["a"]},
             {"step": 5, "entries": [{"id": "c", "tokens": [c[21]], "want": [0]}], "end": ["c"]}]
    dtype = "bfloat16" if place[1] == torch.bfloat16 else "float32"
    out = tmp_path / "out"
    argv = ["--model", d, "--dtype", dtype, "--out", str(out), "--max-tokens", "64", "--device", place[0]]
    assert trace_run.main(argv, [json.dumps(s) for s in steps]) == 0
    assert capsys.readouterr().out.split() == [x for s in steps for x in ("done", str(s["step"]))]
    got = torch.cat([torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).reshape(-1, 88) for i in (0, 1, 2, 4, 5)])
    ea, eb, ec = (expected("mixed", t) for t in (a, b, c))
    close(got, torch.stack([ea[0], ea[19], eb[11], eb[12], eb[13], ea[22], ec[21]]), place[1])
