"""Kinetar end to end: configuration and weights, whole prompts, decoding through the session, batches of unequal requests, generation
through the framework's loop and command line, and trace replay, against the plain implementation in ``kinetar_oracle``."""
import json

import pytest
import torch

import kinetar_oracle as O
from tyr_b200.cli import model_runner, trace_run
from tyr_b200.io import safetensors as st
from tyr_b200.models import kinetar as K
from tyr_b200.models import registry
from tyr_b200.models.generation import SamplingStrategy

GPU = pytest.mark.gpu
PLACES = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU), pytest.param(("cuda", torch.bfloat16), marks=GPU)]


def par(heads, kv_heads, dim, conv, scale, temp, inner, state, dt_rank, rconv, ls, rs, ff):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "scale": scale, "q_temp": {"coef": temp[0], "every": temp[1]}},
        "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": rconv}, "left_scale": ls, "right_scale": rs},
        "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads, kv_heads, dim, vdim, conv, ff):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(vocab, width, eps, scale, logit_scale, layers):
    return {"architecture": "Kinetar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "logit_scale": logit_scale,
            "layers": layers}


CONFIGS = {
    # unequal sizes everywhere, layers without feed-forward, grouped keys in both mixers
    "mixed": config(88, 48, 1e-3, 1.7, 0.4, [
        delta(4, 2, 16, 24, 3, 40), par(6, 3, 24, 2, 0.3, (0.7, 9), 56, 12, 5, 4, 0.8, 1.3, 72), par(4, 4, 16, 5, 0.25, (0.2, 30), 32, 20, 8, 3, 1.5, 0.5, 0),
        delta(3, 3, 40, 8, 2, 0)]),
    # every count that can be one is one
    "ones": config(40, 16, 1e-6, 1.0, 1.0, [delta(1, 1, 8, 8, 1, 8), par(1, 1, 8, 1, 1.0, (1.0, 1), 1, 1, 1, 1, 1.0, 1.0, 1)]),
    # sizes no tensor-core kernel tiles
    "odd": config(77, 50, 1e-5, 0.9, 1.1, [
        par(18, 1, 20, 6, 0.2, (0.3, 4), 37, 70, 9, 5, 0.7, 0.9, 13), delta(3, 1, 10, 14, 2, 21), par(2, 1, 130, 3, 0.1, (0.4, 11), 50, 3, 50, 2, 1.1, 0.6, 30),
        delta(2, 2, 12, 130, 9, 0)]),
    # head sizes of the fused kernels, a first layer that is not followed by its own kind
    "wide": config(120, 128, 1e-5, 0.8, 1.5, [
        par(4, 2, 128, 4, 0.09, (0.5, 50), 128, 16, 24, 4, 0.9, 1.2, 192), delta(2, 1, 128, 128, 4, 128), delta(2, 2, 64, 128, 3, 64),
        par(3, 1, 64, 2, 0.15, (0.25, 16), 64, 32, 32, 4, 1.2, 0.7, 128)]),
}
RANKS = {"mixed": (5, 20), "ones": (1, 1), "odd": (7, 33), "wide": (32, 48)}
TOL = {torch.float32: 1e-4, torch.bfloat16: 0.08}


def weights(name, seed=0):
    """Exact in bf16.  Sharp queries and keys, sinks that matter, decays from forgetful to nearly lossless, norms off one."""
    cfg, gen = CONFIGS[name], torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in K.tensor_shapes(K.KinetarConfig.from_json(cfg)).items():
        last = n.rsplit(".", 1)[-1]
        shape = tuple(RANKS[name]["g" in last] if s is None else s for s in shape)
        t = torch.randn(shape, generator=gen)
        if last in ("norm1",) or n == "final.norm":
            t = 0.3 * t
        elif n.endswith("mix.norm") or last == "D":
            t = 1.0 + 0.3 * t
        elif last == "A_log":
            t = torch.linspace(-5.0, 0.5, t.numel()).reshape(shape) if t.numel() > 1 else torch.tensor([-1.0]).reshape(shape)
        elif last == "dt_bias" or n.endswith("dt.b"):
            t = -2.0 + 0.6 * t
        elif last == "sink":
            t = 1.0 + 1.5 * t
        elif n.endswith("conv.b"):
            t = 0.2 * t
        elif n.endswith(".conv"):
            t = t * shape[-1] ** -0.5 + 0.3
        elif n != "embed":
            t = t * shape[-1] ** -0.5
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
    return K.build(K.KinetarConfig.from_json(CONFIGS[name]), weights(name).__getitem__, *place)


def close(got, want, dtype):
    """Root mean square of the logits' difference at every position."""
    d = got.detach().double().cpu() - want
    err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std()
    assert bool((err < TOL[dtype]).all()) and float(err.median()) < TOL[dtype] / 3, err


# ---- configuration, weights, registry -----------------------------------------------------------------------------
@pytest.mark.parametrize("name", CONFIGS)
def test_config_round_trip(name):
    cfg = K.KinetarConfig.from_json(CONFIGS[name])
    assert K.KinetarConfig.from_json(cfg.to_json()) == cfg
    assert registry.detect(CONFIGS[name]).name == "kinetar"


def test_config_errors():
    def broken(edit, match):
        j = json.loads(json.dumps(CONFIGS["mixed"]))
        edit(j["layers"])
        with pytest.raises(ValueError, match=match):
            K.KinetarConfig.from_json(j)
    broken(lambda l: l[0].update(type="delta"), "unknown type")
    broken(lambda l: l[1]["mixer"]["left"].pop("scale"), "lacks scale")
    broken(lambda l: l[1]["mixer"]["left"].update(window=3), "unknown window")
    broken(lambda l: l[1]["mixer"]["left"].update(heads=5), "multiple of kv_heads")
    broken(lambda l: l[1]["mixer"]["left"].update(vdim=8), "vdim must equal dim")
    broken(lambda l: l[1]["mixer"]["left"]["q_temp"].update(every=0), "every must be positive")
    broken(lambda l: l[1]["mixer"]["right"].update(state=0), "sizes of the scan")
    broken(lambda l: l[1]["mixer"]["right"].update(conv=0), "at least one tap")
    broken(lambda l: l[0]["mixer"].update(kv_heads=3), "multiple of kv_heads")
    broken(lambda l: l[0]["mlp"].update(kind="moe"), "unknown mlp kind")
    broken(lambda l: l[0]["mlp"].update(ff=0), "ff must be positive")


def save(tmp_path, name):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS[name]))
    st.save_file(weights(name), str(tmp_path / "model.safetensors"))
    return str(tmp_path)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", CONFIGS)
def test_weights_round_trip(tmp_path, name, dtype):
    m = registry.detect_dir(save(tmp_path, name)).load(str(tmp_path), "cpu", dtype)
    sd, w = K.state_dict(m), weights(name)
    assert set(sd) == set(w)
    for k in w:
        assert sd[k].shape == w[k].shape and torch.equal(sd[k].float(), w[k].float()), k


def test_missing_or_misshapen_weights_are_named(tmp_path):
    cfg = K.KinetarConfig.from_json(CONFIGS["mixed"])

    def broken(name, edit, match):
        w = weights("mixed")
        w[name] = edit(w[name])
        with pytest.raises(st.SafeTensorsError, match=match):
            K.build(cfg, w.__getitem__, "cpu", torch.float32)
    broken("l1.mix.left.q", lambda t: t[:4], "l1.mix.left.q: expected shape")
    broken("l0.mix.a2", lambda t: t[:, :2], "ranks of a pair differ")
    w = weights("mixed")
    del w["l1.mix.right.D"]
    st.save_file(w, str(tmp_path / "model.safetensors"))
    with pytest.raises(Exception, match="l1.mix.right.D"):
        K.load(cfg, str(tmp_path / "model.safetensors"), "cpu", torch.float32)


# ---- whole prompts and decoding -----------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name,n", [("mixed", 75), ("ones", 20), ("odd", 40), ("wide", 200), ("mixed", 1), ("mixed", 2), ("wide", 3), ("wide", 64)])
def test_whole_prompt(place, name, n):
    toks = tokens(name, n)
    got = K.forward(model(name, place), torch.tensor([toks], device=place[0]))
    close(got[0], expected(name, toks), place[1])


@pytest.mark.parametrize("place", PLACES)
def test_residual_stream_after_every_layer(place):
    toks = tokens("mixed", 30)
    m, seen = model("mixed", place), []
    K.CacheSession(m, 1, 30).hidden(torch.tensor([toks], device=m.device), layer_done=lambda i, x: seen.append((i, x[0].clone())))
    want = O.residual_stream(CONFIGS["mixed"], {k: v.double() for k, v in weights("mixed").items()}, toks)
    assert [i for i, _ in seen] == list(range(len(want))) and all(x.dtype == torch.float32 for _, x in seen)
    for (_, x), w in zip(seen, want):
        close(x, w, place[1])


def run_split(m, toks, first):
    """Logits of every position from ``first`` - 1 on: a prompt of ``first`` tokens, then one by one."""
    s = K.CacheSession(m, 1, len(toks))
    out = [s.prefill(torch.tensor([toks[:first]], device=m.device))[0].clone()]
    for t in toks[first:]:
        out.append(s.step(torch.tensor([t], device=m.device))[0].clone())
    return torch.stack(out)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name,n,first", [("mixed", 75, 1), ("mixed", 75, 2), ("mixed", 75, 4), ("mixed", 75, 40), ("ones", 20, 1), ("odd", 40, 5), ("wide", 200, 1),
                                          ("wide", 200, 63), ("wide", 200, 128), ("wide", 200, 149)])
def test_decoding_continues_a_prompt(place, name, n, first):
    """Cuts inside the convolutions' reach, at and past a chunk, around the query temperature's steps."""
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
    sess = K.CacheSession(m, len(lens), pad + steps)
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


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding(place, name):
    toks = tokens(name, 280, seed=3)
    close(run_split(model(name, place), toks, 4)[-120:], expected(name, toks)[-120:], place[1])


@pytest.mark.parametrize("place", PLACES)
def test_a_new_session_sees_nothing_of_the_last(place):
    """The same memory used again: a session's logits do not depend on what ran before it, and other rows do not matter."""
    m = model("wide", place)
    toks = tokens("wide", 90, seed=5)
    alone = run_split(m, toks, 80)
    noise = K.CacheSession(m, 3, 200)
    noise.prefill(torch.tensor([tokens("wide", 150, seed=s) for s in (6, 7, 8)], device=m.device))
    noise.step(torch.tensor([1, 2, 3], device=m.device))
    del noise
    close(run_split(m, toks, 80), alone.double().cpu(), torch.float32)


@pytest.mark.parametrize("place", PLACES)
def test_session_rules(place):
    m = model("mixed", place)
    s = K.CacheSession(m, 2, 10)
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
        K.CacheSession(m, 1, 0)


def test_one_store_serves_keys_and_values():
    s = K.CacheSession(model("mixed", ("cpu", torch.float32)), 3, 20)
    assert [c is not None for c in s.kv] == [False, True, True, False]
    assert all(c is None or c.v is c.k for c in s.kv)
    s.retain([2, 0])
    assert all(c is None or (c.v is c.k and c.k.shape[0] == 2) for c in s.kv) and all(t.shape[0] == 2 for l in s.lin for t in l.tensors())


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
    out = K.generate_greedy(m, ids.to(place[0]), 8, lengths=lengths)[:, ids.shape[1]:].tolist()
    for p, row in zip(prompts, out):
        assert row == greedy_oracle("mixed", p, 8)


@GPU
def test_generation_through_the_captured_step():
    """16-bit generation: every token is the argmax of the session's own logits, and those are the oracle's."""
    m = model("wide", ("cuda", torch.bfloat16))
    p = tokens("wide", 30, seed=9)
    got = K.generate_greedy(m, torch.tensor([p], device="cuda"), 12)[0].tolist()
    assert got[:30] == p
    lg = run_split(m, got, 30)
    assert lg[:-1].argmax(-1).tolist() == got[30:]
    close(lg, expected("wide", got)[29:], torch.bfloat16)


def test_sampling_and_stop_tokens():
    m = model("mixed", ("cpu", torch.float32))
    ids = torch.tensor([tokens("mixed", 5)])
    first = greedy_oracle("mixed", ids[0].tolist(), 1)[0]
    assert K.generate(m, ids, 6, SamplingStrategy.greedy(), eos_token_ids=[first]).shape[1] == 6
    g = lambda: torch.Generator().manual_seed(5)
    a, b = (K.generate(m, ids, 6, SamplingStrategy.multinomial(0.8, 20, 0.9), generator=g()) for _ in range(2))
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
