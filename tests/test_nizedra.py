"""Nizedra end to end: configuration and weights, whole prompts, decoding through the session, batches of unequal requests, loops of
layers, generation through the framework's loop and command line, and trace replay, against the plain implementation in
``nizedra_oracle``."""
import json

import pytest
import torch

import nizedra_oracle as O
from tyr_b200.cli import model_runner, trace_run
from tyr_b200.io import safetensors as st
from tyr_b200.models import nizedra as K
from tyr_b200.models import registry
from tyr_b200.models.generation import SamplingStrategy

GPU = pytest.mark.gpu
PLACES = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU), pytest.param(("cuda", torch.bfloat16), marks=GPU)]


def layer(kind, ff, **mixer):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def light(heads, dim, vdim, decay, ff):
    return layer("lightning", ff, heads=heads, dim=dim, vdim=vdim, decay=list(decay))


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, base, ff, dims=None):
    return layer("latent_attention", ff, heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale, mask={"size": window},
                 rot={"base": base, "dims": rot_dim if dims is None else dims})


def talk(heads, kv_heads, dim, vdim, scale, softcap, bias_max, ff):
    return layer("attention", ff, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=softcap, bias_max=bias_max)


def config(vocab, width, eps, layers, loop=None):
    out = {"architecture": "Nizedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CONFIGS = {
    # unequal sizes everywhere, layers without feed-forward, every kind of layer in the loop
    "mixed": config(88, 48, 1e-3, [
        talk(6, 3, 24, 40, 0.3, 4.0, 20, 40), light(3, 16, 24, (0.5, 0.97, 0.999), 72), latent(4, 24, 8, 40, 20, 36, 0.25, 7, 300.0, 0), talk(4, 4, 16, 8, 0.5, 9.0, 30, 0),
        latent(2, 8, 6, 16, 9, 17, 0.4, 11, 50.0, 33)], (1, 4, 2)),
    # every count that can be one is one; the loop spans the whole model
    "ones": config(40, 16, 1e-6, [light(1, 8, 8, (0.9,), 8), latent(1, 8, 2, 8, 1, 1, 1.0, 1, 10.0, 1), talk(1, 1, 8, 1, 1.0, 1.0, 2, 0)], (0, 3, 1)),
    # sizes no tensor-core kernel tiles; no loop
    "odd": config(77, 50, 1e-5, [
        latent(3, 130, 20, 17, 33, 41, 0.1, 13, 2000.0, 13), talk(18, 1, 20, 6, 0.2, 2.0, 9, 21), light(2, 10, 14, (0.8, 0.95), 0), latent(1, 40, 10, 270, 30, 24, 0.15, 30, 80.0, 30, 4),
        light(5, 33, 9, (0.3, 0.6, 0.9, 0.99, 1.0), 25)]),
    # sizes of the fused kernels; a loop that starts the model and one that ends it are "start" and "end"
    "wide": config(120, 128, 1e-5, [
        talk(8, 2, 64, 64, 0.125, 20.0, 100, 192), latent(4, 64, 32, 64, 64, 96, 0.1, 40, 1e4, 128), light(2, 128, 128, (0.9, 0.999), 64),
        latent(2, 96, 32, 128, 96, 64, 0.09, 70, 1e5, 0), talk(4, 4, 128, 128, 0.09, 30.0, 64, 128)], (1, 3, 3)),
    "start": config(96, 64, 1e-5, [latent(2, 32, 16, 32, 32, 48, 0.15, 9, 1e3, 64), light(1, 64, 64, (0.98,), 96), talk(2, 1, 32, 32, 0.2, 5.0, 12, 64)], (0, 1, 4)),
    "end": config(96, 64, 1e-5, [light(2, 32, 64, (0.7, 0.99), 64), talk(3, 3, 16, 32, 0.25, 8.0, 40, 0), light(1, 16, 16, (0.95,), 0)], (2, 3, 2)),
}
ROWS = {"mixed": 10, "ones": 2, "odd": 7, "wide": 16, "start": 8, "end": 16}
TOL = {torch.float32: 1e-4, torch.bfloat16: 0.08}


def weights(name, seed=0):
    """Exact in bf16.  Norms off one, temperatures and mixes that matter, distance tables that outweigh a score, biases everywhere."""
    cfg, gen = CONFIGS[name], torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in K.tensor_shapes(K.NizedraConfig.from_json(cfg)).items():
        last = n.rsplit(".", 1)[-1]
        shape = tuple(ROWS[name] if s is None else s for s in shape)
        t = torch.randn(shape, generator=gen)
        if "norm" in last:
            t = 1.0 + 0.3 * t
        elif last == "temp":
            t = 2.0 + 0.7 * t
        elif last == "talk":
            t = torch.eye(shape[0]) + 0.4 * shape[0] ** -0.5 * t
        elif last in ("rel", "act"):
            pass
        elif last == "b":
            t = 0.3 * t
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
    return K.build(K.NizedraConfig.from_json(CONFIGS[name]), weights(name).__getitem__, *place)


def close(got, want, dtype):
    """Root mean square of the logits' difference at every position."""
    d = got.detach().double().cpu() - want
    err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std()
    assert bool((err < TOL[dtype]).all()) and (err.numel() < 8 or float(err.median()) < TOL[dtype] / 3), err


# ---- configuration, weights, registry -----------------------------------------------------------------------------
@pytest.mark.parametrize("name", CONFIGS)
def test_config_round_trip(name):
    cfg = K.NizedraConfig.from_json(CONFIGS[name])
    assert K.NizedraConfig.from_json(cfg.to_json()) == cfg
    assert registry.detect(CONFIGS[name]).name == "nizedra"


def test_config_errors():
    def broken(edit, match):
        j = json.loads(json.dumps(CONFIGS["mixed"]))
        edit(j["layers"])
        with pytest.raises(ValueError, match=match):
            K.NizedraConfig.from_json(j)
    broken(lambda l: l[0].update(type="delta"), "unknown type")
    broken(lambda l: l[0]["mixer"].pop("softcap"), "lacks softcap")
    broken(lambda l: l[0]["mixer"].update(mask={"size": 3}), "unknown mask")
    broken(lambda l: l[0]["mixer"].update(heads=5), "multiple of kv_heads")
    broken(lambda l: l[0]["mixer"].update(softcap=0.0), "softcap must be positive")
    broken(lambda l: l[1]["mixer"].update(decay=[0.5]), "one number per head")
    broken(lambda l: l[1]["mixer"].update(vdim=0), "must be positive")
    broken(lambda l: l[2]["mixer"]["rot"].update(dims=10), "at most rot_dim")
    broken(lambda l: l[2]["mixer"]["rot"].update(dims=3), "must be even")
    broken(lambda l: l[2]["mixer"]["rot"].pop("base"), "lacks base")
    broken(lambda l: l[2]["mixer"]["mask"].update(size=0), "mask.size must be positive")
    broken(lambda l: l[0]["mlp"].update(kind="moe"), "unknown mlp kind")
    broken(lambda l: l[0]["mlp"].update(ff=0), "ff must be positive")
    for loop in ({"start": 2, "stop": 2, "times": 3}, {"start": 1, "stop": 6, "times": 3}, {"start": 1, "stop": 2, "times": 0}):
        with pytest.raises(ValueError, match="loop must name"):
            K.NizedraConfig.from_json({**CONFIGS["mixed"], "loop": loop})


def test_layer_runs():
    runs = lambda name: K.NizedraConfig.from_json(CONFIGS[name]).runs()
    assert all(runs(n) == O.layer_runs(CONFIGS[n]) for n in CONFIGS)
    assert runs("mixed") == [(0, False), (1, True), (2, False), (3, False), (1, True), (2, False), (3, False), (4, False)]
    assert runs("end") == [(0, False), (1, False), (2, True), (2, True)]
    assert runs("odd") == [(i, False) for i in range(5)]


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
    cfg = K.NizedraConfig.from_json(CONFIGS["mixed"])

    def broken(name, edit, match):
        w = weights("mixed")
        w[name] = edit(w[name])
        with pytest.raises(st.SafeTensorsError, match=match):
            K.build(cfg, w.__getitem__, "cpu", torch.float32)
    broken("l1.mix.q", lambda t: t[:4], "l1.mix.q: expected shape")
    broken("l0.mix.rel", lambda t: t[:, :2], "l0.mix.rel: expected shape")
    broken("loop.in", lambda t: t[:, :48], "loop.in: expected shape")
    w = weights("mixed")
    del w["l2.mix.dkv.norm"]
    st.save_file(w, str(tmp_path / "model.safetensors"))
    with pytest.raises(Exception, match="l2.mix.dkv.norm"):
        K.load(cfg, str(tmp_path / "model.safetensors"), "cpu", torch.float32)


# ---- whole prompts and decoding -----------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name,n", [("mixed", 75), ("ones", 20), ("odd", 40), ("wide", 200), ("mixed", 1), ("mixed", 2), ("wide", 3), ("wide", 64),
                                    ("start", 50), ("end", 70)])
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
                                          ("wide", 200, 63), ("wide", 200, 128), ("wide", 200, 149), ("start", 50, 8), ("start", 50, 9), ("end", 70, 33)])
def test_decoding_continues_a_prompt(place, name, n, first):
    """Cuts before, at and past the windows and chunks; windows that pass over decoded tokens."""
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


def test_every_pass_has_stores_and_states_of_its_own():
    s = K.CacheSession(model("mixed", ("cpu", torch.float32)), 3, 20)
    assert [c is not None for c in s.kv] == [True, False, True, True, False, True, True, True]
    assert len({c.k.data_ptr() for c in s.kv if c is not None}) == 6 and s.lin[1].rec.data_ptr() != s.lin[4].rec.data_ptr()
    assert [(c.cap, c.ring, c.v is c.k) for c in s.kv if c is not None] == [(20, False, False), (7, True, True), (20, False, False), (7, True, True),
                                                                             (20, False, False), (11, True, True)]
    s.retain([2, 0])
    assert all(c is None or (c.k.shape[0] == 2 and c.v.shape[0] == 2) for c in s.kv) and s.lin[4].rec.shape[0] == 2
    before = [t.clone() for t in (s.lin[1].rec, s.lin[4].rec)]
    s.prefill(torch.tensor([[1, 2, 3]] * 2))
    assert not torch.equal(before[0], s.lin[1].rec) and not torch.equal(s.lin[1].rec, s.lin[4].rec)


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
