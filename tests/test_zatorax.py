"""Zatorax end to end: configuration and weights, whole prompts, decoding through the session, batches of unequal requests, generation
through the framework's loop and command line, and trace replay, against the plain implementation in ``zatorax_oracle``."""
import json

import pytest
import torch

import zatorax_oracle as O
from tyr_b200.cli import model_runner, trace_run
from tyr_b200.io import safetensors as st
from tyr_b200.models import registry
from tyr_b200.models import zatorax as Z
from tyr_b200.models.generation import SamplingStrategy

GPU = pytest.mark.gpu
PLACES = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU), pytest.param(("cuda", torch.bfloat16), marks=GPU)]


def moe(experts=8, top=3, ff=24, groups=None, shared=16):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r, **({"shared": {"ff": shared}} if shared else {})}


def delta(heads, kv_heads, dim, vdim, conv, mlp):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def attn(heads, kv_heads, dim, vdim, scale, size, mlp, kv_from=None):
    mix = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}
    return {"type": "attention", "mixer": {**mix, **({"kv_from": kv_from} if kv_from is not None else {})}, "mlp": mlp}


CONFIGS = {
    # unequal sizes everywhere, a layer without feed-forward, readers of a layer's keys with wider and narrower windows
    "mixed": {"architecture": "Zatorax", "vocab": 88, "width": 48, "norm": {"eps": 1e-4}, "layers": [
        attn(6, 3, 24, 40, 0.21, 9, moe(groups=(4, 2))),
        delta(4, 2, 16, 24, 3, moe(6, 2, 40, None, 8)),
        attn(3, 3, 24, 40, 0.17, 17, None, kv_from=0),
        delta(3, 3, 40, 8, 6, None),
        attn(4, 1, 16, 16, 0.4, 33, moe(12, 4, 16, (3, 1), 0)),
        attn(2, 1, 16, 16, 0.3, 5, moe(4, 1, 8, (2, 2)), kv_from=4)]},
    # every count that can be one is one
    "ones": {"architecture": "Zatorax", "vocab": 40, "width": 16, "norm": {"eps": 1e-6}, "layers": [
        delta(1, 1, 8, 8, 1, moe(1, 1, 8, (1, 1), 8)), attn(1, 1, 8, 8, 1.0, 1, moe(2, 1, 8, (2, 1), 8))]},
    # sizes no tensor-core kernel tiles
    "odd": {"architecture": "Zatorax", "vocab": 77, "width": 50, "norm": {"eps": 1e-5}, "layers": [
        delta(3, 1, 10, 14, 2, moe(5, 2, 20, None, 13)), attn(18, 1, 20, 12, 0.3, 11, moe(9, 3, 17, (3, 2), 20)), delta(2, 2, 12, 130, 9, None),
        attn(2, 1, 130, 30, 0.1, 6, None)]},
    # head sizes of the fused decode kernels
    "wide": {"architecture": "Zatorax", "vocab": 120, "width": 128, "norm": {"eps": 1e-5}, "layers": [
        delta(2, 1, 128, 128, 4, moe(16, 4, 128, (4, 2), 64)), attn(4, 2, 128, 128, 0.09, 150, moe(8, 2, 72, (2, 1), 64)),
        attn(4, 2, 128, 128, 0.08, 60, None, kv_from=1), delta(4, 2, 64, 128, 2, moe(8, 2, 64, None, 32))]},
}
TOL = {torch.float32: 2e-4, torch.bfloat16: 0.12}


def weights(cfg, dtype=torch.float32, seed=0):
    """Exact in bf16.  Sharp queries and keys (scores of several units), decays from forgetful to nearly lossless, negative
    corrections.  For 16-bit arithmetic the corrections outweigh the scores, so that no near-tie of two experts can flip, and the
    attention is less sharp."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in Z.tensor_shapes(Z.ZatoraxConfig.from_json(cfg)).items():
        t = torch.randn(shape, generator=gen)
        last = n.rsplit(".", 1)[-1]
        if n.endswith("q.norm") or n.endswith("k.norm"):
            t = 1.5 + 0.5 * t if dtype == torch.float32 else 1.0 + 0.2 * t
        elif n.endswith("mix.norm"):
            t = 1.0 + 0.3 * t
        elif last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.2 * t
        elif last == "A_log":
            t = torch.linspace(-4.0, 0.5, shape[0]) if shape[0] > 1 else torch.tensor([-1.0])
        elif last == "dt_bias":
            t = -2.5 + 0.5 * t
        elif last == "r1":
            t = torch.linspace(0.02, 2.0, shape[0])
        elif last == "r2":
            t = 0.05 + 0.2 * t.abs()
        elif last == "correction":
            t = -1.5 + 0.4 * t if dtype == torch.float32 else -0.5 - 1.5 * torch.randperm(shape[0], generator=gen)
        elif n != "embed":
            t = t * shape[-1] ** -0.5
        out[n] = t.bfloat16()
    return out


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


_known = {}


def expected(name, toks, dtype=torch.float32):
    key = (name, tuple(toks), dtype)
    if key not in _known:
        _known[key] = O.logits(CONFIGS[name], {k: v.double() for k, v in weights(CONFIGS[name], dtype).items()}, toks)
    return _known[key]


def model(name, place):
    w = weights(CONFIGS[name], place[1])
    return Z.build(Z.ZatoraxConfig.from_json(CONFIGS[name]), w.__getitem__, *place)


def close(got, want, dtype):
    """Root mean square of the logits' difference at every position."""
    d = got.detach().double().cpu() - want
    err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std()
    assert bool((err < TOL[dtype]).all()) and float(err.median()) < TOL[dtype] / 4, err


# ---- configuration, weights, registry -----------------------------------------------------------------------------
@pytest.mark.parametrize("name", CONFIGS)
def test_config_round_trip(name):
    cfg = Z.ZatoraxConfig.from_json(CONFIGS[name])
    assert Z.ZatoraxConfig.from_json(cfg.to_json()) == cfg
    assert registry.detect(CONFIGS[name]).name == "zatorax"


def test_config_errors():
    def broken(edit, match):
        j = json.loads(json.dumps(CONFIGS["mixed"]))
        edit(j["layers"])
        with pytest.raises(ValueError, match=match):
            Z.ZatoraxConfig.from_json(j)
    broken(lambda l: l[0].update(type="conv"), "unknown type")
    broken(lambda l: l[0]["mixer"].pop("scale"), "lacks scale")
    broken(lambda l: l[0]["mixer"].update(rope=3), "unknown rope")
    broken(lambda l: l[0]["mixer"].update(heads=5), "multiple of kv_heads")
    broken(lambda l: l[2]["mixer"].update(kv_from=1), "keys of its own")
    broken(lambda l: l[5]["mixer"].update(kv_from=2), "keys of its own")
    broken(lambda l: l[5]["mixer"].update(kv_from=0), "same kv_heads")
    broken(lambda l: l[0]["mlp"]["router"].update(top=9), "within bounds")
    broken(lambda l: l[4]["mlp"]["router"].update(top=5), "kept groups")
    broken(lambda l: l[0]["mlp"].update(kind="dense"), "unknown mlp kind")
    broken(lambda l: l[0]["mixer"]["mask"].update(size=0), "mask.size")


def test_registry_picks_the_family():
    assert registry.detect({"model_type": "laguna"}).name == "laguna"
    assert registry.detect({"architectures": ["Qwen3ForCausalLM"]}).name == "qwen3"
    assert registry.detect({"architectures": ["Qwen3_5ForCausalLM"], "model_type": "qwen3_5"}).name == "qwen35"
    with pytest.raises(ValueError, match="no model family"):
        registry.detect({"model_type": "other"})


def save(tmp_path, name, dtype=torch.float32):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS[name]))
    st.save_file(weights(CONFIGS[name], dtype), str(tmp_path / "model.safetensors"))
    return str(tmp_path)


@pytest.mark.parametrize("name", CONFIGS)
def test_weights_round_trip(tmp_path, name):
    m = registry.detect_dir(save(tmp_path, name)).load(str(tmp_path), "cpu", torch.float32)
    sd = Z.state_dict(m)
    w = weights(CONFIGS[name])
    assert set(sd) == set(w)
    for k in w:
        assert sd[k].shape == w[k].shape and torch.equal(sd[k].float(), w[k].float()), k


def test_missing_or_misshapen_weights_are_named(tmp_path):
    w = weights(CONFIGS["ones"])
    w["l0.mix.q"] = w["l0.mix.q"][:4]
    cfg = Z.ZatoraxConfig.from_json(CONFIGS["ones"])
    with pytest.raises(st.SafeTensorsError, match="l0.mix.q: expected shape"):
        Z.build(cfg, w.__getitem__, "cpu", torch.float32)
    del w["l0.mix.q"]
    st.save_file(w, str(tmp_path / "model.safetensors"))
    with pytest.raises(Exception, match="l0.mix.q"):
        Z.load(cfg, str(tmp_path / "model.safetensors"), "cpu", torch.float32)


# ---- whole prompts and decoding -----------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name,n", [("mixed", 75), ("ones", 20), ("odd", 40), ("wide", 200), ("mixed", 1), ("mixed", 2), ("wide", 3)])
def test_whole_prompt(place, name, n):
    toks = tokens(CONFIGS[name], n)
    got = Z.forward(model(name, place), torch.tensor([toks], device=place[0]))
    close(got[0], expected(name, toks, place[1]), place[1])


def run_split(m, toks, first):
    """Logits of every position from ``first`` - 1 on: a prompt of ``first`` tokens, then one by one."""
    s = Z.CacheSession(m, 1, len(toks))
    out = [s.prefill(torch.tensor([toks[:first]], device=m.device))[0].clone()]
    for t in toks[first:]:
        out.append(s.step(torch.tensor([t], device=m.device))[0].clone())
    return torch.stack(out)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name,n,first", [("mixed", 75, 1), ("mixed", 75, 2), ("mixed", 75, 9), ("mixed", 75, 40), ("ones", 20, 1), ("odd", 40, 8), ("wide", 200, 1), ("wide", 200, 149),
                                          ("wide", 200, 64)])
def test_decoding_continues_a_prompt(place, name, n, first):
    """Cuts before, at and past the windows, the convolutions' reach and a chunk; rings wrap while decoding."""
    toks = tokens(CONFIGS[name], n)
    close(run_split(model(name, place), toks, first), expected(name, toks, place[1])[first - 1:], place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name,lens", [("mixed", (40, 1, 23, 9)), ("wide", (3, 170, 64))])
def test_unequal_requests_in_one_batch(place, name, lens):
    """Every request of a batch as alone: prompts, 20 decoded tokens, requests that end early and give their rows back."""
    m, steps = model(name, place), 20
    seqs = [tokens(CONFIGS[name], n + steps, seed=7 + i) for i, n in enumerate(lens)]
    pad = max(lens)
    ids = torch.tensor([s[:n] + [0] * (pad - n) for s, n in zip(seqs, lens)], device=m.device)
    sess = Z.CacheSession(m, len(lens), pad + steps)
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
    want = torch.cat([expected(name, s[:n + len(o) - 1], place[1])[n - 1:] for s, n, o in zip(seqs, lens, out)])
    close(got, want, place[1])


@pytest.mark.parametrize("place", PLACES)
def test_long_decoding(place):
    toks = tokens(CONFIGS["mixed"], 260, seed=3)
    close(run_split(model("mixed", place), toks, 4)[-120:], expected("mixed", toks, place[1])[-120:], place[1])


@pytest.mark.parametrize("place", PLACES)
def test_session_rules(place):
    m = model("mixed", place)
    s = Z.CacheSession(m, 2, 10)
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
        Z.CacheSession(m, 1, 0)


def test_stores_follow_the_windows_that_read_them():
    s = Z.CacheSession(model("mixed", ("cpu", torch.float32)), 1, 100)
    assert [None if c is None else c.cap for c in s.kv] == [17, None, None, None, 33, None]        # the widest reader, none for borrowers
    assert [c is None for c in s.lin] == [True, False, True, False, True, True]


# ---- generation ---------------------------------------------------------------------------------------------------
def greedy_oracle(name, prompt, n):
    seq = list(prompt)
    w = {k: v.double() for k, v in weights(CONFIGS[name]).items()}
    for _ in range(n):
        seq.append(int(O.logits(CONFIGS[name], w, seq)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("place", PLACES[:2])
def test_greedy_generation_of_unequal_prompts(place):
    m = model("mixed", place)
    prompts = [tokens(CONFIGS["mixed"], n, seed=20 + n) for n in (11, 3, 18)]
    ids, lengths = model_runner.right_pad(prompts, 0)
    out = Z.generate_greedy(m, ids.to(place[0]), 8, lengths=lengths)[:, ids.shape[1]:].tolist()
    for p, row in zip(prompts, out):
        assert row == greedy_oracle("mixed", p, 8)


def test_sampling_and_stop_tokens():
    m = model("mixed", ("cpu", torch.float32))
    ids = torch.tensor([tokens(CONFIGS["mixed"], 5)])
    first = greedy_oracle("mixed", ids[0].tolist(), 1)[0]
    assert Z.generate(m, ids, 6, SamplingStrategy.greedy(), eos_token_ids=[first]).shape[1] == 6
    g = lambda: torch.Generator().manual_seed(5)
    a, b = (Z.generate(m, ids, 6, SamplingStrategy.multinomial(0.8, 20, 0.9), generator=g()) for _ in range(2))
    assert torch.equal(a, b) and a.shape[1] == 11


def test_command_line_generates_from_token_ids(tmp_path, capsys):
    d = save(tmp_path, "mixed")
    p = tokens(CONFIGS["mixed"], 6)
    (tmp_path / "prompts.txt").write_text(" ".join(map(str, p)) + "\n" + ", ".join(map(str, p[:2])) + "\n")
    assert model_runner.main(["--source", d, "--prompt-file", str(tmp_path / "prompts.txt"), "--batch-size", "2", "--max-new-tokens", "4", "--device", "cpu"]) == 0
    lines = capsys.readouterr().out.splitlines()
    got = [[int(t) for t in l.split()] for l in lines if not l.startswith(">")]
    assert got == [greedy_oracle("mixed", p, 4), greedy_oracle("mixed", p[:2], 4)]
    with pytest.raises(ValueError, match="list of token ids"):
        model_runner.main(["--source", d, "--prompt", "hello", "--device", "cpu"])


# ---- trace replay -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
def test_trace_replay(tmp_path, capsys, place):
    d = save(tmp_path, "mixed", place[1])
    a, b, c = (tokens(CONFIGS["mixed"], n, seed=n) for n in (30, 14, 22))
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
    assert sorted(p.name for p in out.iterdir()) == ["0.f32", "1.f32", "2.f32", "4.f32", "5.f32"]
    got = torch.cat([torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).reshape(-1, 88) for i in (0, 1, 2, 4, 5)])
    ea, eb, ec = (expected("mixed", t, place[1]) for t in (a, b, c))
    close(got, torch.stack([ea[0], ea[19], eb[11], eb[12], eb[13], ea[22], ec[21]]), place[1])


def test_trace_replay_refuses_what_a_batch_cannot_do(tmp_path):
    fam = registry.by_name("zatorax")
    r = trace_run.Replayer(fam, model("ones", ("cpu", torch.float32)), 32)
    r.step([{"id": "a", "tokens": [1, 2]}, {"id": "b", "tokens": [3]}])
    with pytest.raises(ValueError, match="advance together"):
        r.step([{"id": "a", "tokens": [1]}])
    with pytest.raises(ValueError, match="twice"):
        r.step([{"id": "a", "tokens": [1]}, {"id": "a", "tokens": [1]}])
    r.step([{"id": "a", "tokens": [1]}, {"id": "b", "tokens": [3]}], ["a", "b"])
    assert not r.group_of


def test_trace_replay_of_another_family():
    """Families whose sessions take prompts of one length run unequal prompts as separate batches."""
    from tyr_b200.models import qwen35 as Q
    cfg = Q.Qwen35Config(vocab_size=50, hidden_size=32, intermediate_size=48, num_hidden_layers=4, num_attention_heads=2, num_key_value_heads=1, head_dim=16,
                         half_rotary_dim=4, linear_key_head_dim=8, linear_value_head_dim=8, linear_num_key_heads=2, linear_num_value_heads=2)
    m = Q.init(cfg)
    r = trace_run.Replayer(registry.by_name("qwen35"), m, 32)
    a, b = [1, 5, 9, 4], [7, 8, 2]
    got = [r.step([{"id": "a", "tokens": a[:3], "want": [0, 2]}, {"id": "b", "tokens": b[:2], "want": [1]}])]
    got.append(r.step([{"id": "a", "tokens": a[3:], "want": [0]}, {"id": "b", "tokens": b[2:], "want": [0]}], ["a", "b"]))
    fa, fb = (Q.forward(m, torch.tensor([t]))[0] for t in (a, b))
    torch.testing.assert_close(torch.cat(got), torch.stack([fa[0], fa[2], fb[1], fa[3], fb[2]]), atol=2e-4, rtol=1e-3)
