"""The mechanisms of the Kinetar design one by one, against the plain implementation in ``kinetar_oracle``: embedding with positions,
residual add and norm, segmented convolution, query temperature, sink attention with gate over prompts and over stores, selective
scan, delta rule with a decay per key channel."""
import math

import pytest
import torch

import kinetar_oracle as O
from tyr_b200.models.common import KVCache
from tyr_b200.ops import delta_rule as dr
from tyr_b200.ops import selective_scan as ss
from tyr_b200.ops import sink_attention as sa
from tyr_b200.ops.embed import embed_positions, position_turns
from tyr_b200.ops.mix_conv import Segment, mix_prompt, mix_step
from tyr_b200.ops.norm import add_norm

GPU = pytest.mark.gpu
PLACES = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU), pytest.param(("cuda", torch.bfloat16), marks=GPU)]


def near(got, want, dtype, tol32=2e-5, tol16=2e-2):
    got, want = got.detach().double().cpu(), want.double()
    scale = want.abs().max().clamp_min(1e-6)
    err = float((got - want).abs().max() / scale)
    assert err < (tol16 if dtype == torch.bfloat16 else tol32), err


def rnd(*shape, scale=1.0):
    """Values that bf16 holds exactly."""
    return (torch.randn(*shape) * scale).bfloat16().double()


def window(dev, dt, width, *shape):
    """A column window of a wider buffer, filled with a value that must not survive or leak."""
    return torch.full((*shape, width + 16), 3.0, device=dev, dtype=dt)[..., 8:8 + width]


def int32(x, dev):
    return torch.tensor(x, dtype=torch.int32, device=dev)


# ---- embedding, norm ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("width", [6, 33, 64])
def test_embedding_with_positions(place, width):
    dev, dt = place
    table = rnd(20, width)
    ids = torch.randint(0, 20, (2, 70))
    turns = position_turns(width, device=dev)
    x = embed_positions(ids.to(dev), table.to(dev, dt), turns, 0.75)
    assert x.dtype == torch.float32
    for b in range(2):
        near(x[b], O.embedding({"embed": table}, ids[b].tolist(), 0.75), torch.float32, 1e-6)
    far = [0, 1, 69, 4095, 1_000_003]                     # a single token per row at its own position, also far out
    x = embed_positions(ids[0, :5, None].to(dev), table.to(dev, dt), turns, 1.0, int32(far, dev))
    for r, p in enumerate(far):
        angle = [p * 10000.0 ** (-2.0 * (c // 2) / width) for c in range(width)]
        want = table[ids[0, r]] + torch.tensor([math.cos(a) if c % 2 else math.sin(a) for c, a in enumerate(angle)])
        assert float((x[r, 0].double().cpu() - want).abs().max()) < 1e-6


@GPU
def test_embedding_reports_ids_outside_the_table():
    from tyr_b200.ops._common import raise_on_device_error
    embed_positions(torch.tensor([[1, 9]], device="cuda"), torch.ones(8, 16, device="cuda"), position_turns(16, device="cuda"), 1.0)
    with pytest.raises(RuntimeError, match="code=3"):
        raise_on_device_error("cuda")


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("D", [16, 50, 136, 2048])
def test_add_and_norm(place, D):
    dev, dt = place
    x, r, w = rnd(3, 5, D), torch.randn(3, 5, D).double(), rnd(D)
    resid = r.float().to(dev)
    h = add_norm(x.to(dev, dt), (1 + w).float().to(dev), 0.3, resid, dt)      # an eps that matters, inside the root
    near(resid, r + x, torch.float32, 1e-6)
    near(h, O.zero_centred_norm(r + x, w, 0.3), dt)
    before = resid.clone()
    near(add_norm(None, (1 + w).float().to(dev), 0.3, resid, dt), O.zero_centred_norm(r + x, w, 0.3), dt)
    assert torch.equal(before, resid)


# ---- segmented convolution ----------------------------------------------------------------------------------------
# (heads, channels of a head, taps, bias, activation, temperature)
SEGMENTS = {
    "vector": [(4, 16, 3, False, None, (0.5, 7)), (2, 16, 3, False, None, None), (1, 40, 4, True, "silu", None), (1, 24, 0, False, "relu2", None)],
    "plain": [(3, 10, 2, False, None, (0.25, 3)), (1, 10, 6, False, "silu", None), (1, 13, 1, True, "silu", None), (1, 9, 0, False, "relu2", None)],
    "wide taps": [(2, 8, 9, True, "silu", (1.0, 1)), (1, 8, 4, False, None, None)],
}


def segment_oracle(u, h, d, w, bias, act, temp):
    y = u if w is None else O.short_conv(u, w, bias)
    y = O.silu(y) if act == "silu" else torch.clamp(y, min=0) ** 2 if act == "relu2" else y
    return y if temp is None else y * O.query_temperature(len(u), *temp, u.dtype)[:, None]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", SEGMENTS)
@pytest.mark.parametrize("pad", [0, 6])
def test_segments_of_prompts_and_of_single_tokens(place, name, pad):
    """Prompts of unequal length, then single tokens: convolutions carry over, the store holds every row's own tokens, padded channels
    are zero, and nothing outside a segment's window is touched."""
    dev, dt = place
    lens, S, more = [41, 1, 33, 2], 41, 5
    x = rnd(4, S + more, 8 + sum(h * d + 8 for h, d, *_ in SEGMENTS[name]))
    specs, col = [], 8
    for h, d, taps, has_bias, act, temp in SEGMENTS[name]:
        w, bias = (rnd(h * d, taps) if taps else None), (rnd(h * d) if has_bias else None)
        specs.append((col, h, d, w, bias, act, temp))
        col += h * d + 8
    f32 = lambda t: None if t is None else t.float().to(dev)
    wins = [None if s[3] is None else torch.full((4, s[1] * s[2], s[3].shape[1]), 5.0, device=dev, dtype=dt) for s in specs]
    stores = [torch.zeros(4, s[1], S, s[2] + pad, device=dev, dtype=dt) for s in specs]

    def segs(T, step):
        outs = [window(dev, dt, s[1] * (s[2] + pad), 4, T) for s in specs]
        return outs, [Segment(c, h, d, o, d + pad, f32(w), f32(b), win, act, temp, None if step else st)
                      for (c, h, d, w, b, act, temp), o, win, st in zip(specs, outs, wins, stores)]
    xd = x.to(dev, dt)
    outs, sg = segs(S, False)
    mix_prompt(xd[:, :S], sg, int32(lens, dev))
    steps = []
    for t in range(more):
        row = torch.stack([xd[b, n + t] for b, n in enumerate(lens)])[:, None]
        o, sg = segs(1, True)
        mix_step(row, sg, int32([n + t for n in lens], dev))
        steps.append(o)
    for i, (c, h, d, w, b_, act, temp) in enumerate(specs):
        for b, n in enumerate(lens):
            want = segment_oracle(x[b, :n + more, c:c + h * d], h, d, w, b_, act, temp)
            got = torch.cat([outs[i][b, :n], *(s[i][b] for s in steps)]).reshape(n + more, h, d + pad)
            near(got[..., :d].reshape(n + more, h * d), want, dt)
            assert not got[..., d:].any()
            near(stores[i][b, :, :n, :d].transpose(0, 1).reshape(n, h * d), want[:n], dt)
            assert not stores[i][b, :, n:].any() and not stores[i][..., d:].any()
        whole = outs[i]._base
        assert bool((whole[..., :8] == 3).all()) and bool((whole[..., -8:] == 3).all())


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("coef,every", [(0.5, 64), (1.25, 5), (0.3, 1)])
def test_query_temperature_steps(place, coef, every):
    """The factor changes exactly where position + 1 reaches a multiple of ``every``, in prompts and for single tokens."""
    dev, dt = place
    S = 3 * every + 2
    out = torch.empty(1, S, 8, device=dev, dtype=torch.float32 if dt == torch.float32 else dt)
    mix_prompt(torch.ones(1, S, 8, device=dev, dtype=dt), [Segment(0, 1, 8, out, temp=(coef, every))])
    near(out[0, :, 0], O.query_temperature(S, coef, every, torch.float64), dt, 1e-6, 4e-3)
    for edge in (every, 2 * every, 1000 * every):
        pos = [edge - 2, edge - 1, edge] if every > 1 else [edge - 1, edge, edge + 1]
        one = torch.empty(3, 1, 8, device=dev, dtype=dt)
        mix_step(torch.ones(3, 1, 8, device=dev, dtype=dt), [Segment(0, 1, 8, one, temp=(coef, every))], int32(pos, dev))
        near(one[:, 0, 0], torch.tensor([1 + coef * math.log((p + 1) // every + 1) for p in pos]), dt, 1e-6, 4e-3)


# ---- sink attention -----------------------------------------------------------------------------------------------
HEADS = [(4, 2, 16, 16), (3, 3, 24, 24), (9, 3, 88, 88), (2, 1, 128, 128), (5, 1, 40, 40), (18, 1, 20, 20), (2, 2, 130, 130), (4, 4, 64, 64), (4, 2, 32, 72)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,G,dk,dv", HEADS)
def test_prompt_attention(place, H, G, dk, dv):
    """Sinks from negligible to dominant; gate and factor; output into a column window.  With dk == dv the values are the keys."""
    dev, dt = place
    T = 150
    q, k, gate = rnd(2, T, H, dk), rnd(2, T, G, dk), rnd(2, T, H * dv + 8)
    v = k if dk == dv else rnd(2, T, G, dv)
    sink = torch.linspace(-20.0, 12.0, H).bfloat16().double()
    kd = k.to(dev, dt)
    out = window(dev, dt, H * dv, 2, T)
    sa.prompt_attention(q.to(dev, dt), kd, kd if v is k else v.to(dev, dt), scale=0.2, sink=sink.float().to(dev), gate=gate.to(dev, dt)[..., :H * dv],
                        out_scale=0.7, out=out)
    for b in range(2):
        o = O.sink_attention(q[b], k[b], v[b], 0.2, sink).reshape(T, -1)
        near(out[b], 0.7 * o * O.sigmoid(gate[b, :, :H * dv]), dt)
    assert bool((out._base[..., :8] == 3).all()) and bool((out._base[..., -8:] == 3).all())
    plain = sa.prompt_attention(q.to(dev, dt), kd, kd if v is k else v.to(dev, dt), scale=0.2)
    near(plain[0], O.sink_attention(q[0], k[0], v[0], 0.2, torch.full((H,), -1e4).double()).reshape(T, -1), dt)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("d", [24, 88, 128])
def test_a_far_key_and_the_sink_decide(place, d):
    """One key far back (and one at each block's edge) stands out for the last query, and takes its mass from the sink: with the
    score equal to the sink half of it."""
    dev, dt = place
    T = 600
    for at in (0, 1, 127, 128, 300, 511, 512, T - 2, T - 1):
        k = rnd(1, T, 1, d, scale=0.01)
        k[0, at, 0] = 0.0
        k[0, at, 0, 0] = 16.0
        q = torch.zeros(1, T, 2, d).double()
        q[0, T - 1, :, 0] = 1.0
        sink = torch.tensor([16.0, -30.0]).double()
        kd = k.to(dev, dt)
        o = sa.prompt_attention(q.to(dev, dt), kd, kd, scale=1.0, sink=sink.float().to(dev))[0, T - 1].reshape(2, d).double().cpu()
        assert abs(float(o[0, 0]) - 8.0) < 0.1 and abs(float(o[1, 0]) - 16.0) < 0.1, (at, o[:, 0])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,G,d", [(4, 2, 16), (9, 3, 88), (2, 1, 128), (18, 1, 20), (2, 2, 130), (16, 1, 64), (3, 3, 48)])
@pytest.mark.parametrize("shared", [True, False])
def test_step_attention(place, H, G, d, shared):
    """A position per row (first token, edges of the key blocks and splits, a full store); append, sink, gate, factor, window of the
    output.  Positions past a row's own are poisoned."""
    dev, dt = place
    pos = [0, 1, 15, 16, 63, 64, 255, 256, 257, 519]
    B, cap = len(pos), 520
    dp = sa.store_dim(H, G, d, dt, dev)
    k, v = rnd(B, G, cap, d), rnd(B, G, cap, d)
    q, gate, sink = rnd(B, H, d), rnd(B, 1, H * d + 8), torch.linspace(-4.0, 6.0, H).bfloat16().double()
    pad = lambda t: torch.nn.functional.pad(t, (0, dp - d)).to(dev, dt)
    kp, vp = pad(k), pad(v)
    new_k, new_v = (torch.stack([t[b, :, p] for b, p in enumerate(pos)])[:, None].clone() for t in (kp, vp))
    for b, p in enumerate(pos):
        kp[b, :, p:], vp[b, :, p:] = 1e4, 1e4
    store = KVCache(kp, kp if shared else vp)
    out = window(dev, dt, H * d, B, 1)
    got = sa.step_attention(pad(q)[:, None], new_k, new_k if shared else new_v, store, int32(pos, dev), d, scale=0.3, sink=sink.float().to(dev),
                            gate=gate.to(dev, dt)[..., :H * d], out_scale=1.3, out=out)
    for b, p in enumerate(pos):
        kk, vv = k[b, :, :p + 1].transpose(0, 1), (k if shared else v)[b, :, :p + 1].transpose(0, 1)
        qq = torch.zeros(p + 1, H, d).double()
        qq[p] = q[b]
        if p > 64:                                        # the oracle walks every query: keep the last one's keys only
            s = torch.einsum("hd,jhd->hj", q[b], kk.repeat_interleave(H // G, 1)) * 0.3
            e = torch.exp(s - 20)
            o = torch.einsum("hj,jhd->hd", e / (e.sum(1) + torch.exp(sink - 20))[:, None], vv.repeat_interleave(H // G, 1))
        else:
            o = O.sink_attention(qq, kk, vv, 0.3, sink)[p]
        near(got[b, 0], 1.3 * o.reshape(-1) * O.sigmoid(gate[b, 0, :H * d]), dt)
        assert torch.equal(store.k[b, :, p], new_k[b, 0]) and (shared or torch.equal(store.v[b, :, p], new_v[b, 0]))
    assert bool((out._base[..., :8] == 3).all()) and bool((out._base[..., -8:] == 3).all())


@pytest.mark.parametrize("place", PLACES)
def test_step_attention_reads_far_keys(place):
    dev, dt = place
    cap, d = 1500, 64
    for at in (0, 1, 255, 256, 1023, 1024, cap - 2, cap - 1):
        k = torch.zeros(1, 1, cap, d, device=dev, dtype=dt)
        k[0, 0, at, 0] = 16.0
        q = torch.zeros(1, 1, 1, d, device=dev, dtype=dt)
        q[..., 0] = 1.0
        o = sa.step_attention(q, k[:, None, 0, cap - 1].reshape(1, 1, 1, d).clone(), k[:, None, 0, cap - 1].reshape(1, 1, 1, d).clone(), KVCache(k, k),
                              int32([cap - 1], dev), d, scale=1.0, sink=torch.tensor([16.0], device=dev))
        assert abs(float(o[0, 0, 0]) - 8.0) < 0.1, at


# ---- selective scan -----------------------------------------------------------------------------------------------
def scan_inputs(B, T, C, N):
    x, dt, z, bc = rnd(B, T, C + 8), rnd(B, T, C + 8) - 1.0, rnd(B, T, C + 8), rnd(B, T, 2 * N + 8)
    A = -torch.exp(rnd(C, N)).float().double()
    return x, dt.bfloat16().double(), z, bc, A, rnd(C), rnd(C)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("C,N", [(24, 16), (40, 22), (13, 3), (16, 1), (72, 8), (33, 30), (16, 64), (20, 100), (8, 256), (130, 4)])
def test_scan_of_unequal_rows_and_single_tokens(place, C, N):
    """Prompts from a state that an earlier batch left behind, then single tokens from where each row ended."""
    dev, dtp = place
    lens, T, more = [70, 1, 32, 33], 70, 4
    x, dt, z, bc, A, D, bias = scan_inputs(4, T + more, C, N)
    to = lambda t: t.to(dev, dtp)
    f32 = lambda t: t.float().to(dev)
    state = torch.full((4, C, N), 7.0, device=dev)
    out = window(dev, dtp, C, 4, T)
    xd, dd, zd, bd = to(x), to(dt), to(z), to(bc)
    xw, dw, zw, bw = (t[:, :T].contiguous() for t in (xd, dd, zd, bd))
    ss.scan_prompt(xw[..., :C], dw[..., 8:], zw[..., 8:], bw[..., :N], bw[..., N:2 * N], f32(A), f32(D), f32(bias), state, out, int32(lens, dev), 0.6)
    after = state.clone()
    ones = []
    for t in range(more):
        pick = lambda y: torch.stack([y[b, n + t] for b, n in enumerate(lens)])[:, None]
        o = window(dev, dtp, C, 4, 1)
        b_ = pick(bd)
        ss.scan_step(pick(xd)[..., :C], pick(dd)[..., 8:], pick(zd)[..., 8:], b_[..., :N], b_[..., N:2 * N], f32(A), f32(D), f32(bias), state, o, 0.6)
        ones.append(o)
        assert bool((o._base[..., :8] == 3).all()) and bool((o._base[..., -8:] == 3).all())
    for r, n in enumerate(lens):
        m = n + more
        delta = O.softplus(dt[r, :m, 8:] + bias)
        _, st = O.selective_scan(x[r, :n, :C], delta[:n], A, bc[r, :n, :N], bc[r, :n, N:2 * N], D)
        tol = 2e-5 if dtp == torch.float32 else 2e-4
        near(after[r], st, torch.float32, tol)
        y, st = O.selective_scan(x[r, :m, :C], delta, A, bc[r, :m, :N], bc[r, :m, N:2 * N], D)
        got = torch.cat([out[r, :n], *(o[r] for o in ones)])
        near(got, 0.6 * y * O.silu(z[r, :m, 8:]), dtp)
        near(state[r], st, torch.float32, tol)
    assert bool((out._base[..., :8] == 3).all()) and bool((out._base[..., -8:] == 3).all())


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("N", [3, 16])
def test_scan_remembers_far_inputs(place, N):
    """One input enters every state; 900 tokens later the slow states still show it to the expected digit, the fast ones have lost it."""
    dev, dtp = place
    T, C = 901, 8
    z = lambda *s: torch.zeros(1, T, *s).double()
    x, dt, b, c = z(C), z(C), z(N), z(N)
    x[0, 0], b[0, 0], c[0, T - 1] = 1.0, 1.0, 1.0
    A = -torch.linspace(1e-4, 0.05, C * N).reshape(C, N).float().double()
    one = torch.full((1, T, C), 1.0).double()
    state = torch.zeros(1, C, N, device=dev)
    out = torch.empty(1, T, C, device=dev, dtype=dtp)
    to = lambda t: t.to(dev, dtp)
    bc = to(torch.cat([b, c], -1))
    zero = torch.zeros(C, device=dev)
    ss.scan_prompt(to(x), to(dt), to(one), bc[..., :N], bc[..., N:], A.float().to(dev), zero, zero, state, out)
    delta = math.log(2.0)
    want = delta * torch.exp(900 * delta * A)
    near(state[0], want, torch.float32, 2e-5 if dtp == torch.float32 else 3e-4)
    near(out[0, T - 1], want.sum(1) * O.silu(torch.tensor(1.0).double()), dtp)
    assert float(want[-1, -1]) < 1e-9 * float(want[0, 0])


# ---- delta rule with a decay per key channel ----------------------------------------------------------------------
def delta_inputs(B, T, Hk, Hv, dk, dv, strength=1.0):
    q, k, v = rnd(B, T, Hk, dk), rnd(B, T, Hk, dk), rnd(B, T, Hv, dv)
    a, b = rnd(B, T, Hv * dk + 8), rnd(B, T, Hv + 8)
    return q, k, v, a, b, rnd(Hv * dk) - 2.0, (torch.linspace(-3.0, 0.0, Hv) + math.log(strength)).float().double()


def delta_oracle(q, k, v, a, b, dt_bias, a_log, state=None):
    H = v.shape[1]
    return O.channel_delta_recurrence(O.unit_vectors(q) * q.shape[-1] ** -0.5, O.unit_vectors(k), v, O.channel_decay(a, dt_bias, a_log), O.sigmoid(b[:, :H]), state)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("Hk,Hv,dk,dv", [(2, 4, 16, 24), (1, 3, 40, 16), (2, 2, 128, 128), (3, 3, 8, 72), (1, 2, 20, 12), (2, 2, 56, 48), (1, 1, 136, 10)])
@pytest.mark.parametrize("strength", [1.0, 40.0])
def test_delta_prompt_rows_of_unequal_length(place, Hk, Hv, dk, dv, strength):
    """Gentle decays, and decays that empty a channel within a few tokens next to channels that keep it."""
    dev, dt = place
    lens = [150, 1, 64, 65, 2, 17]
    q, k, v, a, b, bias, a_log = delta_inputs(6, 150, Hk, Hv, dk, dv, strength)
    state = torch.full((6, Hv, dk, dv), 7.0, device=dev)  # what an earlier batch left behind must not matter
    to = lambda t: t.to(dev, dt)
    o = dr.channel_delta_prefill(to(q), to(k), to(v), to(a)[..., :Hv * dk], to(b)[..., :Hv], bias.float().to(dev), a_log.float().to(dev), state, int32(lens, dev))
    assert o.dtype == state.dtype == torch.float32
    for r, n in enumerate(lens):
        wo, ws = delta_oracle(q[r, :n], k[r, :n], v[r, :n], a[r, :n, :Hv * dk], b[r, :n], bias, a_log)
        near(o[r, :n], wo, torch.float32, 2e-4)           # bf16 inputs are exact; everything after them is 32-bit
        near(state[r], ws, torch.float32, 2e-4)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("dk,dv", [(16, 24), (64, 128), (128, 128)])
def test_delta_channels_forget_on_their_own(place, dk, dv):
    """Two writes along two key channels, one of which hardly decays: 400 tokens later only that one is read back; writing zero with
    strength one along its key erases it."""
    dev, dt = place
    T = 403
    q, k, v = torch.zeros(1, T, 1, dk).double(), torch.zeros(1, T, 1, dk).double(), torch.zeros(1, T, 1, dv).double()
    k[0, 2:T - 1, 0, 2:] = rnd(T - 3, dk - 2)
    k[0, 0, 0, 0], k[0, 1, 0, 1], k[0, T - 1, 0, 0] = 1.0, 1.0, 1.0
    q[0, T - 3, 0, 0], q[0, T - 2, 0, 1], q[0, T - 1, 0, 0] = 1.0, 1.0, 1.0
    v[0, 0], v[0, 1] = rnd(1, dv), rnd(1, dv)
    a = torch.full((1, T, dk), -9.0).double()
    a[..., 1] = -2.0
    b = torch.full((1, T, 1), 0.0).double()
    b[0, 0], b[0, 1], b[0, T - 1] = 40.0, 40.0, 40.0
    bias, a_log = torch.zeros(dk).double(), torch.zeros(1).double()
    state = torch.zeros(1, 1, dk, dv, device=dev)
    to = lambda t: t.to(dev, dt)
    o = dr.channel_delta_prefill(to(q), to(k), to(v), to(a), to(b), bias.float().to(dev), a_log.float().to(dev), state)
    want, _ = delta_oracle(q[0], k[0], v[0], a[0], b[0], bias, a_log)
    assert want[T - 3].abs().max() > 1e6 * want[T - 2].abs().max() and want[T - 1].abs().max() < 1e-5
    near(o[0, T - 3], want[T - 3], torch.float32, 2e-4)
    assert float(o[0, T - 2].abs().max()) < 1e-5 * float(want[T - 3].abs().max()) and float(o[0, T - 1].abs().max()) < 1e-3 * float(want[T - 3].abs().max())


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("Hk,Hv,dk,dv", [(2, 4, 16, 24), (1, 2, 128, 128), (2, 2, 64, 128), (2, 6, 40, 16), (1, 1, 200, 20)])
def test_delta_step_continues_its_state(place, Hk, Hv, dk, dv):
    """Eight tokens one by one through recurrence, norm and sigmoid gate, from a state that is not zero."""
    dev, dt = place
    B, T, eps = 2, 8, 1e-2
    q, k, v, a, b, bias, a_log = delta_inputs(B, T, Hk, Hv, dk, dv)
    z, nw, st0 = rnd(B, T, Hv * dv + 8), rnd(dv), rnd(B, Hv, dk, dv, scale=0.3)
    rec = st0.float().to(dev)
    to = lambda t: t.to(dev, dt)
    got = []
    for t in range(T):
        one = lambda y: to(y)[:, t:t + 1]
        out = window(dev, dt, Hv * dv, B, 1)
        dr.channel_delta_decode(one(q), one(k), one(v), one(a)[..., :Hv * dk], one(b)[..., :Hv], one(z)[..., :Hv * dv], bias.float().to(dev),
                                a_log.float().to(dev), nw.float().to(dev), to(nw), eps, rec, out)
        got.append(out[:, 0])
        assert bool((out._base[..., :8] == 3).all()) and bool((out._base[..., -8:] == 3).all())
    for r in range(B):
        o, st = delta_oracle(q[r], k[r], v[r], a[r, :, :Hv * dk], b[r], bias, a_log, st0[r])
        want = (O.rms_unit(o, eps) * nw).reshape(T, Hv * dv) * O.sigmoid(z[r, :, :Hv * dv])
        near(torch.stack(got, 1)[r], want, dt)
        near(rec[r], st, torch.float32, 1e-4)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("dv", [10, 32, 128])
def test_gated_norm_with_sigmoid(place, dv):
    dev, dt = place
    o, z, w = torch.randn(2, 3, 4, dv).double(), rnd(2, 3, 4 * dv + 8), rnd(dv)
    out = window(dev, dt, 4 * dv, 2, 3)
    dr.gated_norm(o.float().to(dev), z.to(dev, dt)[..., :4 * dv], w.float().to(dev), 0.2, "sigmoid", out)
    near(out, (O.rms_unit(o, 0.2) * w).reshape(2, 3, -1) * O.sigmoid(z[..., :4 * dv]), dt)
    assert bool((out._base[..., :8] == 3).all()) and bool((out._base[..., -8:] == 3).all())
