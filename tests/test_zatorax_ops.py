"""The mechanisms of the Zatorax design one by one, against the plain implementation in ``zatorax_oracle``: convolution, gates,
delta recurrence, gated norm, penalised window attention over prompts and over stores, group-limited routing, norm-and-add."""
import pytest
import torch

import zatorax_oracle as O
from tyr_b200.models.common import KVCache
from tyr_b200.ops import biased_attention as ba
from tyr_b200.ops import delta_rule as dr
from tyr_b200.ops import moe
from tyr_b200.ops.norm import post_norm_residual

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


# ---- delta layer --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("C,K", [(16, 1), (24, 3), (13, 4), (40, 6)])
def test_short_convolution(place, C, K):
    dev, dt = place
    T = 45
    x, w = rnd(2, T, C + 8), rnd(C, K)
    got = dr.causal_conv1d_silu(x.to(dev, dt)[..., :C], w.to(dev, dt))
    for b in range(2):
        near(got[b], O.short_conv(x[b, :, :C], w), dt)


@pytest.mark.parametrize("place", PLACES)
def test_convolution_window_of_unequal_rows(place):
    dev, dt = place
    x = rnd(3, 9, 5).to(dev, dt)
    win = dr.conv_window(x, 4, torch.tensor([9, 2, 4], device=dev, dtype=torch.int32))
    for b, n in enumerate((9, 2, 4)):
        rows = torch.cat([torch.zeros(4, 5, device=dev, dtype=dt), x[b, :n]])[-4:]
        assert torch.equal(win[b], rows.T)


@pytest.mark.parametrize("place", PLACES)
def test_gates(place):
    dev, dt = place
    y, bias, a_log = rnd(2, 7, 11), rnd(5), rnd(5)
    y[0, 0, 5] = 40.0                                     # softplus far on either side
    y[0, 1, 5] = -40.0
    g, beta = dr.delta_gates(y.to(dev, dt)[..., :5], y.to(dev, dt)[..., 5:10], bias.float().to(dev), a_log.float().to(dev))
    assert g.dtype == beta.dtype == torch.float32
    near(g, -torch.exp(a_log) * O.softplus(y[..., 5:10] + bias), torch.float32)
    near(beta, O.sigmoid(y[..., :5]), torch.float32)


def delta_inputs(B, T, Hk, Hv, dk, dv):
    q, k, v = rnd(B, T, Hk, dk), rnd(B, T, Hk, dk), rnd(B, T, Hv, dv)
    g = -torch.exp(rnd(B, T, Hv) - 2.0).float().double()
    beta = torch.sigmoid(rnd(B, T, Hv)).float().double()
    return q, k, v, g, beta


def delta_oracle(q, k, v, g, beta, state=None):
    return O.delta_recurrence(O.unit_vectors(q) * q.shape[-1] ** -0.5, O.unit_vectors(k), v, torch.exp(g), beta, state)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("Hk,Hv,dk,dv", [(2, 4, 16, 24), (1, 3, 40, 16), (2, 2, 128, 128), (3, 3, 8, 72), (1, 2, 20, 12)])
def test_delta_prompt_rows_of_unequal_length(place, Hk, Hv, dk, dv):
    dev, dt = place
    lens = [70, 1, 64, 2]
    q, k, v, g, beta = delta_inputs(4, 70, Hk, Hv, dk, dv)
    state = torch.full((4, Hv, dk, dv), 7.0, device=dev)  # what an earlier batch left behind must not matter
    to = lambda t: t.to(dev, dt)
    o = dr.delta_prefill(to(q), to(k), to(v), g.float().to(dev), beta.float().to(dev), state, torch.tensor(lens, dtype=torch.int32, device=dev))
    assert o.dtype == state.dtype == torch.float32
    for b, n in enumerate(lens):
        wo, ws = delta_oracle(q[b, :n], k[b, :n], v[b, :n], g[b, :n], beta[b, :n])
        near(o[b, :n], wo, torch.float32, 2e-4)           # bf16 inputs are exact; everything after them is 32-bit
        near(state[b], ws, torch.float32, 2e-4)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("dk,dv", [(16, 24), (64, 128), (128, 128)])
def test_delta_remembers_and_overwrites_far_writes(place, dk, dv):
    """A write is read back 400 tokens later from a head that hardly decays, and not from one that does; writing zero with
    strength one along the same key erases it."""
    dev, dt = place
    T = 402
    q, k, v = rnd(1, T, 1, dk, scale=0.5), rnd(1, T, 1, dk), torch.zeros(1, T, 2, dv).double()
    q[..., 0], k[..., 0] = 0.0, 0.0                       # the marked direction is left alone by the others
    k[0, 0, 0], q[0, T - 1, 0], q[0, T - 2, 0] = 0.0, 0.0, 0.0
    k[0, 0, 0, 0], q[0, T - 2, 0, 0], q[0, T - 1, 0, 0] = 1.0, 1.0, 1.0
    k[0, T - 1, 0] = k[0, 0, 0]
    v[0, 0] = rnd(2, dv)
    g = torch.tensor([-1e-4, -0.1]).double().expand(1, T, 2).contiguous()
    beta = torch.full((1, T, 2), 0.5).double()
    beta[0, 0], beta[0, T - 1] = 1.0, 1.0
    state = torch.zeros(1, 2, dk, dv, device=dev)
    to = lambda t: t.to(dev, dt)
    o = dr.delta_prefill(to(q), to(k), to(v), g.float().to(dev), beta.float().to(dev), state)
    want, _ = delta_oracle(q[0], k[0], v[0], g[0], beta[0])
    assert want[T - 2, 0].abs().max() > 50 * want[T - 2, 1].abs().max() and want[T - 1, 0].abs().max() < 1e-5
    near(o[0], want, torch.float32, 2e-4)
    near(o[0, T - 2, 0], want[T - 2, 0], torch.float32, 2e-4)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("Hk,Hv,dk,dv,K", [(2, 4, 16, 24, 3), (1, 2, 128, 128, 4), (2, 2, 64, 128, 1), (2, 6, 40, 16, 6)])
def test_delta_step_continues_its_state(place, Hk, Hv, dk, dv, K):
    """Eight tokens through the fused step: convolution window, gates, recurrence, gated norm."""
    dev, dt = place
    B, T, C, eps = 2, 8, 2 * Hk * dk + Hv * dv, 1e-4
    y, w, nw, bias, a_log = rnd(B, T, C + Hv * dv + 2 * Hv + 8), rnd(C, K), rnd(dv), rnd(Hv), rnd(Hv)
    y = y[..., :(C + Hv * dv + 2 * Hv + 7) // 8 * 8]
    conv = torch.zeros(B, C, K, device=dev, dtype=dt)
    rec = torch.zeros(B, Hv, dk, dv, device=dev)
    out = []
    yd = y.to(dev, dt)
    z = C + Hv * dv
    for t in range(T):
        r = yd[:, t:t + 1]
        out.append(dr.delta_decode(r[..., :C], r[..., C:z], r[..., z:z + Hv], r[..., z + Hv:z + 2 * Hv], conv, w.to(dev, dt), bias.float().to(dev),
                                   a_log.float().to(dev), nw.to(dev, dt), eps, rec, Hk, Hv, dk, dv)[:, 0])
    got = torch.stack(out, 1)
    for b in range(B):
        c = O.short_conv(y[b, :, :C], w)
        if dt == torch.bfloat16:
            c = c.bfloat16().double()
        q, k, v = c[:, :Hk * dk].reshape(T, Hk, dk), c[:, Hk * dk:2 * Hk * dk].reshape(T, Hk, dk), c[:, 2 * Hk * dk:].reshape(T, Hv, dv)
        g = -torch.exp(a_log) * O.softplus(y[b, :, z + Hv:z + 2 * Hv] + bias)
        o, st = delta_oracle(q, k, v, g, O.sigmoid(y[b, :, z:z + Hv]))
        o = O.rms_unit(o, eps) * nw * O.silu(y[b, :, C:z]).reshape(T, Hv, dv)
        near(got[b], o.reshape(T, -1), dt)
        near(rec[b], st, torch.float32, 5e-3 if dt == torch.bfloat16 else 2e-5)      # bf16 convolution outputs round either way


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("dv", [8, 24, 128, 30])
def test_gated_norm(place, dv):
    dev, dt = place
    o, z, w = torch.randn(2, 5, 3, dv).double() * 1e-3, rnd(2, 5, 3 * dv + 2), rnd(dv)      # small enough for eps to matter
    got = dr.gated_norm(o.float().to(dev), z.to(dev, dt)[..., :3 * dv], w.float().to(dev), 1e-5)
    want = O.rms_unit(o, 1e-5) * w * O.silu(z[..., :3 * dv]).reshape(2, 5, 3, dv)
    near(got.reshape(2, 5, 3, dv), want, dt)


# ---- penalised window attention -----------------------------------------------------------------------------------
def attention_case(T, H, G, dk, dv, B=1):
    q, k, v = rnd(B, T, H, dk), rnd(B, T, G, dk), rnd(B, T, G, dv)
    r1, r2 = rnd(H).abs() + 0.1, rnd(H).abs() * 0.3
    r1[0] = 0.0                                           # a head that sees far keys without loss
    return q, k, v, r1, r2


def prompt_got(place, q, k, v, r1, r2, window, scale):
    dev, dt = place
    return ba.prompt_attention(q.to(dev, dt), k.to(dev, dt), v.to(dev, dt), r1.float().to(dev), r2.float().to(dev), window=window, scale=scale)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("T,H,G,dk,dv,window", [(50, 6, 3, 24, 40, 9), (300, 4, 2, 64, 128, 130), (280, 2, 2, 128, 128, None), (33, 3, 1, 20, 12, 33),
                                                (270, 2, 1, 72, 8, 128), (70, 4, 4, 16, 16, 1), (40, 5, 1, 136, 24, 7)])
def test_prompt_attention(place, T, H, G, dk, dv, window):
    q, k, v, r1, r2 = attention_case(T, H, G, dk, dv, B=2)
    got = prompt_got(place, q, k, v, r1, r2, window, 0.3 * dk ** -0.5)
    for b in range(2):
        near(got[b], O.window_attention(q[b], k[b], v[b], 0.3 * dk ** -0.5, r1, r2, window), place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("T,window", [(400, 150), (300, 127), (300, 128), (300, 129), (600, 256), (40, 12), (400, 390)])
def test_prompt_window_edges(place, T, window):
    """One key carries a score far above all others and a value of its own: the last query that sees it and the first that does
    not tell a window that is one token off; so do keys just behind the query."""
    H, G, d = 2, 1, 64
    q, k, v = rnd(1, T, H, d, scale=0.1), rnd(1, T, G, d, scale=0.1), rnd(1, T, G, d, scale=0.1)
    q[..., 0] = 4.0
    mark = [0, 5, T - window - 2] if T - window - 2 > 5 else [0]
    for m in mark:
        k[0, m, 0, 0] = 8.0
        v[0, m, 0] = float(3 + m % 7)
    r1, r2 = torch.tensor([0.02, 1.0]).double(), torch.tensor([0.3, 0.01]).double()
    got = prompt_got(place, q, k, v, r1, r2, window, 1.0)[0].double().cpu()
    want = O.window_attention(q[0], k[0], v[0], 1.0, r1, r2, window)
    near(got, want, place[1])
    for m in mark:
        if m + window < T:
            inside, outside = want[m + window - 1], want[m + window]
            assert (inside - outside).abs().max() > 0.5
            near(got[m + window - 1], inside, place[1])
            near(got[m + window], outside, place[1], tol16=5e-2)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("window", [200, None])
@pytest.mark.parametrize("r1,r2", [(40.0, 3.0), (15.0, 0.5), (-2.0, 0.4), (0.0, 0.0), (2.0, 50.0)])
def test_prompt_penalty_strengths(place, window, r1, r2):
    """Steep penalties (probabilities that span more than the fp32 range inside one block of keys), growing ones, none."""
    T, d = 300, 64
    q, k, v, _, _ = attention_case(T, 2, 1, d, d)
    r1, r2 = torch.tensor([r1, r1 / 2]).double(), torch.tensor([r2, r2]).double()
    near(prompt_got(place, q, k, v, r1, r2, window, 0.5)[0], O.window_attention(q[0], k[0], v[0], 0.5, r1, r2, window), place[1])


@pytest.mark.parametrize("place", PLACES[1:])
def test_prompt_window_larger_than_the_penalty_table(place):
    T, window = 7000, 6500
    q, k, v, r1, r2 = attention_case(T, 1, 1, 64, 64)
    r1[0], r2[0] = 0.3, 0.2
    k[0, 20, 0] = q[0, 20 + window - 1, 0] * 2
    q[0, 20 + window, 0] = q[0, 20 + window - 1, 0]
    got = prompt_got(place, q, k, v, r1, r2, window, 0.5)[0].double().cpu()
    for i in (0, 1, 127, 128, 5000, 20 + window - 1, 20 + window, T - 1):
        lo = max(0, i - window + 1)
        dist = torch.arange(i - lo, -1, -1).double()
        p = torch.softmax(k[0, lo:i + 1, 0] @ q[0, i, 0] * 0.5 - r1[0] * torch.log(1 + r2[0] * dist), -1)
        near(got[i, 0], p @ v[0, lo:i + 1, 0], place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,G,dk,dv,window,cap,start", [(6, 3, 24, 40, 9, 9, [3, 20, 0]), (4, 2, 64, 128, 40, 64, [100, 7, 63]), (2, 2, 128, 128, None, 90, [60, 0, 5]),
                                                        (18, 2, 128, 64, 33, 33, [32, 33, 34]), (20, 1, 16, 16, 5, 8, [4, 9, 16]), (12, 1, 64, 64, 700, 700, [900, 3, 699])])
def test_step_attention_rows_at_their_own_positions(place, H, G, dk, dv, window, cap, start):
    """Twelve tokens per row from unequal positions, over plain stores and over rings whose windows are as wide or narrower;
    a layer that reads the same keys with half the window and without appending."""
    dev, dt = place
    B, steps, eps, scale = 3, 12, 1e-5, 1.6 * dk ** -0.5
    T = max(start) + steps
    y, qw, kw = rnd(B, T, (H + G) * dk + G * dv), rnd(dk).abs() + 0.5, rnd(dk).abs() + 0.5
    r1, r2 = rnd(H).abs(), rnd(H).abs() * 0.3
    ring = window is not None and cap < T
    dkp, dvp = ba.store_dims(H, G, dk, dv, dt, dev)
    store = KVCache.allocate(B, G, cap, dkp, dev, dt, ring=ring, v_dim=dvp)
    store.k.fill_(9.0)                                    # an earlier request's keys
    store.v.fill_(9.0)
    f = lambda t: t.float().to(dev)
    pre = max(start)
    yd = y.to(dev, dt)
    if pre:
        lens = torch.tensor([max(s, 1) for s in start], dtype=torch.int32, device=dev)
        ba.qk_norm_store(yd[:, :pre].contiguous(), f(qw), f(kw), H, G, dk, dv, eps, dkp=dkp, dvp=dvp, store=store, lens=lens)
    pos = torch.tensor([max(s, 1) for s in start], dtype=torch.int32, device=dev)
    half = None if window is None else (window + 1) // 2
    got, got_half = [], []
    for t in range(steps):
        rows = torch.stack([yd[b, int(pos[b])] for b in range(B)])[:, None]
        q, k, v = ba.qk_norm_store(rows.contiguous(), f(qw), f(kw), H, G, dk, dv, eps, dkp=dkp, dvp=dvp)
        got.append(ba.step_attention(q, k, v, store, pos, f(r1), f(r2), window=window, scale=scale, append=True)[..., :dv])
        got_half.append(ba.step_attention(q, k, v, store, pos, f(r1), f(r2), window=half, scale=scale, append=False)[..., :dv])
        pos += 1
    for b in range(B):
        s = max(start[b], 1)
        n = s + steps
        q = O.rms_unit(y[b, :n, :H * dk].reshape(n, H, dk), eps) * qw
        k = O.rms_unit(y[b, :n, H * dk:(H + G) * dk].reshape(n, G, dk), eps) * kw
        v = y[b, :n, (H + G) * dk:].reshape(n, G, dv)
        for outs, w in ((got, window), (got_half, half)):
            lo = 0 if w is None else max(0, s - w + 1)    # earlier keys are outside every window
            want = O.window_attention(q[lo:], k[lo:], v[lo:], scale, r1, r2, w)[s - lo:]
            near(torch.stack([o[b, 0] for o in outs]), want, dt)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("window", [7, 40, 300])
def test_step_window_edges(place, window):
    """A marked key is read by the last decoded token that sees it and not by the next one, from a ring that has wrapped."""
    dev, dt = place
    d, marked = 64, 10
    first = marked + window - 3                           # decoded tokens at first .. first + 5
    T = first + 6
    k, v = rnd(T, d, scale=0.1), rnd(T, d, scale=0.1)
    q = torch.zeros(T, 1, d).double()
    q[..., 0] = 4.0
    k[marked, 0], v[marked] = 8.0, 5.0
    r1, r2 = torch.tensor([0.02]), torch.tensor([0.3])
    want = O.window_attention(q, k[:, None], v[:, None], 1.0, r1.double(), r2.double(), window)
    store = KVCache.allocate(1, 1, window, d, dev, dt, ring=True)
    for p in range(first):
        store.k[0, 0, p % window], store.v[0, 0, p % window] = k[p].to(dev, dt), v[p].to(dev, dt)
    for p in range(first, T):
        at = lambda t: t[p].to(dev, dt).reshape(1, 1, 1, d)
        o = ba.step_attention(at(q), at(k), at(v), store, torch.tensor([p], dtype=torch.int32, device=dev), r1.to(dev), r2.to(dev), window=window,
                              scale=1.0, append=True)
        near(o[0, 0], want[p], dt, tol16=5e-2)
        assert (want[p].mean() > 1) == (p - marked < window)


# ---- experts ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES[:2])
@pytest.mark.parametrize("E,top,groups,keep", [(8, 4, 4, 2), (8, 2, 1, 1), (16, 3, 4, 1), (64, 8, 8, 4), (6, 6, 3, 3), (1, 1, 1, 1), (96, 5, 32, 2), (12, 2, 6, 6)])
def test_group_limited_routing(place, E, top, groups, keep):
    """Negative choice scores, corrections that only steer the choice, weights left as they are."""
    dev, _ = place
    T = 40
    logits, corr = torch.randn(T, E) * 2, torch.randn(E) * 0.3 - 1.0
    ids, w, counts = moe.route(logits.to(dev), top, softmax=True, bias=corr.to(dev), renorm=False, groups=groups, keep=keep)
    s = torch.softmax(logits.double(), -1)
    seen = torch.zeros(E, dtype=torch.int32)
    for t in range(T):
        want = O.choose_experts(s[t], corr.double(), top, {"count": groups, "keep": keep})
        assert ids[t].tolist() == want
        near(w[t], s[t, want], torch.float32)
        seen[want] += 1
    assert counts.cpu().tolist() == seen.tolist()


@pytest.mark.parametrize("place", PLACES[:2])
def test_group_choice_follows_the_corrected_best_expert(place):
    """Group 1 holds the second best expert of all but a lower best one; group 2 wins by its correction alone."""
    dev, _ = place
    s = torch.tensor([[0.30, 0.01, 0.25, 0.24, 0.02, 0.18]])
    corr = torch.tensor([-2.0, -2.0, -2.0, -2.0, -2.0, -1.0])
    ids, w, _ = moe.route(torch.log(s).to(dev), 2, softmax=True, bias=corr.to(dev), renorm=False, groups=3, keep=1)
    assert ids.tolist() == [[5, 4]]
    near(w, torch.tensor([[0.18, 0.02]]).double(), torch.float32)
    ids, w, _ = moe.route(torch.log(s).to(dev), 3, softmax=True, bias=corr.to(dev), renorm=False, groups=3, keep=2)
    assert ids.tolist() == [[5, 0, 4]]                    # 0.02 of the kept group, not 0.25 of the group that lost


@pytest.mark.gpu
@pytest.mark.parametrize("T", [1, 3, 130])
def test_fused_routing_matches(T):
    h, E = 64, 16
    x, w, corr = torch.randn(T, h).bfloat16().cuda(), torch.randn(E, h).cuda(), (torch.randn(E) * 0.2 - 1).cuda()
    kw = dict(softmax=True, bias=corr, renorm=False, groups=4, keep=2)
    assert moe.route_fused_supported(x, w)
    ids, wt, counts = moe.route_fused(x, w, 3, **kw)
    ids2, wt2, counts2 = moe.route((x.float().cpu().double() @ w.cpu().double().T).float().cuda(), 3, **kw)
    assert torch.equal(ids, ids2) and torch.equal(counts, counts2)
    near(wt, wt2.cpu(), torch.float32)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("h,ff,E,top", [(40, 24, 4, 2), (64, 136, 8, 3), (16, 8, 1, 1)])
def test_expert_bank(place, h, ff, E, top):
    dev, dt = place
    T = 21
    x, gu, dn, add = rnd(T, h), rnd(E, 2 * ff, h, scale=h ** -0.5), rnd(E, h, ff, scale=ff ** -0.5), rnd(T, h)
    ids = torch.stack([torch.randperm(E)[:top] for _ in range(T)])
    wt = torch.rand(T, top)
    bank = moe.ExpertBank(gu.to(dev, dt), dn.to(dev, dt))
    w = {f"e{e}.{n}": t for e in range(E) for n, t in (("gate", gu[e, :ff]), ("up", gu[e, ff:]), ("down", dn[e]))}
    want = torch.stack([sum(wt[t, j].double() * O.gated_ff(w, f"e{ids[t, j]}", x[t]) for j in range(top)) for t in range(T)]) + add
    for _ in range(2):                                    # the second call finds the banks in the GEMM's layout
        near(moe.moe_bank_forward(x.to(dev, dt), ids.int().to(dev), wt.to(dev), bank, add=add.to(dev, dt)), want, dt)
    assert torch.equal(bank.gate_up.cpu().double(), gu) and torch.equal(bank.down.cpu().double(), dn)


def test_interleaved_bank_of_a_reused_address_is_not_taken_for_the_old_one():
    a = torch.randn(2, 16, 8)
    first = moe.interleave_gate_up(a)
    b = a.detach()                                        # another tensor object at the same address
    b.mul_(2)
    assert torch.equal(moe.interleave_gate_up(b), first * 2)


# ---- norm on the sublayer's output --------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("D,gains", [(40, 1), (40, 40), (13, 1), (2048, 1), (5120, 5120), (9000, 1)])
def test_post_norm_residual(place, D, gains):
    dev, dt = place
    x, resid, g = rnd(5, D, scale=1e-3), torch.randn(5, D).double() * 3, rnd(gains)
    want = resid.float().double() + O.rms_unit(x, 1e-5) * g
    r = resid.float().to(dev)
    y = post_norm_residual(x.to(dev, dt), g.float().to(dev), 1e-5, r, dt)
    near(r, want, torch.float32)                          # the stream keeps 32 bits whatever the compute dtype
    near(y, want, dt)
    assert y.dtype == dt
    near(post_norm_residual(r, g.float().to(dev), 1e-5, out_dtype=dt), O.rms_unit(want, 1e-5) * g, dt)
