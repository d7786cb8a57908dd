"""The mechanisms of the Nizedra design one by one, against the plain implementation in ``nizedra_oracle``: the norm between two sublayers,
xIELU and where it is taken, distance buckets, attention with mixed heads over prompts and over stores, latent rows and rotation,
windows, attention over latent rows, a product per head, lightning attention, the norm over all heads with a gate."""
import math

import pytest
import torch

import nizedra_oracle as O
from tyr_b200.models.common import KVCache, xielu_mlp
from tyr_b200.ops import delta_rule as dr
from tyr_b200.ops import flash
from tyr_b200.ops import joint_attention as ja
from tyr_b200.ops import latent as lt
from tyr_b200.ops import lightning as lg
from tyr_b200.ops import skinny
from tyr_b200.ops.biased_attention import qk_norm_store
from tyr_b200.ops.embed import position_turns
from tyr_b200.ops.mix_conv import activate
from tyr_b200.ops.norm import sandwich_norm

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


def f32(x, dev):
    return x.float().contiguous().to(dev)


# ---- norms and activation -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("D", [16, 50, 136, 2048, 9000])
def test_norm_between_two_sublayers(place, D):
    dev, dt = place
    eps = 0.3                                             # one that matters, inside the root
    x, b, post, gain, r = rnd(3, 5, D), rnd(D), rnd(D), rnd(D), torch.randn(3, 5, D).double()
    resid = f32(r, dev)
    h = sandwich_norm(x.to(dev, dt), f32(post, dev), f32(gain, dev), eps, resid, dt, bias=f32(b, dev))
    want = r + O.norm(x + b, post, eps)
    near(resid, want, torch.float32, 1e-6)
    near(h, O.norm(want, gain, eps), dt)
    out = window(dev, dt, D, 3, 5)                        # no norm after it: the stream itself, into a window of a wider buffer
    sandwich_norm(x.to(dev, dt), f32(post, dev), None, eps, resid, dt, out=out)
    want = want + O.norm(x, post, eps)
    near(resid, want, torch.float32, 1e-6)
    near(out, want, dt)
    h = sandwich_norm(x.to(dev, dt), None, f32(gain, dev), eps, resid, dt, replace=True)
    near(resid, x, torch.float32, 1e-7)
    near(h, O.norm(x, gain, eps), dt)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("rows,width,ff", [(3, 64, 96), (20, 64, 40), (12, 50, 33), (200, 64, 136), (300, 40, 75)])
def test_xielu_of_a_product(place, rows, width, ff):
    """In the epilogue of the tensor-core product, of the decode product, and alone."""
    dev, dt = place
    act = torch.tensor([-0.7, 1.3]).double()
    w = {"up": rnd(ff, width, scale=width ** -0.5), "down": rnd(width, ff, scale=ff ** -0.5), "act": act}
    a, b = float(O.softplus(act[0])), 0.5 + float(O.softplus(act[1]))
    h = rnd(rows, width, scale=2.0)
    with torch.no_grad():
        near(xielu_mlp(h.to(dev, dt), w["up"].to(dev, dt), w["down"].to(dev, dt), a, b), O.feed_forward(w, "", h), dt)
    z = torch.cat([torch.linspace(-30, 30, 400), torch.linspace(-1e-3, 1e-3, 401)]).bfloat16().double()[None]
    near(activate(z.to(dev, dt), "xielu", (a, b)), O.xielu(z, act), dt)
    near(activate(z[:, -401:].to(dev, dt).contiguous(), "xielu", (a, b)), O.xielu(z[:, -401:], act), dt)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,dv", [(3, 100), (1, 40), (6, 64), (16, 128), (5, 1000)])
def test_norm_over_all_heads_with_a_gate(place, H, dv):
    dev, dt = place
    o, g, w = torch.randn(2, 7, H * dv).double(), rnd(2, 7, H * dv), rnd(H * dv)
    z = window(dev, dt, H * dv, 2, 7)
    z.copy_(g)
    y = dr.gated_norm(f32(o, dev).unsqueeze(2), z, f32(w, dev), 0.2, "sigmoid")
    near(y, O.norm(o, w, 0.2) * O.sigmoid(g), dt)


# ---- attention with mixed heads -----------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,reach", [(16, 100), (2, 3), (8, 64), (32, 128), (7, 20), (10, 6)])
def test_distance_buckets(rows, reach):
    got = ja.distance_buckets(rows, reach).tolist()
    assert got == [O.distance_bucket(n, rows, reach) for n in range(reach + 1)]
    half = rows // 2
    assert got[:half] == list(range(half)) and got[-1] == rows - 1
    for n in range(half, reach):                           # away from the steps' edges the logarithm itself decides
        x = math.log(n / half) / math.log(reach / half) * (rows - half)
        if abs(x - round(x)) > 1e-9:
            assert got[n] == min(rows - 1, half + math.floor(x))
    # lower ends of steps that are whole numbers belong to the upper step: 8 * 16^(k / 8) for even k
    if (rows, reach) == (16, 128):
        assert [got[8], got[15], got[16], got[31], got[32], got[63], got[64], got[127]] == [8, 9, 10, 11, 12, 13, 14, 15]


def test_distance_buckets_refuse_tables_without_steps():
    for rows, reach in ((1, 5), (16, 8)):
        with pytest.raises(ValueError, match="distance table"):
            ja.distance_buckets(rows, reach)


def talk_case(T, H, G, dk, dv, softcap, rows, reach):
    """Unit queries and keys, a mix with large entries off the diagonal, a distance table with one row that stands out."""
    mix = {"scale": 0.4, "softcap": softcap, "bias_max": reach}
    q, k = (O.rms_unit(torch.randn(T, n, dk).double(), 1e-6).bfloat16().double() for n in (H, G))
    v = rnd(T, G, dv)
    temp, rel, talk = 1 + 0.5 * rnd(H), rnd(rows, H), torch.eye(H).double() + rnd(H, H, scale=0.5 * H ** -0.5)
    return mix, q, k, v, temp.bfloat16().double(), rel, talk.bfloat16().double()


def talk_of(mix, temp, rel, talk, dev):
    return ja.Talk(f32(temp, dev), f32(rel, dev), ja.distance_buckets(rel.shape[0], mix["bias_max"]).to(dev), f32(talk, dev), float(mix["softcap"]))


TALK = [(40, 6, 2, 24, 40, 2.0, 16, 20), (70, 1, 1, 8, 8, 1.0, 2, 2), (33, 5, 5, 130, 20, 30.0, 9, 31), (150, 4, 2, 64, 64, 3.0, 8, 100),
        (150, 8, 2, 128, 128, 5.0, 32, 128), (100, 16, 4, 64, 128, 20.0, 16, 60), (90, 12, 4, 32, 64, 4.0, 10, 300), (60, 32, 8, 128, 64, 4.0, 12, 40),
        (50, 20, 1, 64, 64, 4.0, 12, 40), (37, 40, 8, 16, 24, 4.0, 12, 40), (130, 7, 7, 48, 80, 6.0, 16, 90), (45, 32, 2, 128, 128, 6.0, 16, 90),
        (400, 4, 1, 64, 64, 3.0, 16, 1000), (300, 2, 1, 32, 16, 3.0, 4, 64)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("case", TALK)
def test_talking_heads_over_prompts(place, case):
    dev, dt = place
    T = case[0]
    mix, q, k, v, temp, rel, talk = talk_case(*case)
    want = O.talking_attention(q, k, v, mix, temp, rel, talk).flatten(1)
    # two rows: the whole prompt, and one that ends early (its padding is noise)
    pad = lambda t: torch.cat([t[:T // 2], torch.randn(T - T // 2, *t.shape[1:]).bfloat16().double()])
    dkp, dvp = ja.store_dims(case[3], case[4], dt, dev)
    batch = lambda t, d: torch.nn.functional.pad(torch.stack([t, pad(t)]), (0, d - t.shape[2])).to(dev, dt)
    for bound in (None, 1.02 * case[3]):                   # with and without a known bound of the products: two ways to take the softmax
        got = ja.prompt_attention(batch(q, dkp), batch(k, dkp), batch(v, dvp)[..., :case[4]], scale=mix["scale"], talk=talk_of(mix, temp, rel, talk, dev),
                                  dot_bound=bound)
        near(got[0], want, dt)
        near(got[1, :T // 2], want[:T // 2], dt)


def stores(dev, dt, B, G, cap, dk, dv, shared=False, ring=False):
    st = KVCache.allocate(B, G, cap, dk, dev, dt, ring=ring, v_dim=dv, shared=shared)
    for t in {id(st.k): st.k, id(st.v): st.v}.values():
        t.fill_(2.0)                                      # slots that hold nothing yet must not matter
    return st


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("case", TALK)
def test_talking_heads_one_token_per_row(place, case):
    """Rows at unequal positions, slots past a row's position unwritten."""
    dev, dt = place
    T, H, G, dk, dv = case[:5]
    mix, q, k, v, temp, rel, talk = talk_case(*case)
    want = O.talking_attention(q, k, v, mix, temp, rel, talk)
    dkp, dvp = ja.store_dims(dk, dv, dt, dev)
    st = stores(dev, dt, 4, G, T + 3, dkp, dvp)
    pos = [T - 1, 0, T // 2, 1]                            # in a long store, the early rows leave slices of the keys empty
    fill = lambda t, n, d: torch.nn.functional.pad(t[:n].transpose(0, 1), (0, d - t.shape[2])).to(dev, dt)
    for b, p in enumerate(pos):
        st.k[b, :, :p + 1], st.v[b, :, :p + 1] = fill(k, p + 1, dkp), fill(v, p + 1, dvp)
    qs = torch.nn.functional.pad(torch.stack([q[p][None] for p in pos]), (0, dkp - dk)).to(dev, dt)
    for bound in (None, 1.02 * dk):
        got = ja.step_attention(qs, st, int32(pos, dev), dv, scale=mix["scale"], talk=talk_of(mix, temp, rel, talk, dev), dot_bound=bound)
        near(got[:, 0], want[pos], dt)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("at", [0, 1, 31, 32, 63, 64, 500, 898, 899])
def test_one_far_key_among_many(place, at):
    """One key stands out in one head's score, and the mix carries it to another head; values name their positions."""
    dev, dt = place
    T, H, G, d = 900, 4, 2, 64
    k = 0.05 * torch.randn(T, G, d).double()
    q = 0.05 * torch.randn(T, H, d).double()
    k[at, 0], q[-1, 1] = 4.0, 4.0                          # heads 0 and 1 read key head 0
    v = torch.stack([torch.full((T,), -1.0), torch.arange(T) / T], -1).double()[:, None].repeat(1, G, d // 2)
    k, q, v = (t.bfloat16().double() for t in (k, q, v))
    mix = {"scale": 0.125, "softcap": 40.0, "bias_max": 64}
    rel, temp = torch.zeros(16, H).double(), torch.ones(H).double()
    talk = torch.eye(H).double()
    talk[3, 1] = 1.0
    want = O.talking_attention(q, k, v, mix, temp, rel, talk, T - 1)[-1]
    assert abs(float(want[3, 1]) - at / T) < 0.01 and abs(float(want[0, 1]) - 0.5) < 0.05
    tk = talk_of(mix, temp, rel, talk, dev)
    near(ja.prompt_attention(q[None].to(dev, dt), k[None].to(dev, dt), v[None].to(dev, dt), scale=0.125, talk=tk)[0, -1], want.flatten(), dt, tol16=1e-2)
    st = KVCache(k.transpose(0, 1)[None].to(dev, dt).contiguous(), v.transpose(0, 1)[None].to(dev, dt).contiguous())
    near(ja.step_attention(q[None, -1:].to(dev, dt), st, int32([T - 1], dev), d, scale=0.125, talk=tk)[0, 0], want, dt, tol16=1e-2)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("n", [3, 4, 5, 8, 9, 39, 40, 41])
def test_distance_bias_at_the_edges_of_its_steps(place, n):
    """A table row that outweighs everything: the keys at its distances take all the attention."""
    dev, dt = place
    T, H, d, rows, reach = 120, 2, 32, 8, 40
    q, k, v = torch.zeros(T, H, d).double(), torch.zeros(T, 1, d).double(), rnd(T, 1, d)
    rel = torch.zeros(rows, H).double()
    rel[O.distance_bucket(n, rows, reach), 1] = 30.0
    mix = {"scale": 1.0, "softcap": 5.0, "bias_max": reach}
    want = O.talking_attention(q, k, v, mix, torch.ones(H).double(), rel, torch.eye(H).double())
    tk = talk_of(mix, torch.ones(H), rel, torch.eye(H), dev)
    near(ja.prompt_attention(*(t[None].to(dev, dt) for t in (q, k, v)), scale=1.0, talk=tk)[0], want.flatten(1), dt)
    st = KVCache(k.transpose(0, 1)[None].to(dev, dt).contiguous(), v.transpose(0, 1)[None].to(dev, dt).contiguous())
    near(ja.step_attention(q[None, -1:].to(dev, dt), st, int32([T - 1], dev), d, scale=1.0, talk=tk)[0, 0], want[-1], dt)


@pytest.mark.parametrize("place", PLACES)
def test_biases_and_norms_without_weights(place):
    """Projection biases enter before the norm of queries and keys; padded channels of the rows are zero; the store gets the same."""
    dev, dt = place
    B, S, H, G, dk, dv, dkp, dvp = 2, 9, 4, 2, 20, 12, 32, 16
    y, bias = rnd(B, S, (H + G) * dk + G * dv), rnd((H + G) * dk + G * dv)
    st = stores(dev, dt, B, G, 12, dkp, dvp)
    lens = [9, 4]
    q, k, v = qk_norm_store(y.to(dev, dt), None, None, H, G, dk, dv, 0.1, dkp=dkp, dvp=dvp, store=st, lens=int32(lens, dev), bias=f32(bias, dev))
    z = y + bias
    part = lambda a, n, d: z[..., a:a + n * d].reshape(B, S, n, d)
    wq, wk, wv = O.rms_unit(part(0, H, dk), 0.1), O.rms_unit(part(H * dk, G, dk), 0.1), part((H + G) * dk, G, dv)
    for got, want in ((q, wq), (k, wk), (v, wv)):
        near(got[..., :want.shape[3]], want, dt)
        assert not bool(got[..., want.shape[3]:].any())
    for b, n in enumerate(lens):
        near(st.k[b, :, :n, :dk], wk[b, :n].transpose(0, 1), dt)
        near(st.v[b, :, :n, :dv], wv[b, :n].transpose(0, 1), dt)
        assert bool((st.k[b, :, n:] == 2.0).all())


# ---- latent attention ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("nq,rank,rot,dims,ring", [(40, 48, 16, 16, False), (17, 33, 6, 4, True), (96, 64, 32, 32, True), (8, 8, 2, 2, False), (24, 40, 12, 0, True)])
def test_latent_rows(place, nq, rank, rot, dims, ring):
    """Norms of both latents, rotation by position, rows of the store: prompts of unequal length, then single tokens far out."""
    dev, dt = place
    B, S, cap, base = 2, 21, 8 if ring else 40, 500.0
    y, qw, kw = rnd(B, S, nq + rank + rot), rnd(nq), rnd(rank)
    width, qwidth = rank + rot + 6, nq + 3
    turns = position_turns(dims, base, dev)
    st = stores(dev, dt, B, 1, cap, width, width, shared=True, ring=ring)
    lens = [21, 5]
    cq, rows = lt.latent_norm_store(y.to(dev, dt), f32(qw, dev), f32(kw, dev), turns, rot, 0.2, q_width=qwidth, width=width, store=st, lens=int32(lens, dev))
    for b in range(B):
        want = torch.cat([O.norm(y[b, :, nq:nq + rank], kw, 0.2), O.rotate(y[b, :, nq + rank:], base, dims) if dims else y[b, :, nq + rank:]], -1)
        near(cq[b, :, :nq], O.norm(y[b, :, :nq], qw, 0.2), dt)
        near(rows[b, :, :rank + rot], want, dt)
        assert not bool(rows[b, :, rank + rot:].any()) and not bool(cq[b, :, nq:].any())
        for p in range(lens[b]):
            if not ring or p >= lens[b] - cap:
                assert torch.equal(st.k[b, 0, p % cap], rows[b, p])
        assert ring and lens[b] >= cap or bool((st.k[b, 0, lens[b]:] == 2.0).all())
    far = [70_001, 13] if ring else [39, 13]
    cq, _ = lt.latent_norm_store(y[:, :1].to(dev, dt), f32(qw, dev), f32(kw, dev), turns, rot, 0.2, q_width=qwidth, width=width, store=st, pos=int32(far, dev))
    for b, p in enumerate(far):
        x = y[b, :1, nq + rank:]
        want = torch.cat([O.norm(y[b, :1, nq:nq + rank], kw, 0.2), O.rotate(x, base, dims, p) if dims else x], -1)[0]
        near(st.k[b, 0, p % cap if ring else p, :rank + rot], want, dt)


@pytest.mark.parametrize("place", PLACES)
def test_rotation_of_query_heads(place):
    dev, dt = place
    q, base = rnd(2, 30, 3, 40), 1000.0
    turns = position_turns(8, base, dev)
    x = q.to(dev, dt)
    lt.rotate_heads(x[..., 20:32], turns)                 # in place: 12 channels, of which 8 turn; the rest of the row stays
    want = q.clone()
    for b in range(2):
        want[b, ..., 20:32] = O.rotate(q[b, ..., 20:32], base, 8)
    near(x, want, dt)
    assert torch.equal(x[..., :20].cpu().double(), q[..., :20]) and torch.equal(x[..., 28:].cpu().double(), q[..., 28:])
    out, pos = torch.full((2, 1, 3, 20), 5.0, device=dev, dtype=dt), [1_000_003, 7]
    lt.rotate_heads(q[:, :1, :, 20:32].to(dev, dt), turns, int32(pos, dev), out[..., 2:])
    for b, p in enumerate(pos):
        near(out[b, :, :, 2:14], O.rotate(q[b, :1, :, 20:32], base, 8, p), dt)
    assert bool((out[..., :2] == 5.0).all()) and not bool(out[..., 14:].any())


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("T,H,dk,dv,win", [(40, 3, 24, 16, 7), (300, 2, 96, 64, 140), (300, 2, 96, 64, 128), (260, 4, 64, 128, 1), (140, 2, 128, 40, None),
                                           (150, 1, 200, 136, 30), (50, 2, 300, 20, 12), (500, 2, 48, 48, 131)])
def test_windowed_attention_over_prompts(place, T, H, dk, dv, win):
    dev, dt = place
    q, k, v = rnd(T, H, dk), rnd(T, H, dk), rnd(T, H, dv)
    want = O.window_attention(q, k, v, dk ** -0.5, win).flatten(1)
    q, k, v = (t[None].to(dev, dt) for t in (q, k, v))
    near(ja.prompt_attention(q, k, v, scale=dk ** -0.5, window=win)[0], want, dt)
    if dev == "cuda" and flash.sink_supported(q, k, v, None, None):
        near(flash.flash_fwd_sink(q, k, v, scale=dk ** -0.5, window=win)[0], want, dt)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("win", [2, 16, 100, 128, 129])
def test_key_just_inside_and_just_outside_the_window(place, win):
    """The key at distance window - 1 takes all the attention; the one a position further back would, and is not seen."""
    dev, dt = place
    T, d, i = 300, 64, 270
    for far, seen in ((win - 1, True), (win, False)):
        q, k, v = torch.zeros(T, 1, d).double(), torch.zeros(T, 1, d).double(), torch.zeros(T, 1, d).double()
        q[i], k[i - far], v[i - far] = 4.0, 4.0, 1.0
        want = O.window_attention(q, k, v, 0.1, win)
        assert (float(want[i, 0, 0]) > 0.99) == seen
        a = [t[None].to(dev, dt) for t in (q, k, v)]
        got = [ja.prompt_attention(*a, scale=0.1, window=win)[0, i]]
        if dev == "cuda" and dt == torch.bfloat16:
            got.append(flash.flash_fwd_sink(*a, scale=0.1, window=win)[0, i])
        row = torch.cat([v[:, 0], k[:, 0]], -1)            # the same as latent rows: value channels first
        ql = torch.cat([torch.zeros(d).double(), q[i, 0]])[None, None, None].to(dev, dt)
        for cap in (T, win):
            st = stores(dev, dt, 1, 1, cap, 2 * d, 2 * d, shared=True, ring=cap == win)
            for p in range(i + 1):
                st.k[0, 0, p % cap] = row[p].to(dev, dt)
            got.append(ja.step_attention(ql, st, int32([i], dev), d, scale=0.1, window=win)[0, 0, 0])
        for g in got:
            assert abs(float(g.float().mean()) - float(want[i].mean())) < 1e-2


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("H,rank,rot,win,ring", [(3, 24, 8, 9, True), (4, 112, 32, 40, True), (1, 8, 0, None, False), (20, 64, 32, 33, False), (5, 520, 24, 64, True),
                                                 (33, 96, 32, 50, True), (16, 512, 64, 100, True), (40, 1100, 20, 17, True)])
def test_attention_over_latent_rows(place, H, rank, rot, win, ring):
    """Every head reads the row of a position as its key and the row's first channels as its value; rows at unequal positions."""
    dev, dt = place
    T, width = 200, -(-(rank + rot) // 32) * 32
    rows, scale = rnd(T, rank + rot), (rank + rot) ** -0.5
    cap = win if ring else T
    st = stores(dev, dt, 3, 1, cap, width, width, shared=True, ring=ring)
    pos, q = [T - 1, 5, 90], rnd(3, H, rank + rot)
    for b, p in enumerate(pos):
        for j in range(p + 1):
            st.k[b, 0, j % cap] = torch.nn.functional.pad(rows[j], (0, width - rank - rot)).to(dev, dt)
    out = window(dev, dt, rank, 3, 1, H)
    ql = torch.nn.functional.pad(q, (0, width - rank - rot))[:, None].to(dev, dt)
    ja.step_attention(ql, st, int32(pos, dev), rank, scale=scale, window=win, out=out)
    for b, p in enumerate(pos):
        k = rows[:p + 1, None].expand(-1, H, -1)
        want = O.window_attention(torch.cat([torch.zeros(p, H, rank + rot).double(), q[b][None]]), k, k[..., :rank], scale, win)[-1]
        near(out[b, 0], want, dt)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("M,H,N,K", [(1, 3, 40, 64), (9, 4, 128, 32), (35, 2, 17, 96), (5, 2, 24, 20)])
def test_product_per_head(place, M, H, N, K):
    dev, dt = place
    x, w = rnd(M, H, K + 8), rnd(H, N, K, scale=K ** -0.5)
    out = torch.full((M, H, N + 3), 7.0, device=dev, dtype=dt)
    skinny.head_products(x.to(dev, dt), w.to(dev, dt), out)
    near(out[..., :N], torch.einsum("mhk,hnk->mhn", x[..., :K], w), dt)
    assert bool((out[..., N:] == 7.0).all())


# ---- lightning ----------------------------------------------------------------------------------------------------
LIGHT = [(2, 24, 40, (0.5, 0.99)), (1, 8, 8, (1.0,)), (3, 64, 64, (0.7, 0.999, 1e-3)), (2, 128, 128, (0.9, 0.9995)), (2, 130, 20, (0.8, 0.97)), (2, 96, 72, (0.6, 0.95)),
         (1, 33, 7, (0.9,)), (2, 128, 256, (0.99, 0.0)), (4, 16, 192, (0.2, 0.9, 0.99, 0.999))]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("case", LIGHT)
def test_lightning_over_prompts_and_tokens(place, case):
    """Prompts of unequal length (padding leaves the state alone), then tokens one by one from that state."""
    dev, dt = place
    H, dk, dv, decay = case
    T, lens = 150, [150, 1, 64, 83] if dk != 64 else [77, 65, 128, 150]
    x = rnd(4, T + 3, H * (2 * dk + dv) + 8)
    dec = torch.tensor(decay, dtype=torch.float64)
    cut = lambda t: [t[..., a:b].unflatten(2, (H, -1)) for a, b in ((0, H * dk), (H * dk, 2 * H * dk), (2 * H * dk, H * (2 * dk + dv)))]
    act = (lambda t: O.silu(t).bfloat16().double()) if dt == torch.bfloat16 else O.silu
    y, z = x.to(dev, dt), act(x).to(dev, dt)               # prompts come activated, single tokens do not
    state = torch.full((4, H, dk, dv), 9.0, device=dev)
    out = lg.prefill(*cut(z[:, :T]), dec.to(dev), state, int32(lens, dev))
    for b, n in enumerate(lens):
        seq = torch.cat([x[b, :n], x[b, T:]])
        q, k, v = (act(t[0]) for t in cut(seq[None]))
        want, _ = O.decayed_recurrence(q, k, v, dec)
        _, mid = O.decayed_recurrence(q[:n], k[:n], v[:n], dec)
        near(out[b, :n], want[:n], dt, tol16=2e-5)          # fp32 read-out of 16-bit operands
        near(state[b], mid, dt, tol16=2e-5)
        assert bool(torch.isfinite(out[b]).all())
    for t in range(3):
        o = lg.step(*cut(y[:, T + t:T + t + 1]), dec.to(dev), state)
        for b, n in enumerate(lens):
            q, k, v = (act(a[0]) for a in cut(torch.cat([x[b, :n], x[b, T:T + t + 1]])[None]))
            near(o[b, 0], O.decayed_recurrence(q, k, v, dec)[0][-1], dt, tol16=2e-5)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("T", [1, 2, 63, 64, 65, 128, 1500])
def test_lightning_keeps_a_long_memory(place, T):
    """Nearly lossless decay over many chunks: the first token still counts at the end, and the last chunk may hold any number of tokens."""
    dev, dt = place
    H, d = 1, 64
    x = rnd(1, T, 3 * d, scale=0.2)
    x[0, 0] = 3.0
    dec = torch.tensor([0.9999], dtype=torch.float64)
    cut = lambda t: [t[..., i * d:(i + 1) * d].unflatten(2, (H, -1)) for i in range(3)]
    state = torch.zeros(1, H, d, d, device=dev)
    out = lg.prefill(*cut(x.to(dev, dt)), dec.to(dev), state)
    want, end = O.decayed_recurrence(*(t[0] for t in cut(x)), dec)
    near(out[0], want, dt, tol16=2e-5)
    near(state[0], end, dt, tol16=2e-5)
