"""The mechanisms of Vonulix one by one: rotation, value norm and store, attention with kept first positions and turned values, experts of the
weighted input, gates, token input and depth average, against the plain implementation in ``vonulix_oracle``."""
import math

import pytest
import torch
import torch.nn.functional as F

import vonulix_oracle as O
from tyr_b200.models.common import KVCache
from tyr_b200.ops import gates, kept_attention as ka, moe
from tyr_b200.ops.depth import depth_average
from tyr_b200.ops.embed import embed_positions
from tyr_b200.ops.gemm import gemm

GPU = pytest.mark.gpu
PLACES = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=GPU), pytest.param(("cuda", torch.bfloat16), marks=GPU)]
TOL = {torch.float32: 3e-5, torch.bfloat16: 1.2e-2}


def rnd(*shape, seed=0, dtype=torch.float32):
    """Values that both precisions hold."""
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).bfloat16().to(dtype)


def close(got, want, dtype, tol=None):
    got, want = got.detach().double().cpu(), want.double()
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-6))
    assert err < (tol or TOL[dtype]), err


def at_place(place, *ts):
    return tuple(t.to(device=place[0], dtype=place[1]) if t.is_floating_point() else t.to(place[0]) for t in ts)


# ---- stores -------------------------------------------------------------------------------------------------------
def test_store_with_kept_slots():
    """The first positions stay, the others share a ring; whatever lies at a slot is the position that ``held`` names."""
    c = KVCache.allocate(1, 1, 9, 1, "cpu", torch.float32, ring=True, keep=4)
    seen = {}
    for first, n in ((0, 3), (3, 1), (4, 4), (8, 1), (9, 7), (16, 1)):
        x = torch.arange(first, first + n, dtype=torch.float32).reshape(1, 1, n, 1)
        c.write(x, -x)
        for p in range(first, first + n):
            seen[int(c.slots(torch.tensor([p])))] = p
        at = c.held(0, first + n - 1)
        assert c.k[0, 0, c.slots(at), 0].tolist() == at.tolist() == sorted(seen.values()) and torch.equal(c.v, -c.k)
    assert at.tolist() == [0, 1, 2, 3, 12, 13, 14, 15, 16]
    with pytest.raises(ValueError, match="beyond the kept"):
        KVCache.allocate(1, 1, 4, 1, "cpu", torch.float32, ring=True, keep=4)
    assert c.clone().keep == 4


# ---- rotation, value norm, store ----------------------------------------------------------------------------------
SHAPES = [  # H, G, dk, dv, rot dims, factor
    (6, 2, 32, 48, 16, 1.5), (3, 3, 24, 40, 24, 1.0), (4, 1, 128, 128, 64, 8.0), (16, 4, 96, 64, 96, 2.0), (2, 1, 7, 6, 4, 3.0), (1, 1, 2, 2, 2, 1.0), (2, 2, 140, 130, 20, 1.0),
    (5, 5, 64, 16, 0, 1.0)]


def oracle_qkv(y, H, G, dk, dv, dims, base, factor, eps, p0):
    """y: [S, n] of one row whose first token is at p0."""
    S = y.shape[0]
    q, k, v = y[:, :H * dk].reshape(S, H, dk), y[:, H * dk:(H + G) * dk].reshape(S, G, dk), y[:, (H + G) * dk:(H + G) * dk + G * dv].reshape(S, G, dv)
    v = O.over_rms(v, eps)
    each = lambda x, *a: torch.stack([O.turn(x[t], p0 + t, *a) for t in range(S)])
    return each(q, dims, base, factor), each(k, dims, base, factor), each(v, dv, base)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("shape", SHAPES)
def test_rotation_value_norm_and_store(place, shape):
    """Prompts of unequal length, then one token per row far on; a plain store and one of kept slots and a ring."""
    H, G, dk, dv, dims, factor = shape
    B, S, base, eps, lens = 3, 21, 500.0, 1e-2, [21, 4, 13]
    n = (H + G) * dk + G * dv
    y, y1 = rnd(B, S, n + 16, seed=1), rnd(B, 1, n + 16, seed=2)
    pos = [40, 7, 300]
    kt, vt = (ka.turn_table(d, base, f, 301, place[0]) for d, f in ((dims, factor), (dv, 1.0)))
    dkp, dvp = ka.step_dims(H, G, dk, dv, *reversed(place))
    yd, y1d = at_place(place, y, y1)
    for store in (KVCache.allocate(B, G, 301, dkp, *place, v_dim=dvp), KVCache.allocate(B, G, 3 + 6, dkp, *place, v_dim=dvp, ring=True, keep=3)):
        q, k, v = ka.rotary_store(yd, H, G, dk, dv, kt, vt, eps, store=store, lens=torch.tensor(lens, dtype=torch.int32, device=place[0]))
        assert q.shape == (B, S, H, dk) and k.shape == (B, S, G, dk) and v.shape == (B, S, G, dv)
        for b in range(B):
            wq, wk, wv = oracle_qkv(y[b].double(), H, G, dk, dv, dims, base, factor, eps, 0)
            for got, want in ((q, wq), (k, wk), (v, wv)):
                close(got[b, :lens[b]], want[:lens[b]], place[1])
            at = store.held(0, lens[b] - 1)
            sl = store.slots(at)
            close(store.k[b][:, sl, :dk], wk[at].transpose(0, 1), place[1])
            close(store.v[b][:, sl, :dv], wv[at].transpose(0, 1), place[1])
            rest = sorted(set(range(store.cap)) - set(sl.tolist()))
            assert not store.k[b][:, rest].any() and not store.v[b][:, rest].any()
        q1, _, _ = ka.rotary_store(y1d, H, G, dk, dv, kt, vt, eps, store=store, pos=torch.tensor(pos, dtype=torch.int32, device=place[0]))
        assert q1.shape == (B, 1, H, dkp) and not q1[..., dk:].any() and not store.k[..., dk:].any() and not store.v[..., dv:].any()
        for b in range(B):
            wq, wk, wv = oracle_qkv(y1[b].double(), H, G, dk, dv, dims, base, factor, eps, pos[b])
            sl = int(store.slots(torch.tensor([pos[b]])))
            close(q1[b, :, :, :dk], wq, place[1])
            close(store.k[b][:, sl, :dk], wk[0], place[1])
            close(store.v[b][:, sl, :dv], wv[0], place[1])


def test_far_positions_keep_their_angles():
    """The table reduces angles in double: a fast pair at a position of a million."""
    t = ka.turn_table(8, 100.0, 3.0, 1_000_001, "cpu")
    for i in range(4):
        a = math.fmod(1_000_000 * 100.0 ** (-i / 4) / 3.0, 2 * math.pi)
        assert abs(float(t[-1, i, 0]) - math.cos(a)) < 1e-6 and abs(float(t[-1, i, 1]) - math.sin(a)) < 1e-6
    assert ka.turn_table(0, 10.0, 1.0, 5, "cpu") is None


# ---- attention ----------------------------------------------------------------------------------------------------
def oracle_attention(q, k, v, gate, scale, window, keep, base):
    """One sequence whose keys stand at 0 .. and whose queries are the last ones; values as stored."""
    first = k.shape[0] - q.shape[0]
    o = O.attend(q, k, v, scale, window, keep, first)
    o = torch.stack([O.turn(o[i], -(first + i), v.shape[2], base) for i in range(q.shape[0])])
    return (o * O.sigmoid(gate)[..., None]).flatten(1)


PROMPTS = [  # T, H, G, dk, dv, window, keep
    (70, 6, 2, 32, 48, 9, 4), (300, 2, 1, 96, 96, 50, 7), (700, 2, 2, 64, 128, 130, 3), (530, 2, 1, 128, 64, 129, 140), (300, 1, 1, 128, 128, 128, 128), (400, 1, 1, 64, 32, 20, 0),
    (260, 2, 1, 40, 16, None, 0), (150, 3, 3, 24, 40, 17, 30), (40, 4, 1, 130, 140, 5, 2), (20, 18, 1, 6, 2, 3, 1), (513, 1, 1, 16, 16, 1, 1), (1, 2, 1, 64, 64, 4, 2), (257, 1, 1, 8, 8, 256, 1),
    (900, 1, 1, 64, 64, 100, 260)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("case", PROMPTS)
def test_prompt_attention(place, case):
    T, H, G, dk, dv, window, keep = case
    q, k, v, gate = rnd(1, T, H, dk, seed=3), rnd(1, T, G, dk, seed=4), rnd(1, T, G, dv, seed=5), rnd(1, T, H + 3, seed=6)
    table = ka.turn_table(dv, 200.0, 1.0, T + 5, place[0])
    got = ka.prompt_attention(*at_place(place, q, k, v), scale=0.2, window=window, keep=keep, head_gate=at_place(place, gate)[0][..., 2:2 + H], back=table)
    want = oracle_attention(q[0].double(), k[0].double(), v[0].double(), gate[0, :, 2:2 + H].double(), 0.2, window, keep, 200.0)
    close(got[0], want, place[1])


@pytest.mark.parametrize("place", PLACES)
def test_prompt_attention_without_turns_and_gate(place):
    q, k, v = rnd(2, 200, 4, 64, seed=3), rnd(2, 200, 2, 64, seed=4), rnd(2, 200, 2, 72, seed=5)
    got = ka.prompt_attention(*at_place(place, q, k, v), scale=0.1, window=30, keep=5)
    want = torch.stack([O.attend(q[b].double(), k[b].double(), v[b].double(), 0.1, 30, 5).flatten(1) for b in range(2)])
    close(got, want, place[1])


STEPS = [  # positions of the rows, H, G, dk, dv, window, keep, ring
    ((40, 0, 8), 6, 2, 32, 48, 9, 4, True), ((3, 12, 13, 14), 6, 2, 96, 96, 10, 3, True), ((1500, 700, 129), 8, 2, 128, 128, 600, 6, True), ((1500, 64, 9), 8, 8, 64, 128, 600, 6, False),
    ((900, 2), 16, 1, 128, 64, None, 0, False), ((900, 301), 16, 1, 64, 64, 200, 300, True), ((70, 20, 19), 3, 3, 24, 40, 17, 3, True), ((30, 31), 18, 1, 6, 2, 3, 1, True),
    ((9, 200), 2, 1, 130, 140, 7, 2, True), ((50, 51, 0), 1, 1, 16, 8, 1, 1, True), ((5000, 4095), 4, 2, 64, 64, 4096, 2, True), ((260,), 4, 1, 64, 64, 100, 0, True)]


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("case", STEPS)
def test_step_attention(place, case):
    """A position per row; stores that have wrapped, that have just filled and that have not."""
    pos, H, G, dk, dv, window, keep, ring = case
    B, T = len(pos), max(pos) + 1
    q, k, v, gate = rnd(B, 1, H, dk, seed=7), rnd(B, G, T, dk, seed=8), rnd(B, G, T, dv, seed=9), rnd(B, 1, H, seed=10)
    dkp, dvp = ka.step_dims(H, G, dk, dv, *reversed(place))
    store = KVCache.allocate(B, G, keep + window if ring else T + 2, dkp, *place, ring=ring, v_dim=dvp, keep=keep if ring else 0)
    for b, p in enumerate(pos):
        at = store.held(0, p)
        store.k[b][:, store.slots(at), :dk] = at_place(place, k[b][:, at])[0]
        store.v[b][:, store.slots(at), :dv] = at_place(place, v[b][:, at])[0]
    qd, gd = at_place(place, F.pad(q, (0, dkp - dk)), gate)
    got = ka.step_attention(qd, store, torch.tensor(pos, dtype=torch.int32, device=place[0]), dk, dv, scale=0.2, window=window, keep=keep, head_gate=gd,
                            back=ka.turn_table(dv, 30.0, 1.0, T, place[0]))
    want = torch.stack([oracle_attention(q[b].double(), k[b][:, :p + 1].transpose(0, 1).double(), v[b][:, :p + 1].transpose(0, 1).double(), gate[b].double(), 0.2, window,
                                         keep, 30.0) for b, p in enumerate(pos)])
    close(got, want, place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("window,keep", [(40, 5), (128, 1), (150, 130), (7, 128), (129, 129)])
def test_edges_of_the_window_and_of_the_kept_positions(place, window, keep):
    """One key at a time stands far out: the last query sees it at the window's first place and at the last kept position, and not one
    place off.  Prompts and steps."""
    T, d = 420, 64
    i = T - 1
    q, k, v = rnd(1, T, 1, d, seed=11), rnd(1, T, 1, d, seed=12), rnd(1, T, 1, d, seed=13)
    q[0, i, 0] = 0
    q[0, i, 0, 0] = 4.0
    k[..., 0] = 0
    table = ka.turn_table(d, 50.0, 1.0, T, place[0])
    where = {i - window + 1: True, i - window: i - window < keep, keep - 1: True, keep: i - keep < window, 0: True, i: True, keep + 1: i - keep - 1 < window}
    for j, seen in where.items():
        kk = k.clone()
        kk[0, j, 0, 0] = 8.0
        qd, kd, vd = at_place(place, q, kk, v)
        got = [ka.prompt_attention(qd, kd, vd, scale=0.5, window=window, keep=keep, back=table)[0, i]]
        for ring in (False, True):
            dkp, dvp = ka.step_dims(1, 1, d, d, *reversed(place))
            store = KVCache.allocate(1, 1, keep + window if ring else T, dkp, *place, ring=ring, v_dim=dvp, keep=keep if ring else 0)
            at = store.held(0, i)
            store.k[0][:, store.slots(at)], store.v[0][:, store.slots(at)] = kd[0, at].transpose(0, 1), vd[0, at].transpose(0, 1)
            got.append(ka.step_attention(qd[:, i:], store, torch.tensor([i], dtype=torch.int32, device=place[0]), d, d, scale=0.5, window=window, keep=keep, back=table)[0, 0])
        alone = O.turn(v[0, j, 0].double(), -i, d, 50.0)
        for o in got:
            same = float((o.double().cpu() - alone).abs().max()) < 0.05
            assert same == seen, (j, seen)


@GPU
def test_a_position_outside_store_and_tables_is_recorded():
    """The kernels check the position, skip the row and record it."""
    from tyr_b200.ops._common import raise_on_device_error
    store = KVCache.allocate(1, 1, 8, 64, "cuda", torch.bfloat16)
    y, table = torch.zeros(1, 1, 3 * 64, device="cuda", dtype=torch.bfloat16), ka.turn_table(64, 10.0, 1.0, 8, "cuda")
    pos = torch.tensor([8], dtype=torch.int32, device="cuda")
    q, _, _ = ka.rotary_store(y, 1, 1, 64, 64, table, table, 1e-6, store=store, pos=pos)
    with pytest.raises(RuntimeError, match="code=3"):
        raise_on_device_error("cuda")
    ka.step_attention(q, store, pos, 64, 64, scale=1.0, back=table)
    with pytest.raises(RuntimeError, match="code=3"):
        raise_on_device_error("cuda")
    for dt in (torch.bfloat16, torch.float32):                      # a ring takes any position, the table does not
        ring = KVCache.allocate(1, 1, 6, 64, "cuda", dt, ring=True)
        ka.step_attention(q.to(dt), ring, pos, 64, 64, scale=1.0, window=6, back=table)
        with pytest.raises(RuntimeError, match="code=3"):
            raise_on_device_error("cuda")


# ---- experts ------------------------------------------------------------------------------------------------------
EXPERTS = [  # T, width, experts, top, ff, shared ff
    (1, 64, 8, 3, 96, 32), (5, 64, 8, 3, 96, 160), (33, 96, 4, 2, 40, 0), (64, 128, 16, 4, 128, 256), (65, 64, 8, 3, 96, 160), (140, 64, 8, 3, 96, 160), (300, 128, 3, 1, 200, 72),
    (300, 128, 5, 5, 128, 0), (7, 50, 6, 2, 13, 11), (140, 50, 6, 2, 13, 11), (20, 32, 1, 1, 1, 1), (40, 72, 6, 2, 24, 24), (64, 64, 2, 1, 32, 32), (64, 32, 70, 20, 32, 64)]


def expert_weights(E, ff, sff, h):
    w = {}
    for j, (n, f) in enumerate([(f"e{e}", ff) for e in range(E)] + ([("shared", sff)] if sff else [])):
        for m, (name, shape) in enumerate((("gate", (f, h)), ("up", (f, h)), ("down", (h, f)))):
            w[f"{n}.{name}"] = (rnd(*shape, seed=100 + 3 * j + m) * 1.5 * shape[1] ** -0.5).bfloat16().float()
    return w


def bank(w, names, place):
    return moe.ExpertBank(*at_place(place, torch.stack([torch.cat([w[n + ".gate"], w[n + ".up"]]) for n in names]), torch.stack([w[n + ".down"] for n in names])))


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("case", EXPERTS)
def test_experts_of_the_weighted_input(place, case):
    """The weight enters before the clamps (so it is no factor of the output); limits of their own; added to the stream in place."""
    T, h, E, top, ff, sff = case
    w = expert_weights(E, ff, sff, h)
    x, s = rnd(T, h, seed=20), torch.rand(T, E, generator=torch.Generator().manual_seed(21)) * 0.9 + 0.05
    ids = torch.stack([torch.tensor(O.choose(s[t], top)) for t in range(T)])
    gate, resid = rnd(T, 3, seed=22)[:, 1], rnd(T, h, seed=23)
    f, sf = moe.ClampedExpert(0.7, 1.702), moe.ClampedExpert(1.3, 1.702)
    b, sb = bank(w, [f"e{e}" for e in range(E)], place), bank(w, ["shared"], place) if sff else None
    r = resid.to(place[0]).clone()
    wd = {k: v.double() for k, v in w.items()}
    want = resid.double().clone()
    for t in range(T):
        for e in ids[t].tolist():
            want[t] += O.expert(wd, f"e{e}", 0.7, s[t, e].double() * x[t].double())
        if sff:
            want[t] += O.sigmoid(gate[t].double()) * O.expert(wd, "shared", 1.3, x[t].double())
    wide = torch.zeros(T, 3, device=place[0])
    wide[:, 1] = gate.to(place[0])
    out = moe.weighted_input_experts(at_place(place, x)[0], ids.int().to(place[0]), torch.gather(s, 1, ids).to(place[0]), b, f, r, shared=sb, shared_form=sf if sff else None,
                                     shared_gate=wide[:, 1] if sff else None)
    assert out.dtype == place[1] and r.dtype == torch.float32
    close(r, want, place[1])
    close(out, want, place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("T", [3, 200])
def test_one_more_row_of_the_router(place, T):
    """Scores are sigmoids, not normalised; the last row is no expert but its logit is handed on."""
    from tyr_b200.models import vonulix as V
    E, h = 10, 64
    x, w = rnd(T, h, seed=30), rnd(E + 1, h, seed=31) * 0.25
    w[E] = (w[E] + 0.5 * x[0]).bfloat16().float()                   # the largest logit of token 0 must not be chosen
    m = V.Experts(w.to(place[0]), F.pad(w, (0, 0, 0, 5)).to(*place), None, None, None, None)
    ids, wt, counts, logits = V.route(V.MoeSpec(E, 4, 1, 1.0, 1, 1.0), m, at_place(place, x)[0])
    z = x.double() @ w.double().T
    close(logits[:, :E + 1], z, torch.float32)
    for t in range(T):
        want = O.choose(O.sigmoid(z[t, :E]), 4)
        assert ids[t].tolist() == want
        close(wt[t], O.sigmoid(z[t, want]), torch.float32)
    assert counts.tolist() == torch.bincount(ids.flatten().long().cpu(), minlength=E).tolist()


@GPU
@pytest.mark.parametrize("rows,n,k", [(200, 256, 64), (1, 128, 192), (300, 640, 128)])
def test_clamped_gate_in_the_products_epilogue(rows, n, k):
    x, g, u = rnd(rows, k, seed=40), rnd(n, k, seed=41) * 0.25, rnd(n, k, seed=42) * 0.25
    w = torch.stack([g.reshape(-1, 128, k), u.reshape(-1, 128, k)], 1).reshape(2 * n, k)
    got = gemm(x.bfloat16().cuda(), w.bfloat16().cuda(), act="clamped_swiglu", alpha=0.8, beta=1.702)
    zg, zu = x.double() @ g.double().T, x.double() @ u.double().T
    a = zg.clamp(max=0.8)
    close(got, a * O.sigmoid(1.702 * a) * (zu.clamp(-0.8, 0.8) + 1), torch.bfloat16)


@pytest.mark.parametrize("place", PLACES)
def test_clamped_gate_alone(place):
    z = rnd(9, 2 * 256, seed=43) * 3
    z = z.bfloat16().float()
    for n, block in ((256, 0), (200, 128)):
        zz = z.reshape(9, -1, 2, 128)
        g, u = (z[:, :256], z[:, 256:]) if block == 0 else (zz[:, :, 0].reshape(9, -1)[:, :n], zz[:, :, 1].reshape(9, -1)[:, :n])
        a = g.double().clamp(max=1.1)
        close(gates.clamped_swiglu(at_place(place, z)[0], n, 1.1, 1.702, block), a * O.sigmoid(1.702 * a) * (u.double().clamp(-1.1, 1.1) + 1), place[1])


# ---- token input, depth average, embedding ------------------------------------------------------------------------
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("rows,K,n", [(1, 64, 16), (7, 2048, 32), (16, 96, 24), (40, 64, 16), (200, 64, 16), (150, 50, 12), (3, 50, 5), (300, 128, 200), (2, 16, 1)])
def test_token_input_gate(place, rows, K, n):
    """The embedding is a window of a wider row."""
    x, w, e = rnd(rows, K, seed=50), rnd(n, K, seed=51) * K ** -0.5, rnd(rows, 3 * n, seed=52)
    w = w.bfloat16().float()
    xd, wd, ed = at_place(place, x, w, e)
    got = gates.gelu_mul_project(xd, wd, ed[:, n:2 * n])
    close(got, O.gelu_tanh(x.double() @ w.double().T) * e[:, n:2 * n].double(), place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("rows,D", [(1, 64), (5, 192), (3, 2048), (2, 4096), (3, 8192), (2, 12288), (2, 16392), (4, 50), (3, 2), (200, 128)])
@pytest.mark.parametrize("n", [1, 3, 9])
def test_depth_average(place, rows, D, n):
    eps = 1e-2
    y, x, post, gain = rnd(rows, D, seed=60), rnd(rows, D, seed=61), 1 + 0.3 * rnd(D, seed=62), 1 + 0.3 * rnd(D, seed=63)
    hist, wts = rnd(n + 1, rows, D, seed=64), rnd(n + 1, seed=65)
    for last in (False, True):
        xd, hd = x.to(place[0]).clone(), hist.to(place[0]).clone()
        h = depth_average(at_place(place, y)[0], post.to(place[0]), xd, hd, n, wts.to(place[0]), gain.to(place[0]), eps, place[1], store=not last)
        X = x.double() + O.over_rms(y.double(), eps) * post.double()
        avg = O.depth_average(wts.double(), [*hist[:n].double(), X])
        close(xd, avg, torch.float32)
        close(h, O.over_rms(avg, eps) * gain.double(), place[1])
        close(hd[n], hist[n].double() if last else X, torch.float32)
        assert torch.equal(hd[:n].cpu(), hist[:n])


@pytest.mark.parametrize("place", PLACES)
def test_depth_average_of_a_plain_sum(place):
    y, x, hist = rnd(5, 64, seed=60), rnd(5, 64, seed=61), rnd(3, 5, 64, seed=64)
    one, w = torch.ones(64), torch.tensor([0.5, -0.25, 2.0])
    for add in (y, None):
        xd = x.to(place[0]).clone()
        depth_average(None if add is None else at_place(place, add)[0], None, xd, hist.to(place[0]), 2, w.to(place[0]), one.to(place[0]), 1e-5, place[1])
        close(xd, 0.5 * hist[0].double() - 0.25 * hist[1].double() + 2.0 * (x.double() + (0 if add is None else add.double())), torch.float32)


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("D", [64, 50])
def test_scaled_embedding_without_positions(place, D):
    table, ids = rnd(30, D, seed=70), torch.randint(0, 30, (2, 9), generator=torch.Generator().manual_seed(71))
    out = torch.empty(3, 2, 9, D, device=place[0])
    got = embed_positions(ids.to(place[0]), at_place(place, table)[0], None, 7.25, out=out[1])
    assert got.data_ptr() == out[1].data_ptr()
    close(got, table[ids].double() * 7.25, torch.float32)
