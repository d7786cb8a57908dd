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
