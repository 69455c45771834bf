"""The recurrent mixers' kernels against the plain oracle: short convolution with a carried ring, gated delta rule
(chunked tensor-core kernel, token-by-token kernel, fused decode step) and the real-gated linear recurrent unit; the
norm step of a parallel block."""
import pytest
import torch

from conftest import rel_err
from oracle import razesun_oracle as R

pytestmark = pytest.mark.gpu


def cuts(L, seed, smallest=1):
    g = torch.Generator().manual_seed(seed)
    out, at = [], 0
    while at < L:
        n = min(L - at, max(smallest, int(torch.randint(1, 70, (1,), generator=g))))
        out.append(n)
        at += n
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,taps,bias,silu", [(64, 4, True, False), (40, 4, False, True), (24, 2, True, True), (7, 3, False, False),
                                              (16, 1, True, False), (33, 6, True, True), (128, 3, False, True)])
def test_short_conv(C, taps, bias, silu, dtype):
    from based_b200 import ops
    g = torch.Generator().manual_seed(C + taps)
    B, L = 2, 150
    x = torch.randn(B, L, C + 8, generator=g).to(dtype)
    w, bb = torch.randn(C, taps, generator=g).to(dtype), torch.randn(C, generator=g).to(dtype) if bias else None
    ref = torch.stack([R.short_conv(x[b, :, :C].double(), w.double(), None if bb is None else bb.double()) for b in range(B)])
    ref = R.silu(ref) if silu else ref
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    xd, wd, bd = x.cuda()[..., :C], w.cuda(), bb.cuda() if bias else None
    assert rel_err(ops.short_conv(xd, wd, bd, silu=silu).float().cpu(), ref) < tol
    for seed in range(3):
        ring = torch.full((B, taps, C), 9.0, dtype=dtype, device="cuda")   # what an earlier sequence left is not read
        got, at = [], 0
        for n in ([1] * L if seed == 0 else cuts(L, seed)):
            pos = torch.full((B,), at, dtype=torch.int32, device="cuda") if seed == 2 else at
            got.append(ops.short_conv(xd[:, at:at + n], wd, bd, ring=ring, pos=pos, silu=silu))
            at += n
        assert rel_err(torch.cat(got, 1).float().cpu(), ref) < tol, seed


def delta_inputs(B, L, H, Hk, d, dv, seed, dtype, strong=True):
    """``strong``: decays near 1, large step sizes and keys that come back, so that the state matters and is corrected."""
    g = torch.Generator().manual_seed(seed)
    q, k = torch.randn(B, L, Hk, d, generator=g), torch.randn(B, L, Hk, d, generator=g)
    if strong:
        back = (torch.rand(L, generator=g) * torch.arange(L)).long()
        use = torch.rand(L, generator=g) < 0.4
        for t in range(1, L):
            if use[t]:
                k[:, t] = k[:, back[t]] + 0.05 * k[:, t]
            q[:, t] = k[:, back[t]] + 0.1 * q[:, t]
    v, z = torch.randn(B, L, H, dv, generator=g), torch.randn(B, L, H, dv, generator=g)
    a, b = torch.randn(B, L, H, generator=g) - (3.0 if strong else 0.0), torch.randn(B, L, H, generator=g) + (1.0 if strong else 0.0)
    A_log, dt = 0.5 * torch.randn(H, generator=g), 0.5 * torch.randn(H, generator=g)
    w = 1 + 0.2 * torch.randn(dv, generator=g)
    return [x.to(dtype) for x in (q, k, v, z)] + [a, b, A_log, dt, w.to(dtype)]


def delta_reference(q, k, v, z, a, b, A_log, dt, w, eps):
    outs, states = [], []
    for i in range(q.shape[0]):
        q1, k1, v1, z1, a1, b1 = [t[i].double() for t in (q, k, v, z, a, b)]
        H, Hk, d = v1.shape[1], q1.shape[1], q1.shape[2]
        head = torch.arange(H) // (H // Hk)
        qn, kn = R.unit_vector(q1) * d ** -0.5, R.unit_vector(k1)
        g = torch.exp(-torch.exp(A_log.double()) * R.softplus(a1 + dt.double()))
        o, S = R.delta_rule(qn[:, head], kn[:, head], v1, torch.sigmoid(b1), g)
        outs.append(R.unit_rms(o, eps) * w.double() * R.silu(z1))
        states.append(S)
    return torch.stack(outs), torch.stack(states)


DELTA_SIZES = [(6, 2, 64, 48), (4, 4, 128, 128), (4, 2, 32, 64), (2, 1, 96, 48), (3, 1, 64, 144), (2, 2, 128, 256)]


@pytest.mark.parametrize("H,Hk,d,dv", DELTA_SIZES)
@pytest.mark.parametrize("strong", [True, False])
def test_delta_chunked(H, Hk, d, dv, strong):
    """Lengths around the chunk's edges, whole and in portions; the fp32 state to 16-bit-pair accuracy."""
    from based_b200 import ops
    eps = 1e-5
    for L in (64, 200, 129, 1, 8, 63):
        t = delta_inputs(2, L, H, Hk, d, dv, seed=L, dtype=torch.bfloat16, strong=strong)
        ref, S = delta_reference(*t, eps)
        args = [x.cuda() for x in t]
        for mode in (0, 1, 2):
            state = torch.full((2, H, d, dv), 3.0, device="cuda")
            out = torch.empty(2, L, H * dv, dtype=torch.bfloat16, device="cuda")
            at = 0
            for n in ([L] if mode == 0 else cuts(L, mode, 2)):
                s = slice(at, at + n)
                ops.delta_prefill(*[x[:, s] for x in args[:6]], *args[6:], state, pos=at, eps=eps, out=out[:, s],
                                  impl="auto" if mode == 2 else "tcgen05")
                at += n
            assert rel_err(state.cpu(), S) < 2e-4, (L, mode)
            assert rel_err(out.float().cpu().view(2, L, H, dv), ref) < 1e-2, (L, mode)
    ops.check_status()


@pytest.mark.parametrize("H,Hk,d,dv,dtype", [(4, 2, 64, 32, torch.float32), (3, 1, 20, 12, torch.float32), (2, 2, 33, 300, torch.float32),
                                             (6, 2, 64, 48, torch.bfloat16), (2, 1, 40, 24, torch.bfloat16), (2, 1, 256, 192, torch.bfloat16)])
def test_delta_recurrent(H, Hk, d, dv, dtype):
    from based_b200 import ops
    eps, L = 1e-6, 70
    t = delta_inputs(2, L, H, Hk, d, dv, seed=d, dtype=dtype)
    ref, S = delta_reference(*t, eps)
    args = [x.cuda() for x in t]
    state = torch.full((2, H, d, dv), 3.0, device="cuda")
    out = torch.empty(2, L, H * dv, dtype=dtype, device="cuda")
    for s in (slice(0, 33), slice(33, 35), slice(35, L)):
        ops.delta_prefill(*[x[:, s] for x in args[:6]], *args[6:], state, pos=s.start, eps=eps, out=out[:, s], impl="simt")
    assert rel_err(state.cpu(), S) < 1e-5
    assert rel_err(out.float().cpu().view(2, L, H, dv), ref) < (1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("H,Hk,d,dv,taps", [(6, 2, 64, 48, 4), (4, 4, 128, 128, 4), (2, 1, 40, 24, 2), (3, 1, 96, 48, 3), (2, 2, 256, 64, 5)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_delta_step(H, Hk, d, dv, taps, dtype):
    """Token by token from the packed projection, two sequences at different positions, against convolution + oracle."""
    from based_b200 import ops
    eps, L, B, lag = 1e-6, 40, 2, 13
    g = torch.Generator().manual_seed(d + dv)
    C = 2 * Hk * d + H * dv
    x = torch.randn(B, L, C + H * dv, generator=g).to(dtype)
    cw = (0.7 * torch.randn(C, taps, generator=g)).to(dtype)
    _, _, _, _, a, b, A_log, dt, w = delta_inputs(B, L, H, Hk, d, dv, seed=1, dtype=dtype)
    y = torch.stack([R.silu(R.short_conv(x[i, :, :C].double(), cw.double())) for i in range(B)]).to(dtype)
    n = Hk * d
    parts = (y[..., :n].unflatten(-1, (Hk, d)), y[..., n:2 * n].unflatten(-1, (Hk, d)), y[..., 2 * n:].unflatten(-1, (H, dv)),
             x[..., C:].unflatten(-1, (H, dv)))
    ref, S = delta_reference(*parts, a, b, A_log, dt, w, eps)
    state = torch.full((B, H, d, dv), 3.0, device="cuda")
    ring = torch.full((B, taps, C), 9.0, dtype=dtype, device="cuda")
    xd, ad, bd = x.cuda(), a.cuda(), b.cuda()
    rest = (A_log.cuda(), dt.cuda(), w.cuda())
    got = torch.empty(B, L, H * dv, dtype=dtype, device="cuda")
    # row 0 starts first; row 1 follows `lag` steps later, both in one call from then on
    for t in range(lag):
        assert ops.delta_step(xd[:1, t], cw.cuda(), ring, ad[:1, t], bd[:1, t], *rest, state, Hk, pos=t, eps=eps, out=got[:1, t])
    for t in range(L):
        p = torch.tensor([min(t + lag, L - 1), t], dtype=torch.int32)
        rows = torch.arange(2)
        if t + lag >= L:   # row 0 is finished
            assert ops.delta_step(xd[1:, t], cw.cuda(), ring[1:], ad[1:, t], bd[1:, t], *rest, state[1:], Hk, pos=t, eps=eps, out=got[1:, t])
            continue
        xs, a1, b1 = xd[rows, p.long()], ad[rows, p.long()], bd[rows, p.long()]
        o = torch.empty(2, H * dv, dtype=dtype, device="cuda")
        assert ops.delta_step(xs, cw.cuda(), ring, a1, b1, *rest, state, Hk, pos=p.cuda(), eps=eps, out=o)
        got[rows, p.long()] = o
    tol = 1e-4 if dtype == torch.float32 else 1.5e-2
    assert rel_err(state.cpu(), S) < (1e-4 if dtype == torch.float32 else 5e-3)   # bf16: the convolution's rounding differs by an ulp
    assert rel_err(got.float().cpu().view(B, L, H, dv), ref) < tol


@pytest.mark.parametrize("W,blocks", [(64, 4), (96, 1), (40, 5), (24, 24), (512, 2), (320, 2), (128, 1), (144, 1), (384, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_rglru(W, blocks, dtype):
    from based_b200 import ops
    g = torch.Generator().manual_seed(W)
    B, L, n = 2, 150, W // blocks
    u, y = (torch.randn(B, L, W, generator=g).to(dtype) for _ in range(2))
    ra, ri = ((torch.randn(blocks, n, n, generator=g) / n ** 0.5).to(dtype) for _ in range(2))
    rb, ib = ((torch.randn(blocks, n, generator=g) - 1).to(dtype) for _ in range(2))
    lam = 2 * torch.randn(W, generator=g) - 4
    ref, last = [], []
    for i in range(B):
        ud = u[i].double()
        r, gi = (torch.sigmoid(R.block_linear(ud, m.double(), c.double())) for m, c in ((ra, rb), (ri, ib)))
        S = R.rglru_scan(ud, r, gi, lam.double())
        ref.append(S * R.gelu_tanh(y[i].double()))
        last.append(S[-1])
    ref, last = torch.stack(ref), torch.stack(last)
    gw = torch.stack([ra, ri], 1).contiguous().cuda()
    ud, yd = u.cuda(), y.cuda()
    for seed in range(3):
        state = torch.full((B, W), 5.0, device="cuda")
        out = torch.empty(B, L, W, dtype=dtype, device="cuda")
        at = 0
        for m in ([L] if seed == 0 else [1] * L if seed == 1 else cuts(L, seed)):
            pos = torch.full((B,), at, dtype=torch.int32, device="cuda") if seed == 1 else at
            ops.rglru_gated(ud[:, at:at + m], yd[:, at:at + m], gw, rb.reshape(W).cuda(), ib.reshape(W).cuda(), lam.cuda(), state,
                            pos=pos, out=out[:, at:at + m])
            at += m
        ops.check_status()
        assert rel_err(state.cpu(), last) < 2e-5
        assert rel_err(out.float().cpu(), ref) < (2e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("D", [64, 96, 50, 2048, 1031, 7168])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_stream_norm(D, dtype):
    from based_b200 import ops
    g = torch.Generator().manual_seed(D)
    V, B, L, eps, mult = 37, 2, 5, 1e-3, 0.3
    table, wt, w1, w2 = (torch.randn(V, D, generator=g).to(dtype), *((1 + 0.3 * torch.randn(D, generator=g)).to(dtype) for _ in range(3)))
    ids = torch.randint(0, V, (B, L), generator=g)
    res = torch.empty(B, L, D, device="cuda")
    cu = [t.cuda() for t in (table, wt, w1, w2)]
    o1, o2 = ops.stream_norm(res, cu[2], cu[3], tokens=ids.cuda(), table=cu[0], table_norm=cu[1], eps=eps)
    z = R.rms_norm(table.double()[ids], wt.double(), eps)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert rel_err(res.cpu(), z) < 1e-5
    assert rel_err(o1.float().cpu(), R.rms_norm(z, w1.double(), eps)) < tol and rel_err(o2.float().cpu(), R.rms_norm(z, w2.double(), eps)) < tol
    br = torch.randn(B, L, D, generator=g).to(dtype)
    o1, o2 = ops.stream_norm(res, cu[2], None, branch=br.cuda(), mult=mult, eps=eps)
    z = z + mult * br.double()
    assert o2 is None and rel_err(res.cpu(), z) < 1e-5 and rel_err(o1.float().cpu(), R.rms_norm(z, w1.double(), eps)) < tol
    x = torch.randn(3, 4, D + 3, generator=g).to(dtype)
    assert rel_err(ops.rmsnorm(x.cuda()[..., :D], cu[2], eps).float().cpu(), R.rms_norm(x[..., :D].double(), w1.double(), eps)) < tol
