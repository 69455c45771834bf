"""Linear attention with a constant decay per head against the plain oracle: every kernel form, every way of cutting a
prompt, decays from 0 to 1, far tokens, chunk borders, states that are used again, the fused decode step; and the norm
steps of a post-norm stack."""
import pytest
import torch

from oracle import vubenex_oracle as V

pytestmark = pytest.mark.gpu

EPS = 1e-4
TOL = {torch.float32: 1e-5, torch.bfloat16: 2e-2}


def case(decay, d, dv, T, B=1, seed=0):
    g = torch.Generator().manual_seed(seed)
    H = len(decay)
    return [torch.randn(B, T, n, generator=g).bfloat16() for n in (H * d, H * d, H * dv)] + [decay, d, dv]


def reference(q, k, v, decay, d, dv, after=lambda x: x):
    """fp64: read-out ``[B, T, H dv]`` and final states; ``after`` is applied to the activations."""
    H = len(decay)
    outs, states = [], []
    for qb, kb, vb in zip(q.double(), k.double(), v.double()):
        a, b, c = (after(V.silu(x)).view(-1, H, n) for x, n in ((qb, d), (kb, d), (vb, dv)))
        o, S = V.decayed_outer_products(a, b, c, torch.tensor(decay, dtype=torch.float64))
        outs.append(o.reshape(-1, H * dv))
        states.append(S)
    return torch.stack(outs), torch.stack(states)


def product(q, k, v, decay, d, dv, cuts, impl="auto", dtype=torch.bfloat16, state=None, device_pos=False):
    from based_b200 import ops
    B, T, _ = q.shape
    H = len(decay)
    packed = torch.cat([q, k, v], -1).to(dtype).cuda()
    qs, ks, vs = packed.split([H * d, H * d, H * dv], -1)
    S = torch.full((B, H, d, dv), 1e3, device="cuda") if state is None else state    # a sequence that starts reads no state
    g = torch.tensor(decay, dtype=torch.float32, device="cuda")
    outs, at, n = [], 0, 0
    while at < T:
        L = min(cuts[min(n, len(cuts) - 1)], T - at)
        pos = torch.full((B,), at, dtype=torch.int32, device="cuda") if device_pos else at
        outs.append(ops.lightning(qs[:, at:at + L], ks[:, at:at + L], vs[:, at:at + L], g, S, pos=pos, impl=impl))
        at += L
        n += 1
    ops.check_status()
    return torch.cat(outs, 1).double().cpu(), S.double().cpu()


def check(args, got, dtype):
    """Against the sum of the terms' sizes, which a read-out or a state that cancels is far below."""
    ref, S = reference(*args)
    size, S_size = reference(*args, after=torch.abs)
    e = ((got[0] - ref).abs() / (size + 1e-3)).amax(-1)
    assert float(e.max()) < TOL[dtype], (int(e.argmax()), float(e.max()))
    assert float(((got[1] - S).abs() / (S_size + 1e-3)).max()) < TOL[dtype]


DECAYS = [0.999, 0.6, 0.05, 1.0]


@pytest.mark.parametrize("d,dv", [(32, 16), (64, 48), (128, 128), (20, 11), (200, 24), (300, 8)])
def test_fp32_is_exact(d, dv):
    args = case(DECAYS, d, dv, 150)
    for cuts in ([150], [64, 1, 63, 2], [1]):
        check(args, product(*args, cuts, dtype=torch.float32), torch.float32)


@pytest.mark.parametrize("d,dv", [(16, 16), (32, 64), (64, 32), (48, 80), (128, 128), (112, 112), (128, 64), (96, 16), (64, 256), (128, 160)])
@pytest.mark.parametrize("impl", ["tcgen05", "simt"])
def test_each_form_over_whole_prompts(d, dv, impl):
    for T in (1, 31, 127, 128, 129, 300):
        args = case(DECAYS, d, dv, T, B=2, seed=T)
        check(args, product(*args, [T], impl=impl), torch.bfloat16)


def test_many_heads_fill_the_machine_without_a_split():
    args = case([0.9 + 0.003 * i for i in range(30)], 64, 64, 140, B=5)
    check(args, product(*args, [140], impl="tcgen05"), torch.bfloat16)


def test_portions_and_decoding_agree():
    args = case(DECAYS, 64, 48, 600, B=2)
    for cuts in ([600], [2], [128, 128, 1, 127, 3], [500, 1], [31, 33, 200], [15, 17, 16], [129]):
        check(args, product(*args, cuts), torch.bfloat16)
    few = [x[:, :40] if torch.is_tensor(x) else x for x in args]
    check(few, product(*few, [1], device_pos=True), torch.bfloat16)
    check(few, product(*few, [17, 1], device_pos=True, dtype=torch.float32), torch.float32)


def test_the_state_keeps_32_bits():
    """A large early outer product, then thousands of small ones that a 16-bit state would not take in."""
    from based_b200 import ops
    T, d, dv = 2048, 64, 64
    q, k, v, decay, *_ = args = case([1.0, 0.9999], d, dv, T, seed=5)
    k[:, 0], v[:, 0] = 20.0, 20.0
    for impl, after in (("tcgen05", lambda x: x.bfloat16().double()), ("simt", lambda x: x)):   # chunks round the activations once
        S = reference(*args, after=after)[1]
        assert float(S.max()) > 300
        got = product(*args, [T], impl=impl)[1]
        assert float((got - S).abs().max()) < 0.05, impl      # one rounding of the largest entries to bf16 costs 1.0
    assert ops.check_status() == 0


@pytest.mark.parametrize("impl", ["tcgen05", "simt"])
def test_one_far_token_is_found(impl):
    """Tokens at the first place and at both sides of chunk borders, each with a key direction of its own, asked for at the
    end: the weight is the decay to the power of the distance."""
    T, d, dv, g = 400, 64, 16, 0.997
    where = [0, 1, 31, 32, 127, 128, 129, 255, 256, 383, 384, 398, 399]
    q, k, v = torch.full((1, T, d), -30.0), torch.full((1, T, d), -30.0), torch.full((1, T, dv), 4.0)   # silu(-30) = 0
    for n, t in enumerate(where):
        k[0, t, n] = 8.0
        q[0, T - 13 + n, n] = 8.0
    args = [q.bfloat16(), k.bfloat16(), v.bfloat16(), [g], d, dv]
    got, _ = product(*args, [T], impl=impl)
    sv = lambda x: float(V.silu(torch.tensor(x, dtype=torch.float64)))
    for n, t in enumerate(where):
        i = T - 13 + n
        want = g ** (i - t) * sv(8.0) ** 2 * sv(4.0) if t <= i else 0.0
        assert torch.allclose(got[0, i], torch.full((dv,), want, dtype=torch.float64), rtol=1e-2, atol=1e-3), (n, t)


@pytest.mark.parametrize("decay", [[0.0], [1e-3, 0.3], [1.0]])
def test_extreme_decays(decay):
    for dtype, impl in ((torch.float32, "simt"), (torch.bfloat16, "tcgen05")):
        args = case(decay, 32, 32, 300, seed=7)
        check(args, product(*args, [200, 100], impl=impl, dtype=dtype), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d,dv", [(4, 64, 48), (2, 128, 128), (16, 32, 16), (3, 20, 12), (1, 256, 8), (2, 16, 1024)])
def test_decode_step(dtype, H, d, dv):
    """The fused step against the recurrence, the norm over all heads together and the gate; twice as many steps as batch
    rows, and a batch whose rows are at positions of their own (one of them fresh)."""
    from based_b200 import ops
    B, T = 3, 6
    decay = [0.5 + 0.4 * i / H for i in range(H)]
    q, k, v, *_ = args = case(decay, d, dv, T, B=B, seed=H)
    g = torch.Generator().manual_seed(1)
    gate, w = torch.randn(B, T, H * dv, generator=g).bfloat16(), (1 + 0.2 * torch.randn(H * dv, generator=g)).bfloat16()
    ref, S_ref = reference(*args)
    want = V.rms(ref, EPS, w.double()) * torch.sigmoid(gate.double())
    packed = torch.cat([q, k, v, gate], -1).to(dtype).cuda()
    S = torch.full((B, H, d, dv), 7.0, device="cuda")
    read, count = torch.empty(B, H * dv, device="cuda"), torch.zeros(B, dtype=torch.int32, device="cuda")
    dec = torch.tensor(decay, dtype=torch.float32, device="cuda")
    for t in range(T):
        pos = torch.full((B,), t, dtype=torch.int32, device="cuda") if t % 2 else t
        a, b, c, e = packed[:, t].split([H * d, H * d, H * dv, H * dv], -1)
        out = torch.empty(B, H * dv, dtype=dtype, device="cuda")
        assert ops.lightning_step(a, b, c, e, dec, w.to(dtype).cuda(), S, read, count, pos=pos, eps=EPS, out=out)
        assert float((out.double().cpu() - want[:, t]).abs().max() / want[:, t].abs().max()) < TOL[dtype], t
    assert int(count.abs().sum()) == 0
    assert float((S.double().cpu() - S_ref).abs().max() / S_ref.abs().max()) < TOL[dtype]
    old = S.clone()
    pos = torch.tensor([5, 0, 9], dtype=torch.int32, device="cuda")     # row 1 starts anew
    a, b, c, e = packed[:, 0].split([H * d, H * d, H * dv, H * dv], -1)
    assert ops.lightning_step(a, b, c, e, dec, w.to(dtype).cuda(), S, read, count, pos=pos, eps=EPS, out=out)
    assert float((out[1].double().cpu() - want[1, 0]).abs().max() / want[1, 0].abs().max()) < TOL[dtype]
    assert not torch.equal(S[0], old[0])


def test_decode_step_declines_other_sizes():
    from based_b200 import ops
    z = lambda *s: torch.zeros(*s, device="cuda")
    assert not ops.lightning_step(z(1, 16), z(1, 16), z(1, 10), z(1, 10), z(2), z(10), z(1, 2, 8, 5), z(1, 10), z(1).int(), pos=0, eps=EPS, out=z(1, 10))


@pytest.mark.parametrize("D", [64, 75, 320, 1000, 4096])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_stream_steps(D, dtype):
    from based_b200 import ops
    g = torch.Generator().manual_seed(D)
    rnd = lambda *s: torch.randn(*s, generator=g).bfloat16()
    B, L, vocab, P = 2, 7, 50, 40
    table, pos_table, w, w2 = rnd(vocab, D), rnd(P, D), rnd(D), rnd(D)
    cu = lambda x: x.to(dtype).cuda()
    ids = torch.randint(0, vocab, (B, L), generator=g)
    stream = torch.empty(B, L, D, device="cuda")
    at = torch.tensor([3, 30], dtype=torch.int32)
    for pos, want_pos in ((5, torch.arange(5, 12).expand(B, L)), (at.cuda(), at[:, None] + torch.arange(L))):
        x = ops.stream_embed(stream, ids.cuda(), cu(table), 2.5, cu(pos_table), pos=pos)
        want = table.double()[ids] * 2.5 + pos_table.double()[want_pos]
        assert torch.allclose(stream.double().cpu(), want, rtol=1e-6, atol=1e-6)
        assert x.dtype == dtype and torch.equal(x, stream.to(dtype))
    with pytest.raises(Exception, match="shape"):
        ops.stream_embed(stream, ids.cuda(), cu(table), 1.0, cu(pos_table), pos=P - L + 1)
    wide = rnd(B, L, D + 8)
    branch = cu(wide)[..., :D]                      # a column slice
    want = want + V.rms(wide[..., :D].double(), EPS, w.double())
    x = ops.stream_post_norm(stream, branch, cu(w), eps=EPS)
    assert torch.allclose(stream.double().cpu(), want, rtol=2e-6, atol=2e-6) and torch.equal(x, stream.to(dtype))
    want = want + V.rms(wide[..., :D].double(), EPS, w2.double())
    x = ops.stream_post_norm(stream, branch, cu(w2), out_weight=cu(w), eps=EPS)
    assert torch.allclose(stream.double().cpu(), want, rtol=4e-6, atol=4e-6)
    assert float((x.double().cpu() - V.rms(want, EPS, w.double())).abs().max()) < (2e-5 if dtype == torch.float32 else 4e-2)
    gate = rnd(B, L, D)
    y = ops.norm_gate(branch, cu(w), cu(gate), EPS)
    ref = V.rms(wide[..., :D].double(), EPS, w.double()) * torch.sigmoid(gate.double())
    assert float((y.double().cpu() - ref).abs().max() / ref.abs().max()) < (1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("n", [5, 16, 64])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_token_gate(n, dtype):
    from based_b200 import ops
    g = torch.Generator().manual_seed(n)
    z, table = torch.randn(3, 11, n, generator=g).bfloat16(), torch.randn(20, 4 * n, generator=g).bfloat16()
    ids = torch.randint(0, 20, (3, 11), generator=g)
    for layer in (0, 2, 3):
        got = ops.token_gate(z.to(dtype).cuda(), ids.cuda(), table.to(dtype).cuda(), layer * n)
        want = V.gelu_tanh(z.double()) * table.double()[ids][..., layer * n:(layer + 1) * n]
        assert float((got.double().cpu() - want).abs().max() / want.abs().max()) < (2e-6 if dtype == torch.float32 else 1e-2)
    with pytest.raises(ValueError, match="inside"):
        ops.token_gate(z.to(dtype).cuda(), ids.cuda(), table.to(dtype).cuda(), 3 * n + 1)


@pytest.mark.parametrize("M,W,n", [(1, 64, 8), (5, 320, 24), (16, 512, 64), (17, 512, 256), (33, 96, 16), (64, 2048, 88), (3, 4096, 40), (2, 8192, 8)])
def test_token_input_in_one_launch(M, W, n):
    from based_b200 import ops
    g = torch.Generator().manual_seed(M)
    rnd = lambda *s, scale=1.0: (torch.randn(*s, generator=g) * scale).bfloat16()
    x, wg, wp, table = rnd(M, W), rnd(n, W, scale=W ** -0.5), rnd(W, n, scale=n ** -0.5), rnd(30, 3 * n)
    norm, out_norm, stream = rnd(W), rnd(W), torch.randn(M, W, generator=g)
    ids = torch.randint(0, 30, (M,), generator=g)
    e = table.double()[ids][:, n:2 * n]
    want = stream.double() + V.rms((V.gelu_tanh(x.double() @ wg.double().T) * e) @ wp.double().T, EPS, norm.double())
    for last in (None, out_norm):
        s = stream.cuda()
        y = ops.token_side_step(s, x.cuda(), ids.cuda(), wg.cuda(), wp.cuda(), table.cuda(), n, norm.cuda(), out_weight=None if last is None else last.cuda(), eps=EPS)
        assert float((s.double().cpu() - want).abs().max()) < 5e-2
        ref = s.double().cpu() if last is None else V.rms(s.double().cpu(), EPS, last.double())
        assert float((y.double().cpu() - ref).abs().max() / ref.abs().max()) < 1e-2
        again = stream.cuda()                       # the separate steps
        z = ops.token_gate(torch.nn.functional.linear(x.cuda(), wg.cuda()), ids.cuda(), table.cuda(), n)
        ops.stream_post_norm(again, torch.nn.functional.linear(z, wp.cuda()), norm.cuda(), eps=EPS)
        assert float((again - s).abs().max()) < 8e-2
    assert ops.token_side_step(stream.cuda(), x.float().cuda(), ids.cuda(), wg.float().cuda(), wp.float().cuda(), table.float().cuda(), n, norm.float().cuda()) is None
    big = torch.zeros(128, 2048).bfloat16().cuda()     # too much weight for one cluster
    assert ops.token_side_step(torch.zeros(1, 2048, device="cuda"), big[:1], ids[:1].cuda(), big, big.view(2048, 128), table.cuda().repeat(1, 128), 0, big[0]) is None
