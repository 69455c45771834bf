"""Grouped attention over keys that are the values, mechanism by mechanism against the plain oracle: norms and temperature
of the queries, the cache row and factor of a key, the sink, groups, the output gate, far keys, tile borders; every kernel
form (CUDA cores, decode, tensor cores) and every way of cutting a prompt."""
import pytest
import torch

from oracle import vubenex_oracle as V

pytestmark = pytest.mark.gpu

EPS = 1e-4
TOL = 4e-2   # bf16: queries rounded once, weights rounded once


def rnd(g, *shape, scale=1.0):
    return (torch.randn(*shape, generator=g) * scale).bfloat16()


def reference(q, k, wq, wk, m, gate):
    """One sequence in fp64 from bf16 projections: q ``[T, H d]``, k ``[T, G d]`` -> gated output ``[T, H d]``."""
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    T = q.shape[0]
    q, k, gate = q.double().view(T, H, d), k.double().view(T, G, d), gate.double()
    t = V.query_temperature(T, m["coef"], m["every"])
    o = V.causal_attention(V.rms(q, EPS, wq.double()) * t[:, None, None], V.rms(k, EPS, wk.double()), k, m["scale"])
    return o.reshape(T, H * d) * torch.sigmoid(gate)


def product(q, k, wq, wk, m, gate, cuts, impl="auto", dtype=torch.bfloat16, max_len=None, state=None, device_pos=False):
    """The same for a batch ``[B, T, .]`` through the cache, in calls of the given lengths (the last one repeats)."""
    from based_b200 import ops
    B, T, _ = q.shape
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    cu = lambda x: x.to(dtype).cuda()
    st = state or ops.tied_attention_state(B, H, G, d, max_len or T, dtype, "cuda")
    outs, at, n = [], 0, 0
    packed = torch.cat([cu(q), cu(k), cu(gate)], -1)       # column slices, as the mixer passes them
    qs, ks, gs = packed.split([H * d, G * d, H * d], -1)
    while at < T:
        L = min(cuts[min(n, len(cuts) - 1)], T - at)
        pos = torch.full((B,), at, dtype=torch.int32, device="cuda") if device_pos else at
        x = qs[:, at:at + L]
        ops.tied_prepare_(x, ks[:, at:at + L], cu(wq), cu(wk), st["keys"], st["factor"], pos=pos, eps=EPS, temp_coef=m["coef"],
                          temp_every=m["every"])
        out = torch.empty(B, L, H * d, dtype=dtype, device="cuda")
        ops.tied_attention(x, st["keys"], st["factor"], st["count"], H, m["scale"], gate=gs[:, at:at + L], pos=pos, sink=1.0, out=out, impl=impl)
        outs.append(out)
        at += L
        n += 1
    ops.check_status()
    assert int(st["count"].abs().sum()) == 0
    return torch.cat(outs, 1).double().cpu()


def case(H, G, d, T, B=1, scale=0.2, coef=0.3, every=50, seed=0, sharp=2.0):
    g = torch.Generator().manual_seed(seed)
    m = {"heads": H, "kv_heads": G, "dim": d, "scale": scale, "coef": coef, "every": every}
    return (rnd(g, B, T, H * d), rnd(g, B, T, G * d), (rnd(g, d, scale=0.3) + sharp).bfloat16(), (rnd(g, d, scale=0.3) + 1).bfloat16(), m,
            rnd(g, B, T, H * d))


def check(args, got, tol):
    q, k, wq, wk, m, gate = args
    for b in range(q.shape[0]):
        ref = reference(q[b], k[b], wq, wk, m, gate[b])
        rows = (got[b] - ref).abs().amax(-1) / ref.abs().amax(-1).clamp_min(0.05)
        assert float(rows.max()) < tol, (b, int(rows.argmax()), float(rows.max()))


@pytest.mark.parametrize("H,G,d", [(4, 2, 32), (6, 1, 64), (3, 3, 18), (12, 4, 128), (5, 1, 7), (20, 1, 48), (2, 2, 160), (40, 2, 16)])
def test_fp32_is_exact(H, G, d):
    args = case(H, G, d, 150)
    for cuts in ([150], [64, 1, 63, 2], [1]):
        check(args, product(*args, cuts, dtype=torch.float32), 2e-5)


@pytest.mark.parametrize("H,G,d", [(4, 2, 32), (6, 1, 64), (8, 2, 80), (12, 4, 128), (5, 1, 112), (3, 3, 16), (16, 2, 96)])
@pytest.mark.parametrize("impl", ["decode", "tcgen05", "simt"])
def test_each_form_over_whole_prompts(H, G, d, impl):
    for T in (1, 127, 128, 129, 257, 515):
        args = case(H, G, d, T, B=2, seed=T)
        check(args, product(*args, [T], impl=impl), TOL)


@pytest.mark.parametrize("d", [160, 192, 256])
def test_wide_heads_decode(d):
    args = case(6, 2, d, 70, B=2)
    check(args, product(*args, [67, 1]), TOL)
    check(args, product(*args, [1, 5, 1], impl="decode"), TOL)


def test_portions_and_decoding_agree():
    args = case(8, 2, 64, 700, B=2)
    for cuts in ([700], [2], [128, 128, 1, 127, 3], [500, 1], [31, 33, 200], [15, 17, 16]):
        check(args, product(*args, cuts), TOL)
    check(args, product(*args, [690, 1], max_len=5000), TOL)
    few = tuple(x[:, :40] if torch.is_tensor(x) and x.dim() == 3 else x for x in args)
    check(few, product(*few, [1], device_pos=True), TOL)
    check(few, product(*few, [1], device_pos=True, dtype=torch.float32), 2e-5)


def test_unequal_positions_in_one_decode_step():
    """Rows of a batch at positions of their own: each sees its own keys only."""
    from based_b200 import ops
    lens = [1, 37, 128, 129, 400]
    q, k, wq, wk, m, gate = case(6, 3, 64, 401, B=5)
    H, G, d = 6, 3, 64
    st = ops.tied_attention_state(5, H, G, d, 401, torch.bfloat16, "cuda")
    c = [x.cuda() for x in (q, k, wq, wk, gate)]
    for b, n in enumerate(lens):
        one = {key: st[key][b:b + 1] for key in ("keys", "factor")}
        ops.tied_prepare_(c[0][b:b + 1, :n].clone(), c[1][b:b + 1, :n], c[2], c[3], one["keys"], one["factor"], eps=EPS, temp_coef=0.3, temp_every=50)
    pos = torch.tensor(lens, dtype=torch.int32, device="cuda")
    pick = torch.arange(5)
    x, kk, gg = (t[pick, lens].unsqueeze(1).contiguous() for t in (c[0], c[1], c[4]))
    ops.tied_prepare_(x, kk, c[2], c[3], st["keys"], st["factor"], pos=pos, eps=EPS, temp_coef=0.3, temp_every=50)
    out = ops.tied_attention(x, st["keys"], st["factor"], st["count"], H, m["scale"], gate=gg, pos=pos, sink=1.0, out=torch.empty_like(x))
    for b, n in enumerate(lens):
        ref = reference(q[b, :n + 1], k[b, :n + 1], wq, wk, m, gate[b, :n + 1])[-1]
        assert float((out[b, 0].double().cpu() - ref).abs().max() / ref.abs().max()) < TOL, n


@pytest.mark.parametrize("impl", ["decode", "tcgen05", "simt"])
def test_one_far_key_is_found(impl):
    """One key among hundreds answers one query: at the first token, at both sides of every tile border, and just before
    the query; a wrong place in the cache or a wrong mask shows at once."""
    H, G, d, T = 4, 2, 64, 600
    q, k, wq, wk, m, gate = case(H, G, d, T, coef=0.0, scale=0.4, sharp=1.0)
    q, k = q * 0.02, k * 0.05                       # with eps, small vectors stay small after the norm
    where = [0, 1, 31, 32, 63, 64, 127, 128, 129, 255, 256, 384, 511, 597, 599, 598]   # the query at 598 must not see 599
    v = torch.zeros(G, d)
    for n, t in enumerate(where):
        v.zero_()
        v[:, 2 * n] = 6.0
        k[0, t] = v.reshape(-1).bfloat16()
    for n in range(len(where)):                     # the last 16 queries ask for one of them each
        qq = torch.zeros(H, d)
        qq[:, 2 * n] = 3.0
        q[0, T - 16 + n] = qq.reshape(-1).bfloat16()
    args = (q.bfloat16(), k.bfloat16(), wq, wk, m, gate)
    got = product(*args, [T], impl=impl)
    check(args, got, TOL)
    o = got[0, T - 16:].view(16, H, d) / torch.sigmoid(gate[0, T - 16:].double()).view(16, H, d)
    for n, t in enumerate(where):
        seen = t <= T - 16 + n                      # keys after the query stay hidden
        assert (float(o[n, :, 2 * n].min()) > 4.0) == seen, (n, t)
    for cuts in ([300, 1], [T - 16, 16], [T - 16, 3, 2]):
        check(args, product(*args, cuts), TOL)


@pytest.mark.parametrize("dtype,impl", [(torch.float32, "simt"), (torch.bfloat16, "simt"), (torch.bfloat16, "decode"), (torch.bfloat16, "tcgen05")])
def test_the_sink_takes_its_share(dtype, impl):
    """First tokens with low scores: nearly all of the weight goes to the sink; with high scores none does."""
    H, G, d, T = 4, 2, 32, 20
    q, k, wq, wk, m, gate = case(H, G, d, T, coef=0.0, scale=0.3)
    k = (k.abs() + 0.5).bfloat16()
    for sign, low in ((-1, True), (1, False)):
        args = ((sign * (q.abs() + 0.5)).bfloat16(), k, wq.abs(), wk.abs(), m, gate)
        got = product(*args, [T], impl=impl, dtype=dtype)
        check(args, got, 2e-5 if dtype == torch.float32 else TOL)
        share = got[0, 0].view(H, d) / torch.sigmoid(gate[0, 0].double()).view(H, d) / k[0, 0].double().view(G, d).repeat_interleave(2, 0)
        assert float(share.max()) < 0.05 if low else float(share.min()) > 0.95
        # without a sink the first token's output is its own key, whatever the score
        from based_b200 import ops
        st = ops.tied_attention_state(1, H, G, d, T, dtype, "cuda")
        x = args[0][:, :1].to(dtype).cuda()
        ops.tied_prepare_(x, k[:, :1].to(dtype).cuda(), wq.abs().to(dtype).cuda(), wk.abs().to(dtype).cuda(), st["keys"], st["factor"], eps=EPS)
        one = ops.tied_attention(x, st["keys"], st["factor"], st["count"], H, m["scale"], out=torch.empty_like(x), impl=impl)
        assert torch.allclose(one.cpu().double().view(H, d), k[0, 0].double().view(G, d).repeat_interleave(2, 0), rtol=1e-2)


@pytest.mark.parametrize("impl", ["decode", "tcgen05", "simt"])
def test_scores_of_any_size(impl):
    """Very high and very low scores, rising and falling along the keys: running maxima in every kernel."""
    for scale, order in ((2.0, 1), (2.0, -1), (1e-3, 1)):
        q, k, wq, wk, m, gate = case(4, 2, 64, 400, scale=scale, coef=0.0, seed=3)
        u = torch.randn(64, generator=torch.Generator().manual_seed(4))      # keys turn towards (away from) all queries
        ramp = order * torch.linspace(-1, 1, 400)[None, :, None]
        q = (0.2 * q + u.repeat(4)).bfloat16()
        k = (ramp * u.repeat(2) + (1 - ramp.abs()) * k).bfloat16()
        args = (q, k, wq, wk, m, gate)
        exact = product(*args, [400], dtype=torch.float32)
        check(args, exact, 1e-3)
        if scale < 1:
            check(args, product(*args, [400], impl=impl), TOL)
        else:   # bf16 queries move scores of hundreds by more than one: compare with the same rounded queries
            from based_b200 import ops
            st = ops.tied_attention_state(1, 4, 2, 64, 400, torch.bfloat16, "cuda")
            x = q.cuda().clone()
            ops.tied_prepare_(x, k.cuda(), wq.cuda(), wk.cuda(), st["keys"], st["factor"], eps=EPS)
            a = ops.tied_attention(x, st["keys"], st["factor"], st["count"], 4, scale, sink=1.0, out=torch.empty_like(x), impl=impl)
            f32 = {n: t.float() if n == "keys" else t for n, t in st.items()}
            b = ops.tied_attention(x.float(), f32["keys"], f32["factor"], f32["count"], 4, scale, sink=1.0, out=torch.empty_like(x).float())
            assert float((a.float() - b).abs().max() / b.abs().max()) < 2e-2


@pytest.mark.parametrize("every,coef", [(1, 0.7), (3, 0.5), (64, 1.0), (1000, 0.3), (2.5, 0.4)])
def test_query_temperature_steps(every, coef):
    """The queries' factor at every position, also when the call starts in the middle."""
    from based_b200 import ops
    T, d = 200, 16
    g = torch.Generator().manual_seed(1)
    q, w = torch.randn(1, T, 2 * d, generator=g), torch.rand(d, generator=g) + 0.5
    wk = torch.rand(d, generator=g) + 0.5
    want = V.rms(q[0].double().view(T, 2, d), EPS, w.double()) * wk.double() * V.query_temperature(T, coef, every)[:, None, None]
    for at in (0, 1, 62, 63, 64, 190):
        st = ops.tied_attention_state(1, 2, 1, d, T, torch.float32, "cuda")
        x = q[:, at:].cuda().contiguous()
        ops.tied_prepare_(x, torch.zeros(1, T - at, d, device="cuda"), w.cuda(), wk.cuda(), st["keys"], st["factor"], pos=at, eps=EPS,
                          temp_coef=coef, temp_every=every)
        assert torch.allclose(x[0].cpu().double().view(-1, 2, d), want[at:], rtol=2e-6, atol=2e-6)


def test_cache_rows_and_factors():
    from based_b200 import ops
    for d, dtype in ((64, torch.bfloat16), (18, torch.bfloat16), (40, torch.float32), (300, torch.float32)):
        g = torch.Generator().manual_seed(d)
        k = torch.randn(2, 9, 3 * d, generator=g).to(dtype)
        st = ops.tied_attention_state(2, 6, 3, d, 50, dtype, "cuda")
        ops.tied_prepare_(torch.zeros(2, 9, 6 * d, dtype=dtype, device="cuda"), k.cuda(), torch.ones(d, dtype=dtype, device="cuda"),
                          torch.ones(d, dtype=dtype, device="cuda"), st["keys"], st["factor"], pos=20, eps=EPS)
        assert torch.equal(st["keys"][:, 20:29].cpu(), k) and not st["keys"][:, :20].any() and not st["keys"][:, 29:].any()
        want = ((k.double().view(2, 9, 3, d) ** 2).mean(-1) + EPS).rsqrt().transpose(1, 2)
        assert torch.allclose(st["factor"][:, :, 20:29].cpu().double(), want, rtol=1e-6)
        with pytest.raises(Exception, match="shape"):      # a scalar position past the cache is refused
            ops.tied_prepare_(torch.zeros(2, 9, 6 * d, dtype=dtype, device="cuda"), k.cuda(), torch.ones(d, dtype=dtype, device="cuda"),
                              torch.ones(d, dtype=dtype, device="cuda"), st["keys"], st["factor"], pos=42, eps=EPS)


def test_a_used_cache_is_used_again():
    """A longer sequence's keys and factors are left in the cache of a shorter one."""
    from based_b200 import ops
    st = ops.tied_attention_state(1, 5, 1, 80, 300, torch.bfloat16, "cuda")
    first = case(5, 1, 80, 300, seed=11)
    check(first, product(*first, [300], state=st), TOL)
    second = case(5, 1, 80, 61, seed=12)
    for cuts in ([61], [50, 1], [1]):
        st["keys"][:, 61:] = 50.0                          # whatever is left behind the sequence's end
        st["factor"][..., 61:] = 1e30
        check(second, product(*second, cuts, state=st), TOL)


def test_arguments_are_checked():
    from based_b200 import _capi, ops
    st = ops.tied_attention_state(1, 4, 2, 32, 16, torch.bfloat16, "cuda")
    q = torch.zeros(1, 8, 128, dtype=torch.bfloat16, device="cuda")
    with pytest.raises(_capi.BasedLibraryError, match="shape"):
        ops.tied_attention(q, st["keys"], st["factor"], st["count"], 4, 1.0, pos=9, out=torch.empty_like(q))
    with pytest.raises(_capi.BasedLibraryError):
        ops.tied_attention(q.float(), st["keys"].float(), st["factor"], st["count"], 4, 1.0, out=torch.empty_like(q).float(), impl="tcgen05")
    with pytest.raises(TypeError, match="gate"):
        ops.tied_attention(q, st["keys"], st["factor"], st["count"], 4, 1.0, gate=q.float(), out=torch.empty_like(q))
    with pytest.raises(ValueError, match="factor"):
        ops.tied_attention(q, st["keys"], st["factor"][:, :1], st["count"], 4, 1.0, out=torch.empty_like(q))
    with pytest.raises(RuntimeError, match="CUDA"):
        ops.tied_attention(q.cpu(), st["keys"], st["factor"], st["count"], 4, 1.0, out=torch.empty_like(q))
