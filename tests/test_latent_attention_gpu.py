"""Latent attention kernels against the plain oracle: the expanded form (tensor-core and CUDA-core kernels), the absorbed
form with split keys, and the append / rotate step.  Queries are aimed at single keys (the first, the query's own, the one
right behind it, tile borders, random far ones), so that one key too many or too few changes the answer."""
import pytest
import torch

from conftest import rel_err
from oracle import razesun_oracle as R

pytestmark = pytest.mark.gpu


def aimed(L, T, H, d1, d2, dv, pos, scale, seed, B=1):
    """q1, q2, k1, k2, v (fp32) where query i of head h scores about 25 on one chosen key and far less elsewhere."""
    g = torch.Generator().manual_seed(seed)
    k1 = torch.randn(B, T, H, d1, generator=g)
    k2 = torch.randn(B, T, 1, d2, generator=g).expand(B, T, H, d2)
    v = torch.randn(B, T, H, dv, generator=g)
    i = torch.arange(L)
    own = pos + i
    choices = torch.stack([torch.zeros_like(i), own, torch.minimum(own + 1, torch.tensor(T - 1)), (own // 64) * 64,
                           torch.clamp((own // 128) * 128 - 1, min=0), (torch.rand(L, generator=g) * (own + 1)).long()])
    pick = torch.randint(0, len(choices), (B, H, L), generator=g)
    target = choices.t().unsqueeze(0).unsqueeze(0).expand(B, H, L, -1).gather(-1, pick.unsqueeze(-1)).squeeze(-1)   # [B, H, L]
    s = 25.0 / (scale * (d1 + d2))
    idx = target.permute(0, 2, 1).unsqueeze(-1)
    q1 = s * k1.gather(1, idx.expand(-1, -1, -1, d1)) + 0.2 * torch.randn(B, L, H, d1, generator=g)
    q2 = s * k2.gather(1, idx.expand(-1, -1, -1, d2)) + 0.2 * torch.randn(B, L, H, d2, generator=g)
    gate = torch.randn(B, L, H, generator=g)
    return q1, q2, k1, k2[:, :, 0], v, gate


def expect(q1, q2, k1, k2, v, gate, pos, scale):
    """The oracle for queries at pos .. of longer sequences: pad the queries in front and cut."""
    out = []
    for b in range(q1.shape[0]):
        T, H = k1.shape[1], k1.shape[2]
        L = q1.shape[1]
        q = torch.zeros(T, H, q1.shape[-1] + q2.shape[-1], dtype=torch.float64)
        q[pos:pos + L] = torch.cat([q1[b], q2[b]], -1).double()
        k = torch.cat([k1[b], k2[b].unsqueeze(1).expand(T, H, -1)], -1).double()
        out.append(R.causal_softmax_attention(q, k, v[b].double(), scale)[pos:pos + L] * torch.sigmoid(gate[b].double())[..., None])
    return torch.stack(out)


# (d1, d2, dv): a small model's, a large model's, and sizes that are no multiple of 64
SIZES = [(64, 16, 96), (128, 64, 128), (48, 16, 80), (80, 48, 32), (32, 96, 112)]
CUTS = [(129, 129, 0), (300, 300, 0), (64, 192, 128), (257, 600, 343), (2, 130, 127), (3, 131, 128), (100, 356, 256), (520, 520, 0),
        (31, 31, 0), (1, 1, 0), (255, 640, 384)]


@pytest.mark.parametrize("d1,d2,dv", SIZES)
@pytest.mark.parametrize("impl", ["tcgen05", "simt"])
def test_expanded_form(d1, d2, dv, impl):
    from based_b200 import ops
    scale = 0.7 * (d1 + d2) ** -0.5
    for n, (L, T, pos) in enumerate(CUTS):
        H = 2 if n % 2 else 3
        B = 2 if n % 3 == 0 else 1
        t = [x.bfloat16() for x in aimed(L, T, H, d1, d2, dv, pos, scale, seed=n, B=B)]
        ref = expect(*t, pos, scale)
        q1, q2, k1, k2, v, gate = [x.cuda() for x in t]
        q = torch.cat([q1, q2], -1)
        kv = torch.cat([k1.flatten(2), v.flatten(2)], -1)
        out = torch.full((B, L, H * dv + 8), 7.0, dtype=torch.bfloat16, device="cuda")
        ops.latent_prefill(q[..., :d1], q[..., d1:], kv[..., :H * d1].unflatten(-1, (H, d1)), k2,
                           kv[..., H * d1:].unflatten(-1, (H, dv)), scale, gate=gate, pos=pos, impl=impl,
                           out=out[..., :H * dv].unflatten(-1, (H, dv)))
        assert rel_err(out[..., :H * dv].float().cpu().view(B, L, H, dv), ref) < 1.5e-2, (L, T, pos)
        assert bool((out[..., H * dv:] == 7.0).all())     # nothing beside the slice is written
    ops.check_status()


def test_expanded_form_fp32_and_odd_sizes():
    from based_b200 import ops
    for n, (d1, d2, dv, dtype) in enumerate([(64, 16, 96, torch.float32), (33, 6, 21, torch.float32), (20, 10, 30, torch.bfloat16),
                                             (128, 64, 200, torch.bfloat16)]):
        L, T, pos, H, scale = 77, 177, 100, 3, (d1 + d2) ** -0.5
        t = [x.to(dtype) for x in aimed(L, T, H, d1, d2, dv, pos, scale, seed=n)]
        q1, q2, k1, k2, v, gate = [x.cuda() for x in t]
        out = torch.empty(1, L, H, dv, dtype=dtype, device="cuda")
        ops.latent_prefill(q1, q2, k1, k2, v, scale, gate=gate, pos=pos, out=out)
        assert rel_err(out.float().cpu(), expect(*t, pos, scale)) < (1e-5 if dtype == torch.float32 else 1.5e-2)


def test_long_far_keys():
    """One head, 5000 keys: keys thousands of tokens back, and the running maximum that grows on the way."""
    from based_b200 import ops
    d1, d2, dv, H, L, T = 64, 48, 64, 2, 5000, 5000
    scale = (d1 + d2) ** -0.5
    t = [x.bfloat16() for x in aimed(L, T, H, d1, d2, dv, 0, scale, seed=5)]
    # a slope along the keys makes the running maximum of most rows grow tile by tile
    q1, q2, k1, k2, v, gate = [x.cuda() for x in t]
    out = torch.empty(1, L, H, dv, dtype=torch.bfloat16, device="cuda")
    ops.latent_prefill(q1, q2, k1, k2, v, scale, gate=gate, out=out, impl="tcgen05")
    q1[..., 0], k1[..., 0] = 8.0, (torch.arange(T, device="cuda") * 0.01).view(1, T, 1).bfloat16()
    out2 = torch.empty_like(out)
    ops.latent_prefill(q1, q2, k1, k2, v, scale, gate=gate, out=out2, impl="tcgen05")
    ops.check_status()
    rows = torch.tensor([0, 1, 127, 128, 255, 256, 2047, 4095, 4096, 4999])
    for o, (a, b) in ((out, (t[0], t[2])), (out2, (q1.cpu(), k1.cpu()))):
        q = torch.cat([a[0], t[1][0]], -1).double()[rows]
        k = torch.cat([b[0], t[3][0].unsqueeze(1).expand(T, H, d2)], -1).double()
        s = torch.einsum("ihd,jhd->hij", q, k) * scale
        s = s.masked_fill(torch.arange(T).view(1, 1, T) > rows.view(1, -1, 1), float("-inf"))
        ref = torch.einsum("hij,jhd->ihd", s.softmax(-1), t[4][0].double()) * torch.sigmoid(t[5][0].double()[rows])[..., None]
        assert rel_err(o[0].float().cpu()[rows], ref) < 1.5e-2


@pytest.mark.parametrize("r,rd,H,dtype", [(80, 32, 4, torch.bfloat16), (512, 64, 16, torch.bfloat16), (96, 16, 3, torch.bfloat16),
                                          (200, 24, 5, torch.bfloat16), (80, 32, 4, torch.float32), (33, 6, 2, torch.float32),
                                          (33, 6, 2, torch.bfloat16), (512, 64, 40, torch.bfloat16)])
def test_absorbed_form(r, rd, H, dtype):
    """Positions at and around tile and split borders, one position per row of the batch, several query tokens."""
    from based_b200 import ops
    scale = (r + rd) ** -0.5
    max_len = 1100
    g = torch.Generator().manual_seed(r + H)
    for L, positions in ((1, [0, 1, 62, 63, 64, 65, 127, 128, 500, 1023, 1024, 1099]), (3, [0, 61, 62, 63, 64, 126, 700]), (2, [0, 1098])):
        B = len(positions)
        cache = torch.randn(B, max_len, r + rd, generator=g)
        pos = torch.tensor(positions)
        own = pos.view(B, 1) + torch.arange(L)
        pick = torch.randint(0, 4, (B, L, H), generator=g)
        far = (torch.rand(B, L, H, generator=g) * (own.unsqueeze(-1) + 1)).long()
        o3 = own.unsqueeze(-1).expand(B, L, H)
        target = torch.where(pick == 0, torch.zeros_like(far), torch.where(pick == 1, o3, torch.where(pick == 2, (o3 + 1).clamp(max=max_len - 1), far)))
        q = 25.0 / (scale * (r + rd)) * torch.stack([cache[b][target[b]] for b in range(B)]) + 0.1 * torch.randn(B, L, H, r + rd, generator=g)
        gate = torch.randn(B, L, H, generator=g).to(dtype)
        q, cache = q.to(dtype), cache.to(dtype)
        s = torch.einsum("blhd,btd->blht", q.double(), cache.double()) * scale
        s = s.masked_fill(torch.arange(max_len).view(1, 1, 1, -1) > own.view(B, L, 1, 1), float("-inf"))
        ref = torch.einsum("blht,btd->blhd", s.softmax(-1), cache[..., :r].double()) * torch.sigmoid(gate.double())[..., None]
        qd, cd = q.cuda(), cache.cuda()
        for t in range(B):    # what lies behind a sequence's last token must not matter
            cd[t, positions[t] + L:] = 1e4
        tol = 1e-5 if dtype == torch.float32 else 1.5e-2
        out = torch.empty(H, B, L, r, dtype=dtype, device="cuda").permute(1, 2, 0, 3)
        ops.latent_decode(qd[..., :r], qd[..., r:], cd, scale, gate=gate.cuda(), pos=pos.int().cuda(), out=out)
        assert rel_err(out.float().cpu(), ref) < tol, L
        for b in range(0, B, 3):   # the same from a scalar position, alone
            alone = torch.empty(1, L, H, r, dtype=dtype, device="cuda")
            ops.latent_decode(qd[b:b + 1, ..., :r], qd[b:b + 1, ..., r:], cd[b:b + 1], scale, gate=gate[b:b + 1].cuda(),
                              pos=positions[b], out=alone)
            assert rel_err(alone.float().cpu(), ref[b:b + 1]) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_append_and_rotate(dtype):
    from based_b200 import ops
    from based_b200.mixers import RotaryEmbedding
    g = torch.Generator().manual_seed(3)
    B, L, H, d, rd, r, max_len, eps, base = 2, 5, 3, 24, 16, 40, 64, 1e-5, 777.0
    cos, sin = RotaryEmbedding(rd, base=base).tables_f32(max_len, torch.device("cuda"))
    w = torch.rand(r, generator=g).to(dtype)
    for pos in (0, 7, torch.tensor([3, 40], dtype=torch.int32)):
        z = torch.randn(B, L, r + rd + 3, generator=g).to(dtype)
        q = torch.randn(B, L, H, d + rd, generator=g).to(dtype)
        cache = torch.full((B, max_len, r + rd), 5.0, dtype=dtype, device="cuda")
        qd = q.cuda().clone()
        ops.latent_prepare_(qd, cos, sin, d, z=z.cuda()[..., :r + rd], norm_weight=w.cuda(), cache=cache, kv_rank=r,
                            pos=pos.cuda() if torch.is_tensor(pos) else pos, eps=eps)
        tol = 1e-5 if dtype == torch.float32 else 1e-2
        for b in range(B):
            p0 = int(pos[b]) if torch.is_tensor(pos) else pos
            p = torch.arange(p0, p0 + L)
            qe = torch.cat([q[b, ..., :d].double(), R.rotate_half(q[b, ..., d:].double(), p, base)], -1)
            assert rel_err(qd[b].float().cpu(), qe) < tol
            row = torch.cat([R.rms_norm(z[b, :, :r].double(), w.double(), eps), R.rotate_half(z[b, :, r:r + rd].double(), p, base)], -1)
            assert rel_err(cache[b, p0:p0 + L].float().cpu(), row) < tol
            rest = torch.ones(max_len, dtype=torch.bool)
            rest[p0:p0 + L] = False
            assert bool((cache[b].cpu()[rest] == 5.0).all())
