"""Latent attention: queries through a low-rank latent, keys and values expanded from a cached latent of ``kv_rank``
values plus one rotated key part shared by all heads; a sigmoid gate per head on the output.

The cache holds ``kv_rank + rot_dim`` values per token.  Two forms of the same product, chosen by the number of query
rows: prompts and long portions expand the cached latents to per-head keys and values (one GEMM) and run causal
attention over them; single tokens and short portions absorb ``W_uk`` into the query and ``W_uv`` into the output and
attend over the latent rows themselves.  A mixer with ``kv_from`` has no cache of its own and reads that layer's."""
import torch
import torch.nn as nn

from .. import ops
from .slide_attention import RotaryEmbedding
from .stateful import PackedLinear, StatefulMixer


class LatentAttention(StatefulMixer):
    # query rows (tokens x heads) of one sequence up to which the absorbed form is used
    ABSORB_ROWS = 128

    def __init__(self, width, heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot_base, kv_from=None, eps=1e-6,
                 layer_idx=None, device=None, dtype=None):
        super().__init__(width, heads * vdim, layer_idx, device=device, dtype=dtype)
        self.num_heads, self.dim, self.rot_dim, self.vdim = heads, dim, rot_dim, vdim
        self.q_rank, self.kv_rank, self.scale, self.kv_from, self.eps = q_rank, kv_rank, scale, kv_from, eps
        fk = {"device": device, "dtype": dtype}
        parts = [("dq", q_rank)] + ([("dkv", kv_rank + rot_dim)] if kv_from is None else []) + [("g", heads)]
        self.in_proj = PackedLinear(width, parts, **fk)
        self.q_norm = nn.Parameter(torch.ones(q_rank, **fk))
        self.kv_norm = nn.Parameter(torch.ones(kv_rank, **fk)) if kv_from is None else None
        self.q_up = nn.Linear(q_rank, heads * (dim + rot_dim), bias=False, **fk)
        self.kv_up = nn.Parameter(torch.zeros(heads * (dim + vdim), kv_rank, **fk))   # keys of all heads, then values
        self.rotary_emb = RotaryEmbedding(rot_dim, base=rot_base)

    @classmethod
    def from_config(cls, width, m, eps, layer_idx, **fk):
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError("rot.dims must equal rot_dim: the whole shared key part is rotated")
        return cls(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"],
                   m["rot"]["base"], kv_from=m.get("kv_from"), eps=eps, layer_idx=layer_idx, **fk)

    def load_tensors(self, t, prefix):
        H, d, rd, dv, r, W = self.num_heads, self.dim, self.rot_dim, self.vdim, self.kv_rank, self.width
        with torch.no_grad():
            self.in_proj.set("dq", t.get(prefix + "dq", (self.q_rank, W)))
            if self.kv_from is None:
                self.in_proj.set("dkv", t.get(prefix + "dkv", (r + rd, W)))
                self.kv_norm.copy_(t.get(prefix + "dkv.norm", (r,)))
            self.in_proj.set("g", t.get(prefix + "g", (H, W)))
            self.q_norm.copy_(t.get(prefix + "dq.norm", (self.q_rank,)))
            self.q_up.weight.copy_(t.get(prefix + "uq", (H * (d + rd), self.q_rank)))
            self.kv_up[:H * d].copy_(t.get(prefix + "uk", (H * d, r)))
            self.kv_up[H * d:].copy_(t.get(prefix + "uv", (H * dv, r)))
            self.out_proj.weight.copy_(t.get(prefix + "o", (W, H * dv)))

    def allocate_inference_cache(self, batch_size, max_seqlen, dtype=None, **kwargs):
        if self.kv_from is not None:
            return ()
        return torch.zeros(batch_size, max_seqlen, self.kv_rank + self.rot_dim, dtype=dtype, device=self.kv_up.device)

    def heads(self, h, inference_params, out):
        B, L, _ = h.shape
        H, d, rd, dv, r = self.num_heads, self.dim, self.rot_dim, self.vdim, self.kv_rank
        pos = self.position(inference_params, L)
        if self.kv_from is None:
            cache = self.state(inference_params, h.dtype)
        else:
            cache = inference_params.key_value_memory_dict[self.kv_from]
        x = self.in_proj(h)
        q = ops.linear(ops.rmsnorm(self.in_proj.slice(x, "dq"), self.q_norm, self.eps), self.q_up.weight)
        q = q.view(B, L, H, d + rd)
        cos, sin = self.rotary_emb.tables_f32(inference_params.max_seqlen, h.device)
        z = self.in_proj.slice(x, "dkv") if self.kv_from is None else None
        ops.latent_prepare_(q, cos, sin, d, z=z, norm_weight=self.kv_norm, cache=cache, kv_rank=r, pos=pos, eps=self.eps)
        gate = self.in_proj.slice(x, "g")
        if L * H <= self.ABSORB_ROWS or torch.is_tensor(pos):
            self._absorbed(q, cache[:B], gate, pos, ops.flat_rows(out).view(B * L, H, dv))
        else:
            self._expanded(q, cache[:B], gate, pos, out.unflatten(-1, (H, dv)))

    def _absorbed(self, q, cache, gate, pos, out):
        B, L, H, _ = q.shape
        d, rd, dv, r = self.dim, self.rot_dim, self.vdim, self.kv_rank
        uk, uv = self.kv_up[:H * d].view(H, d, r), self.kv_up[H * d:].view(H, dv, r)
        rows = q.view(B * L, H, d + rd)
        qa = torch.bmm(rows[..., :d].transpose(0, 1), uk)                        # [H, B L, r]
        ctx = torch.empty_like(qa)
        qa4, ctx4 = qa.view(H, B, L, r).permute(1, 2, 0, 3), ctx.view(H, B, L, r).permute(1, 2, 0, 3)
        ops.latent_decode(qa4, q[..., d:], cache, self.scale, gate=gate, pos=pos, out=ctx4)
        # the gate scales a head's context, which commutes with W_uv
        torch.bmm(ctx, uv.transpose(1, 2), out=out.transpose(0, 1))

    def _expanded(self, q, cache, gate, pos, out):
        B, L, H, _ = q.shape
        d, dv, r = self.dim, self.vdim, self.kv_rank
        T = pos + L
        kv = ops.linear(cache[:, :T, :r], self.kv_up)                             # [B, T, H d + H dv]
        k, v = kv[..., :H * d].unflatten(-1, (H, d)), kv[..., H * d:].unflatten(-1, (H, dv))
        ops.latent_prefill(q[..., :d], q[..., d:], k, cache[:, :T, r:], v, self.scale, gate=gate, pos=pos, out=out)
