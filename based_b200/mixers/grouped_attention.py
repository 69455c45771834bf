"""Grouped softmax attention whose values are its keys as projected, before their norm: RMS norms with weights on queries
and keys per head, a query temperature that grows with the position, a sink in the softmax sum, a sigmoid gate per element
on the output.  No rotation.

The cache holds the projected keys once, ``kv_heads * dim`` values per token, and one fp32 factor per key and key head (the
inverse root mean square of the key); the weight of the key norm is multiplied into the query."""
import torch
import torch.nn as nn

from .. import ops
from .stateful import PackedLinear, StatefulMixer


class GroupedAttention(StatefulMixer):
    def __init__(self, width, heads, kv_heads, dim, scale, temp_coef=0.0, temp_every=1.0, sink=1.0, eps=1e-6, layer_idx=None,
                 device=None, dtype=None):
        super().__init__(width, heads * dim, layer_idx, device=device, dtype=dtype)
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if temp_every <= 0:
            raise ValueError("the query temperature's period must be positive")
        self.num_heads, self.kv_heads, self.dim, self.scale, self.sink, self.eps = heads, kv_heads, dim, scale, sink, eps
        self.temp_coef, self.temp_every = temp_coef, temp_every
        fk = {"device": device, "dtype": dtype}
        self.in_proj = PackedLinear(width, [("q", heads * dim), ("k", kv_heads * dim), ("g", heads * dim)], **fk)
        self.q_norm = nn.Parameter(torch.ones(dim, **fk))
        self.k_norm = nn.Parameter(torch.ones(dim, **fk))

    @classmethod
    def from_config(cls, width, m, eps, layer_idx, **fk):
        if m.get("vdim", m["dim"]) != m["dim"]:
            raise ValueError("vdim must equal dim: the values are the keys")
        t = m.get("q_temp") or {"coef": 0.0, "every": 1}
        return cls(width, m["heads"], m["kv_heads"], m["dim"], m["scale"], temp_coef=t["coef"], temp_every=t["every"], eps=eps,
                   layer_idx=layer_idx, **fk)

    def load_tensors(self, t, prefix):
        H, G, d, W = self.num_heads, self.kv_heads, self.dim, self.width
        for name, n in (("q", H * d), ("k", G * d), ("g", H * d)):
            self.in_proj.set(name, t.get(prefix + name, (n, W)))
        with torch.no_grad():
            self.q_norm.copy_(t.get(prefix + "q.norm", (d,)))
            self.k_norm.copy_(t.get(prefix + "k.norm", (d,)))
            self.out_proj.weight.copy_(t.get(prefix + "o", (W, H * d)))

    def allocate_inference_cache(self, batch_size, max_seqlen, dtype=None, **kwargs):
        return ops.tied_attention_state(batch_size, self.num_heads, self.kv_heads, self.dim, max_seqlen, dtype, self.q_norm.device)

    def heads(self, h, inference_params, out):
        B, L, _ = h.shape
        st = self.state(inference_params, h.dtype)
        pos = self.position(inference_params, L)
        x = self.in_proj(h)
        q = self.in_proj.slice(x, "q")
        ops.tied_prepare_(q, self.in_proj.slice(x, "k"), self.q_norm, self.k_norm, st["keys"], st["factor"], pos=pos, eps=self.eps,
                          temp_coef=self.temp_coef, temp_every=self.temp_every)
        ops.tied_attention(q, st["keys"], st["factor"], st["count"], self.num_heads, self.scale, gate=self.in_proj.slice(x, "g"), pos=pos,
                           sink=self.sink, out=out)
