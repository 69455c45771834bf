"""Linear attention with one constant decay per head and a matrix state ``S [dim, vdim]`` in fp32, silu on q, k and v, an
RMS norm over all heads together and a sigmoid gate on the read-out.

    S <- decay S + k v^T;  o = S^T q

Projections of q, k, v and the gate are one GEMM.  Single-token steps are one launch from the packed projection to the
gated output (``ops.lightning_step``)."""
import torch
import torch.nn as nn

from .. import ops
from .stateful import PackedLinear, StatefulMixer


class LightningAttention(StatefulMixer):
    def __init__(self, width, heads, dim, vdim, decay, eps=1e-6, layer_idx=None, device=None, dtype=None):
        super().__init__(width, heads * vdim, layer_idx, device=device, dtype=dtype)
        if len(decay) != heads:
            raise ValueError("one decay per head is needed")
        self.num_heads, self.dim, self.vdim, self.eps = heads, dim, vdim, eps
        fk = {"device": device, "dtype": dtype}
        self.in_proj = PackedLinear(width, [("q", heads * dim), ("k", heads * dim), ("v", heads * vdim), ("g", heads * vdim)], **fk)
        self.norm_weight = nn.Parameter(torch.ones(heads * vdim, **fk))
        self.decay = nn.Parameter(torch.tensor(decay, dtype=torch.float32, device=device), requires_grad=False)

    @classmethod
    def from_config(cls, width, m, eps, layer_idx, **fk):
        return cls(width, m["heads"], m["dim"], m["vdim"], m["decay"], eps=eps, layer_idx=layer_idx, **fk)

    def _apply(self, fn, *args, **kwargs):   # the decay stays fp32 when a model changes its dtype
        super()._apply(fn, *args, **kwargs)
        self.decay.data = self.decay.data.float()
        return self

    def load_tensors(self, t, prefix):
        H, d, dv, W = self.num_heads, self.dim, self.vdim, self.width
        for name, n in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
            self.in_proj.set(name, t.get(prefix + name, (n, W)))
        with torch.no_grad():
            self.norm_weight.copy_(t.get(prefix + "norm", (H * dv,)))
            self.out_proj.weight.copy_(t.get(prefix + "o", (W, H * dv)))

    def allocate_inference_cache(self, batch_size, max_seqlen, dtype=None, **kwargs):
        dev, H, d, dv = self.norm_weight.device, self.num_heads, self.dim, self.vdim
        return {"state": torch.zeros(batch_size, H, d, dv, dtype=torch.float32, device=dev),
                "read": torch.zeros(batch_size, H * dv, dtype=torch.float32, device=dev),     # workspace of a decode step
                "count": torch.zeros(batch_size, dtype=torch.int32, device=dev)}

    def heads(self, h, inference_params, out):
        L = h.shape[1]
        st = self.state(inference_params, h.dtype)
        pos = self.position(inference_params, L)
        x = self.in_proj(h)
        q, k, v, g = (self.in_proj.slice(x, n) for n in "qkvg")
        if L == 1 and ops.lightning_step(q[:, 0], k[:, 0], v[:, 0], g[:, 0], self.decay, self.norm_weight, st["state"], st["read"],
                                         st["count"], pos=pos, eps=self.eps, out=out[:, 0]):
            return
        ops.norm_gate(ops.lightning(q, k, v, self.decay, st["state"], pos=pos), self.norm_weight, g, self.eps, out=out)
