"""Griffin-style recurrent block: a gelu branch times a short convolution followed by a real-gated linear recurrent
unit with fp32 state, gates from block-diagonal matrices.

    log a = -8 r softplus(lam);  S <- a S + sqrt(1 - a^2) i u;  out = S * gelu_tanh(y)"""
import torch
import torch.nn as nn

from .. import ops
from .stateful import PackedLinear, StatefulMixer


class RGLRU(StatefulMixer):
    def __init__(self, width, inner, blocks, conv=4, layer_idx=None, device=None, dtype=None):
        super().__init__(width, inner, layer_idx, device=device, dtype=dtype)
        if inner % blocks:
            raise ValueError("the recurrent width must be a multiple of blocks")
        self.blocks, self.taps = blocks, conv
        n = inner // blocks
        fk = {"device": device, "dtype": dtype}
        self.in_proj = PackedLinear(width, [("x", inner), ("y", inner)], bias=True, **fk)
        self.conv_weight = nn.Parameter(torch.zeros(inner, conv, **fk))
        self.conv_bias = nn.Parameter(torch.zeros(inner, **fk))
        self.gate_weight = nn.Parameter(torch.zeros(blocks, 2, n, n, **fk))    # r and i matrices, [out, in]
        self.r_bias = nn.Parameter(torch.zeros(inner, **fk))
        self.i_bias = nn.Parameter(torch.zeros(inner, **fk))
        self.lam = nn.Parameter(torch.zeros(inner, device=device, dtype=torch.float32))

    @classmethod
    def from_config(cls, width, m, eps, layer_idx, **fk):
        return cls(width, m["width"], m["blocks"], conv=m["conv"], layer_idx=layer_idx, **fk)

    def load_tensors(self, t, prefix):
        W, R, nb = self.width, self.inner, self.blocks
        n = R // nb
        with torch.no_grad():
            for name in ("x", "y"):
                self.in_proj.set(name, t.get(prefix + name, (R, W)), t.get(prefix + name + ".b", (R,)))
            self.conv_weight.copy_(t.get(prefix + "conv", (R, self.taps)))
            self.conv_bias.copy_(t.get(prefix + "conv.b", (R,)))
            self.gate_weight[:, 0].copy_(t.get(prefix + "ra", (nb, n, n)))
            self.gate_weight[:, 1].copy_(t.get(prefix + "ri", (nb, n, n)))
            self.r_bias.copy_(t.get(prefix + "ra.b", (nb, n)).reshape(R))
            self.i_bias.copy_(t.get(prefix + "ri.b", (nb, n)).reshape(R))
            self.lam.copy_(t.get(prefix + "lam", (R,)))
            self.out_proj.weight.copy_(t.get(prefix + "o", (W, R)))

    def allocate_inference_cache(self, batch_size, max_seqlen, dtype=None, **kwargs):
        dev = self.conv_weight.device
        return {"ring": torch.zeros(batch_size, self.taps, self.inner, dtype=dtype, device=dev),
                "state": torch.zeros(batch_size, self.inner, dtype=torch.float32, device=dev)}

    def heads(self, h, inference_params, out):
        L = h.shape[1]
        st = self.state(inference_params, h.dtype)
        pos = self.position(inference_params, L)
        x = self.in_proj(h)
        u = ops.short_conv(self.in_proj.slice(x, "x"), self.conv_weight, self.conv_bias, ring=st["ring"], pos=pos)
        ops.rglru_gated(u, self.in_proj.slice(x, "y"), self.gate_weight, self.r_bias, self.i_bias, self.lam, st["state"], pos=pos,
                        out=out)
