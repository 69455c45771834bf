"""Gated delta rule mixer: per-head matrix state ``S [d, dv]`` in fp32, short convolutions on q, k, v, unit-norm q and
k, one decay per head, gated RMS norm on the read-out.

    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q

Projections of q, k, v and the output gate are one GEMM; step sizes and decays come from a second, fp32-result GEMM.
Single-token steps are one launch from the packed projection to the gated output (``ops.delta_step``)."""
import torch
import torch.nn as nn

from .. import ops
from .stateful import PackedLinear, StatefulMixer, pad_up


class GatedDelta(StatefulMixer):
    def __init__(self, width, heads, kv_heads, dim, vdim, conv=4, eps=1e-6, layer_idx=None, device=None, dtype=None):
        super().__init__(width, heads * vdim, layer_idx, device=device, dtype=dtype)
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        self.num_heads, self.kv_heads, self.dim, self.vdim, self.taps, self.eps = heads, kv_heads, dim, vdim, conv, eps
        fk = {"device": device, "dtype": dtype}
        # q, k, v are adjacent without padding: the convolution runs over them as one tensor
        self.conv_channels = 2 * kv_heads * dim + heads * vdim
        self.in_proj = PackedLinear(width, [("qkv", self.conv_channels), ("g", heads * vdim)], **fk)
        self.z_offset = self.in_proj.offsets["g"][0]
        self.gate_proj = nn.Parameter(torch.zeros(pad_up(2 * heads), width, **fk))   # a, then b
        self.conv_weight = nn.Parameter(torch.zeros(self.conv_channels, conv, **fk))
        self.norm_weight = nn.Parameter(torch.ones(vdim, **fk))
        self.A_log = nn.Parameter(torch.zeros(heads, device=device, dtype=torch.float32))
        self.dt_bias = nn.Parameter(torch.zeros(heads, device=device, dtype=torch.float32))

    @classmethod
    def from_config(cls, width, m, eps, layer_idx, **fk):
        return cls(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], conv=m["conv"], eps=eps, layer_idx=layer_idx, **fk)

    def load_tensors(self, t, prefix):
        H, d, dv, W = self.num_heads, self.dim, self.vdim, self.width
        sizes = {"q": self.kv_heads * d, "k": self.kv_heads * d, "v": H * dv}
        with torch.no_grad():
            at = 0
            for name, n in sizes.items():
                self.in_proj.weight[at:at + n].copy_(t.get(prefix + name, (n, W)))
                self.conv_weight[at:at + n].copy_(t.get(prefix + name + ".conv", (n, self.taps)))
                at += n
            self.in_proj.set("g", t.get(prefix + "g", (H * dv, W)))
            self.gate_proj[:H].copy_(t.get(prefix + "a", (H, W)))
            self.gate_proj[H:2 * H].copy_(t.get(prefix + "b", (H, W)))
            self.A_log.copy_(t.get(prefix + "A_log", (H,)))
            self.dt_bias.copy_(t.get(prefix + "dt_bias", (H,)))
            self.norm_weight.copy_(t.get(prefix + "norm", (dv,)))
            self.out_proj.weight.copy_(t.get(prefix + "o", (W, H * dv)))

    def allocate_inference_cache(self, batch_size, max_seqlen, dtype=None, **kwargs):
        dev = self.conv_weight.device
        return {"ring": torch.zeros(batch_size, self.taps, self.conv_channels, dtype=dtype, device=dev),
                "state": torch.zeros(batch_size, self.num_heads, self.dim, self.vdim, dtype=torch.float32, device=dev)}

    def heads(self, h, inference_params, out):
        B, L, _ = h.shape
        H, Hk, d, dv, C = self.num_heads, self.kv_heads, self.dim, self.vdim, self.conv_channels
        st = self.state(inference_params, h.dtype)
        pos = self.position(inference_params, L)
        x = self.in_proj(h)
        ab = ops.linear_f32(h, self.gate_proj)
        a, b = ab[..., :H], ab[..., H:2 * H]
        if L == 1 and self.z_offset == C:
            if ops.delta_step(x[:, 0], self.conv_weight, st["ring"], a[:, 0], b[:, 0], self.A_log, self.dt_bias,
                              self.norm_weight, st["state"], Hk, pos=pos, eps=self.eps, out=out[:, 0]):
                return
        y = ops.short_conv(x[..., :C], self.conv_weight, ring=st["ring"], pos=pos, silu=True)
        nq = Hk * d
        q, k = y[..., :nq].unflatten(-1, (Hk, d)), y[..., nq:2 * nq].unflatten(-1, (Hk, d))
        v = y[..., 2 * nq:].unflatten(-1, (H, dv))
        z = self.in_proj.slice(x, "g").unflatten(-1, (H, dv))
        ops.delta_prefill(q, k, v, z, a, b, self.A_log, self.dt_bias, self.norm_weight, st["state"], pos=pos, eps=self.eps,
                          out=out)
