"""Shared parts of the mixers of hybrid stacks: packed projections, the position of a call, the state in
``inference_params.key_value_memory_dict``.

These mixers stop before their output projection: ``heads(h, inference_params, out)`` writes ``[B, L, inner]`` and the
block multiplies it by the output matrix together with the MLP's hidden values (one GEMM for both).  ``forward``
applies the output projection on its own."""
import torch
import torch.nn as nn

from .. import ops

ALIGN = 8   # packed row groups start on multiples of this, so that bf16 column slices are 16-byte aligned


def pad_up(n: int, m: int = ALIGN) -> int:
    return (n + m - 1) // m * m


class PackedLinear(nn.Module):
    """Several projections of one input as ONE GEMM.  ``parts`` is ``[(name, rows), ...]``; each part's rows start on a
    multiple of ``ALIGN`` (rows in between are zero), and :meth:`slice` cuts a part out of the product."""

    def __init__(self, in_features, parts, bias=False, device=None, dtype=None):
        super().__init__()
        self.offsets, at = {}, 0
        for name, rows in parts:
            self.offsets[name] = (at, rows)
            at = pad_up(at + rows)
        self.weight = nn.Parameter(torch.zeros(at, in_features, device=device, dtype=dtype))
        self.bias = nn.Parameter(torch.zeros(at, device=device, dtype=dtype)) if bias else None

    def forward(self, x):
        return ops.linear(x, self.weight, self.bias)

    def slice(self, y, name, upto=None):
        """Columns of part ``name`` of the product ``y``; with ``upto``, through the end of that part."""
        a, n = self.offsets[name]
        if upto is not None:
            b, m = self.offsets[upto]
            n = b + m - a
        return y[..., a:a + n]

    def set(self, name, weight, bias=None):
        a, n = self.offsets[name]
        with torch.no_grad():
            self.weight[a:a + n].copy_(weight)
            if bias is not None:
                self.bias[a:a + n].copy_(bias)


class StatefulMixer(nn.Module):
    """Base of the mixers.  ``inner``: width of what ``heads`` writes."""

    def __init__(self, width, inner, layer_idx, device=None, dtype=None):
        super().__init__()
        self.width, self.inner, self.layer_idx = width, inner, layer_idx
        self.out_proj = nn.Linear(inner, width, bias=False, device=device, dtype=dtype)

    def heads(self, h, inference_params, out):
        raise NotImplementedError

    def allocate_inference_cache(self, batch_size, max_seqlen, dtype=None, **kwargs):
        raise NotImplementedError

    def forward(self, h, inference_params=None):
        B, L, _ = h.shape
        out = torch.empty(B, L, self.inner, dtype=h.dtype, device=h.device)
        if inference_params is None:
            from ..generation import InferenceParams
            inference_params = InferenceParams(max_seqlen=L, max_batch_size=B)
        self.heads(h, inference_params, out)
        return ops.linear(out, self.out_proj.weight)

    def state(self, inference_params, dtype):
        """This layer's state, allocated on first use."""
        d = inference_params.key_value_memory_dict
        if self.layer_idx not in d:
            d[self.layer_idx] = self.allocate_inference_cache(inference_params.max_batch_size, inference_params.max_seqlen,
                                                              dtype=dtype)
        return d[self.layer_idx]

    @staticmethod
    def position(inference_params, L):
        """Position of the call's first token: per row on the device for a decode step (so that a captured step can be
        replayed), one number for prompts and portions."""
        lens = inference_params.lengths_per_sample
        if L == 1 and inference_params.seqlen_offset > 0 and lens is not None:
            return lens
        return inference_params.seqlen_offset
