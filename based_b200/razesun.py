"""Razesun: a decoder-only language model whose layers are listed in its config, each with one of three mixers (latent
attention, gated delta rule, real-gated linear recurrent unit) and an optional SwiGLU MLP beside it.

The residual stream is fp32.  A layer is parallel: ``x <- x + m * (mixer(norm1(x)) + mlp(norm2(x)))``, both norms of the
same x, so one launch adds the previous layer's branch sum to the stream and writes both normed inputs
(``ops.stream_norm``), and one GEMM multiplies mixer output and MLP hidden values, side by side in one buffer, by the
two output matrices, side by side in one weight.  The embedding and its norm are the first such launch."""
from dataclasses import dataclass, field
from typing import List

import torch
import torch.nn as nn
import torch.nn.functional as F

from . import ops
from .generation import GenerationMixin, InferenceParams
from .mixers import RGLRU, GatedDelta, LatentAttention
from .mixers.stateful import pad_up
from .modules import GatedMlp

MIXERS = {"latent_attention": LatentAttention, "delta": GatedDelta, "rglru": RGLRU}


@dataclass
class RazesunConfig:
    vocab_size: int
    width: int
    layers: List[dict] = field(default_factory=list)   # {"type", "mixer": {sizes}, "mlp": {"kind", "ff"} or None}
    norm_eps: float = 1e-6
    residual_mult: float = 1.0
    logit_scale: float = 1.0

    @classmethod
    def from_dict(cls, d):
        cfg = cls(vocab_size=d["vocab"], width=d["width"], layers=d["layers"], norm_eps=d["norm"]["eps"],
                  residual_mult=d["residual_mult"], logit_scale=d["logit_scale"])
        for i, layer in enumerate(cfg.layers):
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r} (known: {', '.join(sorted(MIXERS))})")
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown mlp kind {mlp['kind']!r}")
            src = layer["mixer"].get("kv_from")
            if src is not None:
                other = cfg.layers[src] if 0 <= src < i else None
                if (other is None or other["type"] != "latent_attention" or other["mixer"].get("kv_from") is not None
                        or any(other["mixer"][k] != layer["mixer"][k] for k in ("kv_rank", "rot_dim", "rot"))):
                    raise ValueError(f"layer {i}: kv_from must name an earlier latent_attention layer with a cache of its "
                                     "own and the same kv_rank, rot_dim and rotation")
        return cfg


class ParallelBlock(nn.Module):
    """Mixer and MLP of one layer up to their joint output projection: (norm1(x), norm2(x)) -> branch sum."""

    def __init__(self, config: RazesunConfig, layer_idx: int, device=None, dtype=None):
        super().__init__()
        fk = {"device": device, "dtype": dtype}
        spec = config.layers[layer_idx]
        d = config.width
        self.norm1 = nn.Parameter(torch.ones(d, **fk))
        self.mixer = MIXERS[spec["type"]].from_config(d, spec["mixer"], config.norm_eps, layer_idx, **fk)
        self.inner, self.ff, self.mlp, self.norm2 = self.mixer.inner, 0, None, None
        if spec.get("mlp") is not None:
            self.ff = spec["mlp"]["ff"]
            self.norm2 = nn.Parameter(torch.ones(d, **fk))
            self.mlp = GatedMlp(d, hidden_features=self.ff, activation=F.silu, bias1=False, bias2=False, multiple_of=1, **fk)
        # one weight for both output projections; the modules' own weights become views of it
        self.split = pad_up(self.inner) if self.mlp is not None else self.inner
        self.out_weight = nn.Parameter(torch.zeros(d, self.split + self.ff, **fk))
        self._tie()

    def _tie(self):
        self.mixer.out_proj.weight = nn.Parameter(self.out_weight.data[:, :self.inner])
        if self.mlp is not None:
            self.mlp.fc2.weight = nn.Parameter(self.out_weight.data[:, self.split:])

    def _apply(self, fn, *args, **kwargs):   # .to() and the like make new storage: the views follow it
        super()._apply(fn, *args, **kwargs)
        self._tie()
        return self

    def load_tensors(self, t, prefix):
        d = self.norm1.shape[0]
        self.mixer.load_tensors(t, prefix + "mix.")
        with torch.no_grad():
            self.norm1.copy_(t.get(prefix + "norm1", (d,)))
            if self.mlp is None and prefix + "norm2" in t:
                t.get(prefix + "norm2", (d,))   # the second norm of a layer without an MLP has nothing to feed
            if self.mlp is not None:
                self.norm2.copy_(t.get(prefix + "norm2", (d,)))
                self.mlp.fc1.weight[:self.ff].copy_(t.get(prefix + "mlp.up", (self.ff, d)))
                self.mlp.fc1.weight[self.ff:].copy_(t.get(prefix + "mlp.gate", (self.ff, d)))
                self.mlp.fc2.weight.copy_(t.get(prefix + "mlp.down", (d, self.ff)))

    def forward(self, h1, h2, inference_params):
        B, L, _ = h1.shape
        alloc = torch.empty if self.split == self.inner else torch.zeros   # columns between the parts meet zero weights
        both = alloc(B, L, self.split + self.ff, dtype=h1.dtype, device=h1.device)
        if self.mlp is not None:
            self.mlp.hidden(h2, out=both[..., self.split:])
        self.mixer.heads(h1, inference_params, both[..., :self.inner])
        return ops.linear(both, self.out_weight)


class RazesunLMHeadModel(GenerationMixin, nn.Module):
    supports_portions = True

    def __init__(self, config: RazesunConfig, device=None, dtype=None):
        super().__init__()
        self.config = config
        fk = {"device": device, "dtype": dtype}
        self.embed = nn.Parameter(torch.zeros(config.vocab_size, config.width, **fk))
        self.embed_norm = nn.Parameter(torch.ones(config.width, **fk))
        self.layers = nn.ModuleList([ParallelBlock(config, i, **fk) for i in range(len(config.layers))])
        self.final_norm = nn.Parameter(torch.ones(config.width, **fk))
        self.lm_head = nn.Linear(config.width, config.vocab_size, bias=False, **fk)

    @classmethod
    def from_config(cls, d, device=None, dtype=None):
        return cls(RazesunConfig.from_dict(d), device=device, dtype=dtype)

    def load_tensors(self, t):
        V, d = self.config.vocab_size, self.config.width
        with torch.no_grad():
            self.embed.copy_(t.get("embed", (V, d)))
            self.embed_norm.copy_(t.get("embed.norm", (d,)))
            self.final_norm.copy_(t.get("final.norm", (d,)))
            self.lm_head.weight.copy_(t.get("head", (V, d)))
        for i, layer in enumerate(self.layers):
            layer.load_tensors(t, f"l{i}.")
        if t.unused():
            raise ValueError(f"tensors this model does not have: {t.unused()[:5]}")

    def allocate_inference_cache(self, batch_size, max_seqlen, dtype=None, **kwargs):
        return {i: layer.mixer.allocate_inference_cache(batch_size, max_seqlen, dtype=dtype, **kwargs)
                for i, layer in enumerate(self.layers)}

    def forward(self, input_ids, inference_params=None, num_last_tokens=0, positions=None, stream_hook=None):
        """Logits in fp32: of every token ``[B, L, vocab]``, of the last ``num_last_tokens``, or of the tokens at
        ``positions`` (indices into the call's tokens).  ``stream_hook(layer, stream)``, when given, sees the residual
        stream after every layer."""
        B, L = input_ids.shape
        cfg = self.config
        if inference_params is None:
            inference_params = InferenceParams(max_seqlen=L, max_batch_size=B)
        stream = torch.empty(B, L, cfg.width, dtype=torch.float32, device=self.embed.device)
        norms = [(layer.norm1, layer.norm2) for layer in self.layers] + [(self.final_norm, None)]
        h1, h2 = ops.stream_norm(stream, *norms[0], tokens=input_ids, table=self.embed, table_norm=self.embed_norm,
                                 eps=cfg.norm_eps)
        for i, layer in enumerate(self.layers):
            branch = layer(h1, h2, inference_params)
            h1, h2 = ops.stream_norm(stream, *norms[i + 1], branch=branch, mult=cfg.residual_mult, eps=cfg.norm_eps)
            if stream_hook is not None:
                stream_hook(i, stream)
        if positions is not None:
            h1 = h1[:, positions]
        elif num_last_tokens > 0:
            h1 = h1[:, -num_last_tokens:]
        logits = ops.linear_f32(h1, self.lm_head.weight)
        return logits if cfg.logit_scale == 1.0 else logits.mul_(cfg.logit_scale)
