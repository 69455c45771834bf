"""Vubenex: a decoder-only language model whose layers are listed in its config, each with one of two mixers (grouped
attention with keys as values, linear attention with a constant decay), an optional SwiGLU MLP, and an input of its own
per token and layer.

The residual stream is fp32 and starts from the scaled token vector plus a learned position vector.  A layer norms what its
sublayers put out, not what they read: ``x <- x + norm1(mixer(x))``, ``x <- x + norm2(mlp(x))``, and then ``x <- x + norm(proj
(gelu(gate x) * e))`` with the layer's slice ``e`` of the token's second embedding.  One launch norms a sublayer's output,
adds it to the stream and hands the new stream on in the model's dtype (``ops.stream_post_norm``); the last one of the model
applies the final norm as well."""
from dataclasses import dataclass, field
from typing import List

import torch
import torch.nn as nn
import torch.nn.functional as F

from . import ops
from .generation import GenerationMixin, InferenceParams
from .mixers import GroupedAttention, LightningAttention
from .mixers.stateful import StatefulMixer
from .modules import GatedMlp

MIXERS = {"attention": GroupedAttention, "lightning": LightningAttention}


@dataclass
class VubenexConfig:
    vocab_size: int
    width: int
    max_positions: int
    layers: List[dict] = field(default_factory=list)   # {"type", "mixer": {sizes, constants}, "mlp": {"kind", "ff"} or None}
    embedding_scale: float = 1.0
    norm_eps: float = 1e-6
    side_dim: int = 0

    @classmethod
    def from_dict(cls, d):
        cfg = cls(vocab_size=d["vocab"], width=d["width"], max_positions=d["max_positions"], layers=d["layers"],
                  embedding_scale=d["embedding"]["scale"], norm_eps=d["norm"]["eps"], side_dim=d["token_side"]["dim"])
        if not cfg.layers:
            raise ValueError("a model needs at least one layer")
        for i, layer in enumerate(cfg.layers):
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r} (known: {', '.join(sorted(MIXERS))})")
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown mlp kind {mlp['kind']!r}")
        return cfg


class TokenSide(nn.Module):
    """A layer's own input per token: ``proj(gelu(gate x) * e)``, e a slice of the model's second embedding table."""

    def __init__(self, width, dim, column, device=None, dtype=None):
        super().__init__()
        fk = {"device": device, "dtype": dtype}
        self.dim, self.column = dim, column
        self.gate = nn.Linear(width, dim, bias=False, **fk)
        self.proj = nn.Linear(dim, width, bias=False, **fk)
        self.norm = nn.Parameter(torch.ones(width, **fk))

    def load_tensors(self, t, prefix):
        d, W = self.dim, self.norm.shape[0]
        with torch.no_grad():
            self.gate.weight.copy_(t.get(prefix + "gate", (d, W)))
            self.proj.weight.copy_(t.get(prefix + "proj", (W, d)))
            self.norm.copy_(t.get(prefix + "norm", (W,)))

    def forward(self, stream, x, tokens, table, out_norm, eps):
        """Adds to the stream in place; returns it as :func:`ops.stream_post_norm` does."""
        y = ops.token_side_step(stream, x, tokens, self.gate.weight, self.proj.weight, table, self.column, self.norm, out_weight=out_norm, eps=eps)
        if y is None:
            y = ops.linear(ops.token_gate(ops.linear(x, self.gate.weight), tokens, table, self.column), self.proj.weight)
            y = ops.stream_post_norm(stream, y, self.norm, out_weight=out_norm, eps=eps)
        return y


class PostNormBlock(nn.Module):
    """One layer: its sublayers read the stream, and what they put out is normed before it is added."""

    def __init__(self, config: VubenexConfig, layer_idx: int, device=None, dtype=None):
        super().__init__()
        fk = {"device": device, "dtype": dtype}
        spec, d = config.layers[layer_idx], config.width
        self.eps = config.norm_eps
        self.mixer: StatefulMixer = MIXERS[spec["type"]].from_config(d, spec["mixer"], config.norm_eps, layer_idx, **fk)
        self.norm1 = nn.Parameter(torch.ones(d, **fk))
        self.mlp, self.norm2 = None, None
        if spec.get("mlp") is not None:
            self.ff = spec["mlp"]["ff"]
            self.norm2 = nn.Parameter(torch.ones(d, **fk))
            self.mlp = GatedMlp(d, hidden_features=self.ff, activation=F.silu, bias1=False, bias2=False, multiple_of=1, **fk)
        self.side = TokenSide(d, config.side_dim, layer_idx * config.side_dim, **fk)

    def load_tensors(self, t, prefix):
        d = self.norm1.shape[0]
        self.mixer.load_tensors(t, prefix + "mix.")
        self.side.load_tensors(t, prefix + "side.")
        with torch.no_grad():
            self.norm1.copy_(t.get(prefix + "norm1", (d,)))
            if self.mlp is not None:
                self.norm2.copy_(t.get(prefix + "norm2", (d,)))
                self.mlp.fc1.weight[:self.ff].copy_(t.get(prefix + "mlp.up", (self.ff, d)))
                self.mlp.fc1.weight[self.ff:].copy_(t.get(prefix + "mlp.gate", (self.ff, d)))
                self.mlp.fc2.weight.copy_(t.get(prefix + "mlp.down", (d, self.ff)))
            elif prefix + "norm2" in t:
                t.get(prefix + "norm2", (d,))   # a layer without an MLP has nothing for a second norm

    def forward(self, stream, x, tokens, side_table, inference_params, out_norm=None):
        """``x`` is the stream in the model's dtype; returns what the next layer reads (with ``out_norm``, normed)."""
        x = ops.stream_post_norm(stream, self.mixer(x, inference_params), self.norm1, eps=self.eps)
        if self.mlp is not None:
            x = ops.stream_post_norm(stream, self.mlp(x), self.norm2, eps=self.eps)
        return self.side(stream, x, tokens, side_table, out_norm, self.eps)


class VubenexLMHeadModel(GenerationMixin, nn.Module):
    supports_portions = True

    def __init__(self, config: VubenexConfig, device=None, dtype=None):
        super().__init__()
        self.config = config
        fk = {"device": device, "dtype": dtype}
        self.pos_embed = nn.Parameter(torch.zeros(config.max_positions, config.width, **fk))
        self.side_embed = nn.Parameter(torch.zeros(config.vocab_size, len(config.layers) * config.side_dim, **fk))
        self.layers = nn.ModuleList([PostNormBlock(config, i, **fk) for i in range(len(config.layers))])
        self.final_norm = nn.Parameter(torch.ones(config.width, **fk))
        self.lm_head = nn.Linear(config.width, config.vocab_size, bias=False, **fk)   # the embedding table, too

    @classmethod
    def from_config(cls, d, device=None, dtype=None):
        return cls(VubenexConfig.from_dict(d), device=device, dtype=dtype)

    @property
    def max_positions(self):
        return self.config.max_positions

    def load_tensors(self, t):
        cfg = self.config
        with torch.no_grad():
            self.lm_head.weight.copy_(t.get("embed", (cfg.vocab_size, cfg.width)))
            self.pos_embed.copy_(t.get("pos", (cfg.max_positions, cfg.width)))
            self.side_embed.copy_(t.get("side.embed", tuple(self.side_embed.shape)))
            self.final_norm.copy_(t.get("final.norm", (cfg.width,)))
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
        if inference_params.seqlen_offset + L > cfg.max_positions:
            raise ValueError(f"{inference_params.seqlen_offset} + {L} tokens are more than the model's {cfg.max_positions} positions")
        stream = torch.empty(B, L, cfg.width, dtype=torch.float32, device=input_ids.device)
        x = ops.stream_embed(stream, input_ids, self.lm_head.weight, cfg.embedding_scale, self.pos_embed,
                             pos=StatefulMixer.position(inference_params, L))
        last = len(self.layers) - 1
        for i, layer in enumerate(self.layers):
            x = layer(stream, x, input_ids, self.side_embed, inference_params, out_norm=self.final_norm if i == last else None)
            if stream_hook is not None:
                stream_hook(i, stream)
        if positions is not None:
            x = x[:, positions]
        elif num_last_tokens > 0:
            x = x[:, -num_last_tokens:]
        return ops.linear_f32(x, self.lm_head.weight)
