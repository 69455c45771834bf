"""Inference-time state container shared by the mixers, the decoding loop shared by the models, and the pool that
hands state containers to requests.

``InferenceParams`` is a field-for-field mirror of ``InferenceParams`` in the reference (based/generation.py:18-35):
the mixers only read ``seqlen_offset``, ``max_seqlen``, ``max_batch_size``,
``batch_size_offset``, ``lengths_per_sample`` and store their per-layer state in
``key_value_memory_dict[layer_idx]``.  The reference's own class (or any object with these
attributes) can be passed instead; the mixers never check the type.
"""
from dataclasses import dataclass, field
from typing import Optional

import torch
from torch import Tensor

from . import ops


@dataclass
class InferenceParams:
    max_seqlen: int
    max_batch_size: int
    seqlen_offset: int = 0
    batch_size_offset: int = 0
    key_value_memory_dict: dict = field(default_factory=dict)
    lengths_per_sample: Optional[Tensor] = None

    def reset(self, max_seqlen, max_batch_size):
        self.max_seqlen = max_seqlen
        self.max_batch_size = max_batch_size
        self.seqlen_offset = 0
        if self.lengths_per_sample is not None:
            self.lengths_per_sample.zero_()


def sample_token(logits: torch.Tensor, top_k: int = 1, top_p: float = 0.0, temperature: float = 1.0) -> torch.Tensor:
    """Next token per row of ``logits [B, V]``: greedy for ``top_k == 1``; otherwise restrict to the ``top_k`` largest
    logits (all of them for ``top_k <= 0``), divide by ``temperature``, drop the low-probability tail whose
    cumulative probability is at most ``1 - top_p`` (nucleus sampling; no-op for ``top_p`` outside (0, 1)), and draw
    from the softmax of what is left.  Same policy as ``sample`` in based/generation.py:38-92."""
    if top_k == 1:
        return logits.argmax(dim=-1)
    if not 0.0 <= top_p <= 1.0:
        raise ValueError("top_p must be in [0, 1]")
    if top_k > 0:
        vals, idx = torch.topk(logits, min(top_k, logits.size(-1)), dim=-1)       # descending
    else:
        vals, idx = torch.sort(logits, dim=-1, descending=True)
    vals = vals.float()
    if temperature != 1.0:
        vals = vals / temperature
    if 0.0 < top_p < 1.0:
        probs = vals.softmax(dim=-1)
        tail = probs.flip(-1).cumsum(dim=-1).flip(-1)     # mass of this candidate and everything less likely
        vals = vals.masked_fill(tail <= 1.0 - top_p, float("-inf"))
    choice = torch.multinomial(vals.softmax(dim=-1), num_samples=1)
    return idx.gather(-1, choice).squeeze(-1)


class StatePool:
    """State containers for requests that come and go: ``acquire`` hands out an :class:`InferenceParams` with the model's
    caches and states allocated, ``release`` takes it back for the next request.  Nothing is cleared in between: a
    sequence that starts at position 0 reads neither state nor cache."""

    def __init__(self, model, max_seqlen: int, max_batch_size: int = 1):
        self.model, self.max_seqlen, self.max_batch_size = model, max_seqlen, max_batch_size
        self.live, self.free = {}, []

    def acquire(self, request_id) -> InferenceParams:
        if request_id in self.live:
            raise KeyError(f"request {request_id!r} is already live")
        if self.free:
            ip = self.free.pop()
            ip.reset(self.max_seqlen, self.max_batch_size)
        else:
            ip = self.model.new_inference_params(self.max_batch_size, self.max_seqlen)
        self.live[request_id] = ip
        return ip

    def release(self, request_id) -> None:
        self.free.append(self.live.pop(request_id))


class GenerationMixin:
    """Decoding for a model with ``forward(input_ids, inference_params, num_last_tokens)``,
    ``allocate_inference_cache(batch, max_seqlen, dtype)``, ``lm_head`` and ``config.vocab_size``."""

    # whether a call with seqlen_offset > 0 may bring more than one token (a later portion of a prompt)
    supports_portions = False
    # positions a model has learned vectors for; None: no limit
    max_positions = None

    def new_inference_params(self, batch_size: int, max_seqlen: int) -> InferenceParams:
        w = self.lm_head.weight
        ip = InferenceParams(max_seqlen=max_seqlen, max_batch_size=batch_size)
        ip.key_value_memory_dict = self.allocate_inference_cache(batch_size, max_seqlen, dtype=w.dtype)
        ip.lengths_per_sample = torch.zeros(batch_size, dtype=torch.int32, device=w.device)
        return ip

    def advance(self, input_ids, ip: InferenceParams, **kwargs):
        """Run the next tokens ``[B, L]`` of every sequence from the state earlier calls left: a prompt, a portion of
        one, or one decoded token.  Returns what ``forward`` does; the state and the lengths move on by L."""
        L = input_ids.shape[1]
        if ip.seqlen_offset + L > ip.max_seqlen:
            raise ValueError(f"{ip.seqlen_offset} + {L} tokens do not fit the cache of {ip.max_seqlen}")
        if L > 1 and ip.seqlen_offset > 0 and not self.supports_portions:
            raise NotImplementedError(f"{type(self).__name__} takes a prompt in one piece")
        out = self.forward(input_ids, inference_params=ip, **kwargs)
        ip.seqlen_offset += L
        ip.lengths_per_sample.add_(L)
        return out

    @torch.inference_mode()
    def generate(self, input_ids, max_new_tokens: int, cg: bool = False, timings: Optional[dict] = None,
                 top_k: int = 1, top_p: float = 0.0, temperature: float = 1.0, portion: int = 0):
        """Decoding: one prompt pass, then one token per step (generation.py:93-204); greedy by default, top-k /
        nucleus / temperature sampling as :func:`sample_token` otherwise.  With ``cg`` the decode step is
        captured once in a CUDA graph and replayed (:689-739).  Returns ``[B, L + max_new_tokens]``.
        ``timings``, when given, receives device times in ms: ``prefill_ms``, ``decode_ms`` (all steps, with the graph's
        capture), ``steps_ms`` (the steps alone).
        ``portion`` > 0 feeds the prompt that many tokens at a time (models that support portions)."""
        B, L = input_ids.shape
        if self.max_positions is not None and L + max(max_new_tokens - 1, 0) > self.max_positions:
            raise ValueError(f"{L} + {max_new_tokens} tokens are more than the model's {self.max_positions} positions")
        ip = self.new_inference_params(B, L + max_new_tokens)
        ev = [torch.cuda.Event(enable_timing=True) for _ in range(4)]
        out = torch.empty(B, L + max_new_tokens, dtype=input_ids.dtype, device=input_ids.device)
        out[:, :L] = input_ids
        ev[0].record()
        for l0 in range(0, max(L, 1), portion if portion > 0 else max(L, 1)):
            logits = self.advance(input_ids[:, l0:l0 + portion] if portion > 0 else input_ids, ip, num_last_tokens=1)
        token = sample_token(logits[:, -1, : self.config.vocab_size], top_k, top_p, temperature).unsqueeze(-1)
        ev[1].record()
        if max_new_tokens > 0:
            out[:, L] = token[:, 0]
        cur = token.clone()

        def step():
            lg = self.forward(cur, inference_params=ip, num_last_tokens=1)
            cur.copy_(sample_token(lg[:, -1, : self.config.vocab_size], top_k, top_p, temperature).unsqueeze(-1))
            ip.lengths_per_sample.add_(1)

        graph = None
        steps_left = max_new_tokens - 1
        if cg and steps_left > 2:
            # warm-up on a side stream (the first calls may build rotary tables), then capture one step
            s = torch.cuda.Stream()
            s.wait_stream(torch.cuda.current_stream())
            saved = self._snapshot_state(ip, cur)
            with torch.cuda.stream(s):
                for _ in range(2):
                    step()
            torch.cuda.current_stream().wait_stream(s)
            self._restore_state(ip, cur, saved)
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph):
                step()
            self._restore_state(ip, cur, saved)
        ev[3].record()
        for i in range(steps_left):
            if graph is not None:
                graph.replay()
            else:
                step()
            ip.seqlen_offset += 1
            out[:, L + 1 + i] = cur[:, 0]
        ev[2].record()
        if timings is not None:
            torch.cuda.synchronize()
            ops.check_status()   # the device is idle here: a tensor-core kernel that gave up on a wait shows now
            timings["prefill_ms"] = ev[0].elapsed_time(ev[1])
            timings["decode_ms"] = ev[1].elapsed_time(ev[2])
            timings["steps_ms"] = ev[3].elapsed_time(ev[2])
        return out

    @staticmethod
    def _flat_state(ip):
        for v in ip.key_value_memory_dict.values():
            if isinstance(v, dict):
                yield from v.values()
            elif isinstance(v, (tuple, list)):
                yield from v
            else:
                yield v

    def _snapshot_state(self, ip, cur):
        return [t.clone() for t in self._flat_state(ip)] + [ip.lengths_per_sample.clone(), cur.clone()]

    def _restore_state(self, ip, cur, saved):
        tensors = list(self._flat_state(ip)) + [ip.lengths_per_sample, cur]
        for t, s in zip(tensors, saved):
            t.copy_(s)
