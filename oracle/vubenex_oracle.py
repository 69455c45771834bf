"""Plain, slow restatement of the Vubenex design (test infrastructure, CPU).

One function per mechanism, whole sequences only (no cache, no portions, no batch): the framework's portions, caches and
decode steps are compared with slices of what these functions return for the full sequence.  Shares no code with
``based_b200``.  ``x`` is ``[T, width]``; weights are a dict name -> tensor, stored ``[out, in]``.  Everything runs in the
dtype of the tensors it is given (float64 for reference values).
"""
import math

import torch


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def embed(w, tokens, scale):
    """Scaled token vector plus the (unscaled) vector of the position."""
    return w["embed"][tokens] * scale + w["pos"][:len(tokens)]


def query_temperature(T, coef, every):
    """Factor of the query at each position; steps up after every ``every`` tokens."""
    return torch.tensor([1 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(T)], dtype=torch.float64)


def sink_softmax(s):
    """Rows of scores (-inf where hidden) to weights; one more score of 0 takes part in the sum and has no weight here."""
    m = s.amax(-1, keepdim=True).clamp(min=0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def causal_attention(q, k, v, scale):
    """q ``[T, H, d]``, k ``[T, G, d]``, v ``[T, G, dv]`` -> ``[T, H, dv]``; the H / G heads of a group share a key head."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    head = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, head]) * scale
    s = s.masked_fill(~torch.ones(T, T, dtype=torch.bool).tril(), float("-inf"))
    return torch.einsum("hij,jhe->ihe", sink_softmax(s), v[:, head])


def attention_mixer(x, w, pre, m, eps):
    T = x.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (x @ w[pre + "q"].T).view(T, H, d)
    k = (x @ w[pre + "k"].T).view(T, G, d)
    t = query_temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"]).to(x.dtype)
    qn = rms(q, eps, w[pre + "q.norm"]) * t[:, None, None]
    o = causal_attention(qn, rms(k, eps, w[pre + "k.norm"]), k, m["scale"])   # values: keys before their norm
    return (o.reshape(T, H * d) * torch.sigmoid(x @ w[pre + "g"].T)) @ w[pre + "o"].T


def decayed_outer_products(q, k, v, decay, S=None):
    """q, k ``[T, H, d]``, v ``[T, H, dv]``, decay ``[H]``: o ``[T, H, dv]`` and the final state ``[H, d, dv]``."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if S is None else S.clone()
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


def lightning_mixer(x, w, pre, m, eps):
    T = x.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k = (silu(x @ w[pre + n].T).view(T, H, d) for n in "qk")
    v = silu(x @ w[pre + "v"].T).view(T, H, dv)
    o, _ = decayed_outer_products(q, k, v, torch.tensor(m["decay"], dtype=x.dtype))
    o = rms(o.reshape(T, H * dv), eps, w[pre + "norm"]) * torch.sigmoid(x @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def dense_mlp(x, w, pre):
    return (silu(x @ w[pre + "gate"].T) * (x @ w[pre + "up"].T)) @ w[pre + "down"].T


def token_side(x, w, pre, e, eps):
    """What the token's own vector ``e [T, dim]`` of this layer adds to the stream."""
    y = (gelu_tanh(x @ w[pre + "gate"].T) * e) @ w[pre + "proj"].T
    return rms(y, eps, w[pre + "norm"])


MIXERS = {"attention": attention_mixer, "lightning": lightning_mixer}


def forward(cfg, w, tokens, want_layers=False):
    """Logits ``[T, vocab]`` of one sequence; with ``want_layers`` also the residual after every layer."""
    eps, n = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    x = embed(w, tokens, cfg["embedding"]["scale"])
    per_layer = []
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + rms(MIXERS[layer["type"]](x, w, pre + "mix.", layer["mixer"], eps), eps, w[pre + "norm1"])
        if layer.get("mlp"):
            x = x + rms(dense_mlp(x, w, pre + "mlp."), eps, w[pre + "norm2"])
        x = x + token_side(x, w, pre + "side.", w["side.embed"][tokens][:, i * n:(i + 1) * n], eps)
        per_layer.append(x)
    logits = rms(x, eps, w["final.norm"]) @ w["embed"].T
    return (logits, torch.stack(per_layer)) if want_layers else logits
