"""Plain, slow restatement of the Razesun design (test infrastructure, CPU).

One function per mechanism, whole sequences only (no cache, no portions, no batch): the framework's portions,
caches and decode steps are compared with slices of what these functions return for the full sequence.  Shares no
code with ``based_b200``.  ``x`` is ``[T, width]``; weights are a dict name -> tensor, stored ``[out, in]``.
Everything runs in the dtype of the tensors it is given (float64 for reference values).
"""
import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_vector(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def short_conv(x, taps, bias=None):
    """y[t, c] = sum_j taps[c, j] x[t - (n-1) + j, c] (+ bias[c]); x before the start is zero."""
    T, C = x.shape
    n = taps.shape[1]
    y = torch.zeros_like(x) if bias is None else bias.expand(T, C).clone()
    for j in range(n):
        back = n - 1 - j
        if back < T:
            y[back:] += taps[:, j] * x[:T - back]
    return y


def rotate_half(x, positions, base):
    """x ``[T, ..., d]``, dimension i paired with i + d/2, angle position * base^(-2i/d)."""
    d = x.shape[-1]
    i = torch.arange(d // 2, dtype=torch.float64)
    ang = positions.double().reshape(-1, 1) * base ** (-2 * i / d)
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [d // 2]
    c, s = torch.cos(ang).to(x.dtype).reshape(shape), torch.sin(ang).to(x.dtype).reshape(shape)
    u, v = x[..., :d // 2], x[..., d // 2:]
    return torch.cat([u * c - v * s, v * c + u * s], dim=-1)


def causal_softmax_attention(q, k, v, scale):
    """q, k ``[T, H, d]``, v ``[T, H, dv]`` -> ``[T, H, dv]``."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    s = s.masked_fill(~mask, float("-inf"))
    p = torch.softmax(s, dim=-1)
    return torch.einsum("hij,jhd->ihd", p, v)


def latent_of(h, w, pre, m, eps):
    """The cached pair of a latent-attention layer: normed latent ``[T, kv_rank]``, rotated shared key ``[T, rot_dim]``."""
    r = m["kv_rank"]
    z = h @ w[pre + "dkv"].T
    c = rms_norm(z[:, :r], w[pre + "dkv.norm"], eps)
    kr = rotate_half(z[:, r:], torch.arange(h.shape[0]), m["rot"]["base"])
    return c, kr


def latent_attention(h, w, pre, m, eps, latent):
    T = h.shape[0]
    H, d, rd, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = latent
    cq = rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps)
    q = (cq @ w[pre + "uq"].T).view(T, H, d + rd)
    q = torch.cat([q[..., :d], rotate_half(q[..., d:], torch.arange(T), m["rot"]["base"])], dim=-1)
    k = torch.cat([(c @ w[pre + "uk"].T).view(T, H, d), kr[:, None].expand(T, H, rd)], dim=-1)
    v = (c @ w[pre + "uv"].T).view(T, H, dv)
    o = causal_softmax_attention(q, k, v, m["scale"])
    o = o * torch.sigmoid(h @ w[pre + "g"].T)[..., None]
    return o.reshape(T, H * dv) @ w[pre + "o"].T


def delta_rule(q, k, v, beta, g, S=None):
    """q, k ``[T, H, d]`` (unit vectors, q scaled), v ``[T, H, dv]``, beta, g ``[T, H]``.  Returns o, final S ``[H, d, dv]``."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if S is None else S.clone()
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


def delta_mixer(h, w, pre, m, eps):
    T = h.shape[0]
    H, Hk, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ w[pre + n].T, w[pre + n + ".conv"])) for n in "qkv")
    q = unit_vector(q.view(T, Hk, d)) * d ** -0.5
    k = unit_vector(k.view(T, Hk, d))
    head = torch.arange(H) // (H // Hk)
    beta = torch.sigmoid(h @ w[pre + "b"].T)
    g = torch.exp(-torch.exp(w[pre + "A_log"]) * softplus(h @ w[pre + "a"].T + w[pre + "dt_bias"]))
    o, _ = delta_rule(q[:, head], k[:, head], v.view(T, H, dv), beta, g)
    o = unit_rms(o, eps) * w[pre + "norm"] * silu((h @ w[pre + "g"].T).view(T, H, dv))
    return o.reshape(T, H * dv) @ w[pre + "o"].T


def rglru_scan(u, r, i, lam, S=None):
    """u, r, i ``[T, width]`` -> S ``[T, width]``."""
    S = torch.zeros_like(u[0]) if S is None else S.clone()
    out = []
    for t in range(u.shape[0]):
        a = torch.exp(-8 * r[t] * softplus(lam))
        S = a * S + torch.sqrt(1 - a * a) * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def block_linear(u, W, b):
    """W ``[blocks, n, n]`` applied to the equal parts of u ``[T, blocks * n]``, plus b ``[blocks, n]``."""
    T = u.shape[0]
    n = W.shape[-1]
    z = torch.einsum("bon,tbn->tbo", W, u.view(T, -1, n)) + b
    return z.reshape(T, -1)


def rglru_mixer(h, w, pre, m, eps):
    y = gelu_tanh(h @ w[pre + "y"].T + w[pre + "y.b"])
    u = short_conv(h @ w[pre + "x"].T + w[pre + "x.b"], w[pre + "conv"], w[pre + "conv.b"])
    r = torch.sigmoid(block_linear(u, w[pre + "ra"], w[pre + "ra.b"]))
    i = torch.sigmoid(block_linear(u, w[pre + "ri"], w[pre + "ri.b"]))
    return (rglru_scan(u, r, i, w[pre + "lam"]) * y) @ w[pre + "o"].T


def dense_mlp(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def forward(cfg, w, tokens, want_layers=False):
    """Logits ``[T, vocab]`` of one sequence; with ``want_layers`` also the residual after every layer."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = rms_norm(w["embed"][tokens], w["embed.norm"], eps)
    latents, per_layer = {}, []
    for n, layer in enumerate(cfg["layers"]):
        m, pre = layer["mixer"], f"l{n}.mix."
        h = rms_norm(x, w[f"l{n}.norm1"], eps)
        if layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                latents[n] = latent_of(h, w, pre, m, eps)
            y = latent_attention(h, w, pre, m, eps, latents[n if src is None else src])
        elif layer["type"] == "delta":
            y = delta_mixer(h, w, pre, m, eps)
        elif layer["type"] == "rglru":
            y = rglru_mixer(h, w, pre, m, eps)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp"):
            y = y + dense_mlp(rms_norm(x, w[f"l{n}.norm2"], eps), w, f"l{n}.mlp.")
        x = x + mult * y
        per_layer.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"]
    return (logits, torch.stack(per_layer)) if want_layers else logits
