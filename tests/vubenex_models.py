"""Small Vubenex configurations and random weights for the tests."""
import torch

from razesun_models import write_folder, write_safetensors  # noqa: F401


def attention(heads, kv_heads, dim, scale, coef, every):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                           "q_temp": {"coef": coef, "every": every}}}


def lightning(dim, vdim, *decay):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def config(width, vocab, layers, ffs, side, scale=3.0, eps=1e-5, positions=1500):
    layers = [dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff}) for layer, ff in zip(layers, ffs)]
    return {"architecture": "Vubenex", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "max_positions": positions, "token_side": {"dim": side}}


def configs():
    """name -> config.  ``mixed``: sizes the tensor-core kernels take, unequal everywhere; ``order``: recurrence first, layers
    with and without MLP of both types, groups of one and of all heads; ``odd``: sizes that are no multiple of anything;
    ``wide``: the largest head sizes; ``one``: one head, constants 1 (decay) and 0 (temperature)."""
    return {
        "mixed": config(160, 301, [attention(6, 2, 32, 0.2, 0.4, 50), lightning(48, 32, 0.9, 0.997, 0.4), attention(8, 1, 48, 0.15, 0.2, 7),
                                   lightning(64, 80, 0.7, 0.99)], [96, None, 224, 64], 24),
        "order": config(96, 203, [lightning(32, 16, 0.5, 0.95, 0.999, 0.8, 1.0), attention(5, 5, 64, 0.125, 0.7, 100), lightning(16, 64, 0.05, 0.99),
                                  attention(4, 4, 16, 0.3, 0.1, 1)], [128, None, 160, 64], 40, scale=9.8, eps=1e-4),
        "odd": config(75, 97, [attention(3, 1, 18, 0.3, 0.5, 33), lightning(20, 11, 0.6, 0.98, 0.9), attention(6, 3, 7, 0.4, 0.25, 64)],
                      [50, 33, None], 27, scale=1.7, eps=1e-3),
        "wide": config(224, 150, [lightning(128, 128, 0.98, 0.3), attention(4, 2, 128, 0.09, 0.3, 90), attention(12, 2, 96, 0.1, 0.05, 200),
                                  lightning(96, 112, 0.9999, 0.85)], [192, 128, None, None], 40, scale=2.0),
        "one": config(64, 64, [attention(1, 1, 64, 1.0, 0.0, 1), lightning(32, 32, 1.0)], [64, 64], 32, scale=1.0),
    }


def tensors(cfg, seed=0, sharp=1.0):
    """Random weights (values a bfloat16 holds).  Query norm weights are such that scores spread by ``sharp`` (times the
    temperature): attention picks keys instead of averaging them and the sink takes a visible share."""
    g = torch.Generator().manual_seed(seed)
    t = {}

    def put(name, *shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        t[name] = (mean + std * torch.randn(*shape, generator=g)).bfloat16()

    W, V, n = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"]
    put("embed", V, W, std=1.0 / cfg["embedding"]["scale"])
    put("pos", cfg["max_positions"], W, std=0.3)
    put("side.embed", V, len(cfg["layers"]) * n, std=1.0)
    put("final.norm", W, std=0.2, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        put(f"l{i}.norm1", W, std=0.2, mean=0.8)
        if layer["type"] == "attention":
            H, G, d = m["heads"], m["kv_heads"], m["dim"]
            put(p + "q", H * d, W)
            put(p + "k", G * d, W)
            put(p + "g", H * d, W)
            put(p + "o", W, H * d)
            c = sharp / (m["scale"] * d ** 0.5)
            put(p + "q.norm", d, std=0.2 * c, mean=c)
            put(p + "k.norm", d, std=0.3, mean=1.0)
        else:
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            for x, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                put(p + x, rows, W)
            put(p + "norm", H * dv, std=0.2, mean=1.0)
            put(p + "o", W, H * dv)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            put(f"l{i}.norm2", W, std=0.2, mean=0.8)
            put(f"l{i}.mlp.gate", ff, W)
            put(f"l{i}.mlp.up", ff, W)
            put(f"l{i}.mlp.down", W, ff)
        put(f"l{i}.side.gate", n, W)
        put(f"l{i}.side.proj", W, n)
        put(f"l{i}.side.norm", W, std=0.1, mean=0.4)
    return t
