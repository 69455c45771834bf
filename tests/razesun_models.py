"""Small Razesun configurations and random weights for the tests, and a writer of model folders."""
import json
import os
import struct

import torch


def latent(heads, dim, rot, vdim, q_rank, kv_rank, scale, base, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def rglru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def config(width, vocab, layers, ffs, eps=1e-5, mult=0.6, logit_scale=0.3):
    layers = [dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff}) for layer, ff in zip(layers, ffs)]
    return {"architecture": "Razesun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "residual_mult": mult, "logit_scale": logit_scale}


def configs():
    """name -> config.  ``mixed``: sizes the tensor-core kernels take, unequal everywhere; ``order``: latent attention first,
    two readers of one cache with other heads and value sizes, a layer without MLP; ``odd``: sizes that are no multiple of
    anything; ``one``: one head, one block, one tap, multipliers 1."""
    return {
        "mixed": config(160, 301, [delta(4, 2, 32, 48, 3), latent(3, 48, 16, 80, 96, 112, 0.11, 5000.0), rglru(128, 2, 4),
                                   latent(5, 32, 16, 32, 64, 112, 0.2, 5000.0, kv_from=1), delta(3, 3, 64, 16, 4)], [96, 224, 160, 128, 64]),
        "order": config(96, 203, [latent(4, 32, 32, 64, 48, 64, 0.125, 1e5), rglru(96, 3, 2), latent(2, 64, 32, 32, 40, 64, 0.09, 1e5, kv_from=0),
                                  delta(6, 2, 64, 32, 4), latent(6, 16, 32, 16, 32, 64, 0.15, 1e5, kv_from=0)], [64, None, 128, 96, None],
                        mult=0.9),
        "odd": config(75, 97, [rglru(66, 6, 3), delta(3, 1, 20, 12, 5), latent(3, 18, 6, 10, 25, 33, 0.2, 300.0)], [50, 33, 41], eps=1e-3),
        "one": config(64, 64, [rglru(64, 1, 1), delta(1, 1, 32, 32, 1), latent(1, 64, 64, 64, 64, 64, 0.1, 10.0)], [64, 64, 64], mult=1.0,
                      logit_scale=1.0),
    }


def tensors(cfg, seed=0, sharp=3.0):
    """Random weights (values a bfloat16 holds).  Latent queries are scaled by ``sharp``, so that attention picks keys
    instead of averaging them; decays are slow, so that old tokens stay in the states."""
    g = torch.Generator().manual_seed(seed)
    t = {}

    def put(name, *shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        t[name] = (mean + std * torch.randn(*shape, generator=g)).bfloat16()

    W, V = cfg["width"], cfg["vocab"]
    put("embed", V, W, std=1.0)
    put("head", V, W)
    for n in ("embed.norm", "final.norm"):
        put(n, W, std=0.2, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        put(f"l{i}.norm1", W, std=0.2, mean=1.0)
        if layer["type"] == "delta":
            H, Hk, d, dv, c = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, rows in (("q", Hk * d), ("k", Hk * d), ("v", H * dv)):
                put(p + n, rows, W)
                put(p + n + ".conv", rows, c, std=0.6, mean=0.3)
            put(p + "b", H, W)
            put(p + "a", H, W)
            put(p + "A_log", H, std=0.5)
            put(p + "dt_bias", H, std=0.5, mean=-4.0)
            put(p + "norm", dv, std=0.2, mean=1.0)
            put(p + "g", H * dv, W)
            put(p + "o", W, H * dv)
        elif layer["type"] == "rglru":
            R, nb, c = m["width"], m["blocks"], m["conv"]
            n = R // nb
            for x in ("x", "y"):
                put(p + x, R, W)
                put(p + x + ".b", R, std=0.2)
            put(p + "conv", R, c, std=0.5)
            put(p + "conv.b", R, std=0.2)
            for x in ("ra", "ri"):
                put(p + x, nb, n, n)
                put(p + x + ".b", nb, n, std=0.5)
            put(p + "lam", R, std=1.0, mean=-4.0)
            put(p + "o", W, R)
        else:
            H, d, rd, dv, qr, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            put(p + "dq", qr, W)
            put(p + "dq.norm", qr, std=0.2, mean=1.0)
            put(p + "uq", H * (d + rd), qr, std=sharp * qr ** -0.5)
            if m.get("kv_from") is None:
                put(p + "dkv", r + rd, W)
                put(p + "dkv.norm", r, std=0.2, mean=1.0)
            put(p + "uk", H * d, r)
            put(p + "uv", H * dv, r)
            put(p + "g", H, W)
            put(p + "o", W, H * dv)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            put(f"l{i}.norm2", W, std=0.2, mean=1.0)
            put(f"l{i}.mlp.gate", ff, W)
            put(f"l{i}.mlp.up", ff, W)
            put(f"l{i}.mlp.down", W, ff)
    return t


def write_safetensors(path, t):
    names = {torch.bfloat16: "BF16", torch.float32: "F32", torch.int32: "I32"}
    header, data, at = {"__metadata__": {"format": "pt"}}, [], 0
    for name, x in t.items():
        raw = x.contiguous().view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[x.dtype], "shape": list(x.shape), "data_offsets": [at, at + len(raw)]}
        data.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(data))


def write_folder(folder, cfg, t):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), t)
