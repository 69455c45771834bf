"""Host side of the Vubenex design: registry, configuration, weights, and the oracle's mechanisms.  No GPU."""
import math

import pytest
import torch

import vubenex_models as M
from based_b200 import registry, weights
from oracle import vubenex_oracle as V


def test_registry():
    assert "Vubenex" in registry.architectures()
    assert registry.model_class("Vubenex").supports_portions


def test_library_part(tmp_path):
    from based_b200 import build
    cfg = M.configs()["one"]
    M.write_folder(str(tmp_path), cfg, M.tensors(cfg))
    part = registry.library_part(str(tmp_path))
    assert part in build.PARTS and set(build._sources(part)) <= set(build._sources())


@pytest.mark.parametrize("name", sorted(M.configs()))
def test_every_tensor_is_loaded_and_has_its_place(name, tmp_path):
    cfg = M.configs()[name]
    t = M.tensors(cfg)
    M.write_folder(str(tmp_path), cfg, t)
    m = registry.load_model(str(tmp_path), device="cpu", dtype=torch.float32)
    assert torch.equal(m.lm_head.weight, t["embed"].float()) and torch.equal(m.side_embed, t["side.embed"].float())
    assert torch.equal(m.pos_embed, t["pos"].float())
    for i, (layer, spec) in enumerate(zip(m.layers, cfg["layers"])):
        x = layer.mixer
        for n in "qkg" if spec["type"] == "attention" else "qkvg":
            at, rows = x.in_proj.offsets[n]
            assert at % 8 == 0 and torch.equal(x.in_proj.weight[at:at + rows], t[f"l{i}.mix.{n}"].float())
        if spec["type"] == "lightning":
            assert x.decay.tolist() == torch.tensor(spec["mixer"]["decay"]).tolist()
        assert torch.equal(x.out_proj.weight, t[f"l{i}.mix.o"].float())
        assert (layer.mlp is None) == (spec["mlp"] is None)
        assert layer.side.column == i * cfg["token_side"]["dim"]
    bare = [i for i, layer in enumerate(m.layers) if layer.mlp is None]
    m.load_tensors(weights.TensorDict({**t, **{f"l{i}.norm2": t["final.norm"] for i in bare}}))
    with pytest.raises(ValueError, match="does not have"):
        m.load_tensors(weights.TensorDict({**t, "l0.extra": torch.zeros(1)}))
    del t["l0.side.norm"]
    with pytest.raises(KeyError, match="l0.side.norm"):
        m.load_tensors(weights.TensorDict(t))


def test_moving_a_model_keeps_the_decays_in_fp32():
    m = registry.build_model(M.configs()["mixed"], device="cpu", dtype=torch.float32).to(torch.bfloat16)
    assert m.lm_head.weight.dtype == torch.bfloat16
    assert all(layer.mixer.decay.dtype == torch.float32 for layer in m.layers if hasattr(layer.mixer, "decay"))


def test_config_is_checked():
    def change(layer, **kw):
        c = M.configs()["mixed"]
        c["layers"][layer]["mixer"].update(kw)
        return registry.build_model(c, device="cpu")
    change(0)
    with pytest.raises(ValueError, match="vdim"):
        change(0, vdim=16)
    with pytest.raises(ValueError, match="multiple of kv_heads"):
        change(0, kv_heads=4)
    with pytest.raises(ValueError, match="period"):
        change(0, q_temp={"coef": 0.1, "every": 0})
    with pytest.raises(ValueError, match="decay"):
        change(1, decay=[0.5])
    for key, bad in (("type", "other"), ("mlp", {"kind": "sparse", "ff": 8})):
        c = M.configs()["mixed"]
        c["layers"][0][key] = bad
        with pytest.raises(ValueError, match="other|sparse"):
            registry.build_model(c, device="cpu")


def test_generation_stops_at_the_last_position():
    c = M.config(16, 16, [M.lightning(8, 8, 0.5)], [None], 8, positions=10)
    m = registry.build_model(c, device="cpu", dtype=torch.float32)
    with pytest.raises(ValueError, match="10 positions"):
        m.generate(torch.zeros(1, 8, dtype=torch.int64), max_new_tokens=4)


def test_oracle_mechanisms():
    """The oracle against closed forms."""
    g = torch.Generator().manual_seed(0)
    s = torch.randn(3, 5, generator=g, dtype=torch.float64)
    with_sink = torch.softmax(torch.cat([s, torch.zeros(3, 1, dtype=torch.float64)], -1), -1)[:, :-1]
    assert torch.allclose(V.sink_softmax(s), with_sink)
    assert torch.allclose(V.sink_softmax(s - 800), torch.zeros_like(s))
    t = V.query_temperature(9, 0.5, 4)
    assert t[:3].tolist() == [1, 1, 1] and torch.allclose(t[3:7], torch.full((4,), 1 + 0.5 * math.log(2), dtype=torch.float64))
    assert math.isclose(float(t[7]), 1 + 0.5 * math.log(3))
    q, k, v = (torch.randn(6, 2, 4, generator=g, dtype=torch.float64) for _ in range(3))
    decay = torch.tensor([0.5, 1.0], dtype=torch.float64)
    o, S = V.decayed_outer_products(q, k, v, decay)
    i, j = torch.arange(6)[:, None], torch.arange(6)[None]
    for h in range(2):
        w = torch.where(j <= i, decay[h] ** (i - j).clamp(min=0), 0)
        assert torch.allclose(o[:, h], (q[:, h] @ k[:, h].T * w) @ v[:, h])
        assert torch.allclose(S[h], torch.einsum("t,td,te->de", decay[h] ** (5 - torch.arange(6)), k[:, h], v[:, h]))
    half, rest = V.decayed_outer_products(q[:3], k[:3], v[:3], decay), None
    rest = V.decayed_outer_products(q[3:], k[3:], v[3:], decay, half[1])
    assert torch.allclose(torch.cat([half[0], rest[0]]), o) and torch.allclose(rest[1], S)
    # a group's heads see the same key head
    kk = torch.randn(6, 1, 4, generator=g, dtype=torch.float64)
    one = V.causal_attention(q, kk, kk, 0.3)
    assert torch.allclose(one, V.causal_attention(q, kk.expand(6, 2, 4), kk.expand(6, 2, 4), 0.3))
    assert torch.allclose(one[0], kk[0] * V.sink_softmax((q[0] @ kk[0, 0] * 0.3)[:, None]))
