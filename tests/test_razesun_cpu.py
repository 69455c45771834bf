"""Host side of the Razesun design and of model loading: registry, configuration, safetensors, packing.  No GPU."""
import pytest
import torch

import razesun_models as M
from based_b200 import registry, weights
from oracle import razesun_oracle as R


def test_registry():
    assert {"Based", "Razesun"} <= set(registry.architectures())
    assert registry.model_class("Razesun").supports_portions
    with pytest.raises(ValueError, match="Based"):
        registry.model_class("Nothing")
    based = registry.build_model({"architecture": "Based", "n_embd": 32, "n_layer": 2, "n_head": 2, "n_inner": 64, "vocab_size": 40,
                                  "alt_mixer_layers": [], "alt_mixer_2_layers": []}, device="cpu", dtype=torch.float32)
    sd = {k: torch.randn_like(v) for k, v in based.state_dict().items() if k != "lm_head.weight"}
    based.load_tensors(weights.TensorDict(sd))
    assert all(torch.equal(based.state_dict()[k], v) for k, v in sd.items())
    assert based.lm_head.weight is based.transformer.embeddings.word_embeddings.weight


def test_safetensors_roundtrip_and_errors(tmp_path):
    t = {"a": torch.randn(3, 5).bfloat16(), "b.c": torch.randn(7), "i": torch.arange(6, dtype=torch.int32).view(2, 3), "odd": torch.ones(1).bfloat16(),
         "after": torch.randn(4)}
    p = str(tmp_path / "m.safetensors")
    M.write_safetensors(p, t)
    s = weights.SafeTensors(p)
    assert set(s) == set(t) and "a" in s and "z" not in s
    for k, v in t.items():
        assert torch.equal(s.get(k, tuple(v.shape)), v)
    assert s.unused() == []
    assert weights.SafeTensors(p).unused() == sorted(t)
    with pytest.raises(ValueError, match="shape"):
        s.get("a", (5, 3))
    with pytest.raises(KeyError):
        s.get("z")
    raw = open(p, "rb").read()
    short = str(tmp_path / "short.safetensors")
    open(short, "wb").write(raw[:-4])
    with pytest.raises(ValueError, match="past the end"):
        weights.SafeTensors(short)


@pytest.mark.parametrize("name", sorted(M.configs()))
def test_every_tensor_is_loaded_and_has_its_place(name, tmp_path):
    """A model on the CPU (only its parameters): packed weights hold the named tensors, nothing is left over."""
    cfg, t = M.configs()[name], M.tensors(M.configs()[name])
    M.write_folder(str(tmp_path), cfg, t)
    m = registry.load_model(str(tmp_path), device="cpu", dtype=torch.float32)
    for i, layer in enumerate(m.layers):
        assert torch.equal(layer.out_weight[:, :layer.inner], t[f"l{i}.mix.o"].float())
        if layer.mlp is not None:
            assert torch.equal(layer.out_weight[:, layer.split:], t[f"l{i}.mlp.down"].float())
            assert torch.equal(layer.mlp.fc1.weight, torch.cat([t[f"l{i}.mlp.up"], t[f"l{i}.mlp.gate"]]).float())
        assert bool((layer.out_weight[:, layer.inner:layer.split] == 0).all())
    bare = [i for i, layer in enumerate(m.layers) if layer.mlp is None]
    m.load_tensors(weights.TensorDict({**t, **{f"l{i}.norm2": t["final.norm"] for i in bare}}))
    with pytest.raises(ValueError, match="does not have"):
        m.load_tensors(weights.TensorDict({**t, "l0.extra": torch.zeros(1)}))
    del t["final.norm"]
    with pytest.raises(KeyError, match="final.norm"):
        m.load_tensors(weights.TensorDict(t))


def test_moving_a_model_keeps_the_shared_output_weights():
    cfg = M.configs()["mixed"]
    m = registry.build_model(cfg, device="cpu", dtype=torch.float32).to(torch.bfloat16)
    m.load_tensors(weights.TensorDict(M.tensors(cfg)))
    for layer in m.layers:
        assert layer.mixer.out_proj.weight.data_ptr() == layer.out_weight.data_ptr()
        assert torch.equal(layer.mlp.fc2.weight, layer.out_weight[:, layer.split:])


def test_config_is_checked():
    def change(**kw):
        c = M.configs()["mixed"]
        c["layers"][3]["mixer"].update(kw)
        return registry.build_model(c, device="cpu")
    change()
    for bad in ({"kv_from": 0}, {"kv_from": 3}, {"kv_from": 7}, {"kv_rank": 64}, {"rot": {"base": 1.0, "dims": 16}}):
        with pytest.raises(ValueError, match="kv_from"):
            change(**bad)
    c = M.configs()["mixed"]
    c["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="other"):
        registry.build_model(c, device="cpu")
    c = M.configs()["mixed"]
    c["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError, match="sparse"):
        registry.build_model(c, device="cpu")


def test_oracle_mechanisms():
    """The oracle against closed forms: rotation keeps lengths and depends on distance only, the delta rule overwrites a
    key's value, the recurrent unit's closed form, the convolution against torch's."""
    g = torch.Generator().manual_seed(0)
    x = torch.randn(6, 8, generator=g, dtype=torch.float64)
    r = R.rotate_half(x, torch.arange(6), 100.0)
    assert torch.allclose(r.norm(dim=-1), x.norm(dim=-1))
    a = R.rotate_half(x[:2], torch.tensor([3, 9]), 100.0)
    b = R.rotate_half(x[:2], torch.tensor([10, 16]), 100.0)
    assert torch.allclose(a[0] @ a[1], b[0] @ b[1])
    k = torch.eye(4, dtype=torch.float64)[[0, 1, 0]].view(3, 1, 4)
    v = torch.randn(3, 1, 2, generator=g, dtype=torch.float64)
    _, S = R.delta_rule(k, k, v, torch.ones(3, 1, dtype=torch.float64), torch.ones(3, 1, dtype=torch.float64))
    assert torch.allclose(S[0, 0], v[2, 0]) and torch.allclose(S[0, 1], v[1, 0])
    w = torch.randn(8, 3, generator=g, dtype=torch.float64)
    ref = torch.nn.functional.conv1d(x.t().unsqueeze(0), w.unsqueeze(1), padding=2, groups=8)[0, :, :6].t()
    assert torch.allclose(R.short_conv(x, w), ref)
    u, one = torch.ones(5, 1, dtype=torch.float64), torch.ones(5, 1, dtype=torch.float64)
    lam = torch.tensor([-2.0], dtype=torch.float64)
    a = torch.exp(-8 * R.softplus(lam))
    S = R.rglru_scan(u, one, one, lam)
    assert torch.allclose(S[:, 0], torch.sqrt(1 - a * a) * (1 - a ** torch.arange(1, 6)) / (1 - a))
