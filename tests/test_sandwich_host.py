"""Host side of the decoder with norms on both sides of its sublayers, without a GPU: configuration, weights, cache, rotation tables, and
the plain functions that the GPU tests compare with."""

import json
import math

import pytest
import torch

import plain_sandwich as plain
import vllm_rlt_b200 as rlt
from hybrid_cases import prompt, write_model
from sandwich_cases import CONFIGS, latent_layer, make_config, random_weights, windowed_layer
from vllm_rlt_b200 import registry, sandwich_lm


def parse(config):
    return rlt.SandwichLMConfig.from_json(config)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configurations_parse_and_name_every_tensor(name):
    config = parse(CONFIGS[name])
    shapes = sandwich_lm.parameter_shapes(config)
    weights = random_weights(shapes, 0)
    model = rlt.SandwichLM(config, weights, "cpu")
    for i, entry in enumerate(CONFIGS[name]["layers"]):
        layer, p = model.layers[i], f"l{i}."
        assert len(layer.before) == len(layer.behind) == (2 if entry["mlp"] else 1)
        assert (p + "norm2b" in shapes) == (p + "mlp.down" in shapes) == bool(entry["mlp"])
        m, mixer, w = layer.mixer.config, layer.mixer, lambda n: weights[f"{p}mix.{n}"]
        if entry["type"] == "attention":
            for at, n in zip(mixer.columns, "qkv"):
                assert torch.equal(mixer.w_in[at:at + w(n).shape[0]], w(n)) and torch.equal(mixer.bias[at:at + w(n).shape[0]], w(n + ".b"))
            assert torch.equal(mixer.w_in[mixer.g_col:mixer.g_col + m.heads * m.vdim], w("g"))
            assert not mixer.bias[mixer.g_col:].any() and mixer.conv.shape == (entry["mixer"]["conv"], sum(m.projections.values()))
        else:
            second = entry["type"] == "latent_attention_2"
            assert (mixer.sink is not None) == (f"{p}mix.sink" in shapes) == second
            assert torch.equal(mixer.w_down[mixer.kv_col:mixer.kv_col + m.row], w("dkv"))
            assert torch.equal(mixer.w_down[mixer.g_col:mixer.g_col + m.gate_width], w("g"))
            assert w("g").shape[0] == (m.heads if second else m.heads * m.vdim) and mixer.turn["halves"]


def test_every_layer_has_pages_and_convolutions_have_state():
    config = parse(CONFIGS["odd"])
    spec = rlt.SandwichLM(config, random_weights(sandwich_lm.parameter_shapes(config), 0), "cpu").cache_spec()
    assert spec.layers == {0: rlt.KVSpec(1, 17, 0), 1: rlt.KVSpec(1, 10, 7), 2: rlt.KVSpec(1, 5, 3), 3: rlt.KVSpec(1, 6, 0), 4: rlt.KVSpec(1, 13, 0)}
    assert {k: v.shape for k, v in spec.states.items()} == {"l1.conv": (0, 47), "l2.conv": (5, 13)}
    cache = rlt.SequenceCache(spec, max_tokens=100, max_sequences=2, block=spec.block, device="cpu")
    assert cache.key[0].shape == (2, 64, 1, 17) and sorted(cache.value) == [1, 2] and cache.state["l2.conv"].shape == (3, 5, 13)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][2]["mixer"].update(sink=True), "unknown config keys"),
    (lambda c: c["layers"][2]["mixer"].update(mask={"size": 4}), "unknown config keys"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(scaling={"factor": 2.0}), "unknown config keys"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "lacks"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), "positive"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "lacks"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep=2), "unknown config keys"),
    (lambda c: c["layers"][0].update(type="lightning"), "unknown mixer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "feed-forward"),
    (lambda c: c.pop("residual_mult"), "lacks"),
    (lambda c: c.update(logit_softcap=0.0), "logit_softcap"),
    (lambda c: c["norm"].update(offset=1), "unknown config keys"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configurations_that_make_no_sense_are_refused(change, message):
    config = json.loads(json.dumps(CONFIGS["mixed"]))
    change(config)
    with pytest.raises(ValueError, match=message):
        parse(config)


def test_the_registry_loads_a_folder(tmp_path):
    config = parse(CONFIGS["odd"])
    weights = random_weights(sandwich_lm.parameter_shapes(config), 0)
    write_model(tmp_path, CONFIGS["odd"], weights)
    model = rlt.load_model(tmp_path, device="cpu", dtype=torch.float32)
    assert registry.resolve(CONFIGS["odd"]).model_class is rlt.SandwichLM and model.config == config and model.embed.dtype == torch.float32
    del weights["l1.mix.k.conv"]
    with pytest.raises(ValueError, match="lacks"):
        rlt.SandwichLM(config, weights, "cpu")


@pytest.mark.parametrize("base,dims,scaling", [(10000.0, 64, (40.0, 4096, 32.0, 1.0)), (500.0, 24, (3.0, 700, 24.0, 2.0)), (10.0, 2, (2.0, 64, 4.0, 1.0)),
                                               (1e6, 128, (1.0, 8192, 8.0, 2.0)), (1e4, 32, (8.0, 100, 1.0, 1.0)), (1e4, 32, (8.0, 100, 1e6, 1e-9))])
def test_scaled_frequencies(base, dims, scaling):
    entry = dict(zip(("factor", "original", "fast", "slow"), scaling))
    want, amplitude = plain.frequencies(base, dims, entry)
    s = rlt.YarnScaling(*scaling)
    assert torch.allclose(rlt.rotation_frequencies(base, dims, "cpu", s), torch.tensor(want, dtype=torch.float64), rtol=1e-13, atol=0)
    assert s.amplitude == pytest.approx(amplitude, rel=1e-14)


# ---- the plain functions themselves --------------------------------------------------------------
def test_plain_rotation_turns_the_halves_and_depends_on_distance_only():
    g = torch.Generator().manual_seed(0)
    q, k = torch.randn(1, 10, generator=g).double(), torch.randn(1, 10, generator=g).double()
    turns, _ = plain.frequencies(100.0, 8)
    at = lambda x, p: plain.rotate(x, torch.tensor([p]), turns)
    assert torch.allclose((at(q, 17) * at(k, 5)).sum(), (at(q, 112) * at(k, 100)).sum())
    assert torch.equal(at(q, 9)[:, 8:], q[:, 8:])
    unit = torch.zeros(1, 8, dtype=torch.float64)
    unit[0, 1] = 1.0
    turned = plain.rotate(unit, torch.tensor([3]), turns, 2.0)[0]
    angle = 3 * 100.0 ** -0.25
    assert turned[1] == pytest.approx(2 * math.cos(angle)) and turned[5] == pytest.approx(2 * math.sin(angle)) and turned.count_nonzero() == 2


def test_scaled_frequencies_keep_the_fast_pairs_and_divide_the_slow_ones():
    turns, _ = plain.frequencies(10000.0, 64)
    scaled, _ = plain.frequencies(10000.0, 64, {"factor": 16.0, "original": 2048, "fast": 32.0, "slow": 1.0})
    ratio = [s / t for s, t in zip(scaled, turns)]
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(1 / 16) and all(a >= b for a, b in zip(ratio, ratio[1:]))


def test_plain_attention_against_a_dense_softmax():
    g = torch.Generator().manual_seed(1)
    q, k, v = torch.randn(9, 4, 5, generator=g).double(), torch.randn(9, 2, 5, generator=g).double(), torch.randn(9, 2, 3, generator=g).double()
    sink = torch.tensor([0.3, -50.0, 2.0, 60.0]).double()
    out = plain.attention(q, k, v, 0.5, 3, sink)
    for p in range(9):
        seen = [j for j in range(9) if 0 <= p - j < 3]
        for h in range(4):
            w = torch.softmax(torch.cat([k[seen, h // 2] @ q[p, h] * 0.5, sink[h:h + 1]]), 0)[:-1]
            assert torch.allclose(out[p, h], w @ v[seen, h // 2])


def test_plain_convolution_is_causal_and_starts_from_nothing():
    u = torch.tensor([[1.0], [10.0], [100.0], [1000.0]]).double()
    assert plain.short_conv(u, torch.tensor([[3.0, 2.0, 1.0]]).double())[:, 0].tolist() == [1.0, 12.0, 123.0, 1230.0]
    assert torch.equal(plain.short_conv(u, torch.tensor([[2.0]]).double()), 2 * u)


def test_plain_residual_of_a_layer_without_a_feed_forward():
    config = make_config([windowed_layer(2, 1, 8, 4, 3, 5)], vocab=19, width=16, mult=0.25)
    weights = random_weights(sandwich_lm.parameter_shapes(parse(config)), 3)
    model, layers, tokens = plain.PlainSandwich(config, weights), [], prompt(1, 7, 19)
    logits = model(tokens, layers)
    x = model.w["embed"][tokens]
    y = model.windowed("l0.mix.", config["layers"][0]["mixer"], plain.layer_norm(x, model.w["l0.norm1"], 1e-4))
    added = layers[0] - x
    assert torch.allclose(added, 0.25 * plain.layer_norm(y, model.w["l0.norm1b"], 1e-4))
    assert float(logits.abs().max()) < 8.0


def test_a_latent_layer_without_turns_or_sinks_is_ordinary_attention():
    config = make_config([latent_layer(2, 4, 2, 3, 6, 5)], vocab=19, width=16)
    weights = random_weights(sandwich_lm.parameter_shapes(parse(config)), 4)
    model, m = plain.PlainSandwich(config, weights), config["layers"][0]["mixer"]
    h = torch.randn(1, 16, generator=torch.Generator().manual_seed(2)).double()      # one token sees itself alone
    w = lambda n: model.w["l0.mix." + n]
    c = plain.rms_norm(h @ w("dkv")[:5].T, w("dkv.norm"), 1e-4)
    want = (c @ w("uv").T * plain.sigmoid(h @ w("g").T)) @ w("o").T
    assert torch.allclose(model.latent("l0.mix.", m, h, False), want)
