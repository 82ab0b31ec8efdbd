"""Host side of the decoder that norms its sublayers' outputs, without a GPU: configuration, weights, cache, packed key ranges, and the
plain functions that the GPU tests compare with."""

import json
import math

import pytest
import torch

import plain_postnorm as plain
import vllm_rlt_b200 as rlt
from hybrid_cases import prompt, write_model
from postnorm_cases import CONFIGS, attention_layer, delta_layer, make_config, rank_of, random_weights, retention_layer
from vllm_rlt_b200 import postnorm_lm, registry
from vllm_rlt_b200.engine import KeyRanges


def parse(config):
    return rlt.PostNormLMConfig.from_json(config)


def build(name):
    config = parse(CONFIGS[name])
    weights = random_weights(postnorm_lm.parameter_shapes(config, rank_of(name)), 0)
    return rlt.PostNormLM(config, weights, "cpu"), weights


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configurations_parse_and_every_tensor_finds_its_place(name):
    model, weights = build(name)
    used = {"embed", "head", "final.norm"}
    for i, entry in enumerate(CONFIGS[name]["layers"]):
        layer, p = model.layers[i], f"l{entry.get('weights_of', i)}."
        assert layer is model.layers[entry.get("weights_of", i)]
        mixer, w = layer.mixer, lambda n: weights[f"{p}mix.{n}"]
        rows = lambda at, n: mixer.w_in[at:at + w(n).shape[0]]
        if entry["type"] == "channel_delta":
            for at, n in zip((*mixer.columns, mixer.b_col, mixer.a_col, mixer.g_col), ("q", "k", "v", "b", "a1", "g1")):
                assert torch.equal(rows(at, n), w(n)) and at % 8 == 0
            for at, n in zip(mixer.columns, "qkv"):
                assert torch.equal(mixer.conv[at:at + w(n).shape[0]], w(n + ".conv").float())
            assert mixer.ranks == tuple(rank_of(name)(n) for n in ("a1", "g1"))
            assert torch.equal(mixer.norm.view(-1, w("norm").numel()), w("norm").float().expand(entry["mixer"]["heads"], -1))
        elif entry["type"] == "retention":
            keys = w("q").shape[0]
            assert torch.equal(rows(0, "q"), w("q")) and torch.equal(mixer.w_in[keys:2 * keys], w("k"))
            assert torch.equal(rows(mixer.v_col, "v"), w("v")) and torch.equal(rows(mixer.g_col, "g"), w("g"))
        else:
            assert all(torch.equal(rows(at, n), w(n)) for at, n in zip(mixer.columns, "qkv"))
            assert torch.equal(mixer.terms.head_scale, w("temp").float()) and mixer.terms.keep_first == entry["mixer"]["mask"]["keep_first"]
        mlp = entry["mlp"]
        assert (layer.ff is None) == (not mlp)
        if mlp and mlp["kind"] == "moe":
            assert torch.equal(layer.ff.w_gate_up[1, 0::2], weights[p + "mlp.e1.gate"]) and torch.equal(layer.ff.w_gate_up[1, 1::2], weights[p + "mlp.e1.up"])
            assert (layer.ff.shared is not None) == bool(mlp.get("shared")) and layer.ff.bias.dtype == torch.float32
        used.update(n for n in weights if n.startswith(p))
    assert used == set(weights)


def test_layers_that_share_weights_have_pages_and_state_of_their_own():
    model, _ = build("mixed")
    spec = model.cache_spec()
    assert spec.layers == {0: rlt.KVSpec(2, 24, 40), 4: rlt.KVSpec(6, 64, 32), 6: rlt.KVSpec(2, 24, 40)}
    shapes = {k: v.shape for k, v in spec.states.items()}
    assert shapes == {"l1.conv": (3, 384), "l1.state": (6, 24, 40), "l2.state": (3, 40, 24), "l3.conv": (2, 768), "l3.state": (4, 64, 64),
                      "l5.conv": (3, 384), "l5.state": (6, 24, 40)}
    assert all(spec.states[n].dtype == (torch.float32 if n.endswith("state") else None) for n in shapes)
    odd = build("odd")[0].cache_spec()
    assert odd.states["l0.conv"].shape == (5, 16 + 16 + 24) and odd.states["l4.conv"].shape == (0, 8 + 8 + 16)     # projections start at multiples of 8
    rlt.SequenceCache(odd, max_tokens=100, max_sequences=2, block=odd.block, device="cpu")


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0]["mixer"].update(sink=True), "unknown config keys"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(chunk=4), "unknown config keys"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "lacks"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "lacks"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 1.5, 0.1]), "decay"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(limit=1.0), "unknown config keys"),
    (lambda c: c["layers"][0].update(type="lightning"), "unknown mixer type"),
    (lambda c: c["layers"][5].update(weights_of=40), "weights_of"),
    (lambda c: c["layers"][5].update(weights_of=0), "differs"),
    (lambda c: (c["layers"][1].update(weights_of=5)), "circle"),
    (lambda c: c["norm"].update(offset=1), "unknown config keys"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c.update(width=0), "width"),
])
def test_configurations_that_make_no_sense_are_refused(change, message):
    config = json.loads(json.dumps(CONFIGS["mixed"]))
    change(config)
    with pytest.raises(ValueError, match=message):
        parse(config)


def test_weights_may_come_from_a_layer_that_borrows_them_too_and_from_a_later_one():
    layers = [delta_layer(2, 2, 8, 8, 3), attention_layer(2, 1, 8, 8, 4, 1)]
    config = parse(make_config([{**layers[1], "weights_of": 2}, layers[0], layers[1], {**layers[0], "weights_of": 4}, {**layers[0], "weights_of": 1}], vocab=11, width=16))
    assert [layer.weights for layer in config.layers] == [2, 1, 2, 1, 1] and config.own == [1, 2]
    shapes = postnorm_lm.parameter_shapes(config, lambda name: 5)
    assert {n.split(".")[0] for n in shapes} == {"embed", "head", "final", "l1", "l2"} and shapes["l1.mix.a2"] == (16, 5)


def test_the_registry_loads_a_folder(tmp_path):
    _, weights = build("odd")
    write_model(tmp_path, CONFIGS["odd"], weights)
    model = rlt.load_model(tmp_path, device="cpu", dtype=torch.float32)
    assert registry.resolve(CONFIGS["odd"]).model_class is rlt.PostNormLM and model.head.dtype == torch.float32
    for missing in ("l0.mix.k.conv", "l0.mix.a1", "head"):
        rest = {n: t for n, t in weights.items() if n != missing}
        with pytest.raises(ValueError, match="lacks"):
            rlt.PostNormLM(parse(CONFIGS["odd"]), rest, "cpu")
    with pytest.raises(ValueError, match="shape"):
        rlt.PostNormLM(parse(CONFIGS["odd"]), weights | {"l0.mix.a2": weights["l0.mix.a2"][:, :1]}, "cpu")


@pytest.mark.parametrize("window,keep", [(10, 4), (10, 40), (1, 0), (300, 3)])
def test_packed_ranges_hold_the_kept_positions_and_those_of_the_window(window, keep):
    portions, rows = [(0, 20), (5, 300), (100, 130), (7, 1)], 128
    ranges = KeyRanges.of(portions, window, torch.device("cpu"), keep, rows)
    first, cu = ranges.first.tolist(), ranges.cu.tolist()
    position = lambda s, row: row if row < min(keep, first[s]) else first[s] + row - min(keep, first[s])
    for s, (start, n) in enumerate(portions):
        packed = [position(s, r) for r in range(cu[s + 1] - cu[s])]
        seen = {j for p in range(start, start + n) for j in range(p + 1) if p - j < window or j < keep}
        assert packed == sorted(set(packed)) and seen <= set(packed) <= set(range(start + n))
    assert cu[-1] == ranges.rows and ranges.keep == keep
    covered = []
    for q_row, count, start, key_row, key_first, kept, *_ in ranges.tiles.tolist():
        s = max(i for i in range(4) if sum(n for _, n in portions[:i]) <= q_row)
        assert count <= rows and key_first == first[s] and kept == min(keep, first[s]) and key_row == cu[s] + kept
        assert start - portions[s][0] == q_row - sum(n for _, n in portions[:s])
        covered += range(q_row, q_row + count)
    assert sorted(covered) == list(range(sum(n for _, n in portions)))


# ---- the plain functions themselves --------------------------------------------------------------
def generator(seed=0):
    return torch.Generator().manual_seed(seed)


def test_plain_delta_rule_overwrites_what_a_key_holds():
    """With a unit key, full strength and no decay, a second write replaces the first and the token reads its own write."""
    k = plain.unit_vector(torch.randn(1, 1, 4, generator=generator()).double()).expand(2, 1, 4)
    v = torch.tensor([[[1.0, 2.0]], [[5.0, -1.0]]]).double()
    out, state = plain.delta_rule(k, k, v, torch.zeros(2, 1, 4).double(), torch.ones(2, 1).double())
    assert torch.allclose(out, v, atol=1e-5) and torch.allclose(torch.einsum("de,d->e", state[0], k[0, 0]), v[1, 0], atol=1e-5)


def test_plain_delta_rule_decays_key_channels():
    q, k = torch.tensor([[[1.0, 1.0]], [[1.0, 1.0]]]).double(), torch.tensor([[[1.0, 0.0]], [[0.0, 0.0]]]).double()
    v, log_decay = torch.tensor([[[3.0]], [[0.0]]]).double(), torch.tensor([[[0.0, 0.0]], [[math.log(0.25), 0.0]]]).double()
    out, _ = plain.delta_rule(q, k, v, log_decay, torch.ones(2, 1).double())
    assert out[:, 0, 0].tolist() == pytest.approx([3.0, 0.75])


def test_plain_retention_is_a_decayed_sum():
    q, k, v = (torch.randn(6, 2, 3, generator=generator(i)).double() for i in range(3))
    decay = torch.tensor([0.5, 1.0]).double()
    out = plain.retention(q, k, v, decay)
    for t in range(6):
        for h in range(2):
            assert torch.allclose(out[t, h], sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1)))


def test_plain_talking_attention_against_dense_weights():
    q, k, v = torch.randn(9, 4, 5, generator=generator(1)).double(), torch.randn(9, 2, 5, generator=generator(2)).double(), torch.randn(9, 2, 3, generator=generator(3)).double()
    talk, temp = torch.randn(4, 4, generator=generator(4)).double(), torch.tensor([1.0, 0.5, 2.0, -1.0]).double()
    out = plain.talking_attention(q, k, v, 0.7, temp, 3.0, 3, 2, talk)
    for p in range(9):
        seen = [j for j in range(p + 1) if p - j < 3 or j < 2]
        weights = torch.stack([torch.softmax(3.0 * torch.tanh(k[seen, h // 2] @ q[p, h] * 0.7 * temp[h] / 3.0), 0) for h in range(4)])
        for h in range(4):
            assert torch.allclose(out[p, h], (talk[h] @ weights) @ v[seen, h // 2])


def test_mixing_outputs_is_mixing_weights():
    """What the kernels do: every head over the values of every key/value head, mixed afterwards."""
    weights, v, talk = torch.softmax(torch.randn(6, 7, generator=generator(1)).double(), 1), torch.randn(7, 2, 3, generator=generator(2)).double(), torch.randn(6, 6, generator=generator(3)).double()
    spread = torch.einsum("gt,tce->gce", weights, v)
    for h in range(6):
        assert torch.allclose(torch.einsum("g,ge->e", talk[h], spread[:, h // 3]), (talk[h] @ weights) @ v[:, h // 3])


def test_plain_experts_weigh_the_chosen_logits_alone():
    h, router, bias = torch.randn(3, 4, generator=generator(1)).double(), torch.randn(5, 4, generator=generator(2)).double(), torch.tensor([0.0, 9.0, 0.0, 0.0, -9.0]).double()
    out = plain.experts(h, router, bias, 2, lambda e, rows: torch.full_like(rows, float(e)))
    z = h @ router.T + bias
    for i in range(3):
        best, chosen = z[i].topk(2)
        assert float(out[i, 0]) == pytest.approx(float((torch.softmax(best, 0) * chosen).sum())) and 1 in chosen


def test_plain_rotations_turn_neighbours_or_halves():
    x = torch.zeros(1, 1, 8, dtype=torch.float64)
    x[0, 0, 1] = 1.0
    angle = lambda i, p: p * 100.0 ** (-2 * i / 6)
    pairs = plain.rotate(x, torch.tensor([3]), 100.0, 6, False)[0, 0]
    halves = plain.rotate(x, torch.tensor([3]), 100.0, 6, True)[0, 0]
    assert pairs[:2].tolist() == pytest.approx([-math.sin(angle(0, 3)), math.cos(angle(0, 3))]) and pairs.count_nonzero() == 2
    assert halves[[1, 4]].tolist() == pytest.approx([math.cos(angle(1, 3)), math.sin(angle(1, 3))]) and halves.count_nonzero() == 2


def test_plain_sublayers_read_the_residual_and_norms_stand_behind_them():
    config = make_config([retention_layer(2, 4, 6, mlp={"kind": "dense", "ff": 9})], vocab=19, width=16)
    parsed = parse(config)
    weights = random_weights(postnorm_lm.parameter_shapes(parsed, lambda name: 3), 3)
    model, layers, tokens = plain.PlainPostNorm(config, weights), [], prompt(1, 7, 19)
    logits = model(tokens, layers)
    x = model.w["embed"][tokens]
    x = x + plain.rms_norm(model.retention("l0.mix.", config["layers"][0]["mixer"], x), 1e-4, model.w["l0.norm1"])
    x = x + plain.rms_norm(plain.gated_unit(x, *(model.w[f"l0.mlp.{n}"] for n in ("gate", "up", "down"))), 1e-4, model.w["l0.norm2"])
    assert torch.allclose(layers[0], x) and torch.allclose(logits, plain.rms_norm(x, 1e-4, model.w["final.norm"]) @ model.w["head"].T)
