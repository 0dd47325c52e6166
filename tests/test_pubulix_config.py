"""Pubulix on the CPU: its config.json reader, the tensors it asks for, which caches its layers keep,
and properties of the plain implementation's own mechanisms that the tests on the GPU lean on."""
import copy

import pytest
import torch

import plain_pubulix as plain
import tiny_pubulix as tiny
from vosti_b200.config import ConfigError, model_spec_from_config, model_spec_from_dir
from vosti_b200.models import build_model, expected_weights
from vosti_b200.weights import check_tensors, draw_tensors
from vosti_b200.weights.loader import WeightError


def test_spec_kinds_sizes_and_names(tmp_path):
    spec = model_spec_from_config(tiny.A)
    assert spec.architecture == "Pubulix" and spec.hidden_size == 72 and spec.vocab_size == 211 and not spec.tie_word_embeddings
    assert spec.embedding["scale"] == 2.5 and spec.embedding["publish_ids"] and spec.head["softcap"] == 9.0
    assert all(layer.arrangement == "gated_pre_norm_stream" and layer.residual_scale == 0.7 and layer.input_conv == 3 and layer.norm["scalar"]
               for layer in spec.layers)
    assert [layer.mixer.kind for layer in spec.layers] == ["latent_attention", "sink_attention", "latent_attention", "sink_attention",
                                                           "latent_attention", "latent_attention"]
    assert [entry.cache_from for entry in spec.run_order] == [None, None, 0, None, 0, None]
    first, second, third = (layer.mixer for layer in spec.layers[:3])
    assert first["sink"] and first["out_gate"] and not first["gate"] and first["own_latent"] and first["window"] == 11
    assert first["position"]["interleaved"] and first["position"]["rotary_dim"] == 6
    assert not third["own_latent"] and third["window"] == 29
    assert second["softcap"] == 4.0 and second["window"] == 7 and not second["position"]["interleaved"] and second["position"]["rotary_dim"] == 8
    ff = spec.layers[1].feed_forward
    assert (ff.kind, ff["route"], ff["experts"], ff["top"], ff["intermediate_size"], ff["limit"], ff["activation"]) == \
        ("moe", "table", 7, 3, 24, 0.9, "clamped")
    assert spec.layers[3].feed_forward is None
    names = expected_weights(spec)
    for name, shape in {"embed": (211, 72), "head": (211, 72), "final.norm": (), "l0.norm1": (), "l0.norm2": (), "l0.canon1": (72, 3),
                        "l0.rg1": (72, 72), "l0.rg1.b": (72,), "l0.rg2": (72, 72), "l0.rg2.b": (72,),
                        "l0.mix.q": (3 * 16, 72), "l0.mix.dkv": (26, 72), "l0.mix.dkv.norm": (20,), "l0.mix.uk": (30, 20), "l0.mix.uv": (42, 20),
                        "l0.mix.sink": (3,), "l0.mix.g": (42, 72), "l0.mix.o": (72, 42), "l0.mlp.table": (211, 2), "l0.mlp.e4.gate": (20, 72),
                        "l0.mlp.e4.up": (20, 72), "l0.mlp.e4.down": (72, 20), "l1.mix.q": (96, 72), "l1.mix.k": (48, 72), "l1.mix.v": (32, 72),
                        "l1.mix.o": (72, 64), "l1.mlp.table": (211, 3), "l2.mix.uk": (48, 20), "l2.mix.g": (40, 72)}.items():
        assert tuple(names[name].shape) == shape, name
    for absent in ("l2.mix.dkv", "l2.mix.dkv.norm", "l1.mix.sink", "l1.mix.g", "l0.mlp.router", "l0.mlp.e5.up", "l3.mlp.table", "l1.mix.q.b"):
        assert absent not in names, absent
    assert sorted(n for n, w in names.items() if w.optional) == ["l3.norm2", "l3.rg2", "l3.rg2.b"]
    assert names["l0.mlp.table"].integer
    folder = tiny.write_model(tmp_path / "m", tiny.A, 3)
    assert model_spec_from_dir(folder) == spec


def test_layers_that_read_anothers_latents_keep_state_but_no_pages_and_widen_its_window():
    caches, states = build_model(model_spec_from_config(tiny.A)).cache_specs()
    assert [None if c is None else c.window for c in caches] == [29, 7, None, 40, None, 23]      # layer 0: the widest of 11, 29 and 5
    assert caches[0].widths == (20, 6) and caches[5].widths == (33, 10)
    assert all(s is not None and s.shape == (2 * 72,) for s in states)
    no_window = copy.deepcopy(tiny.A)
    del no_window["layers"][4]["mixer"]["mask"]
    assert build_model(model_spec_from_config(no_window)).cache_specs()[0][0].window == 0        # a reader of everything


def test_optional_blocks_and_defaults():
    config = copy.deepcopy(tiny.A)
    del config["embedding"], config["logit_softcap"]
    del config["layers"][1]["mixer"]["softcap"], config["layers"][1]["mixer"]["mask"], config["layers"][0]["mixer"]["rot"]["dims"]
    config["layers"][3].pop("mlp")
    spec = model_spec_from_config(config)
    assert spec.embedding["scale"] == 1.0 and spec.head["softcap"] == 0.0
    assert spec.layers[1].mixer["softcap"] == 0.0 and spec.layers[1].mixer["window"] == 0 and spec.layers[3].feed_forward is None


def test_checkpoints_with_and_without_unused_tensors_load():
    for unused in (True, False):
        spec, tensors = tiny.tensors_for(tiny.A, 5, unused)
        check_tensors(tensors, expected_weights(spec))
    spec, tensors = tiny.tensors_for(tiny.A, 5)
    del tensors["l0.mlp.table"], tensors["l1.canon1"]
    with pytest.raises(WeightError) as error:
        check_tensors(tensors, expected_weights(spec))
    assert error.value.missing == ["l0.mlp.table", "l1.canon1"]


def test_random_tables_hold_distinct_experts():
    spec = model_spec_from_config(tiny.A)
    table = draw_tensors(expected_weights(spec), 4)["l1.mlp.table"]
    assert table.dtype == torch.int32 and tuple(table.shape) == (211, 3) and int(table.min()) >= 0 and int(table.max()) < 7
    ordered = table.sort(dim=1).values
    assert not (ordered[:, 1:] == ordered[:, :-1]).any()
    assert len(table.unique()) == 7


def test_config_errors_name_the_key():
    for path, message in ((("norm",), "norm"), (("canon", "taps"), "taps"), (("residual_mult",), "residual_mult"), (("vocab",), "vocab"),
                          (("layers", 0, "mixer", "kv_rank"), "kv_rank"), (("layers", 0, "mixer", "rot", "base"), "base"),
                          (("layers", 1, "mixer", "rot", "dims"), "dims"), (("layers", 1, "mixer", "kv_heads"), "kv_heads"),
                          (("layers", 0, "mlp", "expert", "limit"), "limit"), (("layers", 0, "mlp", "router", "top"), "top"),
                          (("layers", 0, "mlp", "kind"), "kind"), (("layers", 1, "mixer", "scale"), "scale"), (("layers", 2, "type"), "type")):
        config = copy.deepcopy(tiny.A)
        block = config
        for key in path[:-1]:
            block = block[key]
        del block[path[-1]]
        with pytest.raises(ConfigError, match=message):
            model_spec_from_config(config)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][2].update(type="attention_3"), "attention_3"),
    (lambda c: c["layers"][1].update(mlp=dict(kind="dense", ff=8)), "dense"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),              # not a latent layer
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "kv_from"),              # it keeps none itself
    (lambda c: c["layers"][2]["mixer"].update(kv_from=5), "kv_from"),              # a later layer
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=16), "differ"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(base=7.0), "differ"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4), "dims"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0), "limit"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].update(mask=dict(size=0)), "size"),
    (lambda c: c.update(layers=[]), "layers")])
def test_unusable_values_are_refused(change, message):
    config = copy.deepcopy(tiny.A)
    change(config)
    with pytest.raises(ConfigError, match=message):
        model_spec_from_config(config)


def test_plain_mechanisms():
    gen = torch.Generator().manual_seed(1)
    h = torch.randn(6, 3, generator=gen, dtype=torch.float64)
    w = torch.randn(3, 4, generator=gen, dtype=torch.float64)
    conv = plain.causal_convolution(h, w)
    want = sum(w[1, j] * h[5 - 3 + j, 1] for j in range(4))
    assert torch.allclose(conv[5, 1], want) and torch.allclose(conv[0], w[:, 3] * h[0])
    assert torch.allclose(conv[1], w[:, 2] * h[0] + w[:, 3] * h[1])
    x = torch.randn(5, 8, generator=gen, dtype=torch.float64)
    for neighbours in (True, False):
        turned = plain.rotate(x, torch.arange(5), 100.0, 6, neighbours)
        assert torch.equal(turned[0], x[0]) and torch.equal(turned[:, 6:], x[:, 6:])
        assert torch.allclose(turned.norm(dim=1), x.norm(dim=1))
        # the product of a query and a key depends on their distance alone
        far = plain.rotate(x, torch.arange(5) + 40, 100.0, 6, neighbours)
        assert torch.allclose(turned @ turned.T, far @ far.T)
    assert plain.visible(5, 2).long().sum(dim=1).tolist() == [1, 2, 2, 2, 2]
    scores = torch.tensor([[1.0, 2.0]], dtype=torch.float64)
    p = plain.softmax_with_sink(scores, torch.ones(1, 2, dtype=torch.bool), 3.0)
    e = torch.exp(torch.tensor([1.0, 2.0, 3.0], dtype=torch.float64))
    assert torch.allclose(p[0], e[:2] / e.sum())
    one = torch.ones(1, 1, dtype=torch.float64)
    y = plain.clamped_expert(one, 5.0 * one, -7.0 * one, one, 2.0)
    assert torch.allclose(y, 2.0 * torch.sigmoid(torch.tensor(3.404, dtype=torch.float64)) * (-2.0 + 1.0) * one)
    low = plain.clamped_expert(one, -5.0 * one, 0.5 * one, one, 2.0)                # the gate has no lower clamp
    assert torch.allclose(low, -5.0 * torch.sigmoid(torch.tensor(-8.51, dtype=torch.float64)) * 1.5 * one)


def test_every_mechanism_matters_in_the_small_configurations():
    """Leaving a mechanism out of the plain implementation moves the logits of configuration A by far more
    than any tolerance of the tests, so that an engine without it cannot pass."""
    _, W = tiny.tensors_for(tiny.A, 51)
    tokens = torch.randint(0, 211, (60,), generator=torch.Generator().manual_seed(2)).tolist()
    want = plain.forward(tiny.A, W, tokens)
    size = want.pow(2).mean().sqrt()

    def moved(config=tiny.A, weights=W):
        return float((plain.forward(config, weights, tokens) - want).pow(2).mean().sqrt() / size)

    def changed(fn):
        config = copy.deepcopy(tiny.A)
        fn(config)
        return config

    without = lambda *names: {k: (torch.zeros_like(v) if k in names else v) for k, v in W.items()}
    assert moved(weights=without("l0.canon1", "l1.canon1")) > 0.02
    assert moved(weights={k: (v - 50.0 if k.endswith(".sink") else v) for k, v in W.items()}) > 0.01
    assert moved(weights=without("l2.rg1", "l2.rg1.b")) > 0.01
    assert moved(weights=without("l0.mix.g")) > 0.01
    assert moved(changed(lambda c: c["layers"][0]["mixer"]["mask"].update(size=12))) > 0.003
    assert moved(changed(lambda c: c["layers"][2]["mixer"]["mask"].update(size=28))) > 0.003
    assert moved(changed(lambda c: c["layers"][1]["mixer"].update(softcap=8.0))) > 0.003
    assert moved(changed(lambda c: c["layers"][0]["mlp"]["expert"].update(limit=3.0))) > 0.003
    assert moved(changed(lambda c: c.update(residual_mult=0.8))) > 0.01
