"""Difavik on the CPU: its config.json reader, the tensors it asks for, layers that share tensors, which pages a
window with kept first tokens gives back, how a step is cut into chunks, and properties of the plain mechanisms."""
import copy

import pytest
import torch

import plain_difavik as plain
import tiny_difavik as tiny
from vosti_b200 import ops
from vosti_b200.cache import CacheManager
from vosti_b200.config import ConfigError, model_spec_from_config, model_spec_from_dir
from vosti_b200.models import build_model, expected_weights
from vosti_b200.parts import PagedCacheSpec
from vosti_b200.weights import check_tensors
from vosti_b200.weights.loader import WeightError


def test_spec_kinds_sizes_and_names(tmp_path):
    spec = model_spec_from_config(tiny.A)
    assert spec.architecture == "Difavik" and spec.hidden_size == 72 and spec.vocab_size == 197 and spec.tie_word_embeddings
    assert (spec.embedding.kind, spec.embedding["buckets"], spec.embedding["mul_prev"], spec.embedding["mul_cur"]) == ("pair_hash", 31, 5, 17)
    assert [layer.number for layer in spec.layers] == [0, 1, 3, 5]
    assert [(entry.layer, entry.instance) for entry in spec.run_order] == [(0, 0), (1, 0), (0, 1), (2, 0), (0, 2), (3, 0)]
    assert all(layer.arrangement == "out_norm_stream" and layer.layer_scale and layer.norm["unit_offset"] for layer in spec.layers)
    (_, attention), (_, retention) = spec.layers[0].mixer["branches"]
    assert (attention["window"], attention["keep_first"], attention["value_is_key"], attention["head_gate"]) == (13, 11, True, True)
    assert retention["decay"] == (0.9, 0.97, 0.6) and retention["key_scale"] == 10 ** -0.5 and retention["out_norm"] == "head"
    light = spec.layers[1].mixer
    assert (light.kind, light["activation"], light["out_norm"], light["gate_activation"]) == ("decay_attention", "silu", "all", "sigmoid")
    ff = spec.layers[0].feed_forward
    assert (ff["route"], ff["experts"], ff["top"], ff["limit"], ff["activation"]) == ("softmax", 5, 2, 0.9, "clamped")
    assert spec.layers[2].feed_forward is None and spec.layers[1].feed_forward["bias"]
    names = expected_weights(spec)
    for name, shape in {"embed": (197, 72), "bigram": (32, 72), "final.norm": (72,), "l0.norm1": (72,), "l0.ls2": (72,),
                        "l0.mix.left.q": (84, 72), "l0.mix.left.q.b": (84,), "l0.mix.left.k": (42, 72), "l0.mix.left.k.b": (42,),
                        "l0.mix.left.q.norm": (84,), "l0.mix.left.k.norm": (42,), "l0.mix.left.g": (6, 72), "l0.mix.left.o": (72, 84),
                        "l0.mix.left.out": (72,), "l0.mix.right.q": (30, 72), "l0.mix.right.v": (21, 72), "l0.mix.right.o": (72, 21),
                        "l0.mix.right.out": (72,), "l1.mix.norm": (33,), "l1.mix.g": (33, 72), "l1.mlp.gate.b": (52,), "l1.mlp.down.b": (72,),
                        "l0.mlp.router": (5, 72), "l5.mlp.e5.down": (72, 28), "l3.mix.right.k": (12, 72)}.items():
        assert tuple(names[name].shape) == shape, name
    for absent in ("head", "l0.mix.left.v", "l0.mix.right.norm", "l0.mix.right.q.b", "l2.norm1", "l4.norm1", "l3.mlp.router", "l1.mix.left.q"):
        assert absent not in names, absent
    assert sorted(n for n, w in names.items() if w.optional) == ["l3.ls2", "l3.norm2"]
    folder = tiny.write_model(tmp_path / "m", tiny.A, 3)
    assert model_spec_from_dir(folder) == spec


def test_runs_of_a_shared_layer_keep_caches_and_states_of_their_own():
    model = build_model(model_spec_from_config(tiny.A))
    caches, states = model.cache_specs()
    reach = [None if c is None else (c.window, c.keep_first) for c in caches]
    assert reach.count((13, 11)) == 3 and reach.count((37, 3)) == 1
    assert sum(s is not None for s in states) == 7          # six layer runs and the embedding's last token
    indices = [model.cache_index[(e.layer, e.instance)] for e in model.spec.run_order]
    assert len(set(indices)) == 6


def test_optional_blocks_and_defaults():
    config = copy.deepcopy(tiny.A)
    del config["embedding"]
    for i in (0, 2, 4):
        del config["layers"][i]["mixer"]["left"]["mask"]["keep_first"]
    del config["layers"][3]["mixer"]["left"]["mask"], config["layers"][3]["mlp"]
    spec = model_spec_from_config(config)
    assert spec.embedding.kind == "table"
    left = [dict(layer.mixer["branches"])["left"] for layer in spec.layers if layer.mixer.kind == "branches"]
    assert [(m["window"], m["keep_first"]) for m in left] == [(13, 0), (0, 0)]


def test_checkpoints_with_and_without_unused_tensors_load():
    for unused in (True, False):
        spec, tensors = tiny.tensors_for(tiny.A, 5, unused)
        check_tensors(tensors, expected_weights(spec))
    spec, tensors = tiny.tensors_for(tiny.A, 5)
    del tensors["l0.mix.left.q.norm"], tensors["bigram"]
    with pytest.raises(WeightError) as error:
        check_tensors(tensors, expected_weights(spec))
    assert error.value.missing == ["bigram", "l0.mix.left.q.norm"]


def test_config_errors_name_the_key():
    for path in (("norm", "eps"), ("vocab",), ("embedding", "bigram", "buckets"), ("embedding", "bigram", "mul_cur"), ("layers", 0, "type"),
                 ("layers", 1, "mixer", "decay"), ("layers", 1, "mixer", "vdim"), ("layers", 1, "mlp", "limit"), ("layers", 1, "mlp", "ff"),
                 ("layers", 3, "mixer", "left", "scale"), ("layers", 3, "mixer", "left", "mask", "size"), ("layers", 3, "mixer", "right", "rot"),
                 ("layers", 5, "mlp", "router", "top"), ("layers", 5, "mlp", "expert", "limit"), ("layers", 5, "mlp", "kind")):
        config = copy.deepcopy(tiny.A)
        config["layers"] = [dict(e) for e in config["layers"] if "weights_of" not in e]
        where = list(path)
        if where[0] == "layers":
            where[1] = {0: 0, 1: 1, 3: 2, 5: 3}[where[1]]
        block = config
        for key in where[:-1]:
            block = block[key]
        del block[where[-1]]
        with pytest.raises(ConfigError, match=str(path[-1])):
            model_spec_from_config(config)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][1].update(type="lightning_2"), "lightning_2"),
    (lambda c: c["layers"][5]["mlp"].update(kind="mixture"), "mixture"),
    (lambda c: c["layers"][3]["mixer"]["left"].update(vdim=11), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.9, 0.9]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.9, 0.9, 1.5]), "decay"),
    (lambda c: c["layers"][1]["mlp"].update(limit=0), "limit"),
    (lambda c: c["layers"][5]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][2].update(weights_of=2), "weights_of"),
    (lambda c: c["layers"][2].update(weights_of=4), "weights_of"),                 # a circle: layer 4 names layer 2
    (lambda c: c["layers"][2].update(weights_of=9), "weights_of"),
    (lambda c: c["layers"][2].update(weights_of=1), "differs"),
    (lambda c: c.update(layers=[]), "layers")])
def test_unusable_values_are_refused(change, message):
    config = copy.deepcopy(tiny.A)
    change(config)
    with pytest.raises(ConfigError, match=message):
        model_spec_from_config(config)


def test_a_window_that_keeps_first_tokens_gives_back_the_pages_between():
    spec = PagedCacheSpec(entries=2, heads=1, width=8, window=10, keep_first=5)
    manager = CacheManager([spec, PagedCacheSpec(entries=2, heads=1, width=8, window=10)], [None, None], num_pages=12, page_size=4, max_requests=1)
    assert [(g.window, g.keep_first) for g in manager.groups] == [(10, 5), (10, 0)]
    manager.begin("r")
    for length in range(1, 41):
        manager.extend("r", 1)
        manager.trim("r")
        held = [[i for i, page in enumerate(manager.block_row("r", g)) if page >= 0] for g in (0, 1)]
        # the next query, at position `length`, reads keys > length - 10 and, in the first group, keys < 5
        window = set(range(max(0, length - 9) // 4, (length - 1) // 4 + 1))
        assert set(held[1]) == window
        assert set(held[0]) == window | {i for i in (0, 1) if i * 4 < length}
    manager.check()
    manager.finish("r")
    assert manager.available_pages() == 12


def test_a_step_is_cut_into_chunks_of_long_requests():
    arrays, host = ops.decay_step_layout([1, 300, 16, 17])
    assert arrays == {"chunk_request": [1, 1, 1, 3], "chunk_first": [0, 128, 256, 0], "long_requests": [1, 3], "long_chunk0": [0, 3]}
    assert host == {"chunks": 4, "longs": 2, "shorts": 2}
    assert ops.decay_step_layout([1, 1]) == ({}, {"chunks": 0, "longs": 0, "shorts": 2})


def test_plain_mechanisms():
    gen = torch.Generator().manual_seed(1)
    x = torch.randn(5, 8, generator=gen, dtype=torch.float64)
    turned = plain.rotate_half(x, torch.arange(5), 100.0, 6)
    assert torch.equal(turned[0], x[0]) and torch.equal(turned[:, 6:], x[:, 6:]) and torch.allclose(turned.norm(dim=1), x.norm(dim=1))
    far = plain.rotate_half(x, torch.arange(5) + 40, 100.0, 6)
    assert torch.allclose(turned @ turned.T, far @ far.T)
    assert plain.window_keeping_first(6, 2, 1).long().tolist() == [[1, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0],
                                                                   [1, 0, 1, 1, 0, 0], [1, 0, 0, 1, 1, 0], [1, 0, 0, 0, 1, 1]]
    assert plain.slopes(4) == [0.25, 0.0625, 0.015625, 0.00390625]
    assert plain.pair_rows([3, 1, 4], 10, 2, 5) == [10, (6 + 5) % 10, (2 + 20) % 10]
    # the recurrence is a masked product with powers of the decay
    q, k, v = (torch.randn(7, n, generator=gen, dtype=torch.float64) for n in (4, 4, 3))
    i, j = torch.arange(7)[:, None], torch.arange(7)[None, :]
    weights = torch.where(i >= j, 0.8 ** (i - j).double(), torch.zeros((), dtype=torch.float64))
    assert torch.allclose(plain.fixed_decay_recurrence(q, k, v, 0.8), ((q @ k.T) * weights) @ v)
    one = torch.ones(1, dtype=torch.float64)
    assert torch.allclose(plain.clamped_gate(5 * one, -7 * one, 2.0), 2.0 * torch.sigmoid(3.404 * one) * (-2.0 + 1.0))
    assert torch.allclose(plain.clamped_gate(-5 * one, 0.5 * one, 2.0), -5.0 * torch.sigmoid(-8.51 * one) * 1.5)


def test_every_mechanism_matters_in_the_small_configurations():
    """Leaving a mechanism out of the plain implementation moves the logits of configuration A by far more than any
    tolerance of the tests, so that an engine without it cannot pass."""
    _, W = tiny.tensors_for(tiny.A, 61)
    tokens = torch.randint(0, 197, (60,), generator=torch.Generator().manual_seed(2)).tolist()
    want = plain.forward(tiny.A, W, tokens)
    size = want.pow(2).mean().sqrt()

    def moved(config=tiny.A, weights=W):
        return float((plain.forward(config, weights, tokens) - want).pow(2).mean().sqrt() / size)

    def changed(fn):
        config = copy.deepcopy(tiny.A)
        fn(config)
        return config

    without = lambda *names: {k: (torch.zeros_like(v) if k in names else v) for k, v in W.items()}
    every = lambda fn: changed(lambda c: [fn(c["layers"][i]["mixer"]) for i in (0, 2, 4)])
    assert moved(weights=without("bigram")) > 0.05
    assert moved(weights=without("l0.mix.left.g")) > 0.003
    assert moved(weights=without("l0.mix.left.q.b")) > 0.003
    assert moved(weights=without("l0.mix.left.k.b")) > 0.003
    assert moved(weights=without("l1.mlp.down.b")) > 0.003
    assert moved(weights=without("l1.mlp.up.b")) > 0.003
    assert moved(weights={k: (torch.ones_like(v) if k.endswith("ls1") else v) for k, v in W.items()}) > 0.05
    assert moved(every(lambda m: m["left"]["mask"].update(size=12))) > 0.002
    assert moved(every(lambda m: m["left"]["mask"].update(keep_first=10))) > 0.002
    assert moved(every(lambda m: m["right"].update(decay=[0.9, 0.97, 0.7]))) > 0.002
    assert moved(every(lambda m: m["right"]["rot"].update(dims=4))) > 0.002
    assert moved(changed(lambda c: c["layers"][1]["mlp"].update(limit=2.6))) > 0.002
