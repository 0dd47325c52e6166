"""The Difavik design, read from its own config.json.

A decoder over a float32 residual stream whose sublayers read the stream itself and are normed
and scaled as they join it (root-mean-square norms with a weight stored around zero, a learned
vector per sublayer),

    x <- x + ls1 * norm1(mixer(x));   x <- x + ls2 * norm2(ff(x))

Token rows have a second embedding added, chosen by the token and the one before it; the head is
the embedding table. A layer may have no tensors of its own and run an earlier layer's with a cache
and a state of its own (`weights_of`). Two kinds of layer, in any order:

  "parallel"   two mixers side by side, the mean of their normed outputs: grouped-query attention
               whose values are its keys before their norm (norms over the whole query and key
               projections, a penalty linear in the distance, a sliding window that keeps a
               sequence's first tokens, a sigmoid gate per head) and retention (a fixed decay per
               head, rotated queries and keys, unit heads, a SiLU gate);
  "lightning"  linear attention over SiLU'd projections with a fixed decay per head, one norm over
               the concatenated heads, a sigmoid gate.

Feed-forwards are gated with clamped inputs: dense with biases, or a mixture of experts weighted by
their shares of a softmax over all experts; or absent.

Keys (a missing one is an error unless marked optional; optional blocks may be absent or null):

    architecture  "Difavik"
    vocab, width
    norm.eps
    embedding.bigram                    optional: buckets, mul_prev, mul_cur
    layers[i].type                      "parallel" | "lightning"
    layers[i].weights_of                optional: the layer whose tensors this one uses
    layers[i].mixer (parallel)          left: heads, kv_heads, dim, vdim (equal to dim), scale,
                                              mask (optional): size, keep_first (optional, 0)
                                        right: heads, dim, vdim, rot.base, rot.dims, decay
    layers[i].mixer (lightning)         heads, dim, vdim, decay
    layers[i].mlp                       optional: {kind: "dense", ff, limit} |
                                        {kind: "moe", expert: {ff, limit}, router: {experts, top}}
"""
from __future__ import annotations

from typing import Any, Mapping, Optional, Tuple

from .schema import ConfigError, LayerSpec, ModelSpec, PartSpec, RunEntry

ARCHITECTURE = "Difavik"
MAX_POSITIONS = 1 << 30        # the design sets no limit (angles are formed from the position); the cache pool does
SIGMOID_SCALE = 1.702          # of the feed-forwards' gate activation g * sigmoid(1.702 g)
SLOPE_RANGE = 8.0              # head h of H takes distance * 2^(-8 (h + 1) / H) off its scores


def _need(block: Mapping[str, Any], key: str, where: str):
    if not isinstance(block, Mapping) or key not in block:
        raise ConfigError(f"Difavik config: {where} lacks '{key}'")
    return block[key]


def _int(block, key, where, lowest: int = 1) -> int:
    value = _need(block, key, where)
    if isinstance(value, bool) or not isinstance(value, int) or value < lowest:
        what = "a positive integer" if lowest == 1 else f"an integer >= {lowest}"
        raise ConfigError(f"Difavik config: {where}.{key} must be {what}, got {value!r}")
    return value


def _number(block, key, where) -> float:
    value = _need(block, key, where)
    if isinstance(value, bool) or not isinstance(value, (int, float)) or value != value:
        raise ConfigError(f"Difavik config: {where}.{key} must be a number, got {value!r}")
    return float(value)


def _limit(block, where) -> float:
    value = _number(block, "limit", where)
    if not value > 0:
        raise ConfigError(f"Difavik config: {where}.limit must be positive, got {value!r}")
    return value


def _decay(block, heads: int, where: str) -> Tuple[float, ...]:
    values = _need(block, "decay", where)
    if not isinstance(values, (list, tuple)) or len(values) != heads or \
            any(isinstance(v, bool) or not isinstance(v, (int, float)) or not 0 < v <= 1 for v in values):
        raise ConfigError(f"Difavik config: {where}.decay must list {heads} numbers in (0, 1], got {values!r}")
    return tuple(float(v) for v in values)


def _sloped_attention(block: Mapping[str, Any], eps: float, where: str) -> PartSpec:
    dim = _int(block, "dim", where)
    if _int(block, "vdim", where) != dim:
        raise ConfigError(f"Difavik config: {where}.vdim must equal dim {dim} (the values are the keys)")
    mask = block.get("mask")
    window = 0 if mask is None else _int(mask, "size", where + ".mask")
    keep = 0 if mask is None or mask.get("keep_first") is None else _int(mask, "keep_first", where + ".mask", lowest=0)
    return PartSpec.make(
        "sink_attention", num_heads=_int(block, "heads", where), num_kv_heads=_int(block, "kv_heads", where), head_dim=dim,
        v_head_dim=dim, scale=_number(block, "scale", where), window=window, keep_first=keep, chunk=0, sink=False, qk_bias=True,
        value_is_key=True, joint_norm_eps=eps, slope_range=SLOPE_RANGE, head_gate=True, partial_out=True)


def _retention(block: Mapping[str, Any], eps: float, where: str) -> PartSpec:
    heads, dim, rot = _int(block, "heads", where), _int(block, "dim", where), _need(block, "rot", where)
    return PartSpec.make(
        "decay_attention", num_heads=heads, head_dim=dim, v_head_dim=_int(block, "vdim", where), decay=_decay(block, heads, where),
        position=PartSpec.make("rope", theta=_number(rot, "base", where + ".rot"), rotary_dim=_int(rot, "dims", where + ".rot"),
                               scaling=None, max_positions=0),
        key_scale=dim ** -0.5, eps=eps, out_norm="head", gate_activation="silu", partial_out=True)


def _lightning(block: Mapping[str, Any], eps: float, where: str) -> PartSpec:
    heads = _int(block, "heads", where)
    return PartSpec.make(
        "decay_attention", num_heads=heads, head_dim=_int(block, "dim", where), v_head_dim=_int(block, "vdim", where),
        decay=_decay(block, heads, where), activation="silu", eps=eps, out_norm="all", gate_activation="sigmoid", partial_out=True)


def _mixer(kind: str, block: Mapping[str, Any], eps: float, where: str) -> PartSpec:
    if kind == "lightning":
        return _lightning(block, eps, where)
    if kind == "parallel":
        return PartSpec.make("branches", eps=eps, defer=True, branches=(
            ("left", _sloped_attention(_need(block, "left", where), eps, where + ".left")),
            ("right", _retention(_need(block, "right", where), eps, where + ".right"))))
    raise ConfigError(f"Difavik config: {where.rsplit('.', 1)[0]}.type is {kind!r}; 'parallel' and 'lightning' are known")


def _feed_forward(block: Optional[Mapping[str, Any]], where: str) -> Optional[PartSpec]:
    if block is None:
        return None
    kind = _need(block, "kind", where)
    if kind == "dense":
        return PartSpec.make("swiglu", intermediate_size=_int(block, "ff", where), tensor_names=("gate", "up", "down"),
                             activation="clamped", limit=_limit(block, where), sigmoid_scale=SIGMOID_SCALE, bias=True,
                             float32_out=True, partial_out=True)
    if kind == "moe":
        router, expert = _need(block, "router", where), _need(block, "expert", where)
        experts, top = _int(router, "experts", where + ".router"), _int(router, "top", where + ".router")
        if top > experts:
            raise ConfigError(f"Difavik config: {where}.router.top {top} exceeds its {experts} experts")
        return PartSpec.make("moe", experts=experts, top=top, intermediate_size=_int(expert, "ff", where + ".expert"), gated=True,
                             activation="clamped", limit=_limit(expert, where + ".expert"), sigmoid_scale=SIGMOID_SCALE,
                             route="softmax", float32_out=True, partial_out=True)
    raise ConfigError(f"Difavik config: {where}.kind is {kind!r}; 'dense' and 'moe' are known")


def _owner(i: int, layers) -> int:
    """The layer whose tensors layer i uses (itself, unless `weights_of` names another)."""
    seen, at = [], i
    while layers[at].get("weights_of") is not None:
        seen.append(at)
        source = layers[at]["weights_of"]
        if isinstance(source, bool) or not isinstance(source, int) or not 0 <= source < len(layers) or source in seen:
            raise ConfigError(f"Difavik config: layers[{at}].weights_of must name another layer, got {source!r}")
        at = source
    if any(layers[i].get(key) != layers[at].get(key) for key in ("type", "mixer", "mlp")):
        raise ConfigError(f"Difavik config: layers[{i}] uses the tensors of layer {at} but its entry differs from it")
    return at


def spec_from_config(raw: Mapping[str, Any]) -> ModelSpec:
    if not isinstance(raw, Mapping) or raw.get("architecture") != ARCHITECTURE:
        raise ConfigError("Difavik config: 'architecture' must be 'Difavik'")
    width, vocab = _int(raw, "width", "config"), _int(raw, "vocab", "config")
    eps = _number(_need(raw, "norm", "config"), "eps", "norm")
    norm = PartSpec.make("rms_stream", eps=eps, unit_offset=True)
    layers = _need(raw, "layers", "config")
    if not isinstance(layers, list) or not layers or not all(isinstance(layer, Mapping) for layer in layers):
        raise ConfigError("Difavik config: 'layers' must be a nonempty list of blocks")
    names = (("mixer_out_norm", "norm1"), ("ff_out_norm", "norm2"), ("mixer", "mix"), ("feed_forward", "mlp"), ("mixer_scale", "ls1"),
             ("ff_scale", "ls2"))
    specs, place, runs, order = [], {}, {}, []
    owners = [_owner(i, layers) for i in range(len(layers))]
    for i in sorted(set(owners)):
        layer, where = layers[i], f"layers[{i}]"
        mixer = _mixer(_need(layer, "type", where), _need(layer, "mixer", where), eps, where + ".mixer")
        place[i] = len(specs)
        specs.append(LayerSpec(mixer=mixer, feed_forward=_feed_forward(layer.get("mlp"), where + ".mlp"), norm=norm, position=None,
                               arrangement="out_norm_stream", names=names, layer_scale=True, number=i))
    for owner in owners:
        runs[owner] = runs.get(owner, -1) + 1
        order.append(RunEntry(place[owner], instance=runs[owner]))
    pairs = (raw.get("embedding") or {}).get("bigram")
    if pairs is None:
        embedding = PartSpec.make("table", out_dtype="float32")
    else:
        where = "embedding.bigram"
        embedding = PartSpec.make("pair_hash", buckets=_int(pairs, "buckets", where), mul_prev=_int(pairs, "mul_prev", where, lowest=0),
                                  mul_cur=_int(pairs, "mul_cur", where, lowest=0), rounded=True, names=(("pairs", "bigram"),))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=width, vocab_size=vocab, max_positions=MAX_POSITIONS, layers=tuple(specs),
        run_order=tuple(order), final_norm=norm, tie_word_embeddings=True, embed_name="embed", final_norm_name="final.norm",
        lm_head_name="head", layer_prefix="l{i}.", embedding=embedding)
