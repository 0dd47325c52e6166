"""The Pubulix design, read from its own config.json.

A pre-norm decoder over a float32 residual stream whose sublayers join it through gates,

    h = norm1(x),  x <- x + m sigmoid(R1 h + r1) * mixer(h + conv(h))
    h = norm2(x),  x <- x + m sigmoid(R2 h + r2) * ff(h)

with root-mean-square norms of one number each, one constant m for the model, and a short causal
convolution over time (per channel) on what every mixer reads. Embedding rows are multiplied by
a constant; logits pass a soft cap. Two kinds of layer, in any order:

  "latent_attention"  attention over a sliding window whose keys and values are made from one
                      cached latent per token and a rotated key part the heads share (pairs
                      (2i, 2i + 1)), with a learned sink per head and a sigmoid gate on every
                      element of the concatenated heads; a layer with `kv_from` reads the cache of
                      an earlier layer of this kind instead of keeping one;
  "attention"         grouped-query attention over a sliding window, a rotation of the first
                      elements of each head (pairs (i, i + dims / 2)), scores under a soft cap.

Feed-forwards are mixtures of gated experts with clamped inputs, assigned to token ids by a
table (no router), all of a token's experts weighing the same; or absent.

Keys (a missing one is an error unless marked optional; optional blocks may be absent or null):

    architecture  "Pubulix"
    vocab, width, residual_mult
    norm.eps, canon.taps
    embedding.scale                        optional (1)
    logit_softcap                          optional
    layers[i].type                         "latent_attention" | "attention"
    layers[i].mixer (latent_attention)     heads, dim, rot_dim, vdim, kv_rank, scale, rot.base, rot.dims (equal to
                                           rot_dim; optional), mask.size (optional), kv_from (optional)
    layers[i].mixer (attention)            heads, kv_heads, dim, vdim, scale, rot.base, rot.dims, mask.size (optional),
                                           softcap (optional)
    layers[i].mlp                          optional: {kind: "moe", expert: {ff, limit}, router: {experts, top}}
"""
from __future__ import annotations

from typing import Any, Mapping, Optional

from .schema import ConfigError, LayerSpec, ModelSpec, PartSpec, RunEntry

ARCHITECTURE = "Pubulix"
MAX_POSITIONS = 1 << 30        # the design sets no limit (angles are formed from the position); the cache pool does
SIGMOID_SCALE = 1.702          # of the experts' gate activation g * sigmoid(1.702 g)


def _need(block: Mapping[str, Any], key: str, where: str):
    if not isinstance(block, Mapping) or key not in block:
        raise ConfigError(f"Pubulix config: {where} lacks '{key}'")
    return block[key]


def _positive_int(block, key, where) -> int:
    value = _need(block, key, where)
    if isinstance(value, bool) or not isinstance(value, int) or value <= 0:
        raise ConfigError(f"Pubulix config: {where}.{key} must be a positive integer, got {value!r}")
    return value


def _number(block, key, where) -> float:
    value = _need(block, key, where)
    if isinstance(value, bool) or not isinstance(value, (int, float)) or value != value:
        raise ConfigError(f"Pubulix config: {where}.{key} must be a number, got {value!r}")
    return float(value)


def _cap(block, key, where) -> float:
    """An optional soft cap: absent, null and 0 mean none."""
    if block.get(key) is None:
        return 0.0
    value = _number(block, key, where)
    if value < 0:
        raise ConfigError(f"Pubulix config: {where}.{key} must be a number >= 0, got {value!r}")
    return value


def _window(block, where) -> int:
    mask = block.get("mask")
    return 0 if mask is None else _positive_int(mask, "size", where + ".mask")


def _rotation(block, dims: int, where: str, interleaved: bool) -> PartSpec:
    return PartSpec.make("rope", theta=_number(_need(block, "rot", where), "base", where + ".rot"), rotary_dim=dims,
                         scaling=None, max_positions=0, interleaved=interleaved)


def _latent(i: int, block: Mapping[str, Any], eps: float) -> PartSpec:
    where = f"layers[{i}].mixer"
    rot_dim = _positive_int(block, "rot_dim", where)
    rot = _need(block, "rot", where)
    if isinstance(rot, Mapping) and rot.get("dims") is not None and _positive_int(rot, "dims", where + ".rot") != rot_dim:
        raise ConfigError(f"Pubulix config: {where}.rot.dims must equal rot_dim {rot_dim}")
    return PartSpec.make(
        "latent_attention", num_heads=_positive_int(block, "heads", where), head_dim=_positive_int(block, "dim", where),
        rot_dim=rot_dim, v_head_dim=_positive_int(block, "vdim", where), kv_rank=_positive_int(block, "kv_rank", where),
        scale=_number(block, "scale", where), eps=eps, gate=False, out_gate=True, sink=True, window=_window(block, where),
        own_latent=block.get("kv_from") is None, partial_out=True, position=_rotation(block, rot_dim, where, interleaved=True))


def _attention(i: int, block: Mapping[str, Any]) -> PartSpec:
    where = f"layers[{i}].mixer"
    dims = _positive_int(_need(block, "rot", where), "dims", where + ".rot")
    return PartSpec.make(
        "sink_attention", num_heads=_positive_int(block, "heads", where), num_kv_heads=_positive_int(block, "kv_heads", where),
        head_dim=_positive_int(block, "dim", where), v_head_dim=_positive_int(block, "vdim", where),
        scale=_number(block, "scale", where), window=_window(block, where), chunk=0, sink=False,
        softcap=_cap(block, "softcap", where), partial_out=True, position=_rotation(block, dims, where, interleaved=False))


def _feed_forward(i: int, block: Optional[Mapping[str, Any]], vocab: int) -> Optional[PartSpec]:
    if block is None:
        return None
    where = f"layers[{i}].mlp"
    kind = _need(block, "kind", where)
    if kind != "moe":
        raise ConfigError(f"Pubulix config: {where}.kind is {kind!r}; 'moe' is known")
    router, expert = _need(block, "router", where), _need(block, "expert", where)
    limit = _number(expert, "limit", where + ".expert")
    if not limit > 0:
        raise ConfigError(f"Pubulix config: {where}.expert.limit must be positive, got {limit!r}")
    return PartSpec.make(
        "moe", experts=_positive_int(router, "experts", where + ".router"), top=_positive_int(router, "top", where + ".router"),
        intermediate_size=_positive_int(expert, "ff", where + ".expert"), gated=True, activation="clamped",
        limit=limit, sigmoid_scale=SIGMOID_SCALE, route="table", vocab=vocab, float32_out=True,
        partial_out=True)


def _source(i: int, layers, where: str) -> Optional[int]:
    """The layer whose latents layer i reads, checked against it, or None."""
    block = layers[i]["mixer"]
    source = block.get("kv_from")
    if source is None:
        return None
    if isinstance(source, bool) or not isinstance(source, int) or not 0 <= source < i:
        raise ConfigError(f"Pubulix config: {where}.kv_from must name an earlier layer, got {source!r}")
    other = layers[source]
    theirs = other.get("mixer") or {}
    if other.get("type") != "latent_attention" or theirs.get("kv_from") is not None:
        raise ConfigError(f"Pubulix config: {where}.kv_from names layer {source}, which keeps no latents of its own")
    same = ("kv_rank", "rot_dim")
    if any(theirs.get(key) != block.get(key) for key in same) or \
            _number(theirs.get("rot"), "base", f"layers[{source}].mixer.rot") != _number(block.get("rot"), "base", where + ".rot"):
        raise ConfigError(f"Pubulix config: {where} and layer {source}, whose latents it reads, differ in kv_rank, rot_dim or rotation")
    return source


def spec_from_config(raw: Mapping[str, Any]) -> ModelSpec:
    if not isinstance(raw, Mapping) or raw.get("architecture") != ARCHITECTURE:
        raise ConfigError("Pubulix config: 'architecture' must be 'Pubulix'")
    width, vocab = _positive_int(raw, "width", "config"), _positive_int(raw, "vocab", "config")
    eps = _number(_need(raw, "norm", "config"), "eps", "norm")
    taps = _positive_int(_need(raw, "canon", "config"), "taps", "canon")
    mult = _number(raw, "residual_mult", "config")
    embedding = raw.get("embedding")
    scale = 1.0 if embedding is None or embedding.get("scale") is None else _number(embedding, "scale", "embedding")
    norm = PartSpec.make("rms_stream", eps=eps, scalar=True)
    layers = _need(raw, "layers", "config")
    if not isinstance(layers, list) or not layers:
        raise ConfigError("Pubulix config: 'layers' must be a nonempty list")
    names = (("input_norm", "norm1"), ("post_norm", "norm2"), ("mixer", "mix"), ("feed_forward", "mlp"), ("input_conv", "canon1"),
             ("mixer_gate", "rg1"), ("ff_gate", "rg2"))
    specs, order = [], []
    for i, layer in enumerate(layers):
        kind = _need(layer, "type", f"layers[{i}]")
        block = _need(layer, "mixer", f"layers[{i}]")
        source = None
        if kind == "latent_attention":
            mixer, source = _latent(i, block, eps), _source(i, layers, f"layers[{i}].mixer")
        elif kind == "attention":
            mixer = _attention(i, block)
        else:
            raise ConfigError(f"Pubulix config: layers[{i}].type is {kind!r}; 'latent_attention' and 'attention' are known")
        specs.append(LayerSpec(mixer=mixer, feed_forward=_feed_forward(i, layer.get("mlp"), vocab), norm=norm, position=None,
                               arrangement="gated_pre_norm_stream", names=names, residual_scale=mult, input_conv=taps))
        order.append(RunEntry(i, cache_from=source))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=width, vocab_size=vocab, max_positions=MAX_POSITIONS, layers=tuple(specs),
        run_order=tuple(order), final_norm=norm, tie_word_embeddings=False, embed_name="embed", final_norm_name="final.norm",
        lm_head_name="head", layer_prefix="l{i}.",
        embedding=PartSpec.make("table", scale=scale, out_dtype="float32", rounded=False, publish_ids=True),
        head=PartSpec.make("linear", softcap=_cap(raw, "logit_softcap", "config")))
