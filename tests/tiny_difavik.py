"""Small Difavik configurations for the tests, with weights of a size that makes every mechanism matter (scores of
several units, gates away from one half, feed-forward inputs that reach their limit, routers with clear picks),
written as a model folder.

A: odd sizes everywhere; both kinds of layer; layers that use the tensors of an earlier one (one of them named
   through another), a window shorter and one longer than a page, kept first tokens that end inside a page, a dense
   layer, mixtures, a layer without a feed-forward between others.
B: values of one: one head, one kv head, heads of one and two elements, a window of one token, no kept tokens, one
   bucket, a decay of one, one expert, all of three experts.
C: the sizes the tensor-core kernels take in bfloat16 (heads of 64 and 128, several query heads a kv head, expert
   widths in whole blocks of 16, pages of 16), windows longer than the pieces decoding cuts contexts into.
"""
import json
from pathlib import Path

import torch

from vosti_b200.config import model_spec_from_config
from vosti_b200.models import expected_weights
from vosti_b200.weights import write_safetensors


def parallel(left, right, mlp, weights_of=None):
    entry = dict(type="parallel", mixer=dict(left=left, right=right), mlp=mlp)
    if weights_of is not None:
        entry["weights_of"] = weights_of
    return entry


def left(heads, kv, dim, scale, window, keep):
    return dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale, mask=dict(size=window, keep_first=keep))


def right(heads, dim, vdim, base, dims, decay):
    return dict(heads=heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=dims), decay=decay)


def lightning(heads, dim, vdim, decay, mlp):
    return dict(type="lightning", mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=decay), mlp=mlp)


def dense(ff, limit):
    return dict(kind="dense", ff=ff, limit=limit)


def moe(experts, top, ff, limit):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))


def model(vocab, width, eps, buckets, prev, cur, layers):
    layers = json.loads(json.dumps(layers))          # entries that start out equal are objects of their own
    return dict(architecture="Difavik", vocab=vocab, width=width, norm=dict(eps=eps),
                embedding=dict(bigram=dict(buckets=buckets, mul_prev=prev, mul_cur=cur)), layers=layers)


_A_SHARED = (left(6, 3, 14, 0.4, 13, 11), right(3, 10, 7, 60.0, 6, [0.9, 0.97, 0.6]), moe(5, 2, 20, 0.9))
A = model(197, 72, 3e-6, 31, 5, 17, [
    parallel(*_A_SHARED),
    lightning(3, 9, 11, [0.8, 0.95, 0.99], dense(52, 1.3)),
    parallel(*_A_SHARED, weights_of=0),
    parallel(left(4, 2, 10, 0.5, 37, 3), right(2, 6, 15, 200.0, 4, [0.93, 0.999]), None),
    parallel(*_A_SHARED, weights_of=2),
    lightning(2, 12, 5, [0.7, 0.98], moe(6, 4, 28, 1.1)),
])
B = model(96, 64, 1e-5, 1, 3, 2, [
    lightning(1, 1, 1, [1.0], moe(1, 1, 48, 1.0)),
    parallel(left(1, 1, 1, 1.0, 1, 0), right(1, 2, 1, 30.0, 2, [0.5]), moe(3, 3, 16, 0.8)),
    parallel(left(1, 1, 2, 0.8, 2, 1), right(1, 4, 3, 30.0, 2, [1.0]), dense(17, 0.7)),
    lightning(1, 8, 4, [0.9], None),
])
_C_SHARED = (left(4, 2, 64, 0.16, 300, 40), right(3, 64, 48, 5000.0, 32, [0.95, 0.99, 0.9995]), moe(8, 3, 64, 1.4))
C = model(160, 128, 1e-6, 61, 7, 11, [
    parallel(*_C_SHARED),
    lightning(2, 128, 72, [0.9, 0.998], dense(160, 1.5)),
    parallel(*_C_SHARED, weights_of=0),
    parallel(left(4, 1, 128, 0.1, 70, 17), right(1, 128, 128, 300.0, 128, [0.97]), dense(96, 1.0)),
    lightning(3, 32, 64, [0.6, 0.97, 0.999], moe(6, 2, 80, 1.0)),
])
ALL = {"a": (A, 61), "b": (B, 62), "c": (C, 63)}      # config, seed
PAGE = {"a": 8, "b": 4, "c": 16}


def windows(config):
    """(window, kept) of every layer that has one."""
    return [(e["mixer"]["left"]["mask"]["size"], e["mixer"]["left"]["mask"]["keep_first"]) for e in config["layers"] if e["type"] == "parallel"]


def draw(name, spec, gen):
    """One tensor by its role, float32 (the caller rounds to bfloat16)."""
    shape = tuple(spec.shape)
    n = lambda std, mean=0.0: mean + std * torch.randn(shape, generator=gen)
    last = name.split(".")[-1]
    if name in ("embed", "bigram"):
        return n(0.8)
    if last == "b":
        return n(0.5)
    if last in ("ls1", "ls2"):
        return n(0.3, 0.8)
    if last in ("norm1", "norm2") or name == "final.norm":       # stored around zero
        return n(0.3)
    if last in ("norm", "out"):
        return n(0.3, 1.2)
    if last == "router":
        return n(1.5 / shape[1] ** 0.5)
    if last in ("g", "gate", "up"):
        return n(1.5 / shape[1] ** 0.5)
    return n(1.0 / shape[1] ** 0.5)


def tensors_for(config, seed, unused=True):
    """`unused` false leaves out the tensors the model never reads (the second norm and scale of a layer without a
    feed-forward); a checkpoint may have them or not."""
    spec = model_spec_from_config(config)
    gen = torch.Generator().manual_seed(seed)
    expected = expected_weights(spec)
    drawn = {name: draw(name, w, gen).to(torch.bfloat16) for name, w in expected.items()}
    return spec, {name: t for name, t in drawn.items() if unused or not expected[name].optional}


def write_model(folder, config, seed, unused=True):
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    _, tensors = tensors_for(config, seed, unused)
    (folder / "config.json").write_text(json.dumps(config))
    write_safetensors(folder / "model.safetensors", tensors, metadata={"format": "pt"})
    return str(folder)
