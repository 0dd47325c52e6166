"""Small Pubulix configurations for the tests, with weights of a size that makes every mechanism
matter (scores of several units, sinks that take a share, experts whose inputs reach their limit,
gates away from one half), written as a model folder.

A: odd sizes everywhere; both kinds of layer; two layers that read an earlier layer's latents, one
   through a wider window than that layer's own and with other heads, one through a narrower one;
   a layer without a feed-forward between others; windows of several lengths; three taps; expert
   counts and picks that differ from layer to layer.
B: values of one: one head, one kv head, a rotated part of two elements, a window of one token and
   one of two, one tap, one expert, all of three experts, one pick.
C: the sizes the tensor-core kernels take in bfloat16 (latents of 128, rotated parts of 32 and 64,
   heads of 64 and 128, expert widths in whole blocks of 16, pages of 16), windows longer than the
   pieces decoding cuts contexts into, nine taps.
"""
import json
from pathlib import Path

import torch

from vosti_b200.config import model_spec_from_config
from vosti_b200.models import expected_weights
from vosti_b200.weights import write_safetensors


def latent(heads, dim, rot, vdim, rank, window, scale, base, mlp, kv_from=None):
    mixer = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, scale=scale, mask=dict(size=window), rot=dict(base=base, dims=rot))
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=mixer, mlp=mlp)


def capped(heads, kv, dim, vdim, window, scale, base, dims, softcap, mlp):
    return dict(type="attention", mlp=mlp, mixer=dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, softcap=softcap,
                                                      mask=dict(size=window), rot=dict(base=base, dims=dims)))


def moe(experts, top, ff, limit):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))


def model(vocab, width, taps, mult, scale, cap, eps, layers):
    return dict(architecture="Pubulix", vocab=vocab, width=width, canon=dict(taps=taps), residual_mult=mult, embedding=dict(scale=scale),
                logit_softcap=cap, norm=dict(eps=eps), layers=layers)


A = model(211, 72, 3, 0.7, 2.5, 9.0, 2e-6, [
    latent(3, 10, 6, 14, 20, 11, 0.5, 100.0, moe(5, 2, 20, 1.1)),
    capped(4, 2, 24, 16, 7, 0.35, 300.0, 8, 4.0, moe(7, 3, 24, 0.9)),
    latent(4, 12, 6, 10, 20, 29, 0.45, 100.0, moe(5, 1, 28, 2.0), kv_from=0),
    capped(6, 3, 14, 22, 40, 0.4, 1000.0, 14, 7.0, None),
    latent(2, 18, 6, 8, 20, 5, 0.4, 100.0, moe(4, 2, 36, 1.3), kv_from=0),
    latent(5, 8, 10, 6, 33, 23, 0.5, 5000.0, moe(6, 4, 16, 0.6)),
])
B = model(128, 64, 1, 1.0, 1.0, 30.0, 1e-5, [
    latent(1, 1, 2, 1, 1, 2, 1.0, 50.0, moe(1, 1, 48, 1.0)),
    capped(1, 1, 2, 3, 1, 1.0, 1000.0, 2, 1.0, moe(3, 3, 16, 1.0)),
    latent(1, 16, 2, 24, 8, 3, 0.5, 50.0, moe(2, 1, 64, 0.8)),
    latent(1, 6, 2, 1, 8, 1, 0.5, 50.0, moe(3, 1, 16, 1.0), kv_from=2),
])
C = model(160, 128, 9, 0.4, 7.0, 12.0, 1e-6, [
    latent(4, 64, 32, 32, 128, 300, 0.12, 10000.0, moe(8, 2, 64, 1.4)),
    capped(4, 2, 64, 64, 290, 0.15, 10000.0, 32, 6.0, moe(6, 3, 80, 1.0)),
    latent(16, 32, 32, 64, 128, 131, 0.14, 10000.0, moe(4, 1, 96, 1.2), kv_from=0),
    capped(2, 1, 128, 128, 64, 0.1, 50000.0, 128, 9.0, moe(8, 2, 64, 1.1)),
    latent(3, 32, 64, 48, 128, 40, 0.15, 500.0, moe(12, 2, 64, 0.9)),
])
ALL = {"a": (A, 51), "b": (B, 52), "c": (C, 53)}      # config, seed
PAGE = {"a": 8, "b": 4, "c": 16}


def draw(name, spec, gen):
    """One tensor by its role, float32 (the caller rounds to bfloat16); integer tables int32."""
    shape = tuple(spec.shape)
    n = lambda std, mean=0.0: mean + std * torch.randn(shape, generator=gen)
    last = name.split(".")[-1]
    if spec.integer:
        return torch.rand((shape[0], spec.distinct_below), generator=gen).argsort(dim=-1)[:, : shape[1]].to(torch.int32)
    if name == "embed":
        return n(1.0)
    if last == "sink":
        return n(1.5)
    if last.startswith("canon"):
        return n(0.6)
    if last == "b":                          # biases of the residual gates
        return n(0.7)
    if len(shape) < 2:                       # weights of norms: one number, or a vector
        return n(0.2, 1.3)
    if last in ("g", "rg1", "rg2", "gate", "up"):
        return n(2.0 / shape[1] ** 0.5)
    return n(1.0 / shape[1] ** 0.5)


def tensors_for(config, seed, unused=True):
    """`unused` false leaves out the tensors the model never reads (the second norm and gate of a
    layer without a feed-forward); a checkpoint may have them or not."""
    spec = model_spec_from_config(config)
    gen = torch.Generator().manual_seed(seed)
    expected = expected_weights(spec)
    drawn = {name: draw(name, w, gen) for name, w in expected.items()}
    drawn = {name: t if expected[name].integer else t.to(torch.bfloat16) for name, t in drawn.items()}
    return spec, {name: t for name, t in drawn.items() if unused or not expected[name].optional}


def write_model(folder, config, seed, unused=True):
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    _, tensors = tensors_for(config, seed, unused)
    (folder / "config.json").write_text(json.dumps(config))
    write_safetensors(folder / "model.safetensors", tensors, metadata={"format": "pt"})
    return str(folder)
