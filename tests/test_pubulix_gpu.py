"""The Pubulix design on the GPU against the plain implementation (tests/plain_pubulix.py).

Mechanisms alone (the boundary kernel between gated sublayers with its norm, its picked rows and
its convolution step; the convolution over portions and its state; windowed latent attention with
sink, gate and neighbouring pairs, also over another layer's latents; capped windowed attention;
the token-table experts: sorting, grouped products, clamped activation), then whole models of
three small configurations: whole prompts, prefill against token-by-token decoding, portions down
to two tokens, unequal requests in one batch against each alone, pages and slots used again, the
first tokens of a sequence, long decoding past every window, and greedy generation through
`Engine` (scheduler, CUDA graphs, asynchronous scheduling, preemption).

Where random inputs would hide a fault, the inputs are made so that it shows: one key that stands
out just inside and just outside a window, at page borders and at the borders of the pieces that
decoding cuts long windows into; sinks that outweigh the keys; a token's experts made unlike all
others.

Exactness is tested in float32 (differences of rounding order only); bfloat16 serving is
compared with the float32 oracle with a bound on the error of rounding.
"""
import math

import pytest
import torch

import plain_pubulix as plain
import tiny_pubulix as tiny
from gpu_util import Harness
from vosti_b200 import Engine, ops
from vosti_b200.config import ConfigError
from vosti_b200.config.pubulix import _attention, _feed_forward, _latent
from vosti_b200.engine.batch import StepEntry
from vosti_b200.engine.runner import ModelRunner
from vosti_b200.parts import StateSpec, build_feed_forward, build_mixer
from vosti_b200.parts.feed_forward import interleave_gate_up

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32 = dict(atol=3e-4, rtol=3e-4)
EPS = 2e-6


def rounded(*shape, gen, std=1.0, mean=0.0):
    """Random values that bfloat16 holds exactly, as float32 on the CPU."""
    return (mean + std * torch.randn(tuple(shape), generator=gen)).to(torch.bfloat16).float()


def give(part, W, dtype):
    """Hand a part its tensors (keys of `weight_specs`) on the device in the serving layout."""
    assert set(W) == set(part.weight_specs()), (sorted(W), sorted(part.weight_specs()))
    store = torch.bfloat16 if dtype == torch.bfloat16 else torch.float32
    part.load({k: (v.to(DEV, store) if v.is_floating_point() else v.to(DEV)).contiguous() for k, v in W.items()}, dtype)
    part.setup(torch.device(DEV), dtype)


def weights_of(part, gen, prefix="l0.mix."):
    drawn = {key: tiny.draw(prefix + key, w, gen) for key, w in part.weight_specs().items()}
    return {k: v.to(torch.bfloat16).float() if v.is_floating_point() else v for k, v in drawn.items()}


def double(W):
    return {k: v.double() if v.is_floating_point() else v for k, v in W.items()}


def close(got, want, dtype, what=None):
    if dtype == torch.float32:
        assert torch.allclose(got, want, **F32), (what, float((got - want).abs().max()))
    else:
        assert float((got - want).abs().mean() / want.abs().mean()) < 0.04, what


def run_mixer(mixer, harness, x, sizes, dtype, rid="r", lender=None, lender_x=None):
    """The mixer over x in portions. `lender`: a mixer that keeps the latents this one reads; it runs
    over `lender_x` first in every step."""
    outs, at = [], 0
    for size in sizes:
        ctx = harness.context([StepEntry(rid, [0] * size)])
        cache = harness.cache.layer_caches[0]
        if lender is not None:
            ops.materialize(lender.forward(ctx, lender_x[at:at + size].to(DEV, dtype).contiguous(), cache))
        out = mixer.forward(ctx, x[at:at + size].to(DEV, dtype).contiguous(), cache, lender is None)
        outs.append(ops.materialize(out).float().cpu())
        harness.cache.trim(rid)
        at += size
    assert int(harness.status.item()) == 0
    return torch.cat(outs)


CUTS = lambda T: ((T,), (T - 33,) + (1,) * 33, (2, 5, 1, 1, 17, 2, 3, T - 31))


# ---------------------------------------------------------------- the boundary between gated sublayers
def partial_of(x, splits, gen, scratch):
    """x as the unsummed K splits of a product."""
    parts = torch.randn((splits, *x.shape), generator=gen)
    parts[-1] = x - parts[:-1].sum(0)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    return ops.PartialSum(parts.to(DEV), splits, x.shape[0], x.shape[1], torch.float32, status, scratch)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,rows", [(200, 9), (67, 5), (1, 3), (4, 2), (1028, 70), (4099, 3), (12544, 2), (12545, 2)])
def test_boundary_gates_adds_and_norms(dtype, width, rows):
    gen = torch.Generator().manual_seed(width)
    stream, y = 1.5 * torch.randn(rows, width, generator=gen), torch.randn(rows, width, generator=gen)
    z, bias = 2.0 * torch.randn(rows, width, generator=gen), rounded(width, gen=gen)
    w, mult, gain = rounded(width, gen=gen, std=0.2, mean=1.0), 0.45, 1.37
    store = torch.bfloat16 if dtype == torch.bfloat16 else torch.float32
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    total = stream.double() + mult * torch.sigmoid(z.double() + bias.double()) * y.double()
    tol = dict(atol=3e-5, rtol=3e-5) if dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)
    for splits in (1, 3, 12):
        pending = lambda: ops.DeferredGated(
            y.to(DEV) if splits == 1 else partial_of(y, splits, gen, "split_k"),
            z.to(DEV) if splits == 1 else partial_of(z, splits + 1, gen, "split_k_gate"), bias.to(DEV, store), mult)
        s = stream.to(DEV).clone()
        h = ops.gated_rms_stream(s, pending(), EPS, dtype, gain=gain, status=status)
        assert h.dtype == dtype and torch.allclose(s.cpu(), total.float(), atol=3e-5, rtol=3e-5)
        assert torch.allclose(h.float().cpu(), plain.rms_norm(total, gain, EPS).float(), **tol)
        # a weight vector, rows asked for one by one (also twice), the stream left alone
        picks = torch.tensor([rows - 1, 0, rows - 1], dtype=torch.int32, device=DEV)
        s = stream.to(DEV).clone()
        h = ops.gated_rms_stream(s, pending(), EPS, dtype, weight=w.to(DEV, store), offset=1.0, rows=picks, status=status)
        want = plain.rms_norm(total, 1.0 + w.double(), EPS).float()[picks.cpu().long()]
        assert torch.allclose(h.float().cpu(), want, **tol) and torch.equal(s.cpu(), stream)
    nothing = ops.gated_rms_stream(stream.to(DEV), None, EPS, dtype, gain=gain, status=status)
    assert torch.allclose(nothing.float().cpu(), plain.rms_norm(stream.double(), gain, EPS).float(), **tol)
    assert int(status.item()) == 0


@pytest.mark.parametrize("width", [48, 37])
def test_boundary_adds_a_tokens_picked_rows(width):
    """y spread over the rows of sorted experts: token t's output is a share of the sum of its rows."""
    gen = torch.Generator().manual_seed(width)
    rows, picks = 6, 3
    y, stream, z = (torch.randn(n, width, generator=gen) for n in (rows * picks, rows, rows))
    where = torch.randperm(rows * picks, generator=gen).view(rows, picks).to(torch.int32)
    total = stream.double() + 0.6 * torch.sigmoid(z.double()) * y.double()[where.long()].sum(1) / picks
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    for splits in (1, 5):
        source = y.to(DEV) if splits == 1 else partial_of(y, splits, gen, "split_k")
        picked = ops.PickedSum(source, where.to(DEV), 1.0 / picks)
        assert torch.allclose(picked.materialize().cpu(), y[where.long()].mean(1), atol=1e-5)
        s = stream.to(DEV).clone()
        h = ops.gated_rms_stream(s, ops.DeferredGated(picked, z.to(DEV), None, 0.6), EPS, torch.float32, gain=0.9, status=status)
        assert torch.allclose(s.cpu(), total.float(), atol=1e-5, rtol=1e-5)
        assert torch.allclose(h.cpu(), plain.rms_norm(total, 0.9, EPS).float(), atol=1e-5, rtol=1e-5)


def test_a_result_overwritten_by_a_later_product_is_refused():
    gen = torch.Generator().manual_seed(1)
    y = partial_of(torch.randn(2, 8, generator=gen), 2, gen, "split_k")
    with pytest.raises(ops.KernelError, match="scratch"):
        ops.DeferredGated(y, partial_of(torch.randn(2, 8, generator=gen), 2, gen, "split_k"), None, 1.0)
    ops._SPLIT_GENERATION["split_k"] = ops._SPLIT_GENERATION.get("split_k", 0) + 1
    with pytest.raises(ops.KernelError, match="overwrote"):
        y.check()


# ---------------------------------------------------------------- the convolution and its state
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps,width", [(1, 24), (2, 24), (3, 37), (4, 64), (4, 1030), (5, 20), (8, 33), (9, 32), (9, 7)])
def test_convolution_over_portions_and_single_tokens(dtype, taps, width):
    """h + conv(h) of two interleaved requests (the second one shorter than the taps at first): portions by
    the portion kernel, single tokens by the boundary kernel; a slot that is used again starts from
    zeros. The two kernels give a token the same bits."""
    gen = torch.Generator().manual_seed(taps * 100 + width)
    w = rounded(width, taps, gen=gen, std=0.6)
    size = max(4, ((taps - 1) * width + 3) // 4 * 4)
    conv = lambda state: ops.StreamConv(w.t().contiguous().to(DEV), state)
    store = torch.bfloat16 if dtype == torch.bfloat16 else torch.float32
    xs = {r: torch.randn(n, width, generator=gen) for r, n in (("a", 41), ("b", 13), ("c", 9))}
    # what the norm makes of the stream, as the kernels round it, is the convolution's input
    hs = {r: ops.gated_rms_stream(x.to(DEV), None, EPS, dtype, gain=1.1).float().cpu() for r, x in xs.items()}
    want = {r: (h.double() + plain.causal_convolution(h.double(), w.double())).float() for r, h in hs.items()}
    schedules = [
        [("a", 41)], [("a", 40), ("a", 1)], [("a", 2)] * 3 + [("a", 35)],
        [("a", 1)] * 12 + [("a", 29)],
    ]
    results = []
    for schedule in schedules:
        harness = Harness([None], [StateSpec((size,))], dtype, max_requests=2)
        state = harness.cache.layer_caches[0].state
        out, at = [], 0
        for _, n in schedule:
            ctx = harness.context([StepEntry("a", [0] * n)])
            s = xs["a"][at:at + n].to(DEV)
            if n == 1:
                h, u = ops.gated_rms_stream(s, None, EPS, dtype, gain=1.1, conv=conv(state), ctx=ctx)
            else:
                h = ops.gated_rms_stream(s, None, EPS, dtype, gain=1.1)
                u = ops.scan_conv(h, w.to(DEV, store), None, state, 0, ctx, inner=width, taps=taps, plain=True)
            assert torch.equal(h.float().cpu(), hs["a"][at:at + n])
            out.append(u.float().cpu())
            at += n
        assert int(harness.status.item()) == 0
        results.append(torch.cat(out))
        tol = dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)
        assert torch.allclose(results[-1], want["a"], **tol), schedule
        assert torch.equal(results[-1], results[0]), schedule
    # several requests in a step, and a slot used again
    harness = Harness([None], [StateSpec((size,))], dtype, max_requests=2)
    state = harness.cache.layer_caches[0].state
    at, got = {r: 0 for r in xs}, {r: [] for r in xs}
    for step in ([("a", 5), ("b", 1)], [("b", 1), ("a", 1)], [("a", 1), ("b", 1)], [("b", 2), ("a", 7)], [("a", 1), ("b", 1)],
                 [("a", 20), ("b", 7)], "end b", [("c", 1), ("a", 1)], [("a", 5), ("c", 2)], [("c", 6)]):
        if step == "end b":
            harness.cache.finish("b")
            continue
        ctx = harness.context([StepEntry(r, [0] * n) for r, n in step])
        s = torch.cat([xs[r][at[r]:at[r] + n] for r, n in step]).to(DEV)
        if all(n == 1 for _, n in step):
            _, u = ops.gated_rms_stream(s, None, EPS, dtype, gain=1.1, conv=conv(state), ctx=ctx)
        else:
            h = ops.gated_rms_stream(s, None, EPS, dtype, gain=1.1)
            u = ops.scan_conv(h, w.to(DEV, store), None, state, 0, ctx, inner=width, taps=taps, plain=True)
        row = 0
        for r, n in step:
            got[r].append(u[row:row + n].float().cpu())
            row += n
            at[r] += n
    assert int(harness.status.item()) == 0
    for r in xs:
        rows = torch.cat(got[r])
        assert torch.allclose(rows, want[r][: rows.shape[0]], **tol), r


# ---------------------------------------------------------------- latent attention
LATENT_SIZES = [
    (3, 20, 6, 10, 40, 17, 8), (1, 8, 2, 8, 8, 1, 4), (5, 12, 10, 24, 24, 40, 8), (4, 32, 16, 48, 64, 64, 16), (2, 7, 4, 5, 33, 2, 4),
    (2, 64, 32, 64, 160, 400, 16), (1, 16, 8, 16, 300, 33, 8),
    # sizes the tensor-core kernel takes in bfloat16: a tile of 16 rows is one token, four tokens, or cuts across tokens
    (16, 128, 64, 128, 512, 100, 16), (4, 32, 32, 48, 128, 70, 16), (3, 64, 32, 64, 256, 130, 8), (40, 16, 64, 16, 128, 31, 4), (1, 32, 32, 8, 128, 65, 16)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,rot,dv,rank,window,page", LATENT_SIZES)
def test_latent_attention_mixer_against_plain(dtype, heads, dim, rot, dv, rank, window, page):
    gen = torch.Generator().manual_seed(heads * 100 + rank)
    width, T = 72, 150
    block = tiny.latent(heads, dim, rot, dv, rank, window, 2.5 / math.sqrt(dim + rot), 200.0, None)["mixer"]
    mixer = build_mixer(_latent(0, block, EPS), width, None)
    assert set(mixer.weight_specs()) == {"q", "dkv", "dkv.norm", "uk", "uv", "g", "sink", "o"}
    assert mixer.cache_spec().widths == (rank, rot) and mixer.cache_spec().window == window
    W = weights_of(mixer, gen)
    give(mixer, W, dtype)
    x = rounded(T, width, gen=gen)
    want, cached = plain.latent_attention(x.double(), double(W), block, EPS)
    for sizes in CUTS(T):
        harness = Harness([mixer.cache_spec()], [None], dtype, num_pages=-(-T // page) + 1, page_size=page)
        close(run_mixer(mixer, harness, x, sizes, dtype), want.float(), dtype, sizes)
    # another layer's queries over these latents, with other heads and a wider, then a narrower window than its owner's
    other_x = rounded(T, width, gen=gen)
    for heads2, other_window in ((heads + 1, window + 9), (2 * heads, max(1, window - 3))):
        block2 = tiny.latent(heads2, dim + 3, rot, dv + 2, rank, other_window, block["scale"], 200.0, None, kv_from=0)["mixer"]
        reader = build_mixer(_latent(1, block2, EPS), width, None)
        assert set(reader.weight_specs()) == {"q", "uk", "uv", "g", "sink", "o"}
        W2 = weights_of(reader, gen)
        give(reader, W2, dtype)
        want2 = plain.latent_attention(other_x.double(), double(W2), block2, EPS, cached)[0]
        import dataclasses
        shared = dataclasses.replace(mixer.cache_spec(), window=max(window, other_window))
        for sizes in CUTS(T):
            harness = Harness([shared], [None], dtype, num_pages=-(-T // page) + 1, page_size=page)
            close(run_mixer(reader, harness, other_x, sizes, dtype, lender=mixer, lender_x=x), want2.float(), dtype, (other_window, sizes))
        ctx = harness.context([StepEntry("s", [0])])
        with pytest.raises(ConfigError, match="another layer"):
            reader.forward(ctx, other_x[:1].to(DEV, dtype), harness.cache.layer_caches[0], True)


def test_latent_attention_of_unequal_requests_in_one_step_on_the_tensor_cores():
    """A long request decoding one token, a portion in the middle of another and a whole short
    prompt in one step: every row equals its request alone in the plain form."""
    gen = torch.Generator().manual_seed(12)
    width, page, dtype = 96, 16, torch.bfloat16
    for window in (24, 300):
        block = tiny.latent(16, 32, 32, 16, 128, window, 0.3, 10000.0, None)["mixer"]
        mixer = build_mixer(_latent(0, block, EPS), width, None)
        W = weights_of(mixer, gen)
        give(mixer, W, dtype)
        xs = {r: rounded(n, width, gen=gen) for r, n in (("a", 420), ("b", 77), ("c", 3))}
        want = {r: plain.latent_attention(x.double(), double(W), block, EPS)[0].float() for r, x in xs.items()}
        harness = Harness([mixer.cache_spec()], [None], dtype, num_pages=40, page_size=page)
        cache = harness.cache.layer_caches[0]
        run = lambda ctx, rows: ops.materialize(mixer.forward(ctx, torch.cat(rows).to(DEV, dtype), cache)).float().cpu()
        got = {r: [] for r in xs}
        got["a"].append(run(harness.context([StepEntry("a", [0] * 419)]), [xs["a"][:419]]))
        got["b"].append(run(harness.context([StepEntry("b", [0] * 20)]), [xs["b"][:20]]))
        rows = run(harness.context([StepEntry("a", [0]), StepEntry("b", [0] * 37), StepEntry("c", [0] * 3)]),
                   [xs["a"][419:], xs["b"][20:57], xs["c"]])
        got["a"].append(rows[:1]); got["b"].append(rows[1:38]); got["c"].append(rows[38:])
        got["b"].append(run(harness.context([StepEntry("b", [0] * 20)]), [xs["b"][57:]]))
        assert int(harness.status.item()) == 0
        for r in xs:
            close(torch.cat(got[r]), want[r], dtype, (window, r))


@pytest.mark.parametrize("dtype,rank,rot,window", [(torch.float32, 16, 4, 30), (torch.bfloat16, 16, 4, 600), (torch.bfloat16, 128, 32, 70),
                                                   (torch.bfloat16, 128, 32, 300), (torch.float32, 16, 4, 300), (torch.bfloat16, 128, 32, 128)])
def test_one_latent_stands_out_at_the_edges_of_a_window(dtype, rank, rot, window):
    """The oldest key a window shows, keys next to page borders and to the borders of the pieces the kernels
    cut a long window into must weigh as the plain form says, and the key one step further back must
    not be seen at all. The projections are rows of the identity, so that the mixer's input is the
    q | down row itself (the gate's weight is zero: one half everywhere); the first latent element of
    every token is zero but the target's, head 0's unrotated key matrix reads that element alone, and
    the last query looks for it."""
    heads, dim, dv, page = 2, 8, 8, 16
    gen = torch.Generator().manual_seed(17)
    qw = heads * (dim + rot)
    width = qw + rank + rot
    block = tiny.latent(heads, dim, rot, dv, rank, window, 1.0, 1000.0, None)["mixer"]
    mixer = build_mixer(_latent(0, block, EPS), width, None)
    eye = torch.eye(width)
    W = {"q": eye[:qw], "dkv": eye[qw:], "g": torch.zeros(heads * dv, width), "dkv.norm": torch.ones(rank), "sink": torch.tensor([1.0, -2.0]),
         "uk": rounded(heads * dim, rank, gen=gen, std=0.1), "uv": rounded(heads * dv, rank, gen=gen, std=0.5),
         "o": rounded(width, heads * dv, gen=gen, std=0.3)}
    W["uk"][:dim] = 0.0
    W["uk"][0, 0] = 1.0                                   # head 0: k[0] = c[0], every other unrotated key element is 0
    give(mixer, W, dtype)
    T = 2 * window + 37
    oldest = T - window                                   # the last query is at T - 1 and sees i - j < window
    base = rounded(T, width, gen=gen, std=0.2)
    base[:, qw] = 0.0                                     # the first latent element
    piece = {ops.LATENT_SEGMENT, ops.LATENT_MMA_SEGMENT}
    borders = {b + d for p in piece for b in range(0, T, p) for d in (-1, 0)} | {(oldest // page + 1) * page + d for d in (-1, 0)}
    inside = sorted(({oldest, oldest + 1, T - 2, T - 1} | borders) & set(range(oldest, T)))
    outside = [t for t in (oldest - 1, oldest - 2, oldest - window, 0) if t >= 0]
    for target in inside + outside:
        x = base.clone()
        x[target, qw] = 2.0 * math.sqrt(rank / 16)        # after the unit-RMS norm about 3.7
        x[T - 1, 0] = 16.0                                # head 0's query, first unrotated element
        want = plain.latent_attention(x.double(), double(W), block, EPS)[0].float()
        hidden = x.clone()
        hidden[target, qw] = 0.0
        without = plain.latent_attention(hidden.double(), double(W), block, EPS)[0].float()
        moved = float((want[T - 1] - without[T - 1]).abs().max())
        assert moved > 0.05 if target >= oldest else moved == 0.0, target      # the target decides the oracle's last row, or is unseen
        for sizes in ((T,), (T - 1, 1), (T - 2, 2), (oldest - 1, T - oldest + 1)):
            harness = Harness([mixer.cache_spec()], [None], dtype, num_pages=-(-T // page) + 1, page_size=page)
            got = run_mixer(mixer, harness, x, sizes, dtype)
            tol = 2e-4 if dtype == torch.float32 else 0.02 * float(want[T - 1].abs().max())
            assert torch.allclose(got[T - 1], want[T - 1], atol=tol, rtol=0), (target, sizes)


@pytest.mark.parametrize("dtype,rank,rot", [(torch.float32, 24, 6), (torch.bfloat16, 24, 6), (torch.bfloat16, 128, 32)])
def test_sinks_that_outweigh_the_keys(dtype, rank, rot):
    """A sink of 8 leaves the keys a small share, one of -60 nothing changed, whatever the number of visible
    keys (the first tokens see few) and wherever the kernels join their pieces."""
    gen = torch.Generator().manual_seed(rank)
    width, T, heads, page = 48, 330, 3, 16
    block = tiny.latent(heads, 12, rot, 10, rank, 280, 0.3, 100.0, None)["mixer"]
    mixer = build_mixer(_latent(0, block, EPS), width, None)
    W = weights_of(mixer, gen)
    x = rounded(T, width, gen=gen)
    outs = {}
    for sink in (8.0, 0.5, -60.0):
        W["sink"] = torch.tensor([sink, sink - 1.0, sink])
        give(mixer, W, dtype)
        want = plain.latent_attention(x.double(), double(W), block, EPS)[0].float()
        for sizes in ((T,), (290,) + (1,) * 40):
            harness = Harness([mixer.cache_spec()], [None], dtype, num_pages=-(-T // page) + 1, page_size=page)
            got = run_mixer(mixer, harness, x, sizes, dtype)
            close(got, want, dtype, (sink, sizes))
            close(got[:4], want[:4], dtype, (sink, "first tokens"))
            close(got[-4:], want[-4:], dtype, (sink, "last tokens"))
        outs[sink] = want
    assert float(outs[8.0][:4].abs().mean()) < 0.1 * float(outs[-60.0][:4].abs().mean())


# ---------------------------------------------------------------- capped attention
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv,dk,dv,dims,window,cap,page", [
    (4, 2, 24, 16, 8, 17, 3.0, 8), (2, 1, 16, 40, 2, 1, 5.0, 8), (3, 3, 8, 8, 8, 400, 2.0, 4), (1, 1, 34, 10, 6, 2, 9.0, 4),
    (4, 2, 64, 64, 32, 70, 4.0, 16), (2, 2, 128, 128, 128, 128, 6.0, 16), (6, 1, 64, 64, 64, 33, 3.0, 16), (2, 1, 136, 200, 32, 90, 5.0, 8),
    (8, 1, 128, 128, 64, 400, 2.5, 16), (20, 1, 64, 64, 64, 50, 3.0, 16), (4, 4, 96, 96, 96, 60, 4.0, 16)])
def test_capped_attention_mixer_against_plain(dtype, heads, kv, dk, dv, dims, window, cap, page):
    gen = torch.Generator().manual_seed(heads * 100 + dk)
    width, T = 72, 150
    block = tiny.capped(heads, kv, dk, dv, window, 4.0 / math.sqrt(dk), 300.0, dims, cap, None)["mixer"]
    mixer = build_mixer(_attention(0, block), width, None)
    assert set(mixer.weight_specs()) == {"q", "k", "v", "o"}
    W = weights_of(mixer, gen)
    give(mixer, W, dtype)
    x = rounded(T, width, gen=gen)
    want = plain.capped_attention(x.double(), double(W), block).float()
    uncapped = plain.capped_attention(x.double(), double(W), dict(block, softcap=1e4)).float()
    if window > 2:
        assert float((want - uncapped).abs().mean() / want.abs().mean()) > 0.05          # the cap matters
    for sizes in CUTS(T):
        harness = Harness([mixer.cache_spec()], [None], dtype, num_pages=-(-T // page) + 1, page_size=page)
        close(run_mixer(mixer, harness, x, sizes, dtype), want, dtype, sizes)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dk,window,page", [(24, 40, 8), (64, 48, 16), (64, 120, 16), (128, 16, 16), (32, 300, 4), (64, 300, 16)])
def test_one_capped_key_stands_out_at_the_edges_of_a_window(dtype, dk, window, page):
    """The last query and one key share a large component in a part of the head that does not turn: their
    score reaches the cap. The oldest key of the window, keys next to page borders and to the pieces that
    decoding cuts a window into give the output their value; the key one step further back must not be
    seen at all."""
    heads, kv, dims, cap = 2, 1, 8, 24.0
    gen = torch.Generator().manual_seed(dk + window)
    width = heads * dk + 2 * dk
    block = tiny.capped(heads, kv, dk, dk, window, 1.0, 100.0, dims, cap, None)["mixer"]
    mixer = build_mixer(_attention(0, block), width, None)
    eye = torch.eye(width)
    W = {"q": eye[: heads * dk], "k": eye[heads * dk: heads * dk + dk], "v": eye[heads * dk + dk:], "o": torch.eye(width)[:, : heads * dk]}
    give(mixer, W, dtype)
    T = 2 * window + window // 2 + 3
    oldest = T - window
    base = rounded(T, width, gen=gen, std=0.1)
    base[:, heads * dk + dk:] = rounded(T, dk, gen=gen)                       # values of order one
    border = (oldest // page + 1) * page
    pieces = {b + d for b in range(0, T, ops.SINK_SEGMENT) for d in (-1, 0)}
    inside = sorted(({oldest, oldest + 1, border, border - 1, T - 2} | pieces) & set(range(oldest, T - 1)))
    for target in inside + [oldest - 1, oldest - 2, 0]:
        x = base.clone()
        x[T - 1, dk - 1] = 8.0                            # head 0's query, last element (not rotated)
        x[target, heads * dk + dk - 1] = 8.0              # the key at `target`: a score of 64 before the cap
        want = plain.capped_attention(x.double(), double(W), block).float()
        value = x[target, heads * dk + dk:]
        assert torch.allclose(want[T - 1, :dk], value, atol=1e-3) == (target >= oldest), target
        for sizes in ((T,), (T - 1, 1), (oldest - 1, 3, T - oldest - 2), (T - 2, 2)):
            harness = Harness([mixer.cache_spec()], [None], dtype, num_pages=-(-T // page) + 1, page_size=page)
            got = run_mixer(mixer, harness, x, sizes, dtype)
            tol = 2e-5 if dtype == torch.float32 else 3e-2
            assert torch.allclose(got[T - 1], want[T - 1], atol=tol, rtol=tol), (target, sizes)


def test_caps_on_the_special_function_unit_keep_small_and_large_scores():
    """Two keys whose capped scores differ by less than a tenth while the scores themselves are far above the cap, and
    scores far below it: the tensor-core kernels' weights against the plain ones."""
    gen = torch.Generator().manual_seed(3)
    dk, page, T = 64, 16, 40
    width = 3 * dk
    for scale, cap in ((0.001, 50.0), (0.3, 2.0), (3.0, 30.0), (20.0, 30.0)):
        block = tiny.capped(1, 1, dk, dk, 64, scale, 100.0, 2, cap, None)["mixer"]
        mixer = build_mixer(_attention(0, block), width, None)
        eye = torch.eye(width)
        W = {"q": eye[:dk], "k": eye[dk:2 * dk], "v": eye[2 * dk:], "o": torch.eye(width)[:, :dk]}
        give(mixer, W, torch.bfloat16)
        x = rounded(T, width, gen=gen)
        x[:, 0:2] = x[:, dk:dk + 2] = 0.0                 # what turns is zero: queries and keys are exact in bfloat16
        want = plain.capped_attention(x.double(), double(W), block).float()
        for sizes in ((T,), (T - 8,) + (1,) * 8):
            harness = Harness([mixer.cache_spec()], [None], torch.bfloat16, num_pages=4, page_size=page)
            got = run_mixer(mixer, harness, x, sizes, torch.bfloat16)
            assert torch.allclose(got, want, atol=0.012, rtol=0.012), (scale, cap, sizes, float((got - want).abs().max()))


# ---------------------------------------------------------------- experts by token id
class TokenCtx:
    """What the expert part needs of a step's context."""

    def __init__(self, dtype, ids):
        self.dtype, self.extras = dtype, {"token_ids": ids}
        self.status = torch.zeros(1, dtype=torch.int32, device=DEV)
        self.num_tokens, self.all_decode = ids.shape[0], False


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,ff,width,grouped", [
    (6, 2, 48, 72, False), (6, 2, 64, 72, True), (5, 1, 96, 128, True), (8, 3, 80, 200, True), (3, 3, 64, 128, False), (1, 1, 48, 72, False),
    (7, 2, 20, 72, False), (40, 4, 64, 64, True), (6, 2, 272, 136, True), (2, 1, 64, 67, False)])
def test_table_experts_against_plain(dtype, experts, top, ff, width, grouped):
    gen = torch.Generator().manual_seed(experts * 10 + top)
    vocab = 90
    mlp = tiny.moe(experts, top, ff, 1.2)
    part = build_feed_forward(_feed_forward(0, mlp, vocab), width)
    W = weights_of(part, gen, "l0.mlp.")
    give(part, W, dtype)
    assert (part.grouped is not None) == (grouped and dtype == torch.bfloat16)
    for tokens in (1, 2, 17, 90, 128, 129, 300):
        ids = torch.randint(0, vocab, (tokens,), generator=gen)
        x = rounded(tokens, width, gen=gen)
        want = plain.table_experts(x.double(), ids.tolist(), double(W), mlp).float()
        ctx = TokenCtx(dtype, ids.to(DEV, torch.int32))
        y = part.forward(ctx, x.to(DEV, dtype))
        assert y.dtype == torch.float32
        got = ops.materialize(y).cpu()
        assert int(ctx.status.item()) == 0
        if dtype == torch.float32:
            assert torch.allclose(got, want, atol=3e-4, rtol=3e-4), (tokens, float((got - want).abs().max()))
        else:
            assert float((got - want).abs().mean() / want.abs().mean()) < 0.02, tokens
            assert float((got - want).abs().max() / want.abs().max()) < 0.03, tokens


def test_each_token_gets_its_own_experts_and_no_others():
    """Expert e's down matrix writes into channel e alone: a token's output names its experts. Also tokens
    that all share one expert, which then has as many rows as the step has tokens."""
    experts, top, ff, width, vocab = 9, 2, 64, 64, 50
    gen = torch.Generator().manual_seed(4)
    part = build_feed_forward(_feed_forward(0, tiny.moe(experts, top, ff, 5.0), vocab), width)
    W = weights_of(part, gen, "l0.mlp.")
    W["table"][:, 0] = torch.where(W["table"][:, 1] == 3, W["table"][:, 0], torch.full((vocab,), 3, dtype=torch.int32))     # expert 3 for every token
    for e in range(experts):
        W[f"e{e}.gate"], W[f"e{e}.up"] = torch.ones(ff, width) / width, torch.ones(ff, width) / width
        W[f"e{e}.down"] = torch.zeros(width, ff)
        W[f"e{e}.down"][e] = 1.0 / ff
    for dtype in (torch.bfloat16, torch.float32):
        give(part, W, dtype)
        for tokens in (1, 40, 128, 200):
            ids = torch.randint(0, vocab, (tokens,), generator=gen)
            got = ops.materialize(part.forward(TokenCtx(dtype, ids.to(DEV, torch.int32)), torch.ones(tokens, width, device=DEV, dtype=dtype))).cpu()
            named = [set(row.nonzero().flatten().tolist()) for row in got]
            assert named == [set(W["table"][t].tolist()) for t in ids.tolist()]
            assert torch.allclose(got.sum(1), torch.full((tokens,), 2.0 * float(torch.sigmoid(torch.tensor(1.702)))), rtol=1e-2)


@pytest.mark.parametrize("tokens,experts,top,width", [(1, 3, 1, 16), (5, 6, 3, 24), (148, 7, 1, 40), (149, 5, 2, 8), (700, 8, 2, 64), (1300, 70, 4, 33),
                                                      (9000, 8, 2, 8)])
def test_dispatch_sorts_and_gathers(tokens, experts, top, width):
    gen = torch.Generator().manual_seed(tokens)
    vocab = 60
    table = torch.rand((vocab, experts), generator=gen).argsort(dim=1)[:, :top].to(torch.int32)
    ids = torch.randint(0, vocab, (tokens,), generator=gen).to(torch.int32)
    x = rounded(tokens, width, gen=gen)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    for store in (torch.bfloat16, torch.float32):
        rows, offsets, where = ops.moe_dispatch(ids.to(DEV), table.to(DEV), experts, x.to(DEV, store), status)
        chosen = table[ids.long()].flatten()
        order = torch.argsort(chosen.long(), stable=True)                      # pairs by expert, in their own order inside one
        assert torch.equal(rows.float().cpu(), x[order // top])
        assert offsets.cpu().tolist() == [int((chosen < e).sum()) for e in range(experts + 1)]
        place = torch.empty(tokens * top, dtype=torch.long)
        place[order] = torch.arange(tokens * top)
        assert torch.equal(where.cpu().flatten().long(), place)
    chosen2, weights, dense = ops.moe_table(ids.to(DEV), table.to(DEV), experts, want_dense=True)
    assert torch.equal(chosen2.cpu(), table[ids.long()]) and torch.all(weights.cpu() == 1.0 / top)
    assert torch.allclose(dense.cpu(), torch.zeros(tokens, experts).scatter_(1, table[ids.long()].long(), 1.0 / top))
    act = torch.ones(tokens, experts * 8, device=DEV)
    assert torch.allclose(ops.moe_scale_table(act, ids.to(DEV), table.to(DEV), 8).cpu(), dense.cpu().repeat_interleave(8, dim=1))


@pytest.mark.parametrize("tokens,counts,features,k", [
    (1, [0, 1, 0, 1], 200, 64), (7, [7, 0, 3, 4], 128, 520), (30, [30, 30, 0, 0, 1], 72, 1024), (128, [128, 5, 100], 300, 2048),
    (129, [129, 1, 128], 264, 128), (600, [0, 600, 130, 2, 0, 127], 512, 192), (300, [300], 100, 72)])
def test_grouped_products_against_plain(tokens, counts, features, k):
    """Experts with no row, one row, a whole tile and a tile and one; features and inner extents that are no
    whole tiles; a few tokens (with K splits) and many."""
    gen = torch.Generator().manual_seed(tokens)
    rows, experts = sum(counts), len(counts)
    offsets = torch.tensor([sum(counts[:e]) for e in range(experts + 1)], dtype=torch.int32)
    x = rounded(rows, k, gen=gen)
    ws = [rounded(features, k, gen=gen, std=k ** -0.5) for _ in counts]
    want = torch.cat([x[offsets[e]:offsets[e + 1]].double() @ ws[e].double().T for e in range(experts)]).float()
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    packed = ops.ExpertWeights([w.to(DEV, torch.bfloat16) for w in ws])
    xd, od = x.to(DEV, torch.bfloat16), offsets.to(DEV)
    f32 = ops.gemm_tc_grouped(xd, packed, od, tokens, status, out_dtype=torch.float32)
    assert torch.allclose(f32.cpu(), want, atol=1e-4, rtol=1e-4)
    left = ops.gemm_tc_grouped(xd, packed, od, tokens, status, out_dtype=torch.float32, allow_partial=True)
    assert torch.equal(ops.materialize(left).cpu(), f32.cpu())
    low = ops.gemm_tc_grouped(xd, packed, od, tokens, status)
    assert torch.equal(low.float().cpu(), f32.cpu().to(torch.bfloat16).float())
    if features % 32 == 0:
        half = features // 2
        gate_up = ops.ExpertWeights([interleave_gate_up(w[:half], w[half:]).to(DEV, torch.bfloat16) for w in ws])
        act = ops.gemm_tc_grouped(xd, gate_up, od, tokens, status, activation="clamped", glu=(0.8, 1.702)).float().cpu()
        g, u = want[:, :half].clamp(max=0.8), want[:, half:].clamp(-0.8, 0.8)
        assert torch.allclose(act, g * torch.sigmoid(1.702 * g) * (u + 1.0), atol=1e-2, rtol=1e-2)
    assert int(status.item()) == 0


def test_unusable_tables_are_refused():
    part = build_feed_forward(_feed_forward(0, tiny.moe(4, 2, 16, 1.0), 10), 32)
    W = weights_of(part, torch.Generator().manual_seed(1), "l0.mlp.")
    for row, message in (([1, 4], "outside"), ([-1, 2], "outside"), ([2, 2], "twice")):
        bad = dict(W, table=W["table"].clone())
        bad["table"][3] = torch.tensor(row, dtype=torch.int32)
        with pytest.raises(ConfigError, match=message):
            give(part, bad, torch.float32)


# ---------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (config, seed) in tiny.ALL.items():
        folder = tiny.write_model(tmp_path_factory.mktemp(f"pubulix_{name}"), config, seed)
        _, tensors = tiny.tensors_for(config, seed)
        out[name] = (folder, config, tensors)
    return out


def prompt(config, n, seed):
    return torch.randint(0, config["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def logits_of(config, W, tokens):
    return plain.forward(config, W, tokens).float()


def close_rows(got, want, dtype):
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if dtype == "float32":
        return bool(err.max() < 2e-4)
    return bool(err.median() < 0.03 and err.max() < 0.15)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_whole_prompt_portions_and_decoding_against_plain(models, name, dtype):
    folder, config, W = models[name]
    tokens = prompt(config, 157, 1)
    want = logits_of(config, W, tokens)
    for sizes in ((157,), (125,) + (1,) * 32, (2, 5, 1, 1, 17, 2, 3, 30, 96), (3, 2, 2, 150), (2,) * 78 + (1,)):
        page = tiny.PAGE[name]
        runner = ModelRunner(folder, dtype=dtype, num_pages=176 // page, page_size=page, max_requests=2)
        runner.begin("r")
        rows, at = [], 0
        for size in sizes:
            rows.append(runner.step([StepEntry("r", tokens[at:at + size], list(range(size)))]).cpu())
            at += size
        runner.check_status()
        assert close_rows(torch.cat(rows), want, dtype), sizes


WIDE = tiny.model(512, 1024, 4, 0.5, 30.0, 15.0, 1e-5, [
    tiny.latent(8, 128, 64, 128, 512, 90, 0.08, 10000.0, tiny.moe(8, 2, 1024, 3.0)),
    tiny.capped(8, 2, 128, 128, 70, 0.09, 10000.0, 64, 20.0, tiny.moe(4, 2, 2048, 3.0)),
    tiny.latent(4, 128, 64, 128, 512, 30, 0.08, 10000.0, tiny.moe(8, 1, 512, 3.0), kv_from=0),
])


def test_wide_layers_whose_products_split_their_inner_range(tmp_path):
    """Layer sizes at which the bfloat16 products of a few tokens split their inner range: the boundary
    kernel adds the unsummed splits of the sublayer's output, of the gate and of a token's experts."""
    lib = ops.library()
    assert lib.vosti_gemm_tc_splits(1, 1024, 1024) > 1 and lib.vosti_gemm_tc_grouped_splits(4, 8, 8, 1024, 1024) > 1
    folder = tiny.write_model(tmp_path / "wide", WIDE, 77)
    _, W = tiny.tensors_for(WIDE, 77)
    tokens = prompt(WIDE, 40, 8)
    want = logits_of(WIDE, W, tokens)
    for dtype in ("bfloat16", "float32"):
        runner = ModelRunner(folder, dtype=dtype, num_pages=4, page_size=16, max_requests=2)
        assert all((block.feed_forward.grouped is not None) == (dtype == "bfloat16") for block in runner.model.blocks)
        runner.begin("r")
        rows = [runner.step([StepEntry("r", tokens[:4], [0, 1, 2, 3])]).cpu()]
        rows += [runner.step([StepEntry("r", [t], [0])]).cpu() for t in tokens[4:]]
        runner.check_status()
        assert close_rows(torch.cat(rows), want, dtype), dtype


def test_a_checkpoint_without_the_unused_tensors_gives_the_same_logits(models, tmp_path):
    folder, config, W = models["a"]
    bare = tiny.write_model(tmp_path / "bare", config, tiny.ALL["a"][1], unused=False)
    tokens = prompt(config, 19, 3)
    rows = []
    for f in (folder, bare):
        runner = ModelRunner(f, dtype="float32", num_pages=8, page_size=8, max_requests=1)
        runner.begin("r")
        rows.append(runner.step([StepEntry("r", tokens, list(range(19)))]).cpu())
    assert torch.equal(rows[0], rows[1])


def test_first_tokens_of_a_sequence(models):
    """Requests of one, two and three tokens, and the first rows of a longer one: zeros before the
    convolution, a softmax over one key beside the sink, position zero (no rotation)."""
    for name in ("a", "b", "c"):
        folder, config, W = models[name]
        page = tiny.PAGE[name]
        for dtype in ("float32", "bfloat16"):
            runner = ModelRunner(folder, dtype=dtype, num_pages=32 // page, page_size=page, max_requests=2)
            for n in (1, 2, 3, 9):
                tokens = prompt(config, n, 40 + n)
                for cut in ((n,), (1,) * n):
                    runner.begin("r")
                    rows, at = [], 0
                    for size in cut:
                        rows.append(runner.step([StepEntry("r", tokens[at:at + size], list(range(size)))]).cpu())
                        at += size
                    runner.finish("r")
                    assert close_rows(torch.cat(rows), logits_of(config, W, tokens), dtype), (name, n, cut)
            runner.check_status()


def test_residual_stream_after_every_layer(models):
    for name in ("a", "b", "c"):
        folder, config, W = models[name]
        tokens = prompt(config, 23, 2)
        want = []
        plain.forward(config, W, tokens, streams=want)
        page = tiny.PAGE[name]
        runner = ModelRunner(folder, dtype="float32", num_pages=32 // page, page_size=page, max_requests=1)
        streams = []
        for block in runner.model.blocks:
            inner = block.forward

            def watched(ctx, hidden, residual, cache, writes_cache=True, inner=inner):
                out, stream = inner(ctx, hidden, residual, cache, writes_cache)
                after = stream.clone()
                ops.gated_rms_stream(after, out, 1e-6, torch.float32, status=ctx.status)     # adds what is still pending
                streams.append(after.cpu())
                return out, stream
            block.forward = watched
        runner.begin("r")
        runner.step([StepEntry("r", tokens, [0])])
        assert len(streams) == len(want) == len(config["layers"])
        for i, (got, expected) in enumerate(zip(streams, want)):
            assert torch.allclose(got, expected.float(), atol=5e-4, rtol=3e-4), (name, i)


@pytest.mark.parametrize("name,dtype", [("a", "float32"), ("b", "float32"), ("c", "float32"), ("c", "bfloat16"), ("a", "bfloat16")])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(models, name, dtype):
    """Four requests through two request slots and a pool that holds two of them: portions of some
    beside single tokens of others; every request equals itself alone."""
    folder, config, W = models[name]
    lengths = {"a": 37, "b": 9, "c": 1, "d": 26}
    tokens = {r: prompt(config, n, 10 + i) for i, (r, n) in enumerate(lengths.items())}
    want = {r: logits_of(config, W, t) for r, t in tokens.items()}
    page = tiny.PAGE[name]
    pool = 80 // page
    runner = ModelRunner(folder, dtype=dtype, num_pages=pool, page_size=page, max_requests=2)
    schedule = [
        [("a", 5), ("b", 2)], [("a", 1), ("b", 6)], [("b", 1), ("a", 20)], [("a", 1)],      # b ends in step 2
        [("c", 1), ("a", 1)], [("d", 1), ("a", 1)], [("d", 1), ("a", 8)], [("d", 1)], [("d", 23)],     # c, then a end
    ]
    at = {r: 0 for r in lengths}
    got = {r: [] for r in lengths}
    for step in schedule:
        entries = []
        for r, n in step:
            if r not in runner.cache.live:
                runner.begin(r)
            entries.append(StepEntry(r, tokens[r][at[r]:at[r] + n], list(range(n))))
        logits = runner.step(entries).cpu()
        row = 0
        for r, n in step:
            got[r].append(logits[row:row + n])
            row += n
            at[r] += n
            if at[r] == lengths[r]:
                runner.finish(r)
    runner.check_status()
    runner.cache.check()
    for r in lengths:
        assert at[r] == lengths[r]
        assert close_rows(torch.cat(got[r]), want[r], dtype), r
    assert runner.cache.available_pages() == pool


@pytest.mark.parametrize("name,dtype", [("a", "float32"), ("b", "float32"), ("c", "float32"), ("c", "bfloat16")])
def test_long_decoding_past_every_window(models, name, dtype):
    """A prompt, then token by token far past every window, with a pool that holds little more than the widest one
    (in configuration A that is the window of a layer that reads another layer's latents through a
    wider one than its owner's): pages come back and are used again."""
    folder, config, W = models[name]
    widest = max(layer["mixer"]["mask"]["size"] for layer in config["layers"])
    total = {"a": 260, "b": 120, "c": 460}[name]
    tokens = prompt(config, total, 4)
    want = logits_of(config, W, tokens)
    page = tiny.PAGE[name]
    first = widest + 5
    pool = (first + 2 * page) // page + 1
    assert pool * page < total
    runner = ModelRunner(folder, dtype=dtype, num_pages=pool, page_size=page, max_requests=1)
    runner.begin("r")
    rows = [runner.step([StepEntry("r", tokens[:first], list(range(first)))]).cpu()]
    rows += [runner.step([StepEntry("r", [t], [0])]).cpu() for t in tokens[first:]]
    runner.check_status()
    runner.cache.check()
    assert close_rows(torch.cat(rows), want, dtype)
    runner.finish("r")
    assert runner.cache.available_pages() == pool


@pytest.mark.parametrize("name,dtype,binary", [("a", "float32", True), ("c", "bfloat16", False), ("b", "float32", False), ("c", "float32", False)])
def test_trace_replay_of_a_mixed_schedule(models, name, dtype, binary, tmp_path):
    """The trace runner (the program itself, and the class it wraps) over a schedule of up to four
    live requests, portions beside single tokens, requests that sit a step out and a pool smaller
    than the sum of all requests: every row against the plain implementation of the request alone."""
    import numpy as np
    import replay_util as R
    folder, config, W = models[name]
    requests = {f"q{i}": prompt(config, n, 60 + i) for i, n in enumerate([70, 40, 33, 90, 64, 21])}
    steps = R.number(R.mixed_steps(requests, seed=5))
    max_tokens = R.max_live_tokens(steps)
    assert max_tokens < sum(R.roundup64(len(t)) for t in requests.values())
    if binary:
        R.run_binary(folder, dtype, steps, max_tokens, tmp_path)
    else:
        R.run_in_process(folder, dtype, steps, max_tokens, tiny.PAGE[name], tmp_path)
    rows = R.collect(steps, tmp_path, config["vocab"])
    assert len(rows) == sum(len(t) for t in requests.values())
    for rid, tokens in requests.items():
        got = torch.from_numpy(np.stack([rows[(rid, p)] for p in range(len(tokens))]))
        assert close_rows(got, logits_of(config, W, tokens), dtype), rid


def plain_greedy(config, W, tokens, new_tokens):
    tokens, out = list(tokens), []
    for _ in range(new_tokens):
        out.append(int(plain.forward(config, W, tokens)[-1].argmax()))
        tokens.append(out[-1])
    return out


@pytest.mark.parametrize("name,cuda_graphs,async_scheduling", [("a", False, False), ("a", True, False), ("a", True, True), ("c", True, True)])
def test_greedy_generation_through_the_engine(models, name, cuda_graphs, async_scheduling):
    """The framework's own entry point: scheduler, portions under a token budget, CUDA graphs for
    decode steps (whose experts follow from tokens the host has not read), two slots for five
    requests, so few pages that a request is preempted and computed again from its first token."""
    folder, config, W = models[name]
    prompts = [prompt(config, n, 20 + n) for n in (5, 17, 2, 11, 8)]
    want = [plain_greedy(config, W, p, 10) for p in prompts]
    blocks, size = (9, 4) if name == "a" else (3, 16)
    engine = Engine(folder, dtype="float32", num_blocks=blocks, block_size=size, max_num_seqs=2, max_num_batched_tokens=16,
                    prefill_chunk_size=8 if name == "a" else 16, cuda_graphs=cuda_graphs, async_scheduling=async_scheduling)
    assert engine.runner.spec.architecture == "Pubulix" and engine.runner.cache.has_state
    assert (engine.graphs is not None) == cuda_graphs
    got = engine.generate(prompts, max_tokens=10, arrival_steps=[0, 0, 1, 4, 20])
    assert got == want
    if name == "a":
        assert engine.scheduler.preemptions > 0
    if cuda_graphs:
        assert engine.graphs.replays > 0
    engine.runner.cache.check()
    assert engine.runner.cache.available_pages() == blocks


def test_graphs_give_the_bfloat16_engine_the_same_tokens(models):
    """bfloat16 serving through the grouped products and fused steps, with and without recorded decode steps."""
    folder, config, W = models["c"]
    prompts = [prompt(config, n, 70 + n) for n in (12, 30, 7)]
    tokens = []
    for cuda_graphs in (False, True):
        engine = Engine(folder, dtype="bfloat16", num_blocks=12, block_size=16, max_num_seqs=3, max_num_batched_tokens=64,
                        cuda_graphs=cuda_graphs, async_scheduling=cuda_graphs)
        tokens.append(engine.generate(prompts, max_tokens=16))
        if cuda_graphs:
            assert engine.graphs.replays > 0
    assert tokens[0] == tokens[1]


def test_the_command_line_generates_from_a_pubulix_folder(models, capsys):
    from vosti_b200.engine import cli
    folder, config, W = models["b"]
    tokens = prompt(config, 6, 9)
    want = plain_greedy(config, W, tokens, 4)
    code = cli.main(["--model", folder, "--dtype", "float32", "--prompt-ids", ",".join(map(str, tokens)), "--max-tokens", "4"])
    assert code in (0, None)
    assert ",".join(map(str, want)) in capsys.readouterr().out.replace(" ", "")
